// The tile list of a float product: dense (groups x weight tiles x token tiles) or ragged (the token rows are ordered by
// group and the group sizes are on the device: experts).
#pragma once

#include "fl_epilogue.cuh"

namespace bxf {

struct GemmShape {
  int M, N, K, groups;
  int n_tiles, m_tiles;          // ragged: m_tiles bounds the token tiles over all groups
  const int* counts;             // NULL: dense
};

// Ragged lists: the group and rows of token tile `mt`. Warp-collective; false when the list is shorter.
__device__ __forceinline__ bool locate_ragged(const int* counts, int groups, int ta, int mt, Tile& t) {
  const int lane = threadIdx.x & 31;
  int tiles_before = 0, rows_before = 0;
  for (int e0 = 0; e0 < groups; e0 += 32) {
    const int cnt = e0 + lane < groups ? counts[e0 + lane] : 0;
    const int tiles = (cnt + ta - 1) / ta;
    int it = tiles, ir = cnt;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int a = __shfl_up_sync(0xffffffffu, it, o), b = __shfl_up_sync(0xffffffffu, ir, o);
      if (lane >= o) {
        it += a;
        ir += b;
      }
    }
    const unsigned hit = __ballot_sync(0xffffffffu, mt < tiles_before + it);
    if (hit) {
      const int src = __ffs(hit) - 1;
      const int first_tile = tiles_before + __shfl_sync(0xffffffffu, it - tiles, src);
      const int first_row = rows_before + __shfl_sync(0xffffffffu, ir - cnt, src);
      const int in_group = (mt - first_tile) * ta;
      t.group = e0 + src;
      t.row0 = first_row + in_group;
      t.rows = min(ta, __shfl_sync(0xffffffffu, cnt, src) - in_group);
      return true;
    }
    tiles_before += __shfl_sync(0xffffffffu, it, 31);
    rows_before += __shfl_sync(0xffffffffu, ir, 31);
  }
  return false;
}

// Tile number `tile` of tiles of ta token rows x tn weight rows. Token tiles are the fastest index, so consecutive CTAs
// share a weight tile. Warp-collective.
__device__ __forceinline__ bool locate_tile(const GemmShape& s, int ta, int tile, Tile& t, int tn = NROWS) {
  const int mt = tile % s.m_tiles, rest = tile / s.m_tiles;
  t.n0 = (rest % s.n_tiles) * tn;
  if (s.counts) return locate_ragged(s.counts, s.groups, ta, mt, t);
  t.group = rest / s.n_tiles;
  t.row0 = mt * ta;
  t.rows = min(ta, s.M - t.row0);
  return true;
}

}  // namespace bxf
