// bf16 products on tcgen05 (kind::f16, fp32 accumulators in TMEM).
//
// Warp roles as in limb_gemm.cuh: warp 0 = TMA producer, warp 1 = TMEM allocation + MMA issue, warps 2 .. 17 = epilogue.
// fl_gemm_kernel (short tile lists: decoding, short portions) has the weights on the MMA M side like the limb GEMM: 128
// weight rows (TMEM lanes) x TA token rows, so a batch of 1 .. 16 rows streams the weights once with TA = 16. A cluster of S
// CTAs shares a tile with K split between them; the fp32 partials are exchanged through distributed shared memory and
// every CTA finishes 128 / S weight rows. NP product planes (the three projections of a minGRU layer) share one token
// tile: plane p accumulates into TMEM columns [p TA, (p + 1) TA).
// fl_gemm_persistent_kernel (long tile lists: prompts) has the tokens on the M side: 128 token rows x TN weight rows, two
// TMEM buffers, so that the epilogue of a tile (16-byte stores of consecutive channels) runs behind the MMAs of the next.
// Every wait is bounded; a timeout raises the device status word and the CTA leaves without storing.
#pragma once

#include <cooperative_groups.h>

#include "fl_tiles.cuh"
#include "limb_gemm.cuh"

namespace bxf {

using namespace bx;

constexpr int KE = 64;                  // K elements per stage (128 bytes: one swizzle atom per row)

// CTAS: CTAs that share an SM (shared memory is cut accordingly).
template <int NP, int TA, int CTAS = 1>
struct FlCfg {
  static_assert(TA % 16 == 0 && TA >= 16 && TA <= 256, "MMA N");
  static constexpr int COLS = NP * TA;
  static_assert(COLS <= 512, "TMEM capacity");
  static constexpr int W_BYTES = NP * NROWS * BKB;
  static constexpr int X_BYTES = TA * BKB;
  static constexpr int STAGE_BYTES = W_BYTES + X_BYTES;
  static constexpr int STAGES_MAX = (227 * 1024 / CTAS - 3072) / STAGE_BYTES;
  static constexpr int STAGES = STAGES_MAX > 8 ? 8 : STAGES_MAX;
  static_assert(STAGES >= 2, "at least two stages");
  static constexpr int RING_BYTES = STAGES * STAGE_BYTES;
  static constexpr int PARTIAL_BYTES = NP * TA * NROWS * 4;
  static constexpr int SMEM_BYTES = RING_BYTES + 1024 + 512;
  static __host__ __device__ constexpr int tmem_cols(int c) { return c <= 32 ? 32 : c <= 64 ? 64 : c <= 128 ? 128 : c <= 256 ? 256 : 512; }
};

struct FlShared {
  uint64_t full[8];
  uint64_t empty[8];
  uint64_t acc_full[2];
  uint64_t acc_empty[2];
  uint32_t tmem_base;
  uint32_t abort_flag;
};

// bf16 x bf16 -> fp32, M = 128; b_mn: the B operand is MN-major (its rows are the contraction index).
__host__ __device__ constexpr uint32_t umma_idesc_bf16(int n, bool b_mn = false) {
  return (1u << 4) | (1u << 7) | (1u << 10) | (b_mn ? 1u << 16 : 0u) | (static_cast<uint32_t>(n >> 3) << 17) |
         (static_cast<uint32_t>(128 >> 4) << 24);
}

__device__ __forceinline__ void umma_bf16(uint32_t d_tmem, uint64_t a_desc, uint64_t b_desc, uint32_t idesc,
                                          uint32_t accumulate) {
  asm volatile(
      "{\n\t"
      ".reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t"
      "}\n" ::"r"(d_tmem),
      "l"(a_desc), "l"(b_desc), "r"(idesc), "r"(accumulate)
      : "memory");
}

// ---- accumulator sources of the epilogues ----
struct TmemGet {
  uint32_t base;                        // this warp's lane quarter
  int ta;
  template <int W>
  __device__ __forceinline__ void load(int plane, int c, float (&v)[W]) const {
    uint32_t r[W];
    if constexpr (W == 16) tmem_ld16(base + plane * ta + c, r);
    else tmem_ldn<W>(base + plane * ta + c, r);
    tmem_ld_wait();
#pragma unroll
    for (int i = 0; i < W; ++i) v[i] = __uint_as_float(r[i]);
  }
};

constexpr int FL_SPLIT_MAX = 4;         // clusters of 2 or 4 CTAs

// The partial sums of the S CTAs of a cluster for the rows this one finishes: [S][column][128 / S] in its own shared memory.
template <int S, int COLS>
struct PartialGet {
  const float* part;
  int ta, row;                          // row among the 128 / S
  template <int W>
  __device__ __forceinline__ void load(int plane, int c, float (&v)[W]) const {
    float t[S][W];
#pragma unroll
    for (int r = 0; r < S; ++r)
#pragma unroll
      for (int i = 0; i < W; ++i) t[r][i] = part[(r * COLS + plane * ta + c + i) * (NROWS / S) + row];
#pragma unroll
    for (int i = 0; i < W; ++i) {
      v[i] = t[0][i];
#pragma unroll
      for (int r = 1; r < S; ++r) v[i] += t[r][i];
    }
  }
};

// ---- the two asynchronous roles; `it` counts stages over the life of the CTA ----
// TOKENS_M: the 128-row operand is the token tile (one plane), else the weight tile. Of the CTA's first tile, `ahead`
// stages have their weights under way already (feed_weights).
template <class Cfg, int NP, bool TOKENS_M = false>
__device__ __forceinline__ bool feed_tile(FlShared* sh, uint8_t* ring, const CUtensorMap* mw, const CUtensorMap* mx,
                                          const Tile& t, bool ragged, int kb0, int nkb, int& it, int ahead = 0) {
  for (int i = 0; i < nkb; ++i, ++it) {
    const int s = it % Cfg::STAGES, round = it / Cfg::STAGES;
    if (round > 0 && !mbar_wait(&sh->empty[s], (round - 1) & 1)) return false;
    uint8_t* st = ring + s * Cfg::STAGE_BYTES;
    uint8_t* w_tile = TOKENS_M ? st + Cfg::W_BYTES : st;
    uint8_t* x_tile = TOKENS_M ? st : st + Cfg::W_BYTES;
    if (i >= ahead) {
      mbar_arrive_expect_tx(&sh->full[s], Cfg::STAGE_BYTES);
      tma_load_3d(w_tile, mw, &sh->full[s], (kb0 + i) * KE, t.n0, NP == 1 ? t.group : 0);
    }
    tma_load_3d(x_tile, mx, &sh->full[s], (kb0 + i) * KE, t.row0, ragged ? 0 : t.group);
  }
  return true;
}

// The weight tiles of the first stages of the CTA's first tile, ahead of the previous kernel's end; returns how many.
template <class Cfg, int NP>
__device__ __forceinline__ int feed_weights(FlShared* sh, uint8_t* ring, const CUtensorMap* mw, const Tile& t, int kb0,
                                            int nkb) {
  const int n = min(nkb, Cfg::STAGES);
  for (int s = 0; s < n; ++s) {
    mbar_arrive_expect_tx(&sh->full[s], Cfg::STAGE_BYTES);
    tma_load_3d(ring + s * Cfg::STAGE_BYTES, mw, &sh->full[s], (kb0 + s) * KE, t.n0, NP == 1 ? t.group : 0);
  }
  return n;
}

template <class Cfg, int NP, int TA>
__device__ __forceinline__ bool multiply_tile(FlShared* sh, uint8_t* ring, uint32_t acc, int nkb, int& it) {
  constexpr uint32_t ID = umma_idesc_bf16(TA);
  for (int i = 0; i < nkb; ++i, ++it) {
    const int s = it % Cfg::STAGES;
    if (!mbar_wait(&sh->full[s], (it / Cfg::STAGES) & 1)) return false;
    tc_fence_after();
    const uint32_t wbase = smem_u32(ring + s * Cfg::STAGE_BYTES), xbase = wbase + Cfg::W_BYTES;
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
      const uint64_t xd = umma_desc_sw128(xbase + ks * 32);
#pragma unroll
      for (int p = 0; p < NP; ++p)
        umma_bf16(acc + p * TA, umma_desc_sw128(wbase + p * (NROWS * BKB) + ks * 32), xd, ID, (i | ks) != 0);
    }
    umma_commit(&sh->empty[s]);
  }
  return true;
}

// After a failed wait of the producer: let the copies in flight land before the CTA exits.
template <int STAGES>
__device__ __forceinline__ void drain_ring(FlShared* sh, int it) {
  for (int i = it > STAGES ? it - STAGES : 0; i < it; ++i) mbar_wait(&sh->full[i % STAGES], (i / STAGES) & 1);
}

__device__ __forceinline__ void give_up(FlShared* sh) {
  atomicAdd(&g_wait_timeouts, 1);
  *reinterpret_cast<volatile uint32_t*>(&sh->abort_flag) = 1;
}

__device__ __forceinline__ bool aborted(const FlShared* sh) {
  return *reinterpret_cast<const volatile uint32_t*>(&sh->abort_flag) != 0;
}

template <int TCOLS>
__device__ __forceinline__ uint32_t open_cta(FlShared* sh, int stages, const CUtensorMap* mw, const CUtensorMap* mx) {
  if (threadIdx.x == 0) {
    for (int s = 0; s < stages; ++s) {
      mbar_init(&sh->full[s], 1);
      mbar_init(&sh->empty[s], 1);
    }
    for (int b = 0; b < 2; ++b) {
      mbar_init(&sh->acc_full[b], 1);
      mbar_init(&sh->acc_empty[b], EPI_THREADS / 32);
    }
    sh->abort_flag = *reinterpret_cast<volatile int*>(&g_wait_timeouts) != 0;
    fence_barrier_init();
    tma_prefetch_desc(mw);
    tma_prefetch_desc(mx);
  }
  __syncthreads();
  if ((threadIdx.x >> 5) == 1) {
    tmem_alloc(&sh->tmem_base, TCOLS);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  launch_next();                        // after the TMEM allocation: the next kernel's CTAs allocate too
  return sh->tmem_base;
}

template <int TCOLS>
__device__ __forceinline__ void close_cta(uint32_t tmem) {
  tc_fence_before();
  __syncthreads();
  if ((threadIdx.x >> 5) == 1) {
    __syncwarp();
    tc_fence_after();
    tmem_dealloc(tmem, TCOLS);
  }
}

// ---- one tile per cluster, K split over the cluster's CTAs ----
template <int TA, class Epi>
__global__ void __launch_bounds__(64 + 32 * Epi::warps(TA), Epi::ctas(TA))
fl_gemm_kernel(const __grid_constant__ CUtensorMap mw, const __grid_constant__ CUtensorMap mx, const GemmShape s,
               const __grid_constant__ typename Epi::Params ep) {
  namespace cg = cooperative_groups;
  constexpr int NP = Epi::PLANES, EW = Epi::warps(TA);
  using Cfg = FlCfg<NP, TA, Epi::ctas(TA)>;
  constexpr int TCOLS = Cfg::tmem_cols(Cfg::COLS);
  static_assert(Epi::stash_bytes(TA) <= Cfg::RING_BYTES, "the epilogue's stash lies in the idle ring");
  extern __shared__ uint8_t smem_raw[];
  uint8_t* ring = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  FlShared* sh = reinterpret_cast<FlShared*>(ring + Cfg::RING_BYTES);

  cg::cluster_group cluster = cg::this_cluster();
  const int S = (int)cluster.num_blocks(), rank = (int)cluster.block_rank();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  Tile t;
  if (s.counts) wait_previous();                                        // the group sizes are the previous kernels' work
  if (!locate_tile(s, TA, blockIdx.x / S, t)) return;                  // the same for every CTA of the cluster
  const int nkb_all = (s.K + KE - 1) / KE;
  const int kb0 = rank * nkb_all / S, nkb = (rank + 1) * nkb_all / S - kb0;

  const uint32_t tmem = open_cta<TCOLS>(sh, Cfg::STAGES, &mw, &mx);
  const bool dead = sh->abort_flag != 0;                                // an earlier timeout: no work, all barriers
  __syncthreads();
  bool ok = !dead;
  // What an epilogue thread finishes: straight from TMEM its lane quarter (S = 1), else quarters rank, rank + S, .. of
  // the tile, 4 / S of them
  const int we = warp - 2, quarters = 4 / S, qi = S == 1 ? warp & 3 : we % quarters, group = we / quarters;
  const int row = (rank + S * qi) * 32 + lane, groups = EW / quarters;
  if (warp == 0) {
    if (lane == 0 && !dead) {
      int it = 0;
      const int ahead = feed_weights<Cfg, NP>(sh, ring, &mw, t, kb0, nkb);
      wait_previous();
      if (!feed_tile<Cfg, NP>(sh, ring, &mw, &mx, t, s.counts != nullptr, kb0, nkb, it, ahead)) {
        give_up(sh);
        drain_ring<Cfg::STAGES>(sh, it);
      }
    }
  } else if (warp == 1) {
    if (lane == 0 && !dead) {
      int it = 0;
      if (multiply_tile<Cfg, NP, TA>(sh, ring, tmem, nkb, it)) umma_commit(&sh->acc_full[0]);
      else give_up(sh);
    }
  } else if (!dead) {
    wait_previous();
    Epi::template prefetch<TA>(ep, t, s.N, row, group, groups);
    if (nkb > 0) ok = mbar_wait(&sh->acc_full[0], 0);
    ok = ok && !aborted(sh);
    ok = __all_sync(0xffffffffu, ok);
    if (ok) tc_fence_after();
    else if (lane == 0) atomicAdd(&g_wait_timeouts, 1);
  }

  if (S == 1) {
    __syncthreads();
    if (warp >= 2 && !dead && !aborted(sh) && nkb > 0) {
      TmemGet get{tmem + ((uint32_t)(qi * 32) << 16), TA};
      Epi::template run<bf16, TA, (TA * 4 / EW >= 8 ? 8 : 4)>(get, ep, t, s.N, row, group, groups, ring);
    }
  } else if constexpr (Cfg::PARTIAL_BYTES + Epi::stash_bytes(TA) <= Cfg::RING_BYTES) {
    float* part = reinterpret_cast<float*>(ring);
    __syncthreads();
    cluster.sync();                                                     // every ring of the cluster is idle
    if (warp >= 2) {
      // lane quarter q goes to CTA q mod S, slot of this rank
      const int quarter = warp & 3;
      float* to = cluster.map_shared_rank(part, quarter % S) +
                  (size_t)rank * Cfg::COLS * (NROWS / S) + quarter / S * 32 + lane;
      const TmemGet get{tmem + ((uint32_t)(quarter * 32) << 16), TA};
      for (int c = (we >> 2) * 8; c < Cfg::COLS; c += EW * 2) {
        if (c % TA >= t.rows) continue;                                 // columns of no token
        float v[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) v[i] = 0.0f;
        if (ok && nkb > 0) get.load<8>(0, c, v);
#pragma unroll
        for (int i = 0; i < 8; ++i) to[(c + i) * (NROWS / S)] = v[i];
      }
    }
    cluster.sync();                                                     // every partial is in its owner's ring
    if (warp >= 2) {
      uint8_t* stash = ring + Cfg::PARTIAL_BYTES;
      if (S == 2) {
        constexpr int PER = TA * 2 / EW;                                // columns of a thread
        PartialGet<2, Cfg::COLS> get{part, TA, qi * 32 + lane};
        Epi::template run<bf16, TA, (PER >= 8 ? 8 : PER)>(get, ep, t, s.N, row, group, groups, stash);
      } else {
        constexpr int PER = TA / EW;
        PartialGet<4, Cfg::COLS> get{part, TA, qi * 32 + lane};
        Epi::template run<bf16, TA, (PER >= 8 ? 8 : PER)>(get, ep, t, s.N, row, group, groups, stash);
      }
    }
  }
  close_cta<TCOLS>(tmem);
}

// ---- persistent: every CTA walks the tile list, two TMEM buffers ----
template <int TN, class Epi>
__global__ void __launch_bounds__(GEMM_THREADS, 1)
fl_gemm_persistent_kernel(const __grid_constant__ CUtensorMap mw, const __grid_constant__ CUtensorMap mx,
                          const GemmShape s, const __grid_constant__ typename Epi::Params ep) {
  using Cfg = FlCfg<1, TN>;
  static_assert(2 * Cfg::COLS <= 512 && Epi::PLANES == 1, "two accumulator buffers");
  constexpr int TCOLS = Cfg::tmem_cols(2 * Cfg::COLS);
  extern __shared__ uint8_t smem_raw[];
  uint8_t* ring = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  FlShared* sh = reinterpret_cast<FlShared*>(ring + Cfg::RING_BYTES);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int total = s.n_tiles * s.m_tiles * (s.counts ? 1 : s.groups), nkb = (s.K + KE - 1) / KE;
  const bool ragged = s.counts != nullptr;

  const uint32_t tmem = open_cta<TCOLS>(sh, Cfg::STAGES, &mw, &mx);
  const bool dead = sh->abort_flag != 0;
  __syncthreads();
  wait_previous();
  Tile t;
  if (!dead) {
    if (warp == 0) {
      int it = 0;
      bool ok = true;
      for (int tile = blockIdx.x; tile < total && ok; tile += gridDim.x) {
        if (!locate_tile(s, NROWS, tile, t, TN)) continue;
        if (lane == 0) ok = feed_tile<Cfg, 1, true>(sh, ring, &mw, &mx, t, ragged, 0, nkb, it);
        ok = __all_sync(0xffffffffu, ok);
      }
      if (!ok && lane == 0) {
        give_up(sh);
        drain_ring<Cfg::STAGES>(sh, it);
      }
    } else if (warp == 1) {
      int it = 0, count = 0;
      bool ok = true;
      for (int tile = blockIdx.x; tile < total && ok; tile += gridDim.x) {
        if (!locate_tile(s, NROWS, tile, t, TN)) continue;
        const int buf = count & 1, use = count >> 1;
        if (lane == 0) {
          if (use > 0) ok = mbar_wait(&sh->acc_empty[buf], (use - 1) & 1);
          tc_fence_after();
          ok = ok && multiply_tile<Cfg, 1, TN>(sh, ring, tmem + buf * Cfg::COLS, nkb, it);
          if (ok) umma_commit(&sh->acc_full[buf]);
        }
        ok = __all_sync(0xffffffffu, ok);
        ++count;
      }
      if (!ok && lane == 0) give_up(sh);
    } else {
      const int we = warp - 2, quarter = warp & 3;
      int count = 0;
      bool ok = true;
      for (int tile = blockIdx.x; tile < total; tile += gridDim.x) {
        if (!locate_tile(s, NROWS, tile, t, TN)) continue;
        const int buf = count & 1, use = count >> 1;
        ok = mbar_wait(&sh->acc_full[buf], use & 1) && !aborted(sh);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        tc_fence_after();
        TmemGet get{tmem + buf * Cfg::COLS + ((uint32_t)(quarter * 32) << 16), TN};
        Epi::template run_rows<bf16, TN>(get, ep, t, s.N, quarter * 32 + lane, we >> 2);
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(&sh->acc_empty[buf]);
        ++count;
      }
      if (!ok && lane == 0) atomicAdd(&g_wait_timeouts, 1);
    }
  }
  close_cta<TCOLS>(tmem);
}

}  // namespace bxf
