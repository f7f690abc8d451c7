// Epilogues of the float products, for both orientations of a tile.
// Weight-major (`run`): 128 weight rows x TA token rows; a thread owns ONE weight row (output channel) n and walks token
// columns, so per-channel constants live in registers, a warp stores 32 consecutive channels of a token, a rotated pair
// is two neighbouring lanes, and a recurrence over tokens is a loop of one thread.
// Token-major (`run_rows`, long prompts): 128 token rows x TN weight rows; a thread owns one token and stores runs of
// consecutive channels with 16-byte stores.
// The kernels hand the accumulators over through a `get` object:
//   get.template load<W>(plane, column, v)   W consecutive columns of one product plane
// which reads TMEM, the summed partials of a K-split cluster, or registers. All calls are warp-collective.
#pragma once

#include "fl_common.cuh"

namespace bxf {

constexpr int NROWS = 128;           // rows of the 128-row operand of a tile
constexpr int EPI_THREADS = 512;     // epilogue threads of the kernels with one CTA per SM (16 warps)

struct Tile {
  int group, n0;                     // weight plane, first weight row
  int row0, rows;                    // first token row, token rows that exist
};

// Runs of 32 bytes: one store (load) of a whole sector per thread when the address allows it.
__device__ __forceinline__ bool aligned32(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 31) == 0; }

__device__ __forceinline__ void store32(void* p, const uint32_t (&w)[8]) {
  asm volatile("st.global.v8.b32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8};" ::"l"(p), "r"(w[0]), "r"(w[1]), "r"(w[2]), "r"(w[3]),
               "r"(w[4]), "r"(w[5]), "r"(w[6]), "r"(w[7])
               : "memory");
}

__device__ __forceinline__ void load32(const void* p, uint32_t (&w)[8]) {
  asm volatile("ld.global.v8.b32 {%0, %1, %2, %3, %4, %5, %6, %7}, [%8];"
               : "=r"(w[0]), "=r"(w[1]), "=r"(w[2]), "=r"(w[3]), "=r"(w[4]), "=r"(w[5]), "=r"(w[6]), "=r"(w[7])
               : "l"(p)
               : "memory");
}

// The first n of 16 consecutive values.
__device__ __forceinline__ void store_run(bf16* p, const float (&v)[16], int n) {
  if (n == 16 && aligned32(p)) {
    uint32_t w[8];
#pragma unroll
    for (int k = 0; k < 8; ++k) w[k] = pack_bf16(v[2 * k], v[2 * k + 1]);
    store32(p, w);
  } else {
#pragma unroll
    for (int i = 0; i < 16; ++i)
      if (i < n) st(p + i, v[i]);
  }
}

__device__ __forceinline__ void store_run(float* p, const float (&v)[16], int n) {
  if (n == 16 && aligned32(p)) {
#pragma unroll
    for (int h = 0; h < 16; h += 8) {
      uint32_t w[8];
#pragma unroll
      for (int k = 0; k < 8; ++k) w[k] = __float_as_uint(v[h + k]);
      store32(p + h, w);
    }
  } else {
#pragma unroll
    for (int i = 0; i < 16; ++i)
      if (i < n) p[i] = v[i];
  }
}

// Eight consecutive values.
__device__ __forceinline__ void store_run8(bf16* p, const float (&v)[8], int n) {
  if (n == 8 && (reinterpret_cast<uintptr_t>(p) & 15) == 0) {
    *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
  } else {
#pragma unroll
    for (int i = 0; i < 8; ++i)
      if (i < n) st(p + i, v[i]);
  }
}

__device__ __forceinline__ void store_run8(float* p, const float (&v)[8], int n) {
#pragma unroll
  for (int i = 0; i < 8; ++i)
    if (i < n) p[i] = v[i];
}

// Fixed point at 24 bits.
__device__ __forceinline__ void store_run(i64* p, const float (&v)[16], int n) {
  i64 q[16];
#pragma unroll
  for (int i = 0; i < 16; ++i) q[i] = __double2ll_rn((double)v[i] * 16777216.0);
  if (n == 16 && aligned32(p)) {
#pragma unroll
    for (int h = 0; h < 16; h += 4) bx::st_global_v4(p + h, q[h], q[h + 1], q[h + 2], q[h + 3]);
  } else {
#pragma unroll
    for (int i = 0; i < 16; ++i)
      if (i < n) p[i] = q[i];
  }
}

__device__ __forceinline__ void add_run(float* p, const float (&v)[16], int n) {
  if (n == 16 && aligned32(p)) {
    uint32_t w[2][8];
    load32(p, w[0]);
    load32(p + 8, w[1]);
#pragma unroll
    for (int h = 0; h < 2; ++h) {
#pragma unroll
      for (int k = 0; k < 8; ++k) w[h][k] = __float_as_uint(__uint_as_float(w[h][k]) + v[8 * h + k]);
      store32(p + 8 * h, w[h]);
    }
  } else {
#pragma unroll
    for (int i = 0; i < 16; ++i)
      if (i < n) p[i] += v[i];
  }
}

__device__ __forceinline__ void epi_barrier() { asm volatile("bar.sync 1, 512;" ::: "memory"); }

// ---- elementwise epilogues (bxf_epilogue) ----
struct StageEpi {
  using Params = bxf_epilogue;
  static constexpr int PLANES = 1;
  // Small token tiles: 8 epilogue warps and half of an SM's shared memory, so that a CTA of the next tile or of the next
  // kernel of the step fetches its first weights while this one finishes.
  static __host__ __device__ constexpr int warps(int ta) { return ta <= 32 ? 8 : 16; }
  static __host__ __device__ constexpr int ctas(int ta) { return ta <= 32 ? 2 : 1; }
  static __host__ __device__ constexpr int stash_bytes(int) { return 0; }

  template <class T>
  static __device__ __forceinline__ void chunk(const Params& p, int group, int n, int N, i64 row, int cnt,
                                               const float (&v)[8]) {
    if (p.kind == BXF_EPI_ROPE) {
      const int r = n - p.n_main, j = r >= 0 ? r % p.rot_dim : 0, h = r >= 0 ? r / p.rot_dim : 0;
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const float other = __shfl_xor_sync(0xffffffffu, v[i], 1);
        if (i >= cnt || n >= N) continue;
        if (r < 0) {
          st(static_cast<T*>(p.out) + (row + i) * p.ldo + n, v[i]);
        } else {
          const float2 cs = *reinterpret_cast<const float2*>(p.cs + ((row + i) * (p.rot_dim / 2) + (j >> 1)) * 2);
          st(static_cast<T*>(p.rot_out) + (row + i) * p.ldr + h * p.hsr + j,
             (j & 1) ? v[i] * cs.x + other * cs.y : v[i] * cs.x - other * cs.y);
        }
      }
      return;
    }
    if (p.kind == BXF_EPI_GLU) {
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const float up = __shfl_xor_sync(0xffffffffu, v[i], 1);
        if (i < cnt && n < N && !(n & 1))
          st(static_cast<T*>(p.out) + (row + i) * p.ldo + (n >> 1), activate<T>(p.act, v[i], p.act_p, p.act_q) * up);
      }
      return;
    }
    if (n >= N) return;
    if (p.kind == BXF_EPI_ADD) {
      float* o = static_cast<float*>(p.out) + row * p.ldo + n;
      float old[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) old[i] = i < cnt ? o[i * p.ldo] : 0.0f;
#pragma unroll
      for (int i = 0; i < 8; ++i)
        if (i < cnt) o[i * p.ldo] = old[i] + v[i];
    } else if (p.kind == BXF_EPI_GATE) {
      T* o = static_cast<T*>(p.out) + group * p.gso + row * p.ldo + n;
#pragma unroll
      for (int i = 0; i < 8; ++i)
        if (i < cnt) st(o + i * p.ldo, v[i] * p.gate[(row + i) * p.ldg + group]);
    } else if (n >= p.n_main) {
      const float b = p.bias ? p.bias[n - p.n_main] : 0.0f;
      float* o = p.side + row * p.lds + (n - p.n_main);
#pragma unroll
      for (int i = 0; i < 8; ++i)
        if (i < cnt) o[i * p.lds] = v[i] + b;
    } else {
      const i64 at = group * p.gso + row * p.ldo + n;
      const float b = p.main_bias ? p.main_bias[n] : 0.0f;
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        if (i >= cnt) break;
        const float y = activate<T>(p.act, v[i] + b, p.act_p, p.act_q);
        if (p.out_type == BXF_OUT_T) st(static_cast<T*>(p.out) + at + i * p.ldo, y);
        else if (p.out_type == BXF_OUT_F32) static_cast<float*>(p.out)[at + i * p.ldo] = y;
        else static_cast<i64*>(p.out)[at + i * p.ldo] = __double2ll_rn((double)y * 16777216.0);
      }
    }
  }

  // Channels n .. n + cnt - 1 (n a multiple of 16) of token row m; v holds their accumulators.
  template <class T>
  static __device__ __forceinline__ void chunk_rows(const Params& p, int group, i64 m, int n, int cnt, float (&v)[16]) {
    if (p.kind == BXF_EPI_ADD) {
      add_run(static_cast<float*>(p.out) + m * p.ldo + n, v, cnt);
      return;
    }
    if (p.kind == BXF_EPI_GLU) {
      float o[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) o[i] = activate<T>(p.act, v[2 * i], p.act_p, p.act_q) * v[2 * i + 1];
      store_run8(static_cast<T*>(p.out) + m * p.ldo + (n >> 1), o, cnt >> 1);
      return;
    }
    int main_cnt = cnt;                                                 // of them, below n_main
    if (p.kind == BXF_EPI_GATE) {
      const float g = p.gate[m * p.ldg + group];
#pragma unroll
      for (int i = 0; i < 16; ++i) v[i] *= g;
    } else {
      main_cnt = min(cnt, p.n_main - n);
      if (main_cnt < cnt) {
#pragma unroll
        for (int i = 0; i < 16; i += 2) {                               // n_main is even where channels are rotated
          const int r = n + i - p.n_main;
          if (p.kind == BXF_EPI_ROPE) {
            if (i >= cnt || r < 0) continue;
            const int j = r % p.rot_dim;
            const float2 cs = *reinterpret_cast<const float2*>(p.cs + (m * (p.rot_dim / 2) + (j >> 1)) * 2);
            T* o = static_cast<T*>(p.rot_out) + m * p.ldr + r / p.rot_dim * p.hsr + j;
            st(o, v[i] * cs.x - v[i + 1] * cs.y);
            st(o + 1, v[i + 1] * cs.x + v[i] * cs.y);
          } else {
#pragma unroll
            for (int k = 0; k < 2; ++k)
              if (i + k < cnt && r + k >= 0) p.side[m * p.lds + r + k] = v[i + k] + (p.bias ? p.bias[r + k] : 0.0f);
          }
        }
      }
      if (main_cnt <= 0) return;
      if (p.main_bias) {
#pragma unroll
        for (int i = 0; i < 16; ++i)
          if (i < main_cnt) v[i] += p.main_bias[n + i];
      }
      if (p.act != BXF_ACT_NONE) {
#pragma unroll
        for (int i = 0; i < 16; ++i) v[i] = activate<T>(p.act, v[i], p.act_p, p.act_q);
      }
    }
    const i64 at = group * p.gso + m * p.ldo + n;
    if (p.out_type == BXF_OUT_I64) store_run(static_cast<i64*>(p.out) + at, v, main_cnt);
    else if (p.out_type == BXF_OUT_F32) store_run(static_cast<float*>(p.out) + at, v, main_cnt);
    else store_run(static_cast<T*>(p.out) + at, v, main_cnt);
  }

  // row: the thread's token row of the tile; the four warps of a lane quarter take 16 columns in turn.
  template <class T, int TN, class Get>
  static __device__ __forceinline__ void run_rows(Get& get, const Params& p, const Tile& t, int N, int row, int group_index) {
    for (int c = group_index * 16; c < TN && t.n0 + c < N; c += 64) {
      float v[16];
      get.template load<16>(0, c, v);
      if (row < t.rows) chunk_rows<T>(p, t.group, (i64)t.row0 + row, t.n0 + c, min(16, N - t.n0 - c), v);
    }
  }

  // Into L1 while the products run: the residual lines this thread's warp will add to.
  template <int TA>
  static __device__ __forceinline__ void prefetch(const Params& p, const Tile& t, int N, int row, int group_index, int groups) {
    if (p.kind != BXF_EPI_ADD || t.n0 + row >= N) return;
    for (int c = group_index * 8; c < TA && c < t.rows; c += groups * 8)
      for (int i = 0; i < min(8, t.rows - c); ++i)
        bx::prefetch_l1(static_cast<const float*>(p.out) + ((i64)t.row0 + c + i) * p.ldo + t.n0 + row);
  }

  // groups: how many warps share a row (they take chunks of 8 columns in turn).
  template <class T, int TA, int W, class Get>
  static __device__ __forceinline__ void run(Get& get, const Params& p, const Tile& t, int N, int row, int group_index,
                                             int groups, uint8_t*) {
    for (int c = group_index * 8; c < TA && c < t.rows; c += groups * 8) {
      float v[8];
      get.template load<8>(0, c, v);
      chunk<T>(p, t.group, t.n0 + row, N, (i64)t.row0 + c, min(8, t.rows - c), v);
    }
  }
};

// One minGRU gate pair: S_t = a S_(t-1) + b from the update and candidate pre-activations.
template <class T>
__device__ __forceinline__ void gru_gate(float z, float u, float& a, float& b) {
  float s;
  sigmoid_pair<T>(z, s, a);
  b = s * (u >= 0.0f ? u + 0.5f : sigmoid<T>(u));
}

// The first row of a sequence that does not start here: its state slot is read.
__device__ __forceinline__ bool gru_resumes(int flags) {
  return (flags & (BXF_ROW_FIRST | BXF_ROW_START | BXF_ROW_PAD)) == BXF_ROW_FIRST;
}

// ---- minGRU: gates and recurrence along the token columns, for rows that fit one tile ----
// The recurrence S_t = a_t S_(t-1) + b_t over a tile is a scan split over the warps of a row: every warp folds its
// columns to one (a, b) pair, the pairs of the warps before it give its start, and a second walk produces the states.
// At the first row of a sequence the state of its slot enters b and a becomes 0, so tiles need not know sequences.
// a and b of the first walk stay in shared memory for the second one (the slots of `state` may be rewritten by then).
struct GruEpi {
  using Params = bxf_gru;
  static constexpr int PLANES = 3;
  static __host__ __device__ constexpr int warps(int) { return 16; }
  static __host__ __device__ constexpr int ctas(int) { return 1; }
  static __host__ __device__ constexpr int stash_bytes(int ta) { return 2 * ta * NROWS * 4 + 16 * NROWS * 8; }

  // Into L1 while the products run: the states that the first rows of sequences start from.
  template <int TA>
  static __device__ __forceinline__ void prefetch(const Params& p, const Tile& t, int N, int row, int group_index, int groups) {
    const int per = TA / groups, c0 = group_index * per;
    for (int c = c0; c < min(c0 + per, t.rows); ++c)
      if (gru_resumes(p.flags[t.row0 + c]) && t.n0 + row < N)
        bx::prefetch_l1(p.state + p.seq[t.row0 + c] * N + t.n0 + row);
  }

  template <class T, int TA, int W, class Get>
  static __device__ __forceinline__ void run(Get& get, const Params& p, const Tile& t, int N, int row, int group_index,
                                             int groups, uint8_t* stash) {
    float* sa = reinterpret_cast<float*>(stash);                        // [TA][128]
    float* sb = sa + TA * NROWS;
    float2* fold = reinterpret_cast<float2*>(sb + TA * NROWS);          // [warp of the row][128]
    const int per = TA / groups, c_begin = group_index * per, c_end = min(c_begin + per, t.rows);
    const int n = t.n0 + row;
    const bool live = n < N;
    const float bz = live ? p.bias_z[n] : 0.0f, bx = live ? p.bias_x[n] : 0.0f;
    float A = 1.0f, B = 0.0f;
    for (int c = c_begin; c < c_end; c += W) {
      float z[W], u[W], start[W];
      int f[W];
#pragma unroll
      for (int i = 0; i < W; ++i) f[i] = c + i < c_end ? p.flags[t.row0 + c + i] : BXF_ROW_PAD;
#pragma unroll
      for (int i = 0; i < W; ++i)
        start[i] = live && gru_resumes(f[i]) ? p.state[p.seq[t.row0 + c + i] * N + n] : 0.0f;
      get.template load<W>(0, c, z);
      get.template load<W>(1, c, u);
#pragma unroll
      for (int i = 0; i < W; ++i) {
        if (c + i >= c_end) break;
        float a, b;
        gru_gate<T>(z[i] + bz, u[i] + bx, a, b);
        if (f[i] & BXF_ROW_FIRST) {
          b += a * start[i];
          a = 0.0f;
        }
        sa[(c + i) * NROWS + row] = a;
        sb[(c + i) * NROWS + row] = b;
        B = B * a + b;
        A *= a;
      }
    }
    fold[group_index * NROWS + row] = make_float2(A, B);
    epi_barrier();
    float S = 0.0f;
    for (int k = 0; k < group_index; ++k) {
      const float2 f = fold[k * NROWS + row];
      S = S * f.x + f.y;
    }
    for (int c = c_begin; c < c_end; c += W) {
      float g[W];
      get.template load<W>(2, c, g);
#pragma unroll
      for (int i = 0; i < W; ++i) {
        if (c + i >= c_end) break;
        S = S * sa[(c + i) * NROWS + row] + sb[(c + i) * NROWS + row];
        if (!live) continue;
        const i64 m = t.row0 + c + i;
        st(static_cast<T*>(p.out) + m * p.ldo + n, S * silu<T>(g[i]));
        if (p.flags[m] & BXF_ROW_LAST) p.state[p.seq[m] * N + n] = S;
      }
    }
  }
};

}  // namespace bxf
