// Memory-bound stages of the float models: row flags, embedding / expert combination + layer norm, expert routing and
// gathering, the preparation of latent attention, long minGRU scans. All arithmetic is 32-bit.
#pragma once

#include "fl_epilogue.cuh"

namespace bxf {

__global__ void fl_row_flags_kernel(const i64* seq, const i64* slot, const i64* pos, int* flags, int M) {
  launch_next();
  wait_previous();
  const int m = blockIdx.x * blockDim.x + threadIdx.x;
  if (m >= M) return;
  if (slot[m] < 0) {
    flags[m] = BXF_ROW_PAD | BXF_ROW_FIRST;
    return;
  }
  const bool first = m == 0 || seq[m - 1] != seq[m] || slot[m - 1] < 0;
  const bool last = m == M - 1 || seq[m + 1] != seq[m] || slot[m + 1] < 0;
  flags[m] = (first ? BXF_ROW_FIRST : 0) | (last ? BXF_ROW_LAST : 0) | (pos[m] == 0 ? BXF_ROW_START : 0);
}

constexpr int NORM_THREADS = 256;

// One row per CTA; the row stays in shared memory between the passes.
template <class T>
__global__ void __launch_bounds__(NORM_THREADS)
fl_norm_kernel(float* __restrict__ x, const i64* ids, const T* __restrict__ embed, i64 V, const float* __restrict__ y,
               const int* __restrict__ place, const float* __restrict__ weight, int top, const float* __restrict__ w,
               const float* __restrict__ b, float eps, T* __restrict__ h, i64 ldh, int* zero, int nzero, int D) {
  launch_next();
  wait_previous();
  extern __shared__ float row[];
  __shared__ float red[33];
  const i64 m = blockIdx.x;
  float* xm = x + m * D;
  if (blockIdx.x == 0)
    for (int i = threadIdx.x; i < nzero; i += NORM_THREADS) zero[i] = 0;
  const T* em = nullptr;
  if (ids) {
    const i64 id = ids[m];
    em = embed + (id < 0 || id >= V ? 0 : id) * D;
  }
  float s = 0.0f;
  if (D % 4 == 0) {
    for (int d = threadIdx.x * 4; d < D; d += NORM_THREADS * 4) {
      float4 v;
      if (em) {
        v = make_float4(ld(em + d), ld(em + d + 1), ld(em + d + 2), ld(em + d + 3));
      } else {
        v = *reinterpret_cast<const float4*>(xm + d);
        for (int k = 0; k < top; ++k) {
          const float wk = weight[m * top + k];
          const float4 e = *reinterpret_cast<const float4*>(y + (i64)place[m * top + k] * D + d);
          v.x += wk * e.x;
          v.y += wk * e.y;
          v.z += wk * e.z;
          v.w += wk * e.w;
        }
      }
      if (em || top) *reinterpret_cast<float4*>(xm + d) = v;
      *reinterpret_cast<float4*>(row + d) = v;
      s += (v.x + v.y) + (v.z + v.w);
    }
  } else {
    for (int d = threadIdx.x; d < D; d += NORM_THREADS) {
      float v = em ? ld(em + d) : xm[d];
      if (!em)
        for (int k = 0; k < top; ++k) v += weight[m * top + k] * y[(i64)place[m * top + k] * D + d];
      if (em || top) xm[d] = v;
      row[d] = v;
      s += v;
    }
  }
  if (!h) return;
  const float mean = block_sum(s, red) / D;
  float q = 0.0f;
  if (D % 4 == 0) {                                      // every thread meets its own entries again: no barrier needed
    for (int d = threadIdx.x * 4; d < D; d += NORM_THREADS * 4) {
      const float4 v = *reinterpret_cast<const float4*>(row + d);
      const float c0 = v.x - mean, c1 = v.y - mean, c2 = v.z - mean, c3 = v.w - mean;
      q += (c0 * c0 + c1 * c1) + (c2 * c2 + c3 * c3);
    }
  } else {
    for (int d = threadIdx.x; d < D; d += NORM_THREADS) {
      const float c = row[d] - mean;
      q += c * c;
    }
  }
  const float r = 1.0f / sqrtf(block_sum(q, red) / D + eps);
  if (D % 4 == 0) {
    for (int d = threadIdx.x * 4; d < D; d += NORM_THREADS * 4) {
      const float4 v = *reinterpret_cast<const float4*>(row + d), g = *reinterpret_cast<const float4*>(w + d),
                   c = *reinterpret_cast<const float4*>(b + d);
      st4(h + m * ldh + d, (v.x - mean) * r * g.x + c.x, (v.y - mean) * r * g.y + c.y, (v.z - mean) * r * g.z + c.z,
          (v.w - mean) * r * g.w + c.w);
    }
  } else {
    for (int d = threadIdx.x; d < D; d += NORM_THREADS) st(h + m * ldh + d, (row[d] - mean) * r * w[d] + b[d]);
  }
}

// One warp per row: `top` rounds of (largest, lowest index first).
__global__ void fl_route_kernel(const float* __restrict__ logits, i64 ldl, int E, int top, int* chosen, float* weight,
                                int* rank, int* counts, int M) {
  launch_next();
  wait_previous();
  const int m = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (m >= M) return;
  const float* z = logits + m * ldl;
  constexpr int PER = BXF_MAX_EXPERTS / 32;
  uint32_t taken = 0;                                    // bit j: expert j * 32 + lane is chosen already
  float mine = 0.0f, first = 0.0f, sum = 0.0f;           // lane k keeps the k-th choice
  int pick = 0;
  for (int k = 0; k < top; ++k) {
    float best = -INFINITY;
    int at = E;
    for (int j = 0; j < PER && j * 32 + lane < E; ++j) {
      const float v = z[j * 32 + lane];
      if (!(taken >> j & 1) && (v > best || at == E)) {
        best = v;
        at = j * 32 + lane;
      }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float bo = __shfl_xor_sync(0xffffffffu, best, o);
      const int ao = __shfl_xor_sync(0xffffffffu, at, o);
      if (ao < E && (at >= E || bo > best || (bo == best && ao < at))) {
        best = bo;
        at = ao;
      }
    }
    if (k == 0) first = best;
    const float e = expf(best - first);
    sum += e;
    if (lane == k) {
      mine = e;
      pick = at;
    }
    if (lane == (at & 31)) taken |= 1u << (at >> 5);
  }
  if (lane < top) {
    chosen[m * top + lane] = pick;
    weight[m * top + lane] = mine / sum;
    rank[m * top + lane] = atomicAdd(counts + pick, 1);
  }
}

// One CTA per (row, choice): its place in expert order, and the copy of the row.
template <class T>
__global__ void __launch_bounds__(128)
fl_gather_kernel(const T* __restrict__ h, i64 ldh, int D, const int* chosen, const int* rank, const int* counts, int top,
                 T* __restrict__ hp, int* place) {
  launch_next();
  wait_previous();
  __shared__ int base;
  const int pair = blockIdx.x, e = chosen[pair];
  if (threadIdx.x < 32) {
    int s = 0;
    for (int i = threadIdx.x; i < e; i += 32) s += counts[i];
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
    if (threadIdx.x == 0) {
      base = s + rank[pair];
      place[pair] = base;
    }
  }
  __syncthreads();
  const T* src = h + (i64)(pair / top) * ldh;
  T* dst = hp + (i64)base * ldh;
  constexpr int V = 16 / sizeof(T);
  if (ldh % V == 0) {                                    // the tail of a row lies inside its leading dimension
    for (int d = threadIdx.x * V; d < D; d += blockDim.x * V)
      *reinterpret_cast<uint4*>(dst + d) = *reinterpret_cast<const uint4*>(src + d);
  } else {
    for (int d = threadIdx.x; d < D; d += blockDim.x) dst[d] = src[d];
  }
}

constexpr int PREP_THREADS = 128;

// Two sums over the block of PREP_THREADS threads in one exchange.
__device__ __forceinline__ float2 block_sum2(float a, float b, float2* red) {
  a = warp_sum(a);
  b = warp_sum(b);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = make_float2(a, b);
  __syncthreads();
  return make_float2((red[0].x + red[1].x) + (red[2].x + red[3].x), (red[0].y + red[1].y) + (red[2].y + red[3].y));
}

template <class T>
__global__ void __launch_bounds__(PREP_THREADS)
fl_latent_prepare_kernel(const float* __restrict__ y, i64 ldy, int q_rank, int R, int rot, int H,
                         const float* __restrict__ wq, const float* __restrict__ wkv, float eps,
                         const float* __restrict__ freq, const i64* pos, const i64* slot, T* __restrict__ cq, i64 ldcq,
                         T* __restrict__ cache, i64 ldc, float* __restrict__ cs, float* __restrict__ gate) {
  launch_next();
  wait_previous();
  __shared__ float2 red[4];
  const i64 m = blockIdx.x;
  const float* ym = y + m * ldy;
  const float* yc = ym + q_rank;
  const float* yr = yc + R;
  T* row = cache + (slot[m] < 0 ? 0 : slot[m]) * ldc;
  float sq = 0.0f, sk = 0.0f;
  for (int d = threadIdx.x; d < q_rank; d += PREP_THREADS) sq += ym[d] * ym[d];
  for (int d = threadIdx.x; d < R; d += PREP_THREADS) sk += yc[d] * yc[d];
  const float2 sums = block_sum2(sq, sk, red);
  const float rq = 1.0f / sqrtf(sums.x / q_rank + eps), rk = 1.0f / sqrtf(sums.y / R + eps);
  for (int d = threadIdx.x; d < q_rank; d += PREP_THREADS) st(cq + m * ldcq + d, ym[d] * rq * wq[d]);
  for (int d = threadIdx.x; d < R; d += PREP_THREADS) st(row + d, yc[d] * rk * wkv[d]);
  const float p = (float)pos[m];
  for (int i = threadIdx.x; i < rot / 2; i += PREP_THREADS) {
    float s, c;
    sincosf(p * freq[i], &s, &c);
    cs[(m * (rot / 2) + i) * 2] = c;
    cs[(m * (rot / 2) + i) * 2 + 1] = s;
    const float u = yr[2 * i], v = yr[2 * i + 1];
    st(row + R + 2 * i, u * c - v * s);
    st(row + R + 2 * i + 1, v * c + u * s);
  }
  for (int i = threadIdx.x; i < H; i += PREP_THREADS) gate[m * H + i] = sigmoid<float>(yr[rot + i]);
}

// ---- minGRU over more rows than a product tile takes: y float [M, 3 width] holds the three products, the rows are scanned
// in chunks side by side. The first kernel folds every chunk to S -> A S + B; the second folds the chunks before its own to
// the state it starts from and produces the outputs. Only the first kernel reads state slots: it leaves a first row's
// finished b in place of the row's update pre-activation, since the second kernel's last rows rewrite the slots.
// One thread per channel; rows are read ahead in batches. ----
constexpr int GRU_BATCH = 8;

template <class T, bool APPLY>
__device__ __forceinline__ void gru_rows(const bxf_gru& g, float* __restrict__ y, int width, int n, int m0, int m1,
                                         float& A, float& S) {
  const float bz = g.bias_z[n], bx = g.bias_x[n];
  const i64 ldy = 3 * (i64)width;
  for (int m = m0; m < m1; m += GRU_BATCH) {
    float z[GRU_BATCH], u[GRU_BATCH], x[GRU_BATCH];                     // x: output gate, or the state a first row resumes
    int f[GRU_BATCH];
#pragma unroll
    for (int i = 0; i < GRU_BATCH; ++i) {
      const bool in = m + i < m1;
      const float* row = y + (m + i) * ldy + n;
      f[i] = in ? g.flags[m + i] : 0;
      z[i] = in ? row[0] : 0.0f;
      u[i] = in ? row[width] : 0.0f;
      if (APPLY) x[i] = in ? row[2 * width] : 0.0f;
    }
    if (!APPLY) {
#pragma unroll
      for (int i = 0; i < GRU_BATCH; ++i) x[i] = gru_resumes(f[i]) ? g.state[g.seq[m + i] * width + n] : 0.0f;
    }
#pragma unroll
    for (int i = 0; i < GRU_BATCH; ++i) {
      if (m + i >= m1) break;
      float a, b;
      if (APPLY && (f[i] & BXF_ROW_FIRST)) {
        a = 0.0f;
        b = z[i];
      } else {
        gru_gate<T>(z[i] + bz, u[i] + bx, a, b);
        if (f[i] & BXF_ROW_FIRST) {
          b += a * x[i];
          a = 0.0f;
          y[(m + i) * ldy + n] = b;
        }
      }
      S = S * a + b;
      A *= a;
      if (APPLY) {
        st(static_cast<T*>(g.out) + (i64)(m + i) * g.ldo + n, S * silu<T>(x[i]));
        if (f[i] & BXF_ROW_LAST) g.state[g.seq[m + i] * width + n] = S;
      }
    }
  }
}

template <class T>
__global__ void __launch_bounds__(128)
fl_gru_fold_kernel(const bxf_gru g, float* y, float2* fold, int M, int width, int chunk) {
  launch_next();
  wait_previous();
  const int n = blockIdx.x * 128 + threadIdx.x, j = blockIdx.y;
  if (n >= width) return;
  float A = 1.0f, S = 0.0f;
  gru_rows<T, false>(g, y, width, n, j * chunk, min(M, (j + 1) * chunk), A, S);
  fold[(i64)j * width + n] = make_float2(A, S);
}

template <class T>
__global__ void __launch_bounds__(128)
fl_gru_apply_kernel(const bxf_gru g, float* y, const float2* fold, int M, int width, int chunk) {
  launch_next();
  wait_previous();
  const int n = blockIdx.x * 128 + threadIdx.x, j = blockIdx.y;
  if (n >= width) return;
  float A = 1.0f, S = 0.0f;
  if (!(g.flags[j * chunk] & BXF_ROW_FIRST))
    for (int i = 0; i < j; ++i) {
      const float2 f = fold[(i64)i * width + n];
      S = S * f.x + f.y;
    }
  gru_rows<T, true>(g, y, width, n, j * chunk, min(M, (j + 1) * chunk), A, S);
}

}  // namespace bxf
