// Attention over a paged cache, plain form: one CTA per (query row, head), any sizes, both element types. A cache row serves
// the H query heads of one of G groups: its key is the first W entries, its value the R entries from voff on. Latent
// attention has one group and [latent | rotated key part] rows whose values are part of the keys (voff 0); grouped-query
// attention has [key | value] rows. Keys j of a row at position i: max(0, i - window + 1) .. i. The running maximum starts
// at the head's sink with denominator 1, so the sink counts once and is never scaled.
#pragma once

#include "fl_common.cuh"

namespace bxf {

struct PagedAttn {
  const void* q;                       // [G][M][H] rows of ldq entries
  i64 ldq;
  int M, H, G, W, R, voff;             // H: heads of a group
  const void* cache;                   // [nb][G][bs] rows of ldc entries
  i64 ldc;
  int bs, nb;
  const void* bt;
  int bt64;
  i64 bt_stride;
  int nblk;
  const i64 *seq, *pos;
  const int* tiles;
  int ntiles, window;
  const float* sink;
  float scale;
  void* out;                           // token m, head h (of all): out + m * out_tok + h * out_head
  i64 out_tok, out_head;

  // The page that holds key block `page` of table row `s`.
  __device__ __forceinline__ i64 page_of(i64 s, int page) const {
    const i64 at = s * bt_stride + page;
    const i64 b = bt64 ? static_cast<const i64*>(bt)[at] : static_cast<const int*>(bt)[at];
    return b < 0 || b >= nb ? 0 : b;
  }
  __device__ __forceinline__ int first_key(i64 p) const { return window > 0 && p >= window ? (int)(p - window + 1) : 0; }
};

constexpr int LA_THREADS = 128, LA_KEYS = 128, LA_MAX_R = 1024;

template <class T>
__global__ void __launch_bounds__(LA_THREADS) fl_paged_attention_kernel(const PagedAttn a) {
  extern __shared__ float la_q[];                        // [W]
  __shared__ float p[LA_KEYS], red[2][4];
  __shared__ i64 krow[LA_KEYS];
  const int m = blockIdx.x, h = blockIdx.y, g = h / a.H, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int W = a.W;
  const T* q = static_cast<const T*>(a.q) + (((i64)g * a.M + m) * a.H + h % a.H) * a.ldq;
  const T* cache = static_cast<const T*>(a.cache);
  for (int d = tid; d < W; d += LA_THREADS) la_q[d] = ld(q + d);
  const i64 pos = min(a.pos[m], (i64)a.nblk * a.bs - 1), s = a.seq[m];
  float mx = a.sink ? a.sink[h] : -INFINITY, den = a.sink ? 1.0f : 0.0f;
  float acc[LA_MAX_R / LA_THREADS];
#pragma unroll
  for (int j = 0; j < LA_MAX_R / LA_THREADS; ++j) acc[j] = 0.0f;
  __syncthreads();
  for (int k0 = a.first_key(pos); k0 <= pos; k0 += LA_KEYS) {
    const int n = min(LA_KEYS, (int)(pos - k0 + 1));
    if (tid < n) krow[tid] = ((a.page_of(s, (k0 + tid) / a.bs) * a.G + g) * a.bs + (k0 + tid) % a.bs) * a.ldc;
    __syncthreads();
    float best = -INFINITY;
    for (int k = warp; k < n; k += 4) {
      const T* c = cache + krow[k];
      float v = 0.0f;
      for (int d = lane; d < W; d += 32) v = fmaf(la_q[d], ld(c + d), v);
      v = warp_sum(v) * a.scale;
      if (lane == 0) p[k] = v;
      best = fmaxf(best, v);
    }
    if (lane == 0) red[0][warp] = best;
    __syncthreads();
    const float m2 = fmaxf(fmaxf(mx, fmaxf(red[0][0], red[0][1])), fmaxf(red[0][2], red[0][3]));
    const float corr = mx == -INFINITY ? 0.0f : expf(mx - m2);
    const float e = tid < n ? expf(p[tid] - m2) : 0.0f;
    const float part = warp_sum(e);
    if (lane == 0) red[1][warp] = part;
    if (tid < n) p[tid] = e;
    __syncthreads();
    den = den * corr + ((red[1][0] + red[1][1]) + (red[1][2] + red[1][3]));
    mx = m2;
#pragma unroll
    for (int j = 0; j < LA_MAX_R / LA_THREADS; ++j) {
      const int d = tid + j * LA_THREADS;
      if (d >= a.R) break;
      float o = acc[j] * corr;
      for (int k = 0; k < n; ++k) o = fmaf(p[k], ld(cache + krow[k] + a.voff + d), o);
      acc[j] = o;
    }
    __syncthreads();                                     // p and krow are rewritten by the next block of keys
  }
  T* o = static_cast<T*>(a.out) + m * a.out_tok + h * a.out_head;
#pragma unroll
  for (int j = 0; j < LA_MAX_R / LA_THREADS; ++j)
    if (tid + j * LA_THREADS < a.R) st(o + tid + j * LA_THREADS, acc[j] / den);
}

}  // namespace bxf
