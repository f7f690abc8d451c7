// Stages around the products of the models with several residual streams and grouped-query attention: the streams' mixing
// with the RMS norm of the next sublayer, rotation angles, and what happens to queries, keys and values between their
// projection and attention. All arithmetic is 32-bit.
#pragma once

#include "fl_stages.cuh"

namespace bxf {

// V consecutive values: 16-byte accesses for V = 8 (the address is aligned), single ones for V = 1.
template <int V>
__device__ __forceinline__ void load_v(const uint4& u, float (&v)[V]) {
  static_assert(V == 8, "eight bf16 values");
  const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    v[2 * i] = __uint_as_float(w[i] << 16);
    v[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
  }
}
template <int V>
__device__ __forceinline__ void load_v(const bf16* p, float (&v)[V]) {
  if constexpr (V == 8) {
    load_v<8>(*reinterpret_cast<const uint4*>(p), v);
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] = ld(p + i);
  }
}
template <int V>
__device__ __forceinline__ void load_v(const float* p, float (&v)[V]) {
  if constexpr (V % 4 == 0) {
#pragma unroll
    for (int i = 0; i < V; i += 4) {
      const float4 u = *reinterpret_cast<const float4*>(p + i);
      v[i] = u.x, v[i + 1] = u.y, v[i + 2] = u.z, v[i + 3] = u.w;
    }
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] = p[i];
  }
}
template <int V>
__device__ __forceinline__ void store_v(bf16* p, const float (&v)[V]) {
  if constexpr (V == 8) {
    *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) st(p + i, v[i]);
  }
}
template <int V>
__device__ __forceinline__ void store_v(float* p, const float (&v)[V]) {
  if constexpr (V % 4 == 0) {
#pragma unroll
    for (int i = 0; i < V; i += 4) *reinterpret_cast<float4*>(p + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) p[i] = v[i];
  }
}

// One row per CTA. Every thread keeps its entries of all streams in registers: the streams are read once and written once.
template <class T, int SM, int V>
__global__ void __launch_bounds__(NORM_THREADS) fl_streams_kernel(const bxf_streams_step p) {
  extern __shared__ float row[];
  __shared__ float c_in[SM], c_out[SM], c_mix[SM * SM], red[33];
  launch_next();
  const int S = p.streams, D = p.D;
  const bool update = !p.ids && p.y;
  if (threadIdx.x < S) {
    c_in[threadIdx.x] = p.in ? p.in[threadIdx.x] : 1.0f;
    if (update) c_out[threadIdx.x] = p.out[threadIdx.x];
  }
  if (update && threadIdx.x < S * S) c_mix[threadIdx.x] = p.mix[threadIdx.x];
  __syncthreads();
  wait_previous();
  const i64 m = blockIdx.x;
  float* xm = p.x + m * S * D;
  const T* em = nullptr;
  if (p.ids) {
    const i64 id = p.ids[m];
    em = static_cast<const T*>(p.embed) + (id < 0 || id >= p.vocab ? 0 : id) * D;
  }
  float sq = 0.0f;
  for (int d = threadIdx.x * V; d < D; d += NORM_THREADS * V) {
    float x[SM][V], u[V];
    if (em) {
      float e[V];
#pragma unroll
      for (int i = 0; i < V; ++i) e[i] = ld(em + d + i);
#pragma unroll
      for (int s = 0; s < SM; ++s)
#pragma unroll
        for (int i = 0; i < V; ++i) x[s][i] = e[i];
    } else {
#pragma unroll
      for (int s = 0; s < SM; ++s)
        if (s < S) load_v<V>(xm + s * D + d, x[s]);
    }
    if (update) {
      float y[V], n[SM][V];
      load_v<V>(p.y + m * D + d, y);
#pragma unroll
      for (int t = 0; t < SM; ++t) {
        if (t >= S) continue;
#pragma unroll
        for (int i = 0; i < V; ++i) n[t][i] = c_out[t] * y[i];
#pragma unroll
        for (int s = 0; s < SM; ++s)
          if (s < S)
#pragma unroll
            for (int i = 0; i < V; ++i) n[t][i] += c_mix[s * S + t] * x[s][i];
      }
#pragma unroll
      for (int t = 0; t < SM; ++t)
        if (t < S)
#pragma unroll
          for (int i = 0; i < V; ++i) x[t][i] = n[t][i];
    }
    if ((em || update) && p.h) {
#pragma unroll
      for (int s = 0; s < SM; ++s)
        if (s < S) store_v<V>(xm + s * D + d, x[s]);
    }
#pragma unroll
    for (int i = 0; i < V; ++i) u[i] = 0.0f;
#pragma unroll
    for (int s = 0; s < SM; ++s)
      if (s < S)
#pragma unroll
        for (int i = 0; i < V; ++i) u[i] += c_in[s] * x[s][i];
    if (p.sum) store_v<V>(p.sum + m * D + d, u);
    if (p.h) {
      store_v<V>(row + d, u);
#pragma unroll
      for (int i = 0; i < V; ++i) sq += u[i] * u[i];
    }
  }
  if (!p.h) return;
  const float r = 1.0f / sqrtf(block_sum(sq, red) / D + p.eps);
  T* h = static_cast<T*>(p.h) + m * p.ldh;
  for (int d = threadIdx.x * V; d < D; d += NORM_THREADS * V) {         // every thread meets its own entries again
    float v[V], w[V];
    load_v<V>(row + d, v);
    load_v<V>(p.w + d, w);
    if constexpr (V == 4) st4(h + d, v[0] * r * w[0], v[1] * r * w[1], v[2] * r * w[2], v[3] * r * w[3]);
    else st(h + d, v[0] * r * w[0]);
  }
}

__global__ void fl_angles_kernel(const double* __restrict__ freq, int half, const i64* pos, float* __restrict__ cs, i64 n) {
  launch_next();
  wait_previous();
  const i64 at = (i64)blockIdx.x * blockDim.x + threadIdx.x;
  if (at >= n) return;
  constexpr double TURN = 6.283185307179586476925;
  const double a = (double)pos[at / half] * freq[at % half];
  float s, c;
  sincosf((float)(a - rint(a / TURN) * TURN), &s, &c);
  reinterpret_cast<float2*>(cs)[at] = make_float2(c, s);
}

// One token per CTA.
template <class T, int V>
__global__ void __launch_bounds__(PREP_THREADS) fl_gqa_prepare_kernel(const bxf_gqa_rows p, int M) {
  launch_next();
  wait_previous();
  __shared__ float2 red[4];
  const i64 m = blockIdx.x;
  const int nq = p.heads * p.dim, nk = p.kv_heads * p.dim, nv = p.kv_heads * p.vdim, per = p.heads / p.kv_heads;
  const T* y = static_cast<const T*>(p.y) + m * p.ldy;
  float rq = 1.0f, rk = 1.0f;
  if (p.q_norm || p.k_norm) {
    float sq = 0.0f, sk = 0.0f;
    for (int e = threadIdx.x * V; e < nq + nk; e += PREP_THREADS * V) {
      float v[V], s = 0.0f;
      load_v<V>(y + e, v);
#pragma unroll
      for (int i = 0; i < V; ++i) s += v[i] * v[i];
      if (e < nq) sq += s;
      else sk += s;
    }
    const float2 sums = block_sum2(sq, sk, red);
    if (p.q_norm) rq = 1.0f / sqrtf(sums.x / nq + p.eps);
    if (p.k_norm) rk = 1.0f / sqrtf(sums.y / nk + p.eps);
  }
  const i64 slot = p.slot[m] < 0 ? 0 : p.slot[m];
  T* rows = static_cast<T*>(p.cache) + (slot / p.page * p.kv_heads * p.page + slot % p.page) * p.ldc;   // of group 0
  const i64 group_stride = p.page * p.ldc;
  const int half = p.rot_dims / 2;
  const float* cs = p.cs + m * half * 2;
  for (int e = threadIdx.x * V; e < nq + nk; e += PREP_THREADS * V) {
    const bool is_q = e < nq;
    const float r = is_q ? rq : rk;
    const float* w = is_q ? p.q_norm : p.k_norm ? p.k_norm - nq : nullptr;
    const int h = (is_q ? e : e - nq) / p.dim, d = (is_q ? e : e - nq) % p.dim;
    float v[V];
    const auto normed = [&](int at, float (&o)[V]) {
      load_v<V>(y + at, o);
#pragma unroll
      for (int i = 0; i < V; ++i) o[i] *= r;
      if (w) {
        float g[V];
        load_v<V>(w + at, g);
#pragma unroll
        for (int i = 0; i < V; ++i) o[i] *= g[i];
      }
    };
    normed(e, v);
    if (d < p.rot_dims) {
      float o[V];
      normed(d < half ? e + half : e - half, o);
      float c[2 * V];
      if constexpr (V == 8) {
        load_v<16>(cs + (d < half ? d : d - half) * 2, c);
      } else {
        c[0] = cs[(d < half ? d : d - half) * 2];
        c[1] = cs[(d < half ? d : d - half) * 2 + 1];
      }
#pragma unroll
      for (int i = 0; i < V; ++i) v[i] = d < half ? v[i] * c[2 * i] - o[i] * c[2 * i + 1] : v[i] * c[2 * i] + o[i] * c[2 * i + 1];
    }
    T* to = is_q ? static_cast<T*>(p.q) + (((i64)(h / per) * M + m) * per + h % per) * p.ldq + d : rows + h * group_stride + d;
    store_v<V>(to, v);
  }
  for (int e = threadIdx.x * V; e < nv; e += PREP_THREADS * V) {
    float v[V];
    load_v<V>(y + nq + nk + e, v);
    store_v<V>(rows + e / p.vdim * group_stride + p.voff + e % p.vdim, v);
  }
}

}  // namespace bxf
