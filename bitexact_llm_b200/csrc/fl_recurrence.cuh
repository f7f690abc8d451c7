// Recurrent layers with a matrix state per head: S_t = diag(a_t) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t, with one decay per key
// channel (gated linear attention) or per head (Mamba-2, whose q, k, v pass a causal convolution first), and the gate + norm
// that follows. Decays, step sizes and states are 32-bit everywhere.
#pragma once

#include "fl_streams.cuh"

namespace bxf {

__device__ __forceinline__ float softplus(float v) { return fmaxf(v, 0.0f) + log1pf(expf(-fabsf(v))); }

// ---- causal convolution ----
// One channel of one row; rows of the step behind the first row of the sequence come from its state.
template <class T>
__device__ __forceinline__ float conv_at(const bxf_conv& c, int m, int ch) {
  const T* u = static_cast<const T*>(c.u) + ch;
  const i64 pos = c.pos[m];
  float acc = c.b[ch];
  int first = -1;                                        // rows back to the sequence's first row of the step
  for (int back = 0; back < c.taps && back <= pos; ++back) {
    float v;
    if (first < 0) {
      v = ld(u + (i64)(m - back) * c.ldu);
      if (c.flags[m - back] & BXF_ROW_FIRST) first = back;
    } else {
      v = ld(static_cast<const T*>(c.state) + (c.seq[m] * (c.taps - 1) + first - back + c.taps - 1) * c.channels + ch);
    }
    acc = fmaf(c.w[ch * c.taps + c.taps - 1 - back], v, acc);
  }
  return silu<T>(acc);
}

constexpr int CONV_ROWS = 16, CONV_THREADS = 128;

// Prompts: a thread walks CONV_ROWS rows of 8 channels with the last TAPS inputs in registers.
template <int TAPS>
__global__ void __launch_bounds__(CONV_THREADS) fl_causal_conv_rows_kernel(const bxf_conv c, bf16* __restrict__ out, i64 ldo, int M) {
  launch_next();
  const int ch = (blockIdx.x * CONV_THREADS + threadIdx.x) * 8;
  if (ch >= c.channels) return;
  float w[TAPS][8], b[8], win[TAPS][8];
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    b[i] = c.b[ch + i];
#pragma unroll
    for (int j = 0; j < TAPS; ++j) w[j][i] = c.w[(ch + i) * TAPS + j];
  }
  wait_previous();
  const int m0 = blockIdx.y * CONV_ROWS, m1 = min(M, m0 + CONV_ROWS);
  const bf16* u = static_cast<const bf16*>(c.u) + ch;
  for (int m = m0; m < m1; ++m) {
    const int f = c.flags[m];
    if (f & BXF_ROW_PAD) continue;
    if (m == m0 || (f & BXF_ROW_FIRST)) {                // the inputs before this row: rows of the step, the state, zeros
      int first = (f & BXF_ROW_FIRST) ? 0 : -1;
#pragma unroll
      for (int back = 1; back < TAPS; ++back) {
        float (&v)[8] = win[TAPS - 1 - back];
        if (back > c.pos[m]) {
#pragma unroll
          for (int i = 0; i < 8; ++i) v[i] = 0.0f;
        } else if (first < 0) {
          load_v<8>(u + (i64)(m - back) * c.ldu, v);
          if (c.flags[m - back] & BXF_ROW_FIRST) first = back;
        } else {
          load_v<8>(static_cast<const bf16*>(c.state) + (c.seq[m] * (TAPS - 1) + first - back + TAPS - 1) * c.channels + ch, v);
        }
      }
    }
    load_v<8>(u + (i64)m * c.ldu, win[TAPS - 1]);
    float o[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      o[i] = b[i];
#pragma unroll
      for (int j = 0; j < TAPS; ++j) o[i] = fmaf(w[j][i], win[j][i], o[i]);
      o[i] = silu<bf16>(o[i]);
    }
    store_v<8>(out + m * ldo + ch, o);
#pragma unroll
    for (int j = 0; j + 1 < TAPS; ++j)
#pragma unroll
      for (int i = 0; i < 8; ++i) win[j][i] = win[j + 1][i];
  }
}

template <class T>
__global__ void __launch_bounds__(CONV_THREADS) fl_causal_conv_kernel(const bxf_conv c, T* __restrict__ out, i64 ldo, int M) {
  launch_next();
  wait_previous();
  for (int k = 0; k < 2; ++k) {
    const int ch = blockIdx.x * 2 * CONV_THREADS + k * CONV_THREADS + threadIdx.x;
    if (ch >= c.channels) return;
    for (int m = blockIdx.y * CONV_ROWS; m < min(M, (int)(blockIdx.y + 1) * CONV_ROWS); ++m)
      if (!(c.flags[m] & BXF_ROW_PAD)) st(out + m * ldo + ch, conv_at<T>(c, m, ch));
  }
}

// The state after the step: the last taps - 1 inputs of the sequence that ends in row m.
template <class T>
__device__ __forceinline__ void conv_advance(const bxf_conv& c, int m) {
  const int R = c.taps - 1;
  int n = 1;                                             // rows of the step among them
  while (n < R && !(c.flags[m - n + 1] & BXF_ROW_FIRST)) ++n;
  T* state = static_cast<T*>(c.state) + c.seq[m] * R * c.channels;
  const T* u = static_cast<const T*>(c.u);
  for (int ch = threadIdx.x; ch < c.channels; ch += blockDim.x)
    for (int e = 0; e < R; ++e)
      state[(i64)e * c.channels + ch] = e < R - n ? state[(i64)(e + n) * c.channels + ch] : u[(i64)(m - (R - 1 - e)) * c.ldu + ch];
}

// ---- the recurrence row by row: decoding, short portions, 32-bit, any sizes ----
// One CTA per (sequence of the step, head, 32 value columns) walks the sequence's rows with its part of the state in
// registers: thread = 4 columns x every 32nd key channel. Rows are prepared in shared memory a few at a time.
constexpr int REC_THREADS = 256, REC_COLS = 32, REC_LANES = 32, REC_ROWS = 8;

__host__ __device__ constexpr int recurrence_smem(int K, bool channel) {
  return (REC_ROWS * K * (channel ? 3 : 2) + REC_ROWS * REC_COLS * 9 + REC_ROWS * 2) * 4;
}

template <class T, bool CHANNEL, int KR>
__global__ void __launch_bounds__(REC_THREADS) fl_recurrence_kernel(const bxf_recurrence_rows p, int M) {
  launch_next();
  wait_previous();
  extern __shared__ float rec_smem[];
  const int m0 = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * REC_COLS, tid = threadIdx.x;
  const int f0 = p.flags[m0];
  if ((f0 & (BXF_ROW_FIRST | BXF_ROW_PAD)) != BXF_ROW_FIRST) return;
  const int K = p.K, V = p.V, g = h / (p.heads / p.groups);
  float* sv = rec_smem;                                  // [rows][32]
  float* red = sv + REC_ROWS * REC_COLS;                 // [rows][8 warps][32]
  float* s_dt = red + REC_ROWS * 8 * REC_COLS;           // [rows] step size and decay of the head
  float* s_dec = s_dt + REC_ROWS;
  float* sq = s_dec + REC_ROWS;                          // [rows][K]
  float* sk = sq + REC_ROWS * K;
  float* sa = sk + REC_ROWS * K;                         // CHANNEL: decays
  const int cx = (tid & 7) * 4, kl = tid >> 3, col = c0 + cx;
  float* state = p.state + ((p.seq[m0] * p.heads + h) * K) * (i64)V + col;
  const bool fresh = f0 & BXF_ROW_START, wide = V % 4 == 0 && col < V;
  float s[KR][4];
#pragma unroll
  for (int j = 0; j < KR; ++j) {
    const int k = j * REC_LANES + kl;
#pragma unroll
    for (int i = 0; i < 4; ++i) s[j][i] = 0.0f;
    if (fresh || k >= K) continue;
    if (wide) {
      load_v<4>(state + (i64)k * V, s[j]);
    } else {
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (col + i < V) s[j][i] = state[(i64)k * V + i];
    }
  }
  const auto value = [&](int m, int column) {
    return !CHANNEL && p.conv.w ? conv_at<T>(p.conv, m, column - min(p.q0, min(p.k0, p.v0)))
                                : ld(static_cast<const T*>(p.y) + m * p.ldy + column);
  };
  for (int m = m0;;) {
    int n = 0;
    bool end = false;
    while (n < REC_ROWS && !end) end = p.flags[m + n++] & BXF_ROW_LAST;
    for (int at = tid; at < n * K; at += REC_THREADS) {
      const int r = at / K, k = at % K;
      sq[r * K + k] = value(m + r, p.q0 + g * K + k) * (CHANNEL ? p.q_scale : 1.0f);
      sk[r * K + k] = value(m + r, p.k0 + g * K + k);
    }
    for (int at = tid; at < n * REC_COLS; at += REC_THREADS) {
      const int c = at % REC_COLS;
      sv[at] = c0 + c < V ? value(m + at / REC_COLS, p.v0 + h * V + c0 + c) : 0.0f;
    }
    if (CHANNEL) {
      for (int k = tid; k < K; k += REC_THREADS) {
        const float* a2 = p.a2 + ((i64)h * K + k) * p.rank;
        const float b = p.a2_b[h * K + k];
        float z[REC_ROWS];
#pragma unroll
        for (int r = 0; r < REC_ROWS; ++r) z[r] = b;
        for (int j = 0; j < p.rank; ++j) {
          const float w = a2[j];
#pragma unroll
          for (int r = 0; r < REC_ROWS; ++r)
            if (r < n) z[r] = fmaf(w, p.side[(m + r) * p.lds + j], z[r]);
        }
#pragma unroll
        for (int r = 0; r < REC_ROWS; ++r)
          if (r < n) sa[r * K + k] = expf(-softplus(-z[r]) * p.inv_tau);
      }
    } else if (tid < n) {
      const float dt = softplus(p.side[(m + tid) * p.lds + h]);
      s_dt[tid] = dt;
      s_dec[tid] = expf(-expf(p.A_log[h]) * dt);
    }
    __syncthreads();
    for (int r = 0; r < n; ++r) {
      const float4 x = *reinterpret_cast<const float4*>(sv + r * REC_COLS + cx);
      const float dt = CHANNEL ? 1.0f : s_dt[r], dec = CHANNEL ? 1.0f : s_dec[r];
      const float v[4] = {x.x * dt, x.y * dt, x.z * dt, x.w * dt};
      float o[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
      for (int j = 0; j < KR; ++j) {
        const int k = j * REC_LANES + kl;
        if (k < K) {
          const float a = CHANNEL ? sa[r * K + k] : dec, kv = sk[r * K + k], qv = sq[r * K + k];
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            s[j][i] = fmaf(kv, v[i], a * s[j][i]);
            o[i] = fmaf(qv, s[j][i], o[i]);
          }
        }
      }
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        o[i] += __shfl_xor_sync(0xffffffffu, o[i], 8);
        o[i] += __shfl_xor_sync(0xffffffffu, o[i], 16);
      }
      if ((tid & 31) < 8) store_v<4>(red + (r * 8 + (tid >> 5)) * REC_COLS + cx, o);
    }
    __syncthreads();
    for (int at = tid; at < n * REC_COLS; at += REC_THREADS) {
      const int r = at / REC_COLS, c = at % REC_COLS;
      if (c0 + c >= V) continue;
      float o = 0.0f;
#pragma unroll
      for (int w = 0; w < 8; ++w) o += red[(r * 8 + w) * REC_COLS + c];
      if (!CHANNEL) o = fmaf(p.skip[h], sv[at], o);
      st(static_cast<T*>(p.out) + (m + r) * p.ldo + (i64)h * V + c0 + c, o);
    }
    if (end) break;
    m += n;
    __syncthreads();                                     // the next rows overwrite sv
  }
#pragma unroll
  for (int j = 0; j < KR; ++j) {
    const int k = j * REC_LANES + kl;
    if (k >= K) continue;
    if (wide) {
      store_v<4>(state + (i64)k * V, s[j]);
    } else {
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (col + i < V) state[(i64)k * V + i] = s[j][i];
    }
  }
}

// ---- gate and norm ----
// A part is normed by a warp (WARP: 8 parts per CTA) or by a CTA. The last CTA of a row advances the convolution's state.
constexpr int GATE_THREADS = 256;

template <class T, bool WARP, int V>
__global__ void __launch_bounds__(GATE_THREADS) fl_gated_norm_kernel(const bxf_gate_rows p, int part_ctas) {
  launch_next();
  wait_previous();
  __shared__ float red[33];
  const i64 m = blockIdx.x;
  if ((int)blockIdx.y == part_ctas) {
    if ((p.conv.flags[m] & (BXF_ROW_LAST | BXF_ROW_PAD)) == BXF_ROW_LAST) conv_advance<T>(p.conv, (int)m);
    return;
  }
  const int size = p.n / p.parts, part = WARP ? blockIdx.y * (GATE_THREADS / 32) + (threadIdx.x >> 5) : blockIdx.y;
  const int lane = WARP ? threadIdx.x & 31 : threadIdx.x, lanes = WARP ? 32 : GATE_THREADS;
  if (WARP && part >= p.parts) return;
  const int at = part * size;
  const T* o = static_cast<const T*>(p.o) + m * p.ldo + at;
  const T* z = static_cast<const T*>(p.z) + m * p.ldz + at;
  T* out = static_cast<T*>(p.out) + m * p.ldout + at;
  float sq = 0.0f;
  for (int e = lane * V; e < size; e += lanes * V) {
    float v[V], g[V];
    load_v<V>(o + e, v);
    if (p.gate_first) load_v<V>(z + e, g);
#pragma unroll
    for (int i = 0; i < V; ++i) {
      if (p.gate_first) v[i] *= silu<T>(g[i]);
      sq += v[i] * v[i];
    }
  }
  sq = WARP ? warp_sum(sq) : block_sum(sq, red);
  const float r = 1.0f / sqrtf(sq / size + p.eps);
  for (int e = lane * V; e < size; e += lanes * V) {
    float v[V], g[V], w[V];
    load_v<V>(o + e, v);
    load_v<V>(z + e, g);
    load_v<V>(p.w + (at + e) % p.wn, w);
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] = v[i] * silu<T>(g[i]) * r * w[i];
    store_v<V>(out + e, v);
  }
}

}  // namespace bxf
