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
    acc = fmaf(c.w[(i64)(c.taps - 1 - back) * c.channels + ch], v, acc);
  }
  return silu<T>(acc);
}

constexpr int CONV_ROWS = 16, CONV_THREADS = 128, CONV_BATCH = 4;

// A thread walks up to CONV_ROWS rows (`rows`) of 8 channels with the last TAPS inputs in registers; the rows are read ahead
// a few at a time.
template <int TAPS>
__global__ void __launch_bounds__(CONV_THREADS)
fl_causal_conv_rows_kernel(const bxf_conv c, bf16* __restrict__ out, i64 ldo, int M, int rows) {
  launch_next();
  const int ch = (blockIdx.x * CONV_THREADS + threadIdx.x) * 8;
  if (ch >= c.channels) return;
  float w[TAPS][8], b[8], win[TAPS][8];
  load_v<8>(c.b + ch, b);
#pragma unroll
  for (int j = 0; j < TAPS; ++j) load_v<8>(c.w + (i64)j * c.channels + ch, w[j]);
  wait_previous();
  const int m0 = blockIdx.y * rows, m1 = min(M, m0 + rows);
  const bf16* u = static_cast<const bf16*>(c.u) + ch;
  for (int at = m0; at < m1; at += CONV_BATCH) {
    uint4 raw[CONV_BATCH];
    int flags[CONV_BATCH];
#pragma unroll
    for (int r = 0; r < CONV_BATCH; ++r)
      if (at + r < m1) {
        raw[r] = *reinterpret_cast<const uint4*>(u + (i64)(at + r) * c.ldu);
        flags[r] = c.flags[at + r];
      }
#pragma unroll
    for (int r = 0; r < CONV_BATCH; ++r) {
      const int m = at + r, f = flags[r];
      if (m >= m1 || (f & BXF_ROW_PAD)) continue;
      if (m == m0 || (f & BXF_ROW_FIRST)) {              // the inputs before this row: rows of the step, the state, zeros
        const i64 pos = c.pos[m], slot = c.seq[m];
        int first = (f & BXF_ROW_FIRST) ? 0 : -1;
#pragma unroll
        for (int back = 1; back < TAPS; ++back) {
          float (&v)[8] = win[TAPS - 1 - back];
          if (back > pos) {
#pragma unroll
            for (int i = 0; i < 8; ++i) v[i] = 0.0f;
          } else if (first < 0) {
            load_v<8>(u + (i64)(m - back) * c.ldu, v);
            if (c.flags[m - back] & BXF_ROW_FIRST) first = back;
          } else {
            load_v<8>(static_cast<const bf16*>(c.state) + (slot * (TAPS - 1) + first - back + TAPS - 1) * c.channels + ch, v);
          }
        }
      }
      load_v<8>(raw[r], win[TAPS - 1]);
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

// ---- decays per channel, a thread each for a few rows ----
constexpr int DECAY_RANK = 16, DECAY_ROWS = 8;

// sigmoid(z)^inv_tau, its logarithm first.
__device__ __forceinline__ float log_decay(float z, float inv_tau) { return -softplus(-z) * inv_tau; }

__global__ void __launch_bounds__(256) fl_decay_rows_kernel(const bxf_recurrence_rows p, int M, int rows) {
  launch_next();
  const i64 HK = (i64)p.heads * p.K;
  const int c = blockIdx.x * 256 + threadIdx.x, m0 = blockIdx.y * rows, m1 = min(M, m0 + rows);
  if (c >= HK) return;
  const float bias = p.a2_b[c];
  float z[DECAY_ROWS];
#pragma unroll
  for (int r = 0; r < DECAY_ROWS; ++r) z[r] = bias;
  bool waited = false;
  for (int j0 = 0; j0 < p.rank; j0 += DECAY_RANK) {
    float w[DECAY_RANK];
#pragma unroll
    for (int j = 0; j < DECAY_RANK; ++j) w[j] = j0 + j < p.rank ? p.a2[(j0 + j) * HK + c] : 0.0f;
    if (!waited) wait_previous();
    waited = true;
#pragma unroll
    for (int r = 0; r < DECAY_ROWS; ++r) {
      if (m0 + r >= m1) break;
      const float* side = p.side + (m0 + r) * p.lds + j0;
#pragma unroll
      for (int j = 0; j < DECAY_RANK; ++j)
        if (j0 + j < p.rank) z[r] = fmaf(w[j], side[j], z[r]);
    }
  }
#pragma unroll
  for (int r = 0; r < DECAY_ROWS; ++r)
    if (m0 + r < m1) p.decays[(m0 + r) * HK + c] = expf(log_decay(z[r], p.inv_tau));
}

// ---- the recurrence row by row: decoding, short portions, 32-bit, any sizes ----
// One CTA per (sequence of the step, head, 4 CW value columns) walks the sequence's rows with its part of the state in
// registers: thread = 4 columns x every (256 / CW)th key channel. Rows are prepared in shared memory ROWS at a time (one for
// decoding). Wide
// slices share the preparation, narrow ones spread a small batch over more SMs.
constexpr int REC_THREADS = 256, REC_ROWS = 8;   // REC_ROWS: most rows at a time

__host__ __device__ constexpr int recurrence_smem(int K, int CW, bool channel, int rows) {
  return (rows * K * (channel ? 3 : 2) + rows * 4 * CW * 9 + 2 * REC_ROWS) * 4;
}

template <class T, bool CHANNEL, int CW, int KR, int ROWS>
__global__ void __launch_bounds__(REC_THREADS, KR > 8 ? 1 : KR <= 4 ? 4 : 3) fl_recurrence_kernel(const bxf_recurrence_rows p, int M) {
  launch_next();
  extern __shared__ float rec_smem[];
  constexpr int COLS = 4 * CW, LANES = REC_THREADS / CW;
  const int m0 = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * COLS, tid = threadIdx.x;
  wait_previous();
  const int f0 = p.flags[m0];
  const i64 slot = p.seq[m0];
  if ((f0 & (BXF_ROW_FIRST | BXF_ROW_PAD)) != BXF_ROW_FIRST) return;
  const int K = p.K, V = p.V, g = h / (p.heads / p.groups);
  float* sv = rec_smem;                                  // [rows][COLS]
  float* red = sv + ROWS * COLS;                     // [rows][8 warps][COLS]
  float* s_dt = red + ROWS * 8 * COLS;               // [rows] step size and decay of the head
  float* s_dec = s_dt + REC_ROWS;
  float* sq = s_dec + REC_ROWS;                          // [rows][K]
  float* sk = sq + ROWS * K;
  float* sa = sk + ROWS * K;                         // CHANNEL: decays
  const int cx = (tid % CW) * 4, kl = tid / CW, col = c0 + cx;
  float* state = p.state + ((slot * p.heads + h) * K) * (i64)V + col;
  const bool fresh = f0 & BXF_ROW_START, wide = V % 4 == 0 && col < V;
  float s[KR][4];
#pragma unroll
  for (int j = 0; j < KR; ++j) {
    const int k = j * LANES + kl;
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
  const T* y = static_cast<const T*>(p.y);
  for (int m = m0;;) {
    int n = 0;
    bool end = false;
    while (n < ROWS && !end) end = p.flags[m + n++] & BXF_ROW_LAST;
    for (int r = 0; r < n; ++r) {
      const T* row = y + (i64)(m + r) * p.ldy;
      for (int k = tid; k < K; k += REC_THREADS) {
        sq[r * K + k] = ld(row + p.q0 + g * K + k) * (CHANNEL ? p.q_scale : 1.0f);
        sk[r * K + k] = ld(row + p.k0 + g * K + k);
        if (CHANNEL) sa[r * K + k] = p.decays[((i64)(m + r) * p.heads + h) * K + k];
      }
      if (tid < COLS) sv[r * COLS + tid] = c0 + tid < V ? ld(row + p.v0 + (i64)h * V + c0 + tid) : 0.0f;
    }
    if (!CHANNEL && tid < n) {
      const float dt = softplus(p.side[(m + tid) * p.lds + h]);
      s_dt[tid] = dt;
      s_dec[tid] = expf(-expf(p.A_log[h]) * dt);
    }
    __syncthreads();
    for (int r = 0; r < n; ++r) {
      const float4 x = *reinterpret_cast<const float4*>(sv + r * COLS + cx);
      const float dt = CHANNEL ? 1.0f : s_dt[r], dec = CHANNEL ? 1.0f : s_dec[r];
      const float v[4] = {x.x * dt, x.y * dt, x.z * dt, x.w * dt};
      float o[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
      for (int j = 0; j < KR; ++j) {
        const int k = j * LANES + kl;
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
      for (int d = CW; d < 32; d *= 2)
#pragma unroll
        for (int i = 0; i < 4; ++i) o[i] += __shfl_xor_sync(0xffffffffu, o[i], d);
      if ((tid & 31) < CW) store_v<4>(red + (r * 8 + (tid >> 5)) * COLS + cx, o);
    }
    if (end) {
#pragma unroll
      for (int j = 0; j < KR; ++j) {
        const int k = j * LANES + kl;
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
    __syncthreads();
    for (int at = tid; at < n * COLS; at += REC_THREADS) {
      const int r = at / COLS, c = at % COLS;
      if (c0 + c >= V) continue;
      float o = 0.0f;
#pragma unroll
      for (int w = 0; w < 8; ++w) o += red[(r * 8 + w) * COLS + c];
      if (!CHANNEL) o = fmaf(p.skip[h], sv[at], o);
      st(static_cast<T*>(p.out) + (m + r) * p.ldo + (i64)h * V + c0 + c, o);
    }
    if (end) break;
    m += n;
    __syncthreads();                                     // the next rows overwrite sv
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
