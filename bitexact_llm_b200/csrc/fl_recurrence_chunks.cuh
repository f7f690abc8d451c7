// Linear recurrences (fl_recurrence.cuh) over prompts, in chunks of up to 64 rows on the tensor cores. Within a chunk, with
// c_t the sum of the log decays of the rows after its first one up to t,
//   o_t = (q_t e^(c_t)) S' + sum_(s <= t) (q_t e^(c_t)) . (k_s e^(-c_s)) v_s,     S' = diag(a_first) S,
//   S  <- diag(e^(c_last)) (S' + sum_s (k_s e^(-c_s)) v_s^T).
// One CTA per (run of rows, head, slice of value columns) walks the chunks of its run. Long runs are cut into segments that are
// walked side by side: a first pass makes every segment's own contribution to the state and its decays, a small kernel
// chains them to the states the segments start from, and the second pass produces the outputs. A warp holds the state of 16 value
// columns in registers, 32-bit, transposed (accumulators of V^T K), so that it is at the same time the B operand of Q S.
// Products are bf16 mma with 32-bit accumulation; whatever carries a decay, a step size or a state is split into two bf16
// terms (high and low part, about 17 bits), so only q, k, v themselves have bf16 precision.
//
// BXF_DECAY_HEAD: q, k enter the scores unscaled and every score gets its factor e^(c_t - c_s) <= 1 in 32-bit.
// BXF_DECAY_CHANNEL: the factors belong to the contraction index, so q e^c and k e^-c are made beforehand, by
// fl_decay_prepare_kernel, in high and low parts. e^-c must not overflow: a chunk whose channels decay by more than e^-40
// is cut into shorter pieces there, down to single rows (c = 0), whatever the decays are.
#pragma once

#include "fl_recurrence.cuh"

namespace bxf {

constexpr int RC_ROWS = 64, RC_LDA = RC_ROWS + 8, RC_MAX_K = 256;
constexpr float RC_RANGE = 40.0f;

// ---- warp-level building blocks ----
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], const bf16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(bx::smem_u32(p)));
}
__device__ __forceinline__ void ldsm4_t(uint32_t (&r)[4], const bf16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(bx::smem_u32(p)));
}
// d += a b: 16 x 8 x 16, a rows and b columns along the contraction
__device__ __forceinline__ void mma16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// Two values as bf16 pairs of their high parts and of what is left.
__device__ __forceinline__ void split_pair(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16(x, y);
  lo = pack_bf16(x - __uint_as_float(hi << 16), y - __uint_as_float(hi & 0xffff0000u));
}
__device__ __forceinline__ void copy16(bf16* to, const bf16* from, bool there) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(bx::smem_u32(to)), "l"(from), "r"(there ? 16 : 0) : "memory");
}
__device__ __forceinline__ void copies_done() { asm volatile("cp.async.wait_all;" ::: "memory"); }

// ---- decays per channel: log decays, pieces, scaled queries and keys ----
// One CTA per (chunk, head). planes bf16 [4][M][heads K] = q high, q low, k high, k low; edge float [M][heads K]: in a
// piece's first row its decays, in its last row (of several) e^(c_last); masks [chunks][heads]: bit t = row t starts a piece.
constexpr int RP_THREADS = 256, RP_RANK = 16;

__host__ __device__ constexpr int decay_ranks(int rank) { return (rank + RP_RANK - 1) / RP_RANK * RP_RANK; }
__host__ __device__ constexpr int decay_prepare_smem(int K, int rank) { return RC_ROWS * (K + decay_ranks(rank)) * 4; }

__global__ void __launch_bounds__(RP_THREADS)
fl_decay_prepare_kernel(const bxf_recurrence_rows p, const int* __restrict__ chunks, bf16* __restrict__ planes,
                        float* __restrict__ edge, unsigned long long* __restrict__ masks, int M) {
  launch_next();
  wait_previous();
  extern __shared__ float rp_smem[];
  const int K = p.K, h = blockIdx.y, tid = threadIdx.x, row0 = chunks[blockIdx.x * 2], n = chunks[blockIdx.x * 2 + 1];
  const i64 HK = (i64)p.heads * K;
  float* la = rp_smem;                                   // [64][K] log decays, then c
  float* side = la + RC_ROWS * K;                        // [64][rank], zeros up to a multiple of RP_RANK
  const int R = decay_ranks(p.rank);
  for (int at = tid; at < n * R; at += RP_THREADS)
    side[at] = at % R < p.rank ? p.side[(row0 + at / R) * p.lds + at % R] : 0.0f;
  __syncthreads();
  const int lanes = RP_THREADS / K, t0 = tid / K, k = tid % K;
  if (t0 < lanes) {
    const float* a2 = p.a2 + h * K + k;
    const float bias = p.a2_b[h * K + k];
    for (int j0 = 0; j0 < p.rank; j0 += RP_RANK) {
      float w[RP_RANK];
#pragma unroll
      for (int j = 0; j < RP_RANK; ++j) w[j] = j0 + j < p.rank ? a2[(j0 + j) * HK] : 0.0f;
      for (int t = t0; t < n; t += lanes) {
        float z = j0 == 0 ? bias : la[t * K + k];
        float s[RP_RANK];
        load_v<RP_RANK>(side + t * R + j0, s);
#pragma unroll
        for (int j = 0; j < RP_RANK; ++j) z = fmaf(w[j], s[j], z);
        la[t * K + k] = j0 + RP_RANK >= p.rank ? log_decay(z, p.inv_tau) : z;
      }
    }
  }
  __syncthreads();
  float sum = 0.0f;
  if (tid < K) {
#pragma unroll 8
    for (int t = 1; t < n; ++t) sum += la[t * K + tid];
  }
  const bool one = __syncthreads_and(sum >= -RC_RANGE);
  unsigned long long mask = 1;
  float c = 0.0f;
  int start = 0;
  float* e = edge + (i64)row0 * HK + h * K + tid;
  if (one && tid < K) {
    e[0] = expf(la[tid]);
    for (int t = 0; t < n; t += 8) {
      float l[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) l[i] = t + i > 0 && t + i < n ? la[(t + i) * K + tid] : 0.0f;
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        c += l[i];
        if (t + i < n) la[(t + i) * K + tid] = c;
      }
    }
  }
  for (int t = 0; t < n && !one; ++t) {
    const float l = tid < K ? la[t * K + tid] : 0.0f;
    const bool cut = t > 0 && __syncthreads_or(c + l < -RC_RANGE);
    if (cut) {
      if (tid < K && t - 1 > start) e[(i64)(t - 1) * HK] = expf(c);
      mask |= 1ull << t;
      start = t;
    }
    if (t == start) {
      c = 0.0f;
      if (tid < K) e[(i64)t * HK] = expf(l);
    } else {
      c += l;
    }
    if (tid < K) la[t * K + tid] = c;
  }
  if (tid < K && n - 1 > start) e[(i64)(n - 1) * HK] = expf(c);
  if (tid == 0) masks[(i64)blockIdx.x * p.heads + h] = mask;
  __syncthreads();
  const i64 plane = (i64)M * HK;
  const bf16* y = static_cast<const bf16*>(p.y);
  for (int at = tid; at < n * (K / 8); at += RP_THREADS) {
    const int t = at / (K / 8), d = at % (K / 8) * 8;
    const i64 row = row0 + t;
    float q[8], kk[8];
    load_v<8>(y + row * p.ldy + p.q0 + h * K + d, q);
    load_v<8>(y + row * p.ldy + p.k0 + h * K + d, kk);
    uint32_t o[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float c0 = la[t * K + d + 2 * i], c1 = la[t * K + d + 2 * i + 1];
      const float e0 = expf(c0), e1 = expf(c1);          // e^-40 at the least: the reciprocals stay finite
      split_pair(q[2 * i] * p.q_scale * e0, q[2 * i + 1] * p.q_scale * e1, o[0][i], o[1][i]);
      split_pair(__fdividef(kk[2 * i], e0), __fdividef(kk[2 * i + 1], e1), o[2][i], o[3][i]);
    }
#pragma unroll
    for (int j = 0; j < 4; ++j)
      *reinterpret_cast<uint4*>(planes + j * plane + row * HK + h * K + d) = make_uint4(o[j][0], o[j][1], o[j][2], o[j][3]);
  }
}

// ---- the chunk kernel ----
struct ChunkArgs {
  const int* runs;               // [runs, 3] (first row, rows, first chunk) of what a CTA walks
  const bf16* planes;            // BXF_DECAY_CHANNEL: of fl_decay_prepare_kernel
  const float* edge;
  const unsigned long long* masks;
  float* states;                 // segments: [segments][heads][K][V] contributions, then the states they start from
  float* decays;                 // segments: [segments][heads][K] of the whole segment
  int M;
};

enum ChunkPass { WHOLE_RUN, CONTRIBUTION, OUTPUTS };

template <bool CHANNEL, int KT, int NW, ChunkPass PASS>
struct ChunkCfg {
  static constexpr int KP = 16 * KT, LDK = KP + 8, VS = 16 * NW, LDV = VS + 8, PARTS = CHANNEL ? 2 : 1;
  static constexpr int QK = RC_ROWS * LDK, V = RC_ROWS * LDV;             // bf16 elements
  static constexpr int Q = PASS == CONTRIBUTION ? 0 : PARTS * QK, A = PASS == CONTRIBUTION ? 0 : RC_ROWS * RC_LDA;
  static constexpr int SMEM = (Q + PARTS * QK + V + 2 * A) * 2 + (3 * KP + 2 * RC_ROWS) * 4;
  static constexpr int FIT = 224 * 1024 / SMEM;
  static constexpr int CTAS = KT > 8 || FIT < 2 ? 1 : FIT < 3 ? 2 : PASS == CONTRIBUTION && FIT >= 4 ? 4 : 3;
};

template <bool CHANNEL, int KT, int NW, ChunkPass PASS>
__global__ void __launch_bounds__(32 * NW, ChunkCfg<CHANNEL, KT, NW, PASS>::CTAS)
fl_recurrence_chunk_kernel(const bxf_recurrence_rows p, const ChunkArgs a) {
  using Cfg = ChunkCfg<CHANNEL, KT, NW, PASS>;
  constexpr int LDK = Cfg::LDK, LDV = Cfg::LDV, KP = Cfg::KP, THREADS = 32 * NW;
  launch_next();
  wait_previous();
  extern __shared__ __align__(16) uint8_t rc_smem[];
  bf16* qs = reinterpret_cast<bf16*>(rc_smem);           // [PARTS][64][LDK]
  bf16* ks = qs + Cfg::Q;
  bf16* vs = ks + Cfg::PARTS * Cfg::QK;                  // [64][LDV]
  bf16* as = vs + Cfg::V;                                // [2][64][72] scores, high and low parts
  float* first = reinterpret_cast<float*>(as + 2 * Cfg::A);   // [KP] decays of the piece's first row
  float* last = first + KP;                              // [KP] e^(c_last)
  float* total = last + KP;                              // [KP] decays of the segment so far
  float* cum = total + KP;                               // [64] BXF_DECAY_HEAD: sums of the log decays
  float* dts = cum + RC_ROWS;                            // [64] step sizes
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, quad = lane & 3, lrow = lane >> 2;
  const int h = blockIdx.y, K = p.K, V = p.V, c0 = blockIdx.z * Cfg::VS, v0 = c0 + warp * 16;
  const int g = h / (p.heads / p.groups);
  const int row0 = a.runs[blockIdx.x * 3], rows = a.runs[blockIdx.x * 3 + 1], chunk0 = a.runs[blockIdx.x * 3 + 2];
  const i64 HK = (i64)p.heads * K, plane = a.M * HK;
  const bf16* y = static_cast<const bf16*>(p.y);
  const float neg_rate = CHANNEL ? 0.0f : -expf(p.A_log[h]), skip = CHANNEL ? 0.0f : p.skip[h];
  // row and column of this lane's address in the four 8 x 8 blocks of ldmatrix
  const int lm = lane & 7, b1 = (lane >> 3) & 1, b2 = lane >> 4;

  // the state, transposed: value column v0 + lrow (+ 8), key channel 8 j + 2 quad (+ 1)
  float* state = (PASS == WHOLE_RUN ? p.state + ((p.seq[row0] * p.heads + h) * K) * (i64)V
                                    : a.states + (((i64)blockIdx.x * p.heads + h) * K) * V);
  float S[2 * KT][4];
  const bool fresh = PASS == CONTRIBUTION || (PASS == WHOLE_RUN && (p.flags[row0] & BXF_ROW_START));
  float total_log = 0.0f;
  if (PASS == CONTRIBUTION && CHANNEL)
    for (int k = tid; k < KP; k += THREADS) total[k] = 1.0f;
#pragma unroll
  for (int j = 0; j < 2 * KT; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int k = 8 * j + 2 * quad + (i & 1), v = v0 + lrow + (i >> 1) * 8;
      S[j][i] = !fresh && k < K && v < V ? state[(i64)k * V + v] : 0.0f;
    }

  for (int r0 = 0, n; r0 < rows; r0 += n) {
    n = min(RC_ROWS - r0 % RC_ROWS, rows - r0);
    if (CHANNEL) {
      const unsigned long long ahead = a.masks[(i64)(chunk0 + r0 / RC_ROWS) * p.heads + h] >> (r0 % RC_ROWS) >> 1;
      if (ahead) n = min(n, __ffsll(ahead));
    }
    const i64 m0 = row0 + r0;
    // ---- rows into shared memory, zeros beyond the piece and the sizes ----
    {
      constexpr int PER = KP / 8, STEP = THREADS / PER;                   // 16-byte pieces of a row, rows at a time
      static_assert(THREADS % PER == 0 && RC_ROWS % STEP == 0, "a thread keeps its columns");
      const int t0 = tid / PER, d = tid % PER * 8;
      const int col = d < K ? d : 0;
      const i64 ld = CHANNEL ? HK : p.ldy;
      const bf16* q = CHANNEL ? a.planes + (m0 + t0) * HK + h * K + col : y + (m0 + t0) * p.ldy + p.q0 + g * K + col;
      const bf16* k = CHANNEL ? q + 2 * plane : y + (m0 + t0) * p.ldy + p.k0 + g * K + col;
#pragma unroll
      for (int i = 0; i < RC_ROWS / STEP; ++i) {
        const bool there = t0 + i * STEP < n && d < K;
        const i64 off = there ? i * STEP * ld : -t0 * ld;                 // the segment's first row stands in for none
#pragma unroll
        for (int part = 0; part < Cfg::PARTS; ++part) {
          const int to = part * Cfg::QK + (t0 + i * STEP) * LDK + d;
          if (PASS != CONTRIBUTION) copy16(qs + to, q + part * plane + off, there);
          copy16(ks + to, k + part * plane + off, there);
        }
      }
    }
    {
      constexpr int PER = Cfg::VS / 8, STEP = THREADS / PER;
      const int t0 = tid / PER, d = tid % PER * 8;
      const bf16* v = y + (m0 + t0) * p.ldy + p.v0 + (i64)h * V + (c0 + d < V ? c0 + d : 0);
#pragma unroll
      for (int i = 0; i < RC_ROWS / STEP; ++i) {
        const bool there = t0 + i * STEP < n && c0 + d < V;
        copy16(vs + (t0 + i * STEP) * LDV + d, v + (there ? i * STEP : -t0) * p.ldy, there);
      }
    }
    if (CHANNEL) {
      for (int k = tid; k < KP; k += THREADS) {
        first[k] = k < K ? a.edge[m0 * HK + h * K + k] : 0.0f;
        last[k] = k < K && n > 1 ? a.edge[(m0 + n - 1) * HK + h * K + k] : 1.0f;
        if (PASS == CONTRIBUTION) total[k] *= first[k] * last[k];         // always this thread's
      }
    } else if (warp == 0) {
      const int t = 2 * lane;
      const float d0 = t < n ? softplus(p.side[(m0 + t) * p.lds + h]) : 0.0f;
      const float d1 = t + 1 < n ? softplus(p.side[(m0 + t + 1) * p.lds + h]) : 0.0f;
      float sum = (d0 + d1) * neg_rate;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float below = __shfl_up_sync(0xffffffffu, sum, o);
        if (lane >= o) sum += below;
      }
      dts[t] = d0;
      dts[t + 1] = d1;
      cum[t] = sum - d1 * neg_rate;
      cum[t + 1] = sum;
    }
    copies_done();
    __syncthreads();

    // ---- scores: warp = 16 rows x 64 (32) columns ----
    if (PASS != CONTRIBUTION) {
      constexpr int NT = NW == 8 ? 4 : 8;
      const int rb = warp & 3, cb = NW == 8 ? (warp >> 2) * 4 : 0;
      float acc[NT][4];
#pragma unroll
      for (int j = 0; j < NT; ++j)
#pragma unroll
        for (int i = 0; i < 4; ++i) acc[j][i] = 0.0f;
      for (int kt = 0; kt < KT; ++kt) {
        uint32_t q[2][4];
        const int at_q = (rb * 16 + b1 * 8 + lm) * LDK + kt * 16 + b2 * 8;
        ldsm4(q[0], qs + at_q);
        if (CHANNEL) ldsm4(q[1], qs + Cfg::QK + at_q);
#pragma unroll
        for (int j = 0; j < NT; j += 2) {
          if ((cb + j) / 2 > rb) continue;
          uint32_t k[4];
          const int at_k = ((cb + j) * 8 + b2 * 8 + lm) * LDK + kt * 16 + b1 * 8;
          ldsm4(k, ks + at_k);
          mma16816(acc[j], q[0], k[0], k[1]);
          mma16816(acc[j + 1], q[0], k[2], k[3]);
          if (CHANNEL) {
            mma16816(acc[j], q[1], k[0], k[1]);
            mma16816(acc[j + 1], q[1], k[2], k[3]);
            ldsm4(k, ks + Cfg::QK + at_k);
            mma16816(acc[j], q[0], k[0], k[1]);
            mma16816(acc[j + 1], q[0], k[2], k[3]);
          }
        }
      }
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        if ((cb + j) / 2 > rb) continue;
        const int s = (cb + j) * 8 + 2 * quad;
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int t = rb * 16 + lrow + half * 8;
          float x0 = s <= t ? acc[j][2 * half] : 0.0f, x1 = s + 1 <= t ? acc[j][2 * half + 1] : 0.0f;
          if (!CHANNEL) {
            if (s <= t) x0 *= __expf(cum[t] - cum[s]) * dts[s];
            if (s + 1 <= t) x1 *= __expf(cum[t] - cum[s + 1]) * dts[s + 1];
          }
          uint32_t hi, lo;
          split_pair(x0, x1, hi, lo);
          *reinterpret_cast<uint32_t*>(as + t * RC_LDA + s) = hi;
          *reinterpret_cast<uint32_t*>(as + Cfg::A + t * RC_LDA + s) = lo;
        }
      }
    }
    if (CHANNEL) {
#pragma unroll
      for (int j = 0; j < 2 * KT; ++j)
#pragma unroll
        for (int i = 0; i < 4; ++i) S[j][i] *= first[8 * j + 2 * quad + (i & 1)];
    }
    if (PASS != CONTRIBUTION) {
      __syncthreads();

      // ---- outputs of this warp's 16 columns: state, then scores ----
      float o[4][2][4];
#pragma unroll
      for (int mt = 0; mt < 4; ++mt)
#pragma unroll
        for (int nt = 0; nt < 2; ++nt)
#pragma unroll
          for (int i = 0; i < 4; ++i) o[mt][nt][i] = 0.0f;
#pragma unroll
      for (int kt = 0; kt < KT; ++kt) {
        uint32_t hi[2][2], lo[2][2];
#pragma unroll
        for (int nt = 0; nt < 2; ++nt)
#pragma unroll
          for (int b = 0; b < 2; ++b) split_pair(S[2 * kt + b][2 * nt], S[2 * kt + b][2 * nt + 1], hi[nt][b], lo[nt][b]);
        uint32_t q[4][4];
        const int at_q = (b1 * 8 + lm) * LDK + kt * 16 + b2 * 8;
#pragma unroll
        for (int mt = 0; mt < 4; ++mt) ldsm4(q[mt], qs + at_q + mt * 16 * LDK);
#pragma unroll
        for (int mt = 0; mt < 4; ++mt)
#pragma unroll
          for (int nt = 0; nt < 2; ++nt) mma16816(o[mt][nt], q[mt], hi[nt][0], hi[nt][1]);
#pragma unroll
        for (int mt = 0; mt < 4; ++mt)
#pragma unroll
          for (int nt = 0; nt < 2; ++nt) mma16816(o[mt][nt], q[mt], lo[nt][0], lo[nt][1]);
        if (CHANNEL) {
#pragma unroll
          for (int mt = 0; mt < 4; ++mt) ldsm4(q[mt], qs + Cfg::QK + at_q + mt * 16 * LDK);
#pragma unroll
          for (int mt = 0; mt < 4; ++mt)
#pragma unroll
            for (int nt = 0; nt < 2; ++nt) mma16816(o[mt][nt], q[mt], hi[nt][0], hi[nt][1]);
        }
      }
      if (!CHANNEL) {
#pragma unroll
        for (int mt = 0; mt < 4; ++mt) {
          const float e0 = __expf(cum[mt * 16 + lrow]), e1 = __expf(cum[mt * 16 + lrow + 8]);
#pragma unroll
          for (int nt = 0; nt < 2; ++nt) {
            o[mt][nt][0] *= e0;
            o[mt][nt][1] *= e0;
            o[mt][nt][2] *= e1;
            o[mt][nt][3] *= e1;
          }
        }
      }
#pragma unroll
      for (int sk = 0; sk < 4; ++sk) {
        uint32_t v[4];
        ldsm4_t(v, vs + (sk * 16 + b1 * 8 + lm) * LDV + warp * 16 + b2 * 8);
#pragma unroll
        for (int mt = sk; mt < 4; ++mt)
#pragma unroll
          for (int part = 0; part < 2; ++part) {
            uint32_t s[4];
            ldsm4(s, as + part * Cfg::A + (mt * 16 + b1 * 8 + lm) * RC_LDA + sk * 16 + b2 * 8);
            mma16816(o[mt][0], s, v[0], v[1]);
            mma16816(o[mt][1], s, v[2], v[3]);
          }
      }
#pragma unroll
      for (int mt = 0; mt < 4; ++mt)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int t = mt * 16 + lrow + half * 8;
          if (t >= n) continue;
          bf16* out = static_cast<bf16*>(p.out) + (m0 + t) * p.ldo + (i64)h * V;
#pragma unroll
          for (int nt = 0; nt < 2; ++nt) {
            const int col = v0 + nt * 8 + 2 * quad;
            if (col >= V) continue;
            float x0 = o[mt][nt][2 * half], x1 = o[mt][nt][2 * half + 1];
            if (!CHANNEL) {
              const uint32_t x = *reinterpret_cast<const uint32_t*>(vs + t * LDV + warp * 16 + nt * 8 + 2 * quad);
              x0 = fmaf(skip, __uint_as_float(x << 16), x0);
              x1 = fmaf(skip, __uint_as_float(x & 0xffff0000u), x1);
            }
            *reinterpret_cast<uint32_t*>(out + col) = pack_bf16(x0, x1);
          }
        }

    }

    // ---- the state after the piece ----
    if (PASS == CONTRIBUTION && !CHANNEL) total_log += cum[RC_ROWS - 1];
    if (!CHANNEL) {
      const float e = __expf(cum[RC_ROWS - 1]);
#pragma unroll
      for (int j = 0; j < 2 * KT; ++j)
#pragma unroll
        for (int i = 0; i < 4; ++i) S[j][i] *= e;
    }
#pragma unroll
    for (int sk = 0; sk < 4; ++sk) {
      uint32_t v[2][4];                                  // V^T: rows = value columns, contraction over the chunk's rows
      ldsm4_t(v[0], vs + (sk * 16 + b2 * 8 + lm) * LDV + warp * 16 + b1 * 8);
      if (!CHANNEL) {
#pragma unroll
        for (int b = 0; b < 2; ++b) {
          const int s = sk * 16 + b * 8 + 2 * quad;
          const float w0 = dts[s] * __expf(cum[RC_ROWS - 1] - cum[s]), w1 = dts[s + 1] * __expf(cum[RC_ROWS - 1] - cum[s + 1]);
#pragma unroll
          for (int half = 0; half < 2; ++half) {
            const uint32_t x = v[0][2 * b + half];
            split_pair(__uint_as_float(x << 16) * w0, __uint_as_float(x & 0xffff0000u) * w1, v[0][2 * b + half], v[1][2 * b + half]);
          }
        }
      }
#pragma unroll
      for (int kt = 0; kt < KT; ++kt) {
        uint32_t k[4];
        const int at_k = (sk * 16 + b1 * 8 + lm) * LDK + kt * 16 + b2 * 8;
        ldsm4_t(k, ks + at_k);
        mma16816(S[2 * kt], v[0], k[0], k[1]);
        mma16816(S[2 * kt + 1], v[0], k[2], k[3]);
        if (CHANNEL) {
          ldsm4_t(k, ks + Cfg::QK + at_k);
          mma16816(S[2 * kt], v[0], k[0], k[1]);
          mma16816(S[2 * kt + 1], v[0], k[2], k[3]);
        } else {
          mma16816(S[2 * kt], v[1], k[0], k[1]);
          mma16816(S[2 * kt + 1], v[1], k[2], k[3]);
        }
      }
    }
    if (CHANNEL) {
#pragma unroll
      for (int j = 0; j < 2 * KT; ++j)
#pragma unroll
        for (int i = 0; i < 4; ++i) S[j][i] *= last[8 * j + 2 * quad + (i & 1)];
    }
    __syncthreads();                                     // the next piece overwrites the operands
  }
  if (PASS == OUTPUTS) return;
  if (PASS == CONTRIBUTION && blockIdx.z == 0) {
    float* decays = a.decays + ((i64)blockIdx.x * p.heads + h) * K;
    for (int k = tid; k < K; k += THREADS) decays[k] = CHANNEL ? total[k] : expf(total_log);
  }
#pragma unroll
  for (int j = 0; j < 2 * KT; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int k = 8 * j + 2 * quad + (i & 1), v = v0 + lrow + (i >> 1) * 8;
      if (k < K && v < V) state[(i64)k * V + v] = S[j][i];
    }
}

// The states that the segments of a run start from, in place of their contributions, and the state after the run. spans
// [runs, 3] (first row, first segment, segments). Thread = 4 consecutive values.
__global__ void __launch_bounds__(256) fl_recurrence_chain_kernel(const bxf_recurrence_rows p, const int* spans, float* states,
                                                                  const float* decays) {
  launch_next();
  wait_previous();
  const int row0 = spans[blockIdx.x * 3], seg0 = spans[blockIdx.x * 3 + 1], segs = spans[blockIdx.x * 3 + 2], h = blockIdx.y;
  const int at = (blockIdx.z * 256 + threadIdx.x) * 4, k = at / p.V;
  const i64 size = (i64)p.K * p.V;
  if (at >= size) return;
  float* state = p.state + (p.seq[row0] * p.heads + h) * size + at;
  float S[4] = {0.0f, 0.0f, 0.0f, 0.0f};
  if (!(p.flags[row0] & BXF_ROW_START)) load_v<4>(state, S);
  for (int s0 = 0; s0 < segs; s0 += 4) {                 // four segments' contributions in flight
    float c[4][4], d[4];
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (s0 + j < segs) {
        const i64 n = (i64)(seg0 + s0 + j) * p.heads + h;
        load_v<4>(states + n * size + at, c[j]);
        d[j] = decays[n * p.K + k];
      }
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (s0 + j < segs) {
        store_v<4>(states + ((i64)(seg0 + s0 + j) * p.heads + h) * size + at, S);
#pragma unroll
        for (int i = 0; i < 4; ++i) S[i] = fmaf(d[j], S[i], c[j][i]);
      }
  }
  store_v<4>(state, S);
}

}  // namespace bxf
