// 32-bit products on the CUDA cores (FP32 multiply-adds, no reduced-precision mode), with the epilogues of the bf16
// kernels: a CTA computes 128 weight rows x 32 token rows, 512 threads, one weight row and 8 token columns each.
#pragma once

#include "fl_tiles.cuh"

namespace bxf {

constexpr int SIMT_TA = 32;
constexpr int SIMT_KC = 16;

template <int NP>
struct RegGet {
  float (&acc)[NP][8];
  template <int W>
  __device__ __forceinline__ void load(int plane, int, float (&v)[W]) const {
    static_assert(W == 8, "a thread holds its 8 columns");
#pragma unroll
    for (int p = 0; p < NP; ++p)
      if (p == plane) {
#pragma unroll
        for (int i = 0; i < 8; ++i) v[i] = acc[p][i];
      }
  }
};

template <class Epi>
__global__ void __launch_bounds__(EPI_THREADS, 1)
fl_gemm_simt_kernel(const float* __restrict__ w, i64 ldw, i64 gsw, const float* __restrict__ x, i64 ldx, i64 gsx,
                    const GemmShape s, const typename Epi::Params ep) {
  constexpr int NP = Epi::PLANES;
  __shared__ float ws[NP][SIMT_KC][NROWS + 1];
  __shared__ __align__(16) float xs[SIMT_KC][SIMT_TA];
  extern __shared__ __align__(16) uint8_t simt_stash[];
  Tile t;
  if (!locate_tile(s, SIMT_TA, blockIdx.x, t)) return;
  const int tid = threadIdx.x, row = tid & 127, cg = tid >> 7;          // warp lanes = consecutive weight rows
  const float* wg = w + (NP == 1 ? (i64)t.group * gsw : 0);
  const float* xg = x + (s.counts ? 0 : (i64)t.group * gsx);
  float acc[NP][8];
#pragma unroll
  for (int p = 0; p < NP; ++p)
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[p][i] = 0.0f;
  for (int k0 = 0; k0 < s.K; k0 += SIMT_KC) {
#pragma unroll
    for (int p = 0; p < NP; ++p)
      for (int e = tid; e < NROWS * SIMT_KC; e += EPI_THREADS) {
        const int r = e / SIMT_KC, k = e % SIMT_KC;
        ws[p][k][r] = (t.n0 + r < s.N && k0 + k < s.K) ? wg[p * gsw + (i64)(t.n0 + r) * ldw + k0 + k] : 0.0f;
      }
    {
      const int r = tid / SIMT_KC, k = tid % SIMT_KC;
      xs[k][r] = (r < t.rows && k0 + k < s.K) ? xg[(i64)(t.row0 + r) * ldx + k0 + k] : 0.0f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < SIMT_KC; ++k) {
      const float4 x0 = *reinterpret_cast<const float4*>(&xs[k][cg * 8]);
      const float4 x1 = *reinterpret_cast<const float4*>(&xs[k][cg * 8 + 4]);
      const float xv[8] = {x0.x, x0.y, x0.z, x0.w, x1.x, x1.y, x1.z, x1.w};
#pragma unroll
      for (int p = 0; p < NP; ++p) {
        const float wv = ws[p][k][row];
#pragma unroll
        for (int i = 0; i < 8; ++i) acc[p][i] = fmaf(wv, xv[i], acc[p][i]);
      }
    }
    __syncthreads();
  }
  RegGet<NP> get{acc};
  Epi::template run<float, SIMT_TA, 8>(get, ep, t, s.N, row, cg, 4, simt_stash);
}

}  // namespace bxf
