// Shared pieces of the float-model kernels: element types, scalar functions, row flags.
#pragma once

#include <cuda_bf16.h>
#include <stdint.h>

#include "bx_ptx.cuh"

namespace bxf {

using bf16 = __nv_bfloat16;
using i64 = long long;

// Programmatic dependent launch: the kernels of a step are launched so that the next one may start (barriers, TMEM, the
// first weight tiles) while the last CTAs of the one before it are still running. `launch_next` permits that, as soon as
// every CTA has come this far; `wait_previous` returns when the previous kernel has completed and its writes are visible,
// and stands before the first access to anything another kernel of the step reads or writes. Weights are exempt. A
// kernel that allocates TMEM calls `launch_next` after the allocation: a CTA of the next kernel on the same SM could
// otherwise take the columns first and wait, holding them, for the CTA that needs them.
__device__ __forceinline__ void launch_next() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }
__device__ __forceinline__ void wait_previous() { asm volatile("griddepcontrol.wait;" ::: "memory"); }

template <class T>
__device__ __forceinline__ float ld(const T* p);
template <>
__device__ __forceinline__ float ld<float>(const float* p) { return *p; }
template <>
__device__ __forceinline__ float ld<bf16>(const bf16* p) { return __bfloat162float(*p); }

__device__ __forceinline__ void st(float* p, float v) { *p = v; }
__device__ __forceinline__ void st(bf16* p, float v) { *p = __float2bfloat16(v); }

__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
  const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<const uint32_t*>(&v);
}

// Four consecutive values at an address that is aligned to all four.
__device__ __forceinline__ void st4(float* p, float a, float b, float c, float d) {
  *reinterpret_cast<float4*>(p) = make_float4(a, b, c, d);
}
__device__ __forceinline__ void st4(bf16* p, float a, float b, float c, float d) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(a, b), pack_bf16(c, d));
}

// e^v and 1 / v: the library's full-precision forms for the 32-bit kernels, the hardware's approximations (a few units in the
// last place of a float) for the bf16 ones.
template <class T>
__device__ __forceinline__ float exp_of(float v);
template <>
__device__ __forceinline__ float exp_of<float>(float v) { return expf(v); }
template <>
__device__ __forceinline__ float exp_of<bf16>(float v) { return __expf(v); }

template <class T>
__device__ __forceinline__ float recip(float v);
template <>
__device__ __forceinline__ float recip<float>(float v) { return 1.0f / v; }
template <>
__device__ __forceinline__ float recip<bf16>(float v) { return __fdividef(1.0f, v); }

// sigmoid(v) and 1 - sigmoid(v), both without cancellation.
template <class T>
__device__ __forceinline__ void sigmoid_pair(float v, float& s, float& one_minus_s) {
  const float e = exp_of<T>(-fabsf(v)), r = recip<T>(1.0f + e);
  s = v >= 0.0f ? r : e * r;
  one_minus_s = v >= 0.0f ? e * r : r;
}

// 1 / (1 + e^-v) = e^v / (1 + e^v): the exponent is kept below zero, so nothing overflows.
template <class T>
__device__ __forceinline__ float sigmoid(float v) {
  const float e = exp_of<T>(-fabsf(v)), r = recip<T>(1.0f + e);
  return v >= 0.0f ? r : e * r;
}

template <class T>
__device__ __forceinline__ float silu(float v) { return v * sigmoid<T>(v); }

template <class T>
__device__ __forceinline__ float activate(int act, float z, float p, float q) {
  if (act == BXF_ACT_RELU2) {
    const float r = fmaxf(z, 0.0f);
    return r * r;
  }
  if (act == BXF_ACT_XIELU) return (z > 0.0f ? p * z * z : q * (expm1f(z) - z)) + 0.5f * z;
  // (1 + tanh(a)) / 2 = sigmoid(2 a), a = sqrt(2 / pi) (z + 0.044715 z^3)
  if (act == BXF_ACT_GELU) return z * sigmoid<T>(1.5957691216057308f * (z + 0.044715f * z * z * z));
  if (act == BXF_ACT_SCALE) return p * z;
  if (act == BXF_ACT_SOFTCAP) return q * tanhf(p * z);
  return z;
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}

// Sum over the block (a multiple of 32 threads, at most 1024); `red` holds 33 floats.
__device__ __forceinline__ float block_sum(float v, float* red) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
  v = warp_sum(v);
  __syncthreads();                                       // red may still be read from the previous sum
  if (lane == 0) red[warp] = v;
  __syncthreads();
  if (warp == 0) {
    float t = lane < warps ? red[lane] : 0.0f;
    t = warp_sum(t);
    if (lane == 0) red[32] = t;
  }
  __syncthreads();
  return red[32];
}

}  // namespace bxf
