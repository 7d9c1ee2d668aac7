// Activation element types of the models that run in bf16 or in 32-bit: conversion and 8-wide vector access.
#pragma once
#include <cuda_bf16.h>
#include <stdint.h>

#include "ptx.cuh"

namespace nfb {

__device__ __forceinline__ float elem_to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ float elem_to_f(float v) { return v; }
template <typename A>
__device__ __forceinline__ A elem_from_f(float v);
template <>
__device__ __forceinline__ __nv_bfloat16 elem_from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }
template <>
__device__ __forceinline__ float elem_from_f<float>(float v) { return v; }

// 8 consecutive values at a 16-byte (bf16) / 32-byte (fp32) aligned address.
__device__ __forceinline__ void load8(const __nv_bfloat16* p, float* v) {
  const uint4 r = *reinterpret_cast<const uint4*>(p);
  const uint32_t w[4] = {r.x, r.y, r.z, r.w};
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    v[2 * j] = __uint_as_float(w[j] << 16);
    v[2 * j + 1] = __uint_as_float(w[j] & 0xffff0000u);
  }
}
__device__ __forceinline__ void load8(const float* p, float* v) {
  const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
  v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ void store8(__nv_bfloat16* p, const float* v) {
  *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]),
                                            pack_bf16x2(v[6], v[7]));
}
__device__ __forceinline__ void store8(float* p, const float* v) {
  reinterpret_cast<float4*>(p)[0] = make_float4(v[0], v[1], v[2], v[3]);
  reinterpret_cast<float4*>(p)[1] = make_float4(v[4], v[5], v[6], v[7]);
}

// Hardware 2^x and 1 / x (subnormals flushed): the building blocks of exponentials whose argument is already scaled.
__device__ __forceinline__ float ex2_fast(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float rcp_fast(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
constexpr float kLog2e = 1.4426950408889634f;

// cap * tanh(x * scale / cap) with k = 2 log2(e) scale / cap: cap - 2 cap / (1 + 2^(k x)).
__device__ __forceinline__ float softcap_fast(float x, float k, float cap) {
  return fmaf(-2.f * cap, rcp_fast(ex2_fast(x * k) + 1.f), cap);
}

// exp / tanh / sigmoid in the precision that goes with the element type: the library functions with 32-bit
// activations, the hardware exponential otherwise (absolute error of tanh about 1e-7).
template <typename A>
__device__ __forceinline__ float exp_of(float z) {
  if constexpr (sizeof(A) == 4) return expf(z);
  return __expf(z);
}
template <typename A>
__device__ __forceinline__ float tanh_of(float z) {
  if constexpr (sizeof(A) == 4) return tanhf(z);
  return 1.f - __fdividef(2.f, __expf(fminf(2.f * z, 80.f)) + 1.f);
}
template <typename A>
__device__ __forceinline__ float sigmoid_of(float z) {
  return 1.f / (1.f + exp_of<A>(-z));
}

}  // namespace nfb
