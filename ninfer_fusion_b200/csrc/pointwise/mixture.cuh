// Sublayer outputs put together from their parts (MixtureParts of stream_rows.h), four columns at a time.
#pragma once
#include "../common/elem.cuh"
#include "stream_rows.h"

namespace nfb {

__device__ __forceinline__ void load4(const float* p, float* v) {
  const float4 a = *reinterpret_cast<const float4*>(p);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
}
__device__ __forceinline__ void load4(const __nv_bfloat16* p, float* v) {
  const uint2 r = *reinterpret_cast<const uint2*>(p);
  v[0] = __uint_as_float(r.x << 16); v[1] = __uint_as_float(r.x & 0xffff0000u);
  v[2] = __uint_as_float(r.y << 16); v[3] = __uint_as_float(r.y & 0xffff0000u);
}
__device__ __forceinline__ void store4(float* p, const float* v) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void store4(__nv_bfloat16* p, const float* v) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]));
}

// y[t, c .. c + 3]; `g` is the shared expert's factor
template <typename A>
__device__ __forceinline__ void mixture4(const MixtureParts& p, long long t, int c, int N, float g, float* y) {
  y[0] = y[1] = y[2] = y[3] = 0.f;
  if (p.delta != nullptr) {
    load4(p.delta + t * N + c, y);
    if (p.gate != nullptr) {
#pragma unroll
      for (int e = 0; e < 4; ++e) y[e] *= g;
    }
  }
  if (p.choice == nullptr) return;
#pragma unroll 4
  for (int j = 0; j < p.k; ++j) {
    const int id = p.choice[t * p.k + j];
    const float w = p.weight[t * p.k + j];
    float v[4];
    load4(id < p.n_experts ? static_cast<const A*>(p.ret) + (t * p.k + j) * N + c : static_cast<const A*>(p.h) + t * p.ld_h + c, v);
#pragma unroll
    for (int e = 0; e < 4; ++e) y[e] = fmaf(w, v[e], y[e]);
  }
}
__device__ __forceinline__ float mixture_gate(const MixtureParts& p, long long t) {
  return p.gate == nullptr ? 1.f : 1.f / (1.f + expf(-p.gate[t * p.ld_gate]));
}

inline const char* bad_mixture(const MixtureParts& y) {
  if (y.choice != nullptr && (y.weight == nullptr || y.k < 1 || (y.n_experts > 0 && y.ret == nullptr) || y.h == nullptr || y.ld_h % 8))
    return "expert sum: missing or misaligned parts";
  return nullptr;
}

}  // namespace nfb
