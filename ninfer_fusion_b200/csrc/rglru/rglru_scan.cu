// Gated linear recurrence in steps: the convolution, and the recurrence with one thread per (sequence, channel).
#include "rglru.cuh"

#include "../common/launch.h"

namespace nfb {

namespace {

template <typename A>
__global__ void __launch_bounds__(128) rglru_conv_kernel(const RglruArgs p, A* __restrict__ u) {
  pdl_launch_next();
  pdl_wait_prior();
  const int C = p.blocks * p.width, t = blockIdx.x, seq = p.token_seq[t], i = t - p.cu_seqlens[seq], pos = p.cache_pos[t];
  const float* ring = p.ring + static_cast<long long>(p.state_slot[seq]) * p.taps * C;
  for (int c = blockIdx.y * blockDim.x * 8 + threadIdx.x * 8; c < C; c += gridDim.y * blockDim.x * 8) {
    float v[8];
    rglru_conv8(p, static_cast<const A*>(p.proj) + C, ring, t, i, pos, C, c, v);
    store8(u + static_cast<long long>(t) * C + c, v);
  }
}

template <typename A>
__global__ void __launch_bounds__(128) rglru_scan_kernel(const RglruArgs p, const A* __restrict__ u, const float* __restrict__ raw) {
  pdl_launch_next();
  pdl_wait_prior();
  const int C = p.blocks * p.width, c = blockIdx.x * blockDim.x + threadIdx.x, seq = blockIdx.y;
  if (c >= C) return;
  const int t0 = p.cu_seqlens[seq], t1 = p.cu_seqlens[seq + 1];
  if (t1 <= t0) return;
  const long long slot = p.state_slot[seq];
  const int b = c / p.width, at = c % p.width;
  const float rate = p.rate[c];
  float S = p.S[slot * C + c];
  for (int t = t0; t < t1; ++t) {
    const float* g = raw + (static_cast<long long>(t) * p.blocks + b) * 2 * p.width + at;
    float em, in;
    rglru_gates<A>(g[0], g[p.width], rate, elem_to_f(u[static_cast<long long>(t) * C + c]), em, in);
    S += fmaf(em, S, in);
    const float y = elem_to_f(static_cast<const A*>(p.proj)[t * p.ldp + c]);
    static_cast<A*>(p.out)[t * p.ldo + c] = elem_from_f<A>(S * gelu_tanh_of<A>(y));
  }
  if (!p.write_state) return;
  p.S[slot * C + c] = S;
  float* ring = p.ring + slot * p.taps * C;
  for (int t = max(t0, t1 - p.taps); t < t1; ++t)
    ring[static_cast<long long>(p.cache_pos[t] % p.taps) * C + c] = elem_to_f(static_cast<const A*>(p.proj)[t * p.ldp + C + c]);
}

}  // namespace

const char* rglru_check(const RglruArgs& a) {
  if (a.blocks < 1 || a.width < 16 || a.width % 16 || a.taps < 1) return "rglru: block widths must be multiples of 16";
  const int align = a.f32 ? 4 : 8;
  if (a.ldp % align || a.ldo % align || a.n_seq < 1 || a.n_seq > 65535) return "rglru: misaligned rows or too many sequences";
  return nullptr;
}

const char* rglru_conv(const RglruArgs& a, void* u) {
  if (a.T <= 0) return nullptr;
  if (const char* err = rglru_check(a)) return err;
  const dim3 grid(a.T, (a.blocks * a.width + 1023) / 1024);
  const cudaError_t e = a.f32 ? launch_kernel(rglru_conv_kernel<float>, grid, dim3(128), 0, a.stream, a.pdl, 1, a, static_cast<float*>(u))
                              : launch_kernel(rglru_conv_kernel<__nv_bfloat16>, grid, dim3(128), 0, a.stream, a.pdl, 1, a, static_cast<__nv_bfloat16*>(u));
  return e == cudaSuccess ? nullptr : cudaGetErrorString(e);
}

const char* rglru_scan(const RglruArgs& a, const void* u, const float* raw) {
  if (a.T <= 0) return nullptr;
  if (const char* err = rglru_check(a)) return err;
  const dim3 grid((a.blocks * a.width + 127) / 128, a.n_seq);
  const cudaError_t e = a.f32 ? launch_kernel(rglru_scan_kernel<float>, grid, dim3(128), 0, a.stream, a.pdl, 1, a, static_cast<const float*>(u), raw)
                              : launch_kernel(rglru_scan_kernel<__nv_bfloat16>, grid, dim3(128), 0, a.stream, a.pdl, 1, a,
                                              static_cast<const __nv_bfloat16*>(u), raw);
  return e == cudaSuccess ? nullptr : cudaGetErrorString(e);
}

}  // namespace nfb
