// Row kernels of decoders whose residual is several streams x_1 .. x_S (plain C++ ABI).
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

namespace nfb {

// A sublayer's output y[t] put together from the parts that its kernels leave:
//   y = g delta + sum_j weight_j (choice_j < n_experts ? ret[t, j] : h),   g = sigmoid(gate) where there is a gate, else 1
// (choices of n_experts and more stand for the sublayer's input h).  Without choices y = delta.
struct MixtureParts {
  const float* delta = nullptr;     // [T, N] or null
  const float* gate = nullptr;      // [T] logits, step ld_gate, or null
  int64_t ld_gate = 0;
  const int* choice = nullptr;      // [T, k] or null
  const float* weight = nullptr;    // [T, k]
  const void* ret = nullptr;        // [T, k, N] in the activation type
  const void* h = nullptr;          // [T, N] in the activation type, leading dimension ld_h
  int64_t ld_h = 0;
  int k = 0, n_experts = 0;
};

// The step between two sublayers:
//   x_u <- sum_s mix[s, u] x_s + w_out[u] y                   (mix null: the streams stay)
//   out = rms_norm(sum_s w_in[s] x_s) * w_next
struct StreamArgs {
  const float* x_in = nullptr;      // [T, S, N]; null: every stream is row ids[t] of the table
  const int* ids = nullptr;
  const void* table = nullptr;      // [vocab, N] in the activation type
  int vocab = 0;
  float* x_out = nullptr;           // [T, S, N], may be x_in
  MixtureParts y;
  const float* mix = nullptr;       // [S, S], [from, to]
  const float* w_out = nullptr;     // [S]
  const float* w_in = nullptr;      // [S]
  const float* w_next = nullptr;    // [N]
  void* out = nullptr;              // [T, N] in the activation type, leading dimension ld_out; may be y.h
  int64_t ld_out = 0;
  int T = 0, S = 0, N = 0, n_true = 0;      // columns >= n_true are zero padding
  float eps = 0.f;
  bool f32 = false;
};
constexpr int kMaxStreams = 16;
const char* stream_rows(const StreamArgs& a, cudaStream_t stream, bool pdl);

// out[t] = y[t] (fp32): for residuals whose row step knows nothing of experts.  out may be y.delta.
const char* mixture_rows(const MixtureParts& y, float* out, int T, int N, bool f32, cudaStream_t stream, bool pdl);

// g [T, 2 F] (gate | up columns, fp32) -> out [T, F]: the bounded gated unit of common/glu.cuh, for 32-bit runs.
const char* glu_rows_f32(const float* g, int64_t ldg, float* out, int64_t ldo, int64_t T, int F, float limit, float slope, float shift,
                         cudaStream_t stream, bool pdl);

}  // namespace nfb
