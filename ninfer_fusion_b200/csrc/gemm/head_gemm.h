// One small matrix per head (plain C++ ABI, bf16): out[t, h * N + n] = sum_k w[h, n, k] x[t, h * x_step + k].
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

namespace nfb {

struct HeadGemmArgs {
  const void* x = nullptr;   // [T, >= (H - 1) * x_step + K], leading dimension ldx
  int64_t ldx = 0;
  int x_step = 0;
  const void* w = nullptr;   // [H, N, K]
  void* out = nullptr;       // [T, H * N], leading dimension ldo
  int64_t ldo = 0;
  int T = 0, H = 0, N = 0, K = 0;
  // optional: token tiles that lie inside one sequence of `max_tokens` or more tokens of this step are left out
  const int* token_seq = nullptr;   // [T]
  const int* cu_seqlens = nullptr;
  int max_tokens = 0;
  cudaStream_t stream = nullptr;
  bool pdl = false;
};
const char* head_gemm(const HeadGemmArgs& a);

}  // namespace nfb
