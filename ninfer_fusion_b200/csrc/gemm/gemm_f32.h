// 32-bit GEMM (plain C++ ABI): out = act(x w^T + bias) with fp32 operands and accumulation on the FP32 pipes.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

namespace nfb {

struct GemmF32Args {
  const float* w = nullptr;   // [N, K], leading dimension ldw
  int64_t N = 0, K = 0, ldw = 0;
  const float* x = nullptr;   // [T, K], leading dimension ldx
  int64_t T = 0, ldx = 0;
  float* out = nullptr;       // columns below out2_from
  int64_t ldo = 0;
  float* out2 = nullptr;      // columns from out2_from on (null: none)
  int64_t ldo2 = 0;
  int out2_from = 0;
  const float* bias = nullptr;
  int act = 0;                // GemmActivation (gemm.h)
  const float* act_params = nullptr;
  cudaStream_t stream = nullptr;
};

const char* gemm_f32(const GemmF32Args& a);

}  // namespace nfb
