// Grouped expert GEMM in true 32-bit (no TF32) over the same tile table as moe_grouped_gemm.cu: 64 rows x 64 columns per CTA,
// 16-wide K slices in shared memory, a 4 x 4 register tile per thread.  It exists for exactness, not for the roofline.
#include "moe.h"

namespace nfb {

namespace {

constexpr int kTile = 64, kSlice = 16, kThreads = 256, kPad = 4;

struct Params {
  const float* w;
  const float* x;
  long long ldx;
  int N, K;
  const int* tile_expert;
  const int* tile_row0;
  const int* tile_rows;
  const MoeState* state;
  float* out;
  long long ldo;
  const int* meta;      // null: row r of the result is row r of `out`
};

__global__ void __launch_bounds__(kThreads) moe_gemm_f32_kernel(const Params p) {
  __shared__ __align__(16) float xs[kSlice][kTile + kPad];
  __shared__ __align__(16) float ws[kSlice][kTile + kPad];
  if (static_cast<int>(blockIdx.y) >= p.state->n_tiles) return;
  const int expert = p.tile_expert[blockIdx.y], row0 = p.tile_row0[blockIdx.y], rows = p.tile_rows[blockIdx.y];
  const int n0 = blockIdx.x * kTile, tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const int lr = threadIdx.x >> 2, lk = (threadIdx.x & 3) * 4;
  const float* w = p.w + static_cast<long long>(expert) * p.N * p.K;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < p.K; k0 += kSlice) {
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int k = k0 + lk + j;
      xs[lk + j][lr] = lr < rows && k < p.K ? p.x[(row0 + lr) * p.ldx + k] : 0.f;
      ws[lk + j][lr] = n0 + lr < p.N && k < p.K ? w[static_cast<long long>(n0 + lr) * p.K + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kSlice; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&xs[k][ty * 4]);
      const float4 b = *reinterpret_cast<const float4*>(&ws[k][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int r = ty * 4 + i;
    if (r >= rows) break;
    const long long to = p.meta != nullptr ? p.meta[row0 + r] & 0xffffff : row0 + r;
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (n0 + tx * 4 + j < p.N) p.out[to * p.ldo + n0 + tx * 4 + j] = acc[i][j];
  }
}

}  // namespace

const char* moe_gemm_f32(const MoeGemmArgs& a) {
  if (a.n_local_experts <= 0 || a.rows_per_expert <= 0 || a.K <= 0 || a.cap <= 0) return "moe_gemm_f32: empty problem";
  if (a.tile_tokens != kTile || a.max_tiles < 1 || a.max_tiles > 65535) return "moe_gemm_f32: tiles of 64 rows";
  if (a.ldw != a.K || a.tile_expert == nullptr || a.state == nullptr) return "moe_gemm_f32: weights must be contiguous, with a tile table";
  Params p = {};
  p.w = static_cast<const float*>(a.w); p.x = static_cast<const float*>(a.x); p.ldx = a.ldx;
  p.N = static_cast<int>(a.rows_per_expert); p.K = static_cast<int>(a.K);
  p.tile_expert = a.tile_expert; p.tile_row0 = a.tile_row0; p.tile_rows = a.tile_rows; p.state = a.state;
  if (a.epi == kMoeEpiReturn) {
    if (a.recv_meta == nullptr || a.peer_ret[0] == nullptr) return "moe_gemm_f32: bad return set-up";
    p.out = reinterpret_cast<float*>(a.peer_ret[0]); p.ldo = a.rows_per_expert; p.meta = a.recv_meta;
  } else {
    if (a.out == nullptr) return "moe_gemm_f32: no output";
    p.out = static_cast<float*>(a.out); p.ldo = a.ldo;
  }
  const dim3 grid((p.N + kTile - 1) / kTile, a.max_tiles);
  moe_gemm_f32_kernel<<<grid, kThreads, 0, a.stream>>>(p);
  const cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? nullptr : cudaGetErrorString(e);
}

}  // namespace nfb
