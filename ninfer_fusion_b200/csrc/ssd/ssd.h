// Selective state space with a scalar decay per head (Mamba-2's state-space duality), between its projections (plain C++ ABI).
// The projection's columns are [z: H V | ... | x: H V | B: G N | C: G N]; x, B and C are the K = H V + 2 G N convolved channels.
//   u_t = silu(conv_b + sum_j conv_w[j] in_(t - taps + 1 + j))                     per channel; zeros before the start
//   dt  = softplus(raw_dt),   S_t = exp(-rate dt) S_(t-1) + dt x_t B_t^T,   y_t = S_t C_t + skip x_t      per head, fp32
// (head h reads B and C of group h / (H / G)), and in a step of its own
//   out = rms of each of `norm_groups` equal parts of (y * silu(z)), times norm
// State of a slot: S [H, V, N] and the last `taps` values of the convolved channels, that of position p in row p mod taps (a
// token only reads rows that no other token of its step replaces, unless its sequence brings several tokens).
// V and N are multiples of 16, zero-padded by the producer.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

namespace nfb {

struct SsdArgs {
  const void* proj = nullptr;       // [T, ldp]
  int64_t ldp = 0;
  int x_off = 0;                    // column of the first convolved channel
  const float* dt = nullptr;        // [T, ld_dt] raw step sizes (bias added)
  int64_t ld_dt = 0;
  int T = 0, n_heads = 0, groups = 0, vdim = 0, state = 0, taps = 0;
  const float* conv_w = nullptr;    // [taps, K], the last row multiplies the newest input
  const float* conv_b = nullptr;    // [K]
  const float* rate = nullptr;      // [H]
  const float* skip = nullptr;      // [H]
  const int* cu_seqlens = nullptr;
  const int* token_seq = nullptr;   // [T]
  const int* cache_pos = nullptr;   // [T]
  const int* state_slot = nullptr;
  int n_seq = 0;
  float* ring = nullptr;            // [slots, taps, K]
  float* S = nullptr;               // [slots, H, V, N]
  void* u = nullptr;                // [T, K] convolved channels in the activation type (portions)
  void* out = nullptr;              // [T, ldo] y
  int64_t ldo = 0;
  bool write_state = true;
  bool f32 = false;
  cudaStream_t stream = nullptr;
  bool pdl = false;
};

// One token per sequence: convolution, state and output in one kernel that streams the state.
const char* ssd_decode(const SsdArgs& a);
// Portions: the convolution, then the recurrence token by token with the state in registers (every size, 32-bit runs) ...
const char* ssd_conv(const SsdArgs& a);
const char* ssd_recurrent(const SsdArgs& a);
// ... or in chunks of 64 tokens on the tensor cores (bf16).
constexpr int kSsdChunk = 64;
bool ssd_chunked_supported(int state, int vdim);
int64_t ssd_chunked_workspace_bytes(int T, int n_seq, int n_heads, int state, int vdim);
const char* ssd_chunked(const SsdArgs& a, void* workspace, int64_t workspace_bytes);

// y [T, ldo] in place.  Columns are H heads of `vdim`, the first vdim_true of each count.
struct SsdNormArgs {
  void* y = nullptr;
  int64_t ldo = 0;
  const void* z = nullptr;          // [T, ldz]
  int64_t ldz = 0;
  const float* norm = nullptr;      // [H * vdim]
  int T = 0, n_heads = 0, vdim = 0, vdim_true = 0, norm_groups = 1;
  float eps = 0.f;
  bool f32 = false;
  cudaStream_t stream = nullptr;
  bool pdl = false;
};
const char* ssd_gated_norm(const SsdNormArgs& a);

const char* ssd_check(const SsdArgs& a);

}  // namespace nfb
