// Griffin's recurrent block between its projections (plain C++ ABI).  Per channel, with x the recurrent branch's input and y
// the other branch's:
//   u_t = conv_b + sum_j conv_w[j] x_(t - taps + 1 + j)
//   r = sigmoid(raw_r), i = sigmoid(raw_i)                       raw: block-diagonal maps of u plus biases
//   log a = -r rate,   S <- a S + sqrt(1 - a^2) i u              (rate = 8 softplus(lam), all of this in fp32)
//   out_t = S gelu_tanh(y_t)
// State of a slot: S and the last `taps` values of x, that of position p in row p mod taps (a token only reads rows that no
// token of its step with another position mod taps has to wait for).
// Channels lie in `blocks` parts of `width` (a multiple of 16, zero-padded by the producer).
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

namespace nfb {

struct RglruArgs {
  const void* proj = nullptr;       // [T, ldp]: y at column 0, x at column C = blocks * width
  int64_t ldp = 0;
  int T = 0, blocks = 0, width = 0, taps = 0;
  const float* conv_w = nullptr;    // [taps, C], the last row multiplies the newest input
  const float* conv_b = nullptr;    // [C]
  const void* gate_w = nullptr;     // [blocks, 2 width, width] rows of r, then of i, in the activation type (fused kernels)
  const float* gate_b = nullptr;    // [blocks, 2 width]
  const float* rate = nullptr;      // [C]
  const int* cu_seqlens = nullptr;
  const int* token_seq = nullptr;   // [T]
  const int* cache_pos = nullptr;   // [T]
  const int* state_slot = nullptr;
  int n_seq = 0;
  float* ring = nullptr;            // [slots, taps, C]
  float* S = nullptr;               // [slots, C]
  void* out = nullptr;              // [T, ldo]
  int64_t ldo = 0;
  bool write_state = true;
  bool f32 = false;
  cudaStream_t stream = nullptr;
  bool pdl = false;
};

// In steps, for every size and 32-bit runs: u [T, C] in the activation type; the caller makes the gates' raw values
// [T, blocks, 2 width] (with biases); the recurrence walks a sequence's tokens one by one.
const char* rglru_conv(const RglruArgs& a, void* u);
const char* rglru_scan(const RglruArgs& a, const void* u, const float* raw);

// Convolution and gates inside (bf16; blocks of up to about 500 channels).
bool rglru_fused_supported(int width);
// One token per sequence.
const char* rglru_decode(const RglruArgs& a);
// Query blocks: up to 64 consecutive tokens of one sequence each, a sequence's blocks in order and all but its last of 64.
int64_t rglru_chunked_workspace_bytes(int T, int n_seq, int channels);
const char* rglru_chunked(const RglruArgs& a, const int* blk_start, const int* blk_count, int n_blocks, void* workspace, int64_t bytes);

}  // namespace nfb
