// The row step of decoders with norms around every sublayer: residual update with a grouped norm of the sublayer's output,
// the next sublayer's grouped norm, and the causal convolution in front of a mixer, in one pass over the row.
//
// Without a convolution a CTA is one row.  With one, a CTA walks kBlockTokens consecutive tokens of a sequence and keeps
// the last taps - 1 normed rows in shared memory (every thread reads back only its own columns); the rows before its first
// token are recomputed from the step's inputs, or come from the sequence's slot at the step's start.  The CTA of a
// sequence's first tokens is the only one that reads the slot, so it is also the one that stores the new history.
#include "rows32.h"

#include "../common/elem.cuh"
#include "../common/launch.h"

namespace nfb {

namespace {

constexpr int kBlockTokens = 8;

// How the sum of squares of a group is taken: whole warps lie in one group / whole 8-column vectors do / neither.
enum GroupMode : int { kWarpGroups = 0, kVectorGroups = 1, kColumnGroups = 2 };

// 1 / rms of the group of each of the thread's columns: inv[i][j] for column j of vector i (j = 0 stands for all eight
// unless the mode is kColumnGroups).  `part` and `inv_s` are shared, `part` alternates between two arrays from call to call;
// every thread of the CTA takes part.
template <int KV, int MODE>
__device__ __forceinline__ void group_inv(const float (&v)[KV][8], float (&inv)[KV][MODE == kColumnGroups ? 8 : 1], float* part,
                                          float* inv_s, const SandwichArgs& p, int group_size) {
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, nt = blockDim.x;
  constexpr int kUnit = MODE == kWarpGroups ? 256 : (MODE == kVectorGroups ? 8 : 1);
#pragma unroll
  for (int i = 0; i < KV; ++i) {
    const int vec = tid + i * nt;
    if constexpr (MODE == kColumnGroups) {
      if (vec * 8 < p.N) {
#pragma unroll
        for (int j = 0; j < 8; ++j) part[vec * 8 + j] = v[i][j] * v[i][j];
      }
    } else {
      float s = 0.f;
#pragma unroll
      for (int j = 0; j < 8; ++j) s += v[i][j] * v[i][j];
      if constexpr (MODE == kWarpGroups) {
        s = warp_sum(s);
        if (lane == 0 && vec * 8 < p.N) part[vec >> 5] = s;
      } else if (vec * 8 < p.N) {
        part[vec] = s;
      }
    }
  }
  __syncthreads();
  const int units = group_size / kUnit;
  const float inv_n = 1.f / static_cast<float>(group_size);
  if constexpr (MODE == kWarpGroups) {      // few partial sums per group: every thread adds its own up
#pragma unroll
    for (int i = 0; i < KV; ++i) {
      const int c = (tid + i * nt) * 8;
      if (c < p.N) {
        const float* src = part + c / group_size * units;
        float s = 0.f;
        for (int u = 0; u < units; ++u) s += src[u];
        inv[i][0] = 1.f / sqrtf(s * inv_n + p.eps);
      }
    }
    return;
  }
  for (int g = warp; g < p.groups; g += nt >> 5) {
    float s = 0.f;
    for (int u = lane; u < units; u += 32) s += part[g * units + u];
    s = warp_sum(s);
    if (lane == 0) inv_s[g] = 1.f / sqrtf(s * inv_n + p.eps);
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < KV; ++i) {
    const int c = (tid + i * nt) * 8;
    if (c < p.N) {
#pragma unroll
      for (int j = 0; j < (MODE == kColumnGroups ? 8 : 1); ++j) inv[i][j] = inv_s[min((c + j) / group_size, p.groups - 1)];
    }
  }
}

template <typename A, int KV, int MODE, bool CONV>
__global__ void __launch_bounds__(512, KV == 1 ? 2 : 1) sandwich_kernel(const SandwichArgs p) {
  extern __shared__ __align__(16) float smem[];
  const int group_size = p.n_true / p.groups;
  const int n_part = MODE == kWarpGroups ? (p.N + 255) / 256 : (MODE == kVectorGroups ? p.N / 8 : p.N);
  float* part = smem;
  float* inv_s = part + (2 * n_part + 3) / 4 * 4;
  float* hist = inv_s + (p.groups + 3) / 4 * 4;      // [taps - 1][N], row of token i at i mod (taps - 1)
  const int tid = threadIdx.x, nt = blockDim.x;
  pdl_launch_next();
  pdl_wait_prior();

  float h[KV][8];
  int turn = 0;
  // h of row t; `store`: the row's new residual is kept
  auto row = [&](long long t, bool store) {
    float inv[KV][MODE == kColumnGroups ? 8 : 1];
    float x[KV][8];
#pragma unroll
    for (int i = 0; i < KV; ++i) {
      const int c = (tid + i * nt) * 8;
#pragma unroll
      for (int j = 0; j < 8; ++j) h[i][j] = 0.f;
      if (c < p.N) {
        load8(p.x_in + t * p.N + c, x[i]);
        if (p.delta != nullptr) {
          load8(p.delta + t * p.N + c, h[i]);
        } else {
#pragma unroll
          for (int j = 0; j < 8; ++j) h[i][j] = x[i][j];
        }
      }
    }
    if (p.delta != nullptr) {
      group_inv<KV, MODE>(h, inv, part + (turn ^= 1) * n_part, inv_s, p, group_size);
#pragma unroll
      for (int i = 0; i < KV; ++i) {
        const int c = (tid + i * nt) * 8;
        if (c < p.N) {
          float w[8];
          load8(p.w_post + c, w);
#pragma unroll
          for (int j = 0; j < 8; ++j) h[i][j] = x[i][j] + p.mult * (h[i][j] * inv[i][MODE == kColumnGroups ? j : 0] * w[j]);
          if (store) store8(p.x_out + t * p.N + c, h[i]);
        }
      }
    }
    if (p.w_next != nullptr) {
      group_inv<KV, MODE>(h, inv, part + (turn ^= 1) * n_part, inv_s, p, group_size);
#pragma unroll
      for (int i = 0; i < KV; ++i) {
        const int c = (tid + i * nt) * 8;
        if (c < p.N) {
          float w[8];
          load8(p.w_next + c, w);
#pragma unroll
          for (int j = 0; j < 8; ++j) h[i][j] = h[i][j] * inv[i][MODE == kColumnGroups ? j : 0] * w[j];
        }
      }
    }
  };
  A* out = static_cast<A*>(p.out);
  if constexpr (!CONV) {
    const long long t = blockIdx.x;
    row(t, true);
#pragma unroll
    for (int i = 0; i < KV; ++i) {
      const int c = (tid + i * nt) * 8;
      if (c < p.N) store8(out + t * p.ld_out + c, h[i]);
    }
  } else {
    const int seq = blockIdx.y, tb = p.cu_seqlens[seq], n = p.cu_seqlens[seq + 1] - tb;
    const int K = p.taps - 1, R = max(kBlockTokens, K);
    const int i0 = blockIdx.x * R, i1 = min(n, i0 + R);
    if (i0 >= n) return;
    float* state = K > 0 ? p.conv_state + static_cast<long long>(p.state_slot[seq]) * K * p.N : nullptr;
    auto keep = [&](float* dst) {
#pragma unroll
      for (int i = 0; i < KV; ++i) {
        const int c = (tid + i * nt) * 8;
        if (c < p.N) store8(dst + c, h[i]);
      }
    };
    // history rows of tokens i0 - K .. i0 - 1
    for (int j = 0; j < K; ++j) {
      const int i = i0 - K + j;
      float* dst = hist + ((i + K) % K) * p.N;
      if (i >= 0) {
        row(tb + i, false);
        keep(dst);
      } else {
#pragma unroll
        for (int k = 0; k < KV; ++k) {
          const int c = (tid + k * nt) * 8;
          if (c < p.N) {
            float v[8];
            load8(state + static_cast<long long>(j) * p.N + c, v);
            store8(dst + c, v);
          }
        }
      }
    }
    for (int i = i0; i < i1; ++i) {
      row(tb + i, true);
#pragma unroll
      for (int k = 0; k < KV; ++k) {
        const int c = (tid + k * nt) * 8;
        if (c < p.N) {
          float o[8], w[8];
          load8(p.conv_w + static_cast<long long>(K) * p.N + c, w);
#pragma unroll
          for (int j = 0; j < 8; ++j) o[j] = fmaf(w[j], h[k][j], h[k][j]);
          for (int tap = 0; tap < K; ++tap) {        // tap K - 1 is the token before
            float y[8];
            load8(hist + ((i + tap) % K) * p.N + c, y);
            load8(p.conv_w + static_cast<long long>(tap) * p.N + c, w);
#pragma unroll
            for (int j = 0; j < 8; ++j) o[j] = fmaf(w[j], y[j], o[j]);
          }
          store8(out + (tb + i) * p.ld_out + c, o);
        }
      }
      if (K > 0) keep(hist + (i % K) * p.N);
    }
    if (i0 != 0 || K == 0 || !p.write_state) return;
    for (int j = 0; j < K; ++j) {
      const int i = n - K + j;                        // token whose row becomes state row j
      if (i < i1) {                                   // among the rows kept here (i >= -K)
        const float* src = hist + ((i + K) % K) * p.N;
        if (i1 == n) {
#pragma unroll
          for (int k = 0; k < KV; ++k) {
            const int c = (tid + k * nt) * 8;
            if (c < p.N) {
              float v[8];
              load8(src + c, v);
              store8(state + static_cast<long long>(j) * p.N + c, v);
            }
          }
          continue;
        }
      }
      row(tb + i, false);
      keep(state + static_cast<long long>(j) * p.N);
    }
  }
}

template <typename A, int KV, int MODE>
cudaError_t launch(const SandwichArgs& a, int threads, cudaStream_t stream, bool pdl) {
  const int n_part = MODE == kWarpGroups ? (a.N + 255) / 256 : (MODE == kVectorGroups ? a.N / 8 : a.N);
  size_t smem = sizeof(float) * ((2 * n_part + 3) / 4 * 4 + (a.groups + 3) / 4 * 4);
  if (a.conv_w == nullptr) return launch_kernel(sandwich_kernel<A, KV, MODE, false>, dim3(a.T), dim3(threads), smem, stream, pdl, 1, a);
  smem += sizeof(float) * static_cast<size_t>(a.taps - 1) * a.N;
  auto kern = sandwich_kernel<A, KV, MODE, true>;
  if (smem > 48 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return e;
  }
  const int R = a.taps - 1 > kBlockTokens ? a.taps - 1 : kBlockTokens;
  return launch_kernel(kern, dim3((a.max_seq_tokens + R - 1) / R, a.n_seq), dim3(threads), smem, stream, pdl, 1, a);
}

template <typename A, int KV>
cudaError_t pick_mode(const SandwichArgs& a, int threads, cudaStream_t stream, bool pdl) {
  const int gs = a.n_true / a.groups;
  if (gs % 256 == 0) return launch<A, KV, kWarpGroups>(a, threads, stream, pdl);
  if (gs % 8 == 0) return launch<A, KV, kVectorGroups>(a, threads, stream, pdl);
  return launch<A, KV, kColumnGroups>(a, threads, stream, pdl);
}

template <typename A>
cudaError_t pick_width(const SandwichArgs& a, cudaStream_t stream, bool pdl) {
  const int vecs = a.N / 8;
  if (vecs <= 512) return pick_mode<A, 1>(a, (vecs + 31) / 32 * 32, stream, pdl);
  if (vecs <= 1024) return pick_mode<A, 2>(a, ((vecs + 1) / 2 + 31) / 32 * 32, stream, pdl);
  return pick_mode<A, 4>(a, 512, stream, pdl);
}

}  // namespace

const char* sandwich_rows(const SandwichArgs& a, cudaStream_t stream, bool pdl) {
  if (a.T <= 0) return nullptr;
  if (a.N % 8 || a.ld_out % 8 || a.n_true <= 0 || a.n_true > a.N || a.N > 16384) return "sandwich_rows: bad row width (up to 16384 columns)";
  if (a.groups < 1 || a.n_true % a.groups || a.groups > 4096) return "sandwich_rows: the width is not a multiple of the groups";
  if (a.delta != nullptr && (a.w_post == nullptr || a.x_out == nullptr)) return "sandwich_rows: a sublayer output needs its norm and a destination";
  if (a.conv_w != nullptr) {
    if (a.taps < 1 || a.n_seq <= 0 || a.max_seq_tokens <= 0 || a.n_seq > 65535) return "sandwich_rows: bad convolution";
    if (static_cast<long long>(a.taps - 1) * a.N > 40 * 1024) return "sandwich_rows: (taps - 1) x width exceeds the shared memory of a block";
    if (a.delta != nullptr && a.max_seq_tokens > 1 && a.x_in == a.x_out) return "sandwich_rows: with a convolution the new rows need their own buffer";
  }
  const cudaError_t e = a.f32 ? pick_width<float>(a, stream, pdl) : pick_width<__nv_bfloat16>(a, stream, pdl);
  return e == cudaSuccess ? nullptr : cudaGetErrorString(e);
}

}  // namespace nfb
