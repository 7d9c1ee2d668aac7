// Gated linear memory, token by token.  One thread-block cluster per (sequence, head); each CTA of the cluster owns VC
// value columns and keeps its slice of the state in registers over all tokens of the step: a thread holds four columns of
// every (256 / (VC / 4))-th row.  Per token: the gates of the head's channels, state update and S^T q in one pass over the
// registers, one shuffle + shared-memory reduction, then the head norm (sum of squares exchanged inside the cluster) and
// the store.  Steps with one token per sequence take a variant that streams the state.
#include "gated.h"

#include <cooperative_groups.h>

#include "../common/elem.cuh"
#include "../common/launch.h"

namespace nfb {

namespace cg = cooperative_groups;

namespace {

constexpr int kThreads = 256;

template <typename A>
__device__ __forceinline__ float silu_of(float z) { return z * sigmoid_of<A>(z); }

template <typename A, int VC, int R>
__global__ void __launch_bounds__(kThreads) gated_recurrent_kernel(const GatedArgs p) {
  constexpr int kCg = VC / 4;                 // column groups (at most 32)
  constexpr int kRg = kThreads / kCg;         // row groups; a thread's rows are rg, rg + kRg, ...
  constexpr int kWarps = kThreads / 32;
  extern __shared__ __align__(16) float smem[];
  const int D = p.dim, V = p.vdim, H = p.n_heads;
  float* qs = smem;                           // [2][D]
  float* fs = qs + 2 * D;                     // [2][D]
  float* ks = fs + 2 * D;                     // [2][D]
  float* red = ks + 2 * D;                    // [kWarps][kCg][4]
  __shared__ float ss_part[2];                // sum of squares of this CTA's columns, by token parity
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int c = tid % kCg, rg = tid / kCg;
  const int n_cta = gridDim.x;                // cluster size along x
  const int h = blockIdx.y, seq = blockIdx.z;
  const int col = blockIdx.x * VC + c * 4;
  const bool col_ok = col < V;
  cg::cluster_group cluster = cg::this_cluster();

  pdl_launch_next();
  pdl_wait_prior();
  const int t_begin = p.cu_seqlens[seq], t_end = p.cu_seqlens[seq + 1];
  float* Sg = p.S + (static_cast<long long>(p.state_slot[seq]) * H + h) * D * V;
  float4 S[R];
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int r = rg + i * kRg;
    S[i] = (r < D && col_ok) ? *reinterpret_cast<const float4*>(Sg + static_cast<long long>(r) * V + col)
                             : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  const A* proj = static_cast<const A*>(p.proj);
  auto stage = [&](int t, int b) {
    const A* q = proj + t * p.ldp + p.q_off + h * D;
    const float* g = p.gates + t * p.ldg + h * D;
    for (int i = tid; i < D; i += kThreads) {
      float f, k;
      gated_forget(g[i], p.lower[h * D + i], f, k);
      qs[b * D + i] = silu_of<A>(elem_to_f(q[i]));
      fs[b * D + i] = f;
      ks[b * D + i] = k;
    }
  };
  if (t_begin < t_end) stage(t_begin, 0);
  __syncthreads();
  for (int t = t_begin; t < t_end; ++t) {
    const int b = (t - t_begin) & 1;
    float v4[4] = {0.f, 0.f, 0.f, 0.f};
    if (col_ok) {
      const A* vr = proj + t * p.ldp + p.v_off + h * V + col;
#pragma unroll
      for (int j = 0; j < 4; ++j) v4[j] = elem_to_f(vr[j]);
    }
    if (t + 1 < t_end) stage(t + 1, b ^ 1);
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    const float* q = qs + b * D;
    const float* f = fs + b * D;
    const float* k = ks + b * D;
#pragma unroll
    for (int i = 0; i < R; ++i) {
      const int r = rg + i * kRg;
      if (r < D) {
        const float kr = k[r], fr = f[r], qr = q[r];
        S[i].x = fmaf(fr, S[i].x, kr * v4[0]);
        S[i].y = fmaf(fr, S[i].y, kr * v4[1]);
        S[i].z = fmaf(fr, S[i].z, kr * v4[2]);
        S[i].w = fmaf(fr, S[i].w, kr * v4[3]);
        acc[0] = fmaf(S[i].x, qr, acc[0]);
        acc[1] = fmaf(S[i].y, qr, acc[1]);
        acc[2] = fmaf(S[i].z, qr, acc[2]);
        acc[3] = fmaf(S[i].w, qr, acc[3]);
      }
    }
    if constexpr (kCg < 32) {
#pragma unroll
      for (int e = 0; e < 4; ++e)
#pragma unroll
        for (int o = kCg; o < 32; o <<= 1) acc[e] += __shfl_xor_sync(0xffffffffu, acc[e], o);
    }
    if (lane < kCg) *reinterpret_cast<float4*>(red + (warp * kCg + lane) * 4) = make_float4(acc[0], acc[1], acc[2], acc[3]);
    __syncthreads();
    // one warp finishes the token's columns
    float o4[4] = {0.f, 0.f, 0.f, 0.f};
    if (tid < 32) {
      float sq = 0.f;
      if (tid < kCg) {
#pragma unroll
        for (int w = 0; w < kWarps; ++w) {
          const float4 s = *reinterpret_cast<const float4*>(red + (w * kCg + tid) * 4);
          o4[0] += s.x; o4[1] += s.y; o4[2] += s.z; o4[3] += s.w;
        }
#pragma unroll
        for (int e = 0; e < 4; ++e) sq += o4[e] * o4[e];
      }
      sq = warp_sum(sq);
      if (tid == 0) ss_part[b] = sq;
    }
    float total = 0.f;
    if (n_cta > 1) {
      cluster.sync();
      if (tid < 32) {
        for (int r = 0; r < n_cta; ++r) total += *cluster.map_shared_rank(&ss_part[b], r);
      }
    } else {
      __syncthreads();
      total = ss_part[b];
    }
    if (tid < kCg && col_ok) {
      const float inv = 1.f / sqrtf(total / static_cast<float>(p.vdim_true) + p.eps);
      A* dst = static_cast<A*>(p.out) + t * p.ldo + h * V + col;
#pragma unroll
      for (int e = 0; e < 4; ++e) dst[e] = elem_from_f<A>(o4[e] * inv * p.norm[col + e]);
    }
  }
  if (n_cta > 1) cluster.sync();   // nobody leaves while a neighbour may still read its sum
  if (!p.write_state) return;
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int r = rg + i * kRg;
    if (r < D && col_ok) *reinterpret_cast<float4*>(Sg + static_cast<long long>(r) * V + col) = S[i];
  }
}

// One token per sequence: the state slice is streamed instead of kept (read, updated, written and contracted row by row),
// so few registers and many CTAs keep HBM busy.
template <typename A, int VC>
__global__ void __launch_bounds__(kThreads, 3) gated_decode_kernel(const GatedArgs p) {
  constexpr int kCg = VC / 4, kRg = kThreads / kCg, kAhead = 8, kWarps = kThreads / 32;
  extern __shared__ __align__(16) float smem[];
  const int D = p.dim, V = p.vdim, H = p.n_heads;
  float* qs = smem;            // [D]
  float* fs = qs + D;          // [D]
  float* ks = fs + D;          // [D]
  float* red = ks + D;         // [kWarps][kCg][4]
  __shared__ float ss_part;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int c = tid % kCg, rg = tid / kCg, n_cta = gridDim.x;
  const int h = blockIdx.y, seq = blockIdx.z, col = blockIdx.x * VC + c * 4;
  const bool col_ok = col < V;
  cg::cluster_group cluster = cg::this_cluster();
  pdl_launch_next();
  pdl_wait_prior();
  const int t = p.cu_seqlens[seq];
  float* Sg = p.S + (static_cast<long long>(p.state_slot[seq]) * H + h) * D * V + col;
  float4 S[kAhead];
  auto fetch = [&](int i0) {
#pragma unroll
    for (int j = 0; j < kAhead; ++j) {
      const int r = rg + (i0 + j) * kRg;
      if (r < D && col_ok) S[j] = __ldcs(reinterpret_cast<const float4*>(Sg + static_cast<long long>(r) * V));
    }
  };
  fetch(0);
  const A* row = static_cast<const A*>(p.proj) + t * p.ldp;
  const float* g = p.gates + t * p.ldg + h * D;
  for (int i = tid; i < D; i += kThreads) {
    float f, k;
    gated_forget(g[i], p.lower[h * D + i], f, k);
    qs[i] = silu_of<A>(elem_to_f(row[p.q_off + h * D + i]));
    fs[i] = f;
    ks[i] = k;
  }
  float v4[4] = {0.f, 0.f, 0.f, 0.f};
  if (col_ok) {
#pragma unroll
    for (int j = 0; j < 4; ++j) v4[j] = elem_to_f(row[p.v_off + h * V + col + j]);
  }
  __syncthreads();
  float acc[4] = {0.f, 0.f, 0.f, 0.f};
  const int per = (D + kRg - 1) / kRg;
  for (int i0 = 0; i0 < per; i0 += kAhead) {
#pragma unroll
    for (int j = 0; j < kAhead; ++j) {
      const int r = rg + (i0 + j) * kRg;
      if (r < D && col_ok) {
        const float kr = ks[r], fr = fs[r], qr = qs[r];
        float4 s = S[j];
        s.x = fmaf(fr, s.x, kr * v4[0]);
        s.y = fmaf(fr, s.y, kr * v4[1]);
        s.z = fmaf(fr, s.z, kr * v4[2]);
        s.w = fmaf(fr, s.w, kr * v4[3]);
        if (p.write_state) __stcs(reinterpret_cast<float4*>(Sg + static_cast<long long>(r) * V), s);
        acc[0] = fmaf(s.x, qr, acc[0]);
        acc[1] = fmaf(s.y, qr, acc[1]);
        acc[2] = fmaf(s.z, qr, acc[2]);
        acc[3] = fmaf(s.w, qr, acc[3]);
      }
    }
    if (i0 + kAhead < per) fetch(i0 + kAhead);
  }
  if constexpr (kCg < 32) {
#pragma unroll
    for (int e = 0; e < 4; ++e)
#pragma unroll
      for (int o = kCg; o < 32; o <<= 1) acc[e] += __shfl_xor_sync(0xffffffffu, acc[e], o);
  }
  if (lane < kCg) *reinterpret_cast<float4*>(red + (warp * kCg + lane) * 4) = make_float4(acc[0], acc[1], acc[2], acc[3]);
  __syncthreads();
  float o4[4] = {0.f, 0.f, 0.f, 0.f};
  if (tid < 32) {
    float sq = 0.f;
    if (tid < kCg) {
#pragma unroll
      for (int w = 0; w < kWarps; ++w) {
        const float4 s = *reinterpret_cast<const float4*>(red + (w * kCg + tid) * 4);
        o4[0] += s.x; o4[1] += s.y; o4[2] += s.z; o4[3] += s.w;
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) sq += o4[e] * o4[e];
    }
    sq = warp_sum(sq);
    if (tid == 0) ss_part = sq;
  }
  float total = 0.f;
  if (n_cta > 1) {
    cluster.sync();
    if (tid < 32)
      for (int r = 0; r < n_cta; ++r) total += *cluster.map_shared_rank(&ss_part, r);
  } else {
    __syncthreads();
    total = ss_part;
  }
  if (tid < kCg && col_ok) {
    const float inv = 1.f / sqrtf(total / static_cast<float>(p.vdim_true) + p.eps);
    A* dst = static_cast<A*>(p.out) + t * p.ldo + h * V + col;
#pragma unroll
    for (int e = 0; e < 4; ++e) dst[e] = elem_from_f<A>(o4[e] * inv * p.norm[col + e]);
  }
  if (n_cta > 1) cluster.sync();   // nobody leaves while a neighbour may still read its sum
}

template <typename A, int VC>
cudaError_t launch_decode(const GatedArgs& a) {
  const size_t smem = sizeof(float) * (3 * static_cast<size_t>(a.dim) + kThreads / 32 * VC);
  const int n_cta = (a.vdim + VC - 1) / VC;
  return launch_kernel(gated_decode_kernel<A, VC>, dim3(n_cta, a.n_heads, a.n_seq), dim3(kThreads), smem, a.stream, a.pdl, n_cta, a);
}

template <typename A, int VC, int R>
cudaError_t launch(const GatedArgs& a) {
  const size_t smem = sizeof(float) * (6 * static_cast<size_t>(a.dim) + kThreads / 32 * VC);
  const int n_cta = (a.vdim + VC - 1) / VC;
  return launch_kernel(gated_recurrent_kernel<A, VC, R>, dim3(n_cta, a.n_heads, a.n_seq), dim3(kThreads), smem, a.stream, a.pdl, n_cta, a);
}

template <typename A>
const char* dispatch(const GatedArgs& a) {
  cudaError_t e;
  if (a.one_token) {
    e = a.vdim <= 64 ? launch_decode<A, 64>(a) : launch_decode<A, 128>(a);
    return e == cudaSuccess ? nullptr : cudaGetErrorString(e);
  }
  if (a.vdim <= 8 * 64) {         // 16 row groups
    if (a.dim <= 64) e = launch<A, 64, 4>(a);
    else if (a.dim <= 128) e = launch<A, 64, 8>(a);
    else if (a.dim <= 256) e = launch<A, 64, 16>(a);
    else e = launch<A, 64, 32>(a);
  } else {                        // 8 row groups
    if (a.dim <= 128) e = launch<A, 128, 16>(a);
    else if (a.dim <= 256) e = launch<A, 128, 32>(a);
    else return "gated memory: value width above 512 needs a channel width of at most 256";
  }
  return e == cudaSuccess ? nullptr : cudaGetErrorString(e);
}

}  // namespace

const char* gated_recurrent(const GatedArgs& a) {
  if (a.T <= 0 || a.n_seq <= 0) return nullptr;
  if (a.dim % 16 || a.vdim % 16 || a.dim > 512 || a.vdim > 1024)
    return "gated memory: head widths must be multiples of 16, at most 512 (channels) and 1024 (values)";
  if (a.ldp % 8 || a.ldo % 4 || a.q_off % 8 || a.v_off % 4) return "gated memory: misaligned rows";
  if (a.n_seq > 65535 || a.n_heads > 65535) return "gated memory: too many sequences or heads";
  return a.f32 ? dispatch<float>(a) : dispatch<__nv_bfloat16>(a);
}

}  // namespace nfb
