// mLSTM, token by token.  One thread-block cluster per (sequence, head); each CTA of the cluster owns VC value columns
// and keeps its slice of the matrix memory in registers over all tokens of the step: a thread holds four columns of
// every (256 / (VC / 4))-th row.  Per token: state update and both contractions (S^T q and n . q) in one pass over the
// registers, one shuffle + shared-memory reduction, then the head norm (sum of squares exchanged inside the cluster),
// the output gate and the store.  Steps with one token per sequence take a variant that streams the state.
#include "mlstm.h"

#include <cooperative_groups.h>

#include "../common/elem.cuh"
#include "../common/launch.h"

namespace nfb {

namespace cg = cooperative_groups;

namespace {

constexpr int kThreads = 256;

template <typename A, int VC, int R>
__global__ void __launch_bounds__(kThreads) mlstm_recurrent_kernel(const MlstmArgs p) {
  constexpr int kCg = VC / 4;                 // column groups
  constexpr int kRg = kThreads / kCg;         // row groups; a thread's rows are rg, rg + kRg, ...
  constexpr int kWarps = kThreads / 32;
  constexpr int kPartials = kCg <= 32 ? kWarps : kRg;   // partial sums per column group after the shuffles
  extern __shared__ __align__(16) float smem[];
  const int D = p.dim, V = p.vdim, H = p.n_heads;
  float* qs = smem;                           // [2][D]
  float* ks = qs + 2 * D;                     // [2][D]
  float* red = ks + 2 * D;                    // [kPartials][kCg][5]
  __shared__ float ss_part[2];                // sum of squares of this CTA's columns, by token parity
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int c = tid % kCg, rg = tid / kCg;
  const int n_cta = gridDim.x;                // cluster size along x
  const int v0 = blockIdx.x * VC;
  const int h = blockIdx.y, seq = blockIdx.z;
  const int col = v0 + c * 4;
  const bool col_ok = col < V;
  cg::cluster_group cluster = cg::this_cluster();

  pdl_launch_next();
  pdl_wait_prior();
  const int t_begin = p.cu_seqlens[seq], t_end = p.cu_seqlens[seq + 1];
  const long long slot = p.state_slot[seq];
  float* Sg = p.S + (slot * H + h) * D * V;
  float* ng = p.n + (slot * H + h) * D;
  float* mg = p.m + slot * H + h;
  float4 S[R];
  float n[R];
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int r = rg + i * kRg;
    S[i] = (r < D && col_ok) ? *reinterpret_cast<const float4*>(Sg + static_cast<long long>(r) * V + col)
                             : make_float4(0.f, 0.f, 0.f, 0.f);
    n[i] = r < D ? ng[r] : 0.f;
  }
  float m = *mg;
  const float inv_cap = 1.f / p.gate_cap;
  const A* proj = static_cast<const A*>(p.proj);
  auto stage = [&](int t, int b) {
    const A* row = proj + t * p.ldp;
    for (int i = tid * 8; i < 2 * D; i += kThreads * 8) {
      float v[8];
      if (i < D) {
        load8(row + p.q_off + h * D + i, v);
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] *= p.q_scale;
        store8(qs + b * D + i, v);
      } else {
        load8(row + p.k_off + h * D + i - D, v);
        store8(ks + b * D + i - D, v);
      }
    }
  };
  if (t_begin < t_end) stage(t_begin, 0);
  __syncthreads();
  for (int t = t_begin; t < t_end; ++t) {
    const int b = (t - t_begin) & 1;
    const float ig = p.gate_cap * tanhf(p.gates[t * p.ldg + p.i_off + h] * inv_cap);
    const float fr = p.gate_cap * tanhf(p.gates[t * p.ldg + p.f_off + h] * inv_cap);
    const float fg = fminf(fr, 0.f) - log1pf(expf(-fabsf(fr)));      // log sigmoid
    const float m_new = fmaxf(fg + m, ig);
    const float da = expf(fg + m - m_new), db = expf(ig - m_new);
    m = m_new;
    float v4[4] = {0.f, 0.f, 0.f, 0.f};
    if (col_ok) {
      const A* vr = proj + t * p.ldp + p.v_off + h * V + col;
#pragma unroll
      for (int j = 0; j < 4; ++j) v4[j] = elem_to_f(vr[j]);
    }
    if (t + 1 < t_end) stage(t + 1, b ^ 1);
    float acc[5] = {0.f, 0.f, 0.f, 0.f, 0.f};
    const float* q = qs + b * D;
    const float* k = ks + b * D;
#pragma unroll
    for (int i = 0; i < R; ++i) {
      const int r = rg + i * kRg;
      if (r < D) {
        const float kb = k[r] * db, qr = q[r];
        S[i].x = fmaf(da, S[i].x, kb * v4[0]);
        S[i].y = fmaf(da, S[i].y, kb * v4[1]);
        S[i].z = fmaf(da, S[i].z, kb * v4[2]);
        S[i].w = fmaf(da, S[i].w, kb * v4[3]);
        n[i] = fmaf(da, n[i], kb);
        acc[0] = fmaf(S[i].x, qr, acc[0]);
        acc[1] = fmaf(S[i].y, qr, acc[1]);
        acc[2] = fmaf(S[i].z, qr, acc[2]);
        acc[3] = fmaf(S[i].w, qr, acc[3]);
        acc[4] = fmaf(n[i], qr, acc[4]);
      }
    }
    if constexpr (kCg < 32) {
#pragma unroll
      for (int e = 0; e < 5; ++e)
#pragma unroll
        for (int o = kCg; o < 32; o <<= 1) acc[e] += __shfl_xor_sync(0xffffffffu, acc[e], o);
    }
    if (kCg >= 32 || lane < kCg) {
      float* dst = red + ((kCg <= 32 ? warp : rg) * kCg + c) * 5;
#pragma unroll
      for (int e = 0; e < 5; ++e) dst[e] = acc[e];
    }
    __syncthreads();
    // the first kCg threads (one warp at most) finish the token's columns
    float o4[4] = {0.f, 0.f, 0.f, 0.f};
    if (tid < 32) {
      float sq = 0.f;
      if (tid < kCg) {
        float den = 0.f;
        for (int w = 0; w < kPartials; ++w) {
          const float* src = red + (w * kCg + tid) * 5;
#pragma unroll
          for (int e = 0; e < 4; ++e) o4[e] += src[e];
          den += src[4];
        }
        const float inv = 1.f / (fmaxf(fabsf(den), expf(-m)) + 1e-6f);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          o4[e] *= inv;
          sq += o4[e] * o4[e];
        }
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
      const A* gr = proj + t * p.ldp + p.g_off + h * V + col;
      A* dst = static_cast<A*>(p.out) + t * p.ldo + h * V + col;
#pragma unroll
      for (int e = 0; e < 4; ++e)
        dst[e] = elem_from_f<A>(o4[e] * inv * p.norm[h * V + col + e] * sigmoid_of<A>(elem_to_f(gr[e])));
    }
  }
  // every CTA of the cluster has read n and m, and nobody still reads a neighbour's shared memory
  if (n_cta > 1) cluster.sync();
  if (!p.write_state) return;
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int r = rg + i * kRg;
    if (r < D && col_ok) *reinterpret_cast<float4*>(Sg + static_cast<long long>(r) * V + col) = S[i];
    if (r < D && c == 0 && blockIdx.x == 0) ng[r] = n[i];
  }
  if (tid == 0 && blockIdx.x == 0) *mg = m;
}

// One token per sequence: the state slice is streamed instead of kept (read, updated, written and contracted row by row),
// so few registers and many CTAs keep HBM busy.
template <typename A, int VC>
__global__ void __launch_bounds__(kThreads, 3) mlstm_decode_kernel(const MlstmArgs p) {
  constexpr int kCg = VC / 4, kRg = kThreads / kCg, kAhead = 8;
  constexpr int kPartials = kThreads / 32;
  extern __shared__ __align__(16) float smem[];
  const int D = p.dim, V = p.vdim, H = p.n_heads;
  float* qs = smem;            // [D]
  float* ks = qs + D;          // [D]
  float* ns = ks + D;          // [D] updated normaliser
  float* red = ns + D;         // [kPartials][kCg][5]
  __shared__ float ss_part;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int c = tid % kCg, rg = tid / kCg, n_cta = gridDim.x;
  const int h = blockIdx.y, seq = blockIdx.z, col = blockIdx.x * VC + c * 4;
  const bool col_ok = col < V;
  cg::cluster_group cluster = cg::this_cluster();
  pdl_launch_next();
  pdl_wait_prior();
  const int t = p.cu_seqlens[seq];
  const long long slot = p.state_slot[seq];
  float* Sg = p.S + (slot * H + h) * D * V + col;
  float* ng = p.n + (slot * H + h) * D;
  float* mg = p.m + slot * H + h;
  float4 S[kAhead];
  auto fetch = [&](int i0) {
#pragma unroll
    for (int j = 0; j < kAhead; ++j) {
      const int r = rg + (i0 + j) * kRg;
      if (r < D && col_ok) S[j] = __ldcs(reinterpret_cast<const float4*>(Sg + static_cast<long long>(r) * V));
    }
  };
  fetch(0);
  const float inv_cap = 1.f / p.gate_cap;
  const float ig = p.gate_cap * tanhf(p.gates[t * p.ldg + p.i_off + h] * inv_cap);
  const float fr = p.gate_cap * tanhf(p.gates[t * p.ldg + p.f_off + h] * inv_cap);
  const float fg = fminf(fr, 0.f) - log1pf(expf(-fabsf(fr)));      // log sigmoid
  const float m_old = *mg;
  const float m = fmaxf(fg + m_old, ig);
  const float da = expf(fg + m_old - m), db = expf(ig - m);
  const A* row = static_cast<const A*>(p.proj) + t * p.ldp;
  for (int i = tid; i < D; i += kThreads) {
    const float k = elem_to_f(row[p.k_off + h * D + i]) * db;
    qs[i] = elem_to_f(row[p.q_off + h * D + i]) * p.q_scale;
    ks[i] = k;
    ns[i] = fmaf(da, ng[i], k);
  }
  float v4[4] = {0.f, 0.f, 0.f, 0.f};
  if (col_ok) {
#pragma unroll
    for (int j = 0; j < 4; ++j) v4[j] = elem_to_f(row[p.v_off + h * V + col + j]);
  }
  __syncthreads();
  float acc[5] = {0.f, 0.f, 0.f, 0.f, 0.f};
  const int per = (D + kRg - 1) / kRg;
  for (int i0 = 0; i0 < per; i0 += kAhead) {
#pragma unroll
    for (int j = 0; j < kAhead; ++j) {
      const int r = rg + (i0 + j) * kRg;
      if (r < D) {
        const float kb = ks[r], qr = qs[r];
        if (col_ok) {
          float4 s = S[j];
          s.x = fmaf(da, s.x, kb * v4[0]);
          s.y = fmaf(da, s.y, kb * v4[1]);
          s.z = fmaf(da, s.z, kb * v4[2]);
          s.w = fmaf(da, s.w, kb * v4[3]);
          if (p.write_state) __stcs(reinterpret_cast<float4*>(Sg + static_cast<long long>(r) * V), s);
          acc[0] = fmaf(s.x, qr, acc[0]);
          acc[1] = fmaf(s.y, qr, acc[1]);
          acc[2] = fmaf(s.z, qr, acc[2]);
          acc[3] = fmaf(s.w, qr, acc[3]);
        }
        acc[4] = fmaf(ns[r], qr, acc[4]);
      }
    }
    if (i0 + kAhead < per) fetch(i0 + kAhead);
  }
  if constexpr (kCg < 32) {
#pragma unroll
    for (int e = 0; e < 5; ++e)
#pragma unroll
      for (int o = kCg; o < 32; o <<= 1) acc[e] += __shfl_xor_sync(0xffffffffu, acc[e], o);
  }
  if (lane < kCg) {
    float* dst = red + (warp * kCg + c) * 5;
#pragma unroll
    for (int e = 0; e < 5; ++e) dst[e] = acc[e];
  }
  __syncthreads();
  float o4[4] = {0.f, 0.f, 0.f, 0.f};
  if (tid < 32) {
    float sq = 0.f;
    if (tid < kCg) {
      float den = 0.f;
      for (int w = 0; w < kPartials; ++w) {
        const float* src = red + (w * kCg + tid) * 5;
#pragma unroll
        for (int e = 0; e < 4; ++e) o4[e] += src[e];
        den += src[4];
      }
      const float inv = 1.f / (fmaxf(fabsf(den), expf(-m)) + 1e-6f);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        o4[e] *= inv;
        sq += o4[e] * o4[e];
      }
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
    const A* gr = row + p.g_off + h * V + col;
    A* dst = static_cast<A*>(p.out) + t * p.ldo + h * V + col;
#pragma unroll
    for (int e = 0; e < 4; ++e)
      dst[e] = elem_from_f<A>(o4[e] * inv * p.norm[h * V + col + e] * sigmoid_of<A>(elem_to_f(gr[e])));
  }
  if (blockIdx.x == 0 && p.write_state) {   // (every CTA of the cluster has read n and m: it passed the cluster barrier)
    for (int i = tid; i < D; i += kThreads) ng[i] = ns[i];
    if (tid == 0) *mg = m;
  }
  if (n_cta > 1) cluster.sync();   // nobody leaves while a neighbour may still read its sum
}

template <typename A, int VC>
cudaError_t launch_decode(const MlstmArgs& a) {
  const size_t smem = sizeof(float) * (3 * static_cast<size_t>(a.dim) + kThreads / 32 * (VC / 4) * 5);
  const int n_cta = (a.vdim + VC - 1) / VC;
  return launch_kernel(mlstm_decode_kernel<A, VC>, dim3(n_cta, a.n_heads, a.n_seq), dim3(kThreads), smem, a.stream, a.pdl, n_cta, a);
}

template <typename A, int VC, int R>
cudaError_t launch(const MlstmArgs& a) {
  constexpr int kCg = VC / 4;
  constexpr int kPartials = kCg <= 32 ? kThreads / 32 : kThreads / kCg;
  const size_t smem = sizeof(float) * (4 * static_cast<size_t>(a.dim) + kPartials * kCg * 5);
  const int n_cta = (a.vdim + VC - 1) / VC;
  return launch_kernel(mlstm_recurrent_kernel<A, VC, R>, dim3(n_cta, a.n_heads, a.n_seq), dim3(kThreads), smem, a.stream, a.pdl,
                       n_cta, a);
}

template <typename A>
const char* dispatch(const MlstmArgs& a) {
  cudaError_t e;
  if (a.one_token) {
    e = a.vdim <= 8 * 64 ? launch_decode<A, 64>(a) : launch_decode<A, 128>(a);
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
    else return "mlstm: value width above 512 needs a key width of at most 256";
  }
  return e == cudaSuccess ? nullptr : cudaGetErrorString(e);
}

}  // namespace

const char* mlstm_recurrent(const MlstmArgs& a) {
  if (a.T <= 0 || a.n_seq <= 0) return nullptr;
  if (a.dim % 16 || a.vdim % 16 || a.dim > 512 || a.vdim > 1024)
    return "mlstm: head widths must be multiples of 16, at most 512 (keys) and 1024 (values)";
  if (a.ldp % 8 || a.ldo % 4 || a.q_off % 8 || a.k_off % 8 || a.v_off % 4 || a.g_off % 4) return "mlstm: misaligned rows";
  if (!(a.gate_cap > 0.f)) return "mlstm: the gate cap must be positive";
  if (a.n_seq > 65535 || a.n_heads > 65535) return "mlstm: too many sequences or heads";
  return a.f32 ? dispatch<float>(a) : dispatch<__nv_bfloat16>(a);
}

}  // namespace nfb
