// State space on the FP32 pipes: single tokens, and portions token by token; the convolution; the gated norm.
//
// A state column (one value channel, N numbers) belongs to a group of LP lanes, four consecutive numbers per lane and step, so
// that reads are whole 16-byte vectors and the output's contraction over N stays inside the group.
#include "ssd.cuh"

#include "../common/launch.h"

namespace nfb {

namespace {

constexpr int kThreads = 256;

struct Channels {
  int K, x0, b0, c0;       // convolved channels in all; first x, B and C channel of the head
  __device__ __forceinline__ Channels(const SsdArgs& p, int h) {
    const int HV = p.n_heads * p.vdim, g = h / (p.n_heads / p.groups), GN = p.groups * p.state;
    K = HV + 2 * GN;
    x0 = h * p.vdim;
    b0 = HV + g * p.state;
    c0 = b0 + GN;
  }
};

// RI: 16-byte vectors of a column per lane; U: columns of a lane group in flight.  grid: (column slice, head, sequence)
template <typename A, int RI, int U>
__global__ void __launch_bounds__(kThreads) ssd_decode_kernel(const SsdArgs p, int lp_log, int cols) {
  extern __shared__ __align__(16) float smem[];
  const int N = p.state, V = p.vdim, H = p.n_heads, h = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x;
  float* bs = smem;              // [N]
  float* cs = bs + N;            // [N]
  float* xs = cs + N;            // [cols]
  const int LP = 1 << lp_log, grp = tid >> lp_log, l = tid & (LP - 1), groups = kThreads >> lp_log;
  const Channels ch(p, h);
  const int v0 = blockIdx.x * cols, nv = min(cols, V - v0);
  pdl_launch_next();
  pdl_wait_prior();
  const int t = p.cu_seqlens[seq], pos = p.cache_pos[t];
  const long long slot = p.state_slot[seq];
  float* Sg = p.S + ((slot * H + h) * V + v0) * N + l * 4;
  float4 S[U][RI];
  auto fetch = [&](int c0) {
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int c = c0 + u * groups;
#pragma unroll
      for (int i = 0; i < RI; ++i)
        if (c < nv && l * 4 + i * LP * 4 < N) S[u][i] = __ldcs(reinterpret_cast<const float4*>(Sg + static_cast<long long>(c) * N + i * LP * 4));
    }
  };
  fetch(grp);
  const float dt = softplus_of(p.dt[t * p.ld_dt + h]);
  const float em = expm1f(-p.rate[h] * dt);
  {
    const A* in = static_cast<const A*>(p.proj) + t * p.ldp + p.x_off;
    float* ring = p.ring + slot * p.taps * ch.K;
    const bool first = blockIdx.x == 0 && h % (H / p.groups) == 0;      // keeps the inputs of B and C, which other heads read too
    for (int i = tid; i < nv + 2 * N; i += kThreads) {
      const int c = i < nv ? ch.x0 + v0 + i : (i < nv + N ? ch.b0 + i - nv : ch.c0 + i - nv - N);
      const float now = elem_to_f(in[c]);
      float a = fmaf(p.conv_w[static_cast<long long>(p.taps - 1) * ch.K + c], now, p.conv_b[c]);
      for (int b0 = 1; b0 < p.taps; b0 += 3) {              // three earlier inputs at a time, their loads side by side
        float x[3], w[3];
#pragma unroll
        for (int j = 0; j < 3; ++j) {
          const int back = b0 + j;
          const bool there = back < p.taps && back <= pos;
          x[j] = there ? ring[static_cast<long long>((pos - back) % p.taps) * ch.K + c] : 0.f;
          w[j] = there ? p.conv_w[static_cast<long long>(p.taps - 1 - back) * ch.K + c] : 0.f;
        }
#pragma unroll
        for (int j = 0; j < 3; ++j) a = fmaf(w[j], x[j], a);
      }
      a *= sigmoid_of<A>(a);
      (i < nv ? xs + i : (i < nv + N ? bs + i - nv : cs + i - nv - N))[0] = a;
      if (p.write_state && (i < nv || first)) ring[static_cast<long long>(pos % p.taps) * ch.K + c] = now;
    }
  }
  __syncthreads();
  const float skip = p.skip[h];
  A* out = static_cast<A*>(p.out) + t * p.ldo + h * V + v0;
  for (int c0 = grp; c0 < cols; c0 += groups * U) {       // (all lanes of a warp take the same number of turns: the shuffles need them)
    float acc[U];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int c = c0 + u * groups;
      acc[u] = 0.f;
      if (c < nv) {
        const float xv = xs[c] * dt;
#pragma unroll
        for (int i = 0; i < RI; ++i) {
          const int n = l * 4 + i * LP * 4;
          if (n < N) {
            const float4 b = *reinterpret_cast<const float4*>(bs + n), q = *reinterpret_cast<const float4*>(cs + n);
            float4 s = S[u][i];
            s.x = fmaf(em, s.x, fmaf(xv, b.x, s.x));
            s.y = fmaf(em, s.y, fmaf(xv, b.y, s.y));
            s.z = fmaf(em, s.z, fmaf(xv, b.z, s.z));
            s.w = fmaf(em, s.w, fmaf(xv, b.w, s.w));
            if (p.write_state) __stcs(reinterpret_cast<float4*>(Sg + static_cast<long long>(c) * N + i * LP * 4), s);
            acc[u] = fmaf(s.x, q.x, fmaf(s.y, q.y, fmaf(s.z, q.z, fmaf(s.w, q.w, acc[u]))));
          }
        }
      }
    }
    if (c0 + groups * U < cols) fetch(c0 + groups * U);
#pragma unroll
    for (int u = 0; u < U; ++u) {
      for (int o = LP >> 1; o > 0; o >>= 1) acc[u] += __shfl_xor_sync(0xffffffffu, acc[u], o);
      const int c = c0 + u * groups;
      if (l == 0 && c < nv) out[c] = elem_from_f<A>(fmaf(skip, xs[c], acc[u]));
    }
  }
}

// The same with the columns of the CTA in registers over all tokens of the sequence; u comes from ssd_conv.
template <typename A, int RI, int U>
__global__ void __launch_bounds__(kThreads) ssd_recurrent_kernel(const SsdArgs p, int lp_log) {
  extern __shared__ __align__(16) float smem[];
  const int N = p.state, V = p.vdim, H = p.n_heads, h = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x;
  const int LP = 1 << lp_log, grp = tid >> lp_log, l = tid & (LP - 1), groups = kThreads >> lp_log, cols = groups * U;
  const int stride = 2 * N + cols;       // per buffer: B, C, x
  const Channels ch(p, h);
  const int v0 = blockIdx.x * cols, nv = min(cols, V - v0);
  pdl_launch_next();
  pdl_wait_prior();
  const int t0 = p.cu_seqlens[seq], t1 = p.cu_seqlens[seq + 1];
  if (t1 <= t0) return;
  const long long slot = p.state_slot[seq];
  float* Sg = p.S + ((slot * H + h) * V + v0) * N + l * 4;
  float4 S[U][RI];
#pragma unroll
  for (int u = 0; u < U; ++u)
#pragma unroll
    for (int i = 0; i < RI; ++i) {
      const int c = grp + u * groups;
      S[u][i] = c < nv && l * 4 + i * LP * 4 < N ? *reinterpret_cast<const float4*>(Sg + static_cast<long long>(c) * N + i * LP * 4)
                                                 : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  const A* in = static_cast<const A*>(p.u);
  auto stage = [&](int t, int b) {
    float* dst = smem + b * stride;
    const A* row = in + static_cast<long long>(t) * ch.K;
    for (int i = tid; i < 2 * N + nv; i += kThreads)
      dst[i] = elem_to_f(row[i < N ? ch.b0 + i : (i < 2 * N ? ch.c0 + i - N : ch.x0 + v0 + i - 2 * N)]);
  };
  const float rate = p.rate[h], skip = p.skip[h];
  stage(t0, 0);
  float raw = p.dt[t0 * p.ld_dt + h];
  __syncthreads();
  for (int t = t0; t < t1; ++t) {
    const int b = (t - t0) & 1;
    const float dt = softplus_of(raw), em = expm1f(-rate * dt);
    if (t + 1 < t1) {
      stage(t + 1, b ^ 1);
      raw = p.dt[(t + 1) * p.ld_dt + h];
    }
    const float* bs = smem + b * stride;
    const float *cs = bs + N, *xs = cs + N;
    A* out = static_cast<A*>(p.out) + t * p.ldo + h * V + v0;
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int c = grp + u * groups;
      const bool live = c < nv;
      const float x = live ? xs[c] : 0.f, xv = x * dt;
      float acc = 0.f;
#pragma unroll
      for (int i = 0; i < RI; ++i) {
        const int n = l * 4 + i * LP * 4;
        if (n < N) {
          const float4 k = *reinterpret_cast<const float4*>(bs + n), q = *reinterpret_cast<const float4*>(cs + n);
          float4& s = S[u][i];
          s.x = fmaf(em, s.x, fmaf(xv, k.x, s.x));
          s.y = fmaf(em, s.y, fmaf(xv, k.y, s.y));
          s.z = fmaf(em, s.z, fmaf(xv, k.z, s.z));
          s.w = fmaf(em, s.w, fmaf(xv, k.w, s.w));
          acc = fmaf(s.x, q.x, fmaf(s.y, q.y, fmaf(s.z, q.z, fmaf(s.w, q.w, acc))));
        }
      }
      for (int o = LP >> 1; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
      if (l == 0 && live) out[c] = elem_from_f<A>(fmaf(skip, x, acc));
    }
    __syncthreads();
  }
  if (!p.write_state) return;
#pragma unroll
  for (int u = 0; u < U; ++u)
#pragma unroll
    for (int i = 0; i < RI; ++i) {
      const int c = grp + u * groups;
      if (c < nv && l * 4 + i * LP * 4 < N) *reinterpret_cast<float4*>(Sg + static_cast<long long>(c) * N + i * LP * 4) = S[u][i];
    }
  float* ring = p.ring + slot * p.taps * ch.K;        // (its readers have finished: they are the kernel before this one)
  ssd_keep_inputs<A>(p, ring, ch.K, t0, t1, ch.x0 + v0, nv);
  if (blockIdx.x == 0 && h % (H / p.groups) == 0) {
    ssd_keep_inputs<A>(p, ring, ch.K, t0, t1, ch.b0, N);
    ssd_keep_inputs<A>(p, ring, ch.K, t0, t1, ch.c0, N);
  }
}

// Convolution and SiLU of kTokens consecutive tokens x eight channels per thread; tokens of one sequence share their loads.
constexpr int kTokens = 8, kMaxWindow = 4;

template <typename A, int TAPS>
__global__ void __launch_bounds__(128) ssd_conv_kernel(const SsdArgs p, int K) {
  pdl_launch_next();
  pdl_wait_prior();
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * 8;
  if (c >= K) return;
  const int taps = TAPS > 0 ? TAPS : p.taps;
  const A* in = static_cast<const A*>(p.proj) + p.x_off + c;
  float bias[8], w[TAPS > 0 ? TAPS : 1][8];
  load8(p.conv_b + c, bias);
  if constexpr (TAPS > 0) {
#pragma unroll
    for (int j = 0; j < TAPS; ++j) load8(p.conv_w + static_cast<long long>(j) * K + c, w[j]);
  }
  float win[TAPS > 0 ? TAPS : 1][8];      // inputs of the last TAPS tokens, oldest first
  int seq = -1;
  for (int j = 0; j < kTokens; ++j) {
    const int t = blockIdx.x * kTokens + j;
    if (t >= p.T) return;
    const int s = p.token_seq[t], i = t - p.cu_seqlens[s], pos = p.cache_pos[t];
    auto before = [&](int back, float* v) {   // the input `back` positions earlier
      if (back > pos) {
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] = 0.f;
      } else if (back <= i) {
        load8(in + static_cast<long long>(t - back) * p.ldp, v);
      } else {
        load8(p.ring + (static_cast<long long>(p.state_slot[s]) * taps + (pos - back) % taps) * K + c, v);
      }
    };
    float o[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) o[e] = bias[e];
    if constexpr (TAPS > 0) {
      if (s != seq) {
#pragma unroll
        for (int b = 0; b + 1 < TAPS; ++b) before(TAPS - 1 - b, win[b]);
        seq = s;
      } else {
#pragma unroll
        for (int b = 0; b + 1 < TAPS; ++b)
#pragma unroll
          for (int e = 0; e < 8; ++e) win[b][e] = win[b + 1][e];
      }
      load8(in + static_cast<long long>(t) * p.ldp, win[TAPS - 1]);
#pragma unroll
      for (int b = 0; b < TAPS; ++b)
#pragma unroll
        for (int e = 0; e < 8; ++e) o[e] = fmaf(w[b][e], win[b][e], o[e]);
    } else {
      for (int back = taps - 1; back >= 0; --back) {
        float v[8], k[8];
        before(back, v);
        load8(p.conv_w + static_cast<long long>(taps - 1 - back) * K + c, k);
#pragma unroll
        for (int e = 0; e < 8; ++e) o[e] = fmaf(k[e], v[e], o[e]);
      }
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) o[e] *= sigmoid_of<A>(o[e]);
    store8(static_cast<A*>(p.u) + static_cast<long long>(t) * K + c, o);
  }
}

// One CTA per (part of the row, token).  VEC: parts are whole 16-byte vectors and no head is padded.
constexpr int kNormKeep = 4;     // columns (vectors) per thread that stay in registers
template <typename A, bool VEC>
__global__ void __launch_bounds__(256) ssd_norm_kernel(const SsdNormArgs p) {
  __shared__ float red[8];
  pdl_launch_next();
  pdl_wait_prior();
  constexpr int W = VEC ? 8 : 1;
  const int size = p.n_heads * p.vdim_true / p.norm_groups, first = blockIdx.x * size, tid = threadIdx.x, nt = blockDim.x;
  const long long t = blockIdx.y;
  A* y = static_cast<A*>(p.y) + t * p.ldo;
  const A* z = static_cast<const A*>(p.z) + t * p.ldz;
  auto column = [&](int i) {     // of the i-th value of the part
    const int c = first + i;
    return VEC ? c : c / p.vdim_true * p.vdim + c % p.vdim_true;
  };
  auto gated = [&](int c, float* v) {
    if constexpr (VEC) {
      float g[8];
      load8(y + c, v);
      load8(z + c, g);
#pragma unroll
      for (int e = 0; e < 8; ++e) v[e] *= g[e] * sigmoid_of<A>(g[e]);
    } else {
      const float g = elem_to_f(z[c]);
      v[0] = elem_to_f(y[c]) * (g * sigmoid_of<A>(g));
    }
  };
  float keep[kNormKeep][W], ss = 0.f;
#pragma unroll
  for (int k = 0; k < kNormKeep; ++k) {
    const int i = (tid + k * nt) * W;
    if (i < size) {
      gated(column(i), keep[k]);
#pragma unroll
      for (int e = 0; e < W; ++e) ss = fmaf(keep[k][e], keep[k][e], ss);
    }
  }
  for (int i = (tid + kNormKeep * nt) * W; i < size; i += nt * W) {
    float v[W];
    gated(column(i), v);
#pragma unroll
    for (int e = 0; e < W; ++e) ss = fmaf(v[e], v[e], ss);
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  float total = 0.f;
  for (int w = 0; w < nt >> 5; ++w) total += red[w];
  const float inv = 1.f / sqrtf(total / static_cast<float>(size) + p.eps);
  auto finish = [&](int c, float* v) {
    if constexpr (VEC) {
      float w[8];
      load8(p.norm + c, w);
#pragma unroll
      for (int e = 0; e < 8; ++e) v[e] *= inv * w[e];
      store8(y + c, v);
    } else {
      y[c] = elem_from_f<A>(v[0] * inv * p.norm[c]);
    }
  };
#pragma unroll
  for (int k = 0; k < kNormKeep; ++k) {
    const int i = (tid + k * nt) * W;
    if (i < size) finish(column(i), keep[k]);
  }
  for (int i = (tid + kNormKeep * nt) * W; i < size; i += nt * W) {
    float v[W];
    gated(column(i), v);
    finish(column(i), v);
  }
}

int lane_log(int N) {
  int lg = 2;
  while (lg < 5 && (4 << lg) < N) ++lg;
  return lg;
}

template <typename A, int RI, int U>
cudaError_t launch_decode(const SsdArgs& a) {
  const int lg = lane_log(a.state), cols = a.vdim < 64 ? a.vdim : 64;
  const size_t smem = sizeof(float) * (2 * static_cast<size_t>(a.state) + cols);
  return launch_kernel(ssd_decode_kernel<A, RI, U>, dim3((a.vdim + cols - 1) / cols, a.n_heads, a.n_seq), dim3(kThreads), smem, a.stream, a.pdl,
                       1, a, lg, cols);
}
template <typename A, int RI, int U>
cudaError_t launch_recurrent(const SsdArgs& a) {
  const int lg = lane_log(a.state), cols = (kThreads >> lg) * U;
  const size_t smem = 2 * sizeof(float) * (2 * static_cast<size_t>(a.state) + cols);
  return launch_kernel(ssd_recurrent_kernel<A, RI, U>, dim3((a.vdim + cols - 1) / cols, a.n_heads, a.n_seq), dim3(kThreads), smem, a.stream, a.pdl,
                       1, a, lg);
}
template <typename A>
cudaError_t pick_decode(const SsdArgs& a) {
  if (a.state <= 32) return launch_decode<A, 1, 2>(a);
  if (a.state <= 64) return launch_decode<A, 1, 4>(a);
  if (a.state <= 128) return launch_decode<A, 1, 8>(a);
  if (a.state <= 256) return launch_decode<A, 2, 4>(a);
  return launch_decode<A, 4, 2>(a);
}
template <typename A>
cudaError_t pick_recurrent(const SsdArgs& a) {
  if (a.state <= 64) return launch_recurrent<A, 1, 2>(a);
  if (a.state <= 128) return launch_recurrent<A, 1, 4>(a);
  if (a.state <= 256) return launch_recurrent<A, 2, 4>(a);
  return launch_recurrent<A, 4, 4>(a);
}
template <typename A>
cudaError_t pick_conv(const SsdArgs& a) {
  const int K = a.n_heads * a.vdim + 2 * a.groups * a.state;
  const dim3 grid((a.T + kTokens - 1) / kTokens, (K / 8 + 127) / 128);
  switch (a.taps) {
    case 2: return launch_kernel(ssd_conv_kernel<A, 2>, grid, dim3(128), 0, a.stream, a.pdl, 1, a, K);
    case 3: return launch_kernel(ssd_conv_kernel<A, 3>, grid, dim3(128), 0, a.stream, a.pdl, 1, a, K);
    case kMaxWindow: return launch_kernel(ssd_conv_kernel<A, kMaxWindow>, grid, dim3(128), 0, a.stream, a.pdl, 1, a, K);
    default: return launch_kernel(ssd_conv_kernel<A, 0>, grid, dim3(128), 0, a.stream, a.pdl, 1, a, K);
  }
}
template <typename A>
cudaError_t pick_norm(const SsdNormArgs& a) {
  const int size = a.n_heads * a.vdim_true / a.norm_groups;
  const bool vec = a.vdim == a.vdim_true && size % 8 == 0;
  const int per = vec ? size / 8 : size, threads = per >= 256 ? 256 : (per + 31) / 32 * 32;
  const dim3 grid(a.norm_groups, a.T);
  return vec ? launch_kernel(ssd_norm_kernel<A, true>, grid, dim3(threads), 0, a.stream, a.pdl, 1, a)
             : launch_kernel(ssd_norm_kernel<A, false>, grid, dim3(threads), 0, a.stream, a.pdl, 1, a);
}
const char* text(cudaError_t e) { return e == cudaSuccess ? nullptr : cudaGetErrorString(e); }

}  // namespace

const char* ssd_check(const SsdArgs& a) {
  if (a.state < 16 || a.state % 16 || a.state > 512 || a.vdim < 16 || a.vdim % 16)
    return "ssd: state and value widths must be multiples of 16, the state up to 512";
  if (a.n_heads < 1 || a.groups < 1 || a.n_heads % a.groups || a.taps < 1) return "ssd: bad head geometry";
  const int align = a.f32 ? 4 : 8;
  if (a.ldp % align || a.x_off % 8) return "ssd: misaligned rows";
  if (a.n_seq < 1 || a.n_seq > 65535 || a.n_heads > 65535) return "ssd: too many sequences or heads";
  return nullptr;
}

const char* ssd_decode(const SsdArgs& a) {
  if (a.T <= 0) return nullptr;
  if (const char* err = ssd_check(a)) return err;
  if (a.T != a.n_seq) return "ssd: one token per sequence expected";
  return text(a.f32 ? pick_decode<float>(a) : pick_decode<__nv_bfloat16>(a));
}

const char* ssd_conv(const SsdArgs& a) {
  if (a.T <= 0) return nullptr;
  if (const char* err = ssd_check(a)) return err;
  if (a.u == nullptr) return "ssd: no room for the convolved channels";
  return text(a.f32 ? pick_conv<float>(a) : pick_conv<__nv_bfloat16>(a));
}

const char* ssd_recurrent(const SsdArgs& a) {
  if (a.T <= 0) return nullptr;
  if (const char* err = ssd_check(a)) return err;
  if (a.u == nullptr) return "ssd: the convolved channels are missing";
  return text(a.f32 ? pick_recurrent<float>(a) : pick_recurrent<__nv_bfloat16>(a));
}

const char* ssd_gated_norm(const SsdNormArgs& a) {
  if (a.T <= 0) return nullptr;
  if (a.norm_groups < 1 || a.vdim_true < 1 || a.vdim_true > a.vdim || a.n_heads * a.vdim_true % a.norm_groups)
    return "ssd: the channels are no multiple of the norm's groups";
  if (a.ldo % 8 || a.ldz % 8 || a.vdim % 8) return "ssd: misaligned rows";
  for (int t0 = 0; t0 < a.T; t0 += 65535) {      // grid.y limit
    SsdNormArgs b = a;
    const size_t es = a.f32 ? 4 : 2;
    b.T = a.T - t0 < 65535 ? a.T - t0 : 65535;
    b.y = static_cast<char*>(a.y) + es * t0 * a.ldo;
    b.z = static_cast<const char*>(a.z) + es * t0 * a.ldz;
    const cudaError_t e = a.f32 ? pick_norm<float>(b) : pick_norm<__nv_bfloat16>(b);
    if (e != cudaSuccess) return text(e);
  }
  return nullptr;
}

}  // namespace nfb
