// The row step of decoders with several residual streams: the sublayer's output (a GEMM's result, or the weighted sum over
// its experts) goes into all streams, then the next sublayer's input is read out of them and normed.  One CTA per row; all
// streams of a thread's columns stay in registers, so every stream is read and written once.
#include "stream_rows.h"

#include "../common/glu.cuh"
#include "../common/launch.h"
#include "mixture.cuh"

namespace nfb {

namespace {

// KV: four-column pieces per thread, SM: upper bound of the streams.
template <typename A, int KV, int SM>
__global__ void __launch_bounds__(512) stream_rows_kernel(const StreamArgs p) {
  __shared__ float coef[SM * SM + 2 * SM];     // mix[from][to], w_out, w_in
  __shared__ float red[16];
  const int tid = threadIdx.x, nt = blockDim.x, S = p.S, N = p.N;
  float* w_out = coef + SM * SM;
  float* w_in = w_out + SM;
  for (int i = tid; i < SM * SM; i += nt)
    coef[i] = p.mix != nullptr && i / SM < S && i % SM < S ? p.mix[i / SM * S + i % SM] : 0.f;
  if (tid < SM) {
    w_out[tid] = p.mix != nullptr && tid < S ? p.w_out[tid] : 0.f;
    w_in[tid] = tid < S ? p.w_in[tid] : 0.f;
  }
  pdl_launch_next();
  pdl_wait_prior();
  __syncthreads();
  const long long t = blockIdx.x;
  const A* row = nullptr;
  if (p.x_in == nullptr) {
    int id = p.ids[t];
    id = id < 0 ? 0 : (id >= p.vocab ? p.vocab - 1 : id);
    row = static_cast<const A*>(p.table) + static_cast<long long>(id) * N;
  }
  const float g = p.mix != nullptr ? mixture_gate(p.y, t) : 1.f;
  float u[KV][4], ss = 0.f;
#pragma unroll
  for (int i = 0; i < KV; ++i) {
    const int c = (tid + i * nt) * 4;
#pragma unroll
    for (int e = 0; e < 4; ++e) u[i][e] = 0.f;
    if (c >= N) continue;
    float x[SM][4];
    if (row != nullptr) {
      float v[4];
      load4(row + c, v);
#pragma unroll
      for (int s = 0; s < SM; ++s)
#pragma unroll
        for (int e = 0; e < 4; ++e) x[s][e] = s < S ? v[e] : 0.f;
    } else {
#pragma unroll
      for (int s = 0; s < SM; ++s) {
        if (s < S) {
          load4(p.x_in + (t * S + s) * N + c, x[s]);
        } else {
#pragma unroll
          for (int e = 0; e < 4; ++e) x[s][e] = 0.f;
        }
      }
    }
    if (p.mix != nullptr) {
      float y[4];
      mixture4<A>(p.y, t, c, N, g, y);
#pragma unroll
      for (int to = 0; to < SM; ++to) {
        if (to < S) {
          float v[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) v[e] = w_out[to] * y[e];
#pragma unroll
          for (int s = 0; s < SM; ++s)
#pragma unroll
            for (int e = 0; e < 4; ++e) v[e] = fmaf(coef[s * SM + to], x[s][e], v[e]);
          if (p.x_out != nullptr) store4(p.x_out + (t * S + to) * N + c, v);
#pragma unroll
          for (int e = 0; e < 4; ++e) u[i][e] = fmaf(w_in[to], v[e], u[i][e]);
        }
      }
    } else {
#pragma unroll
      for (int s = 0; s < SM; ++s)
#pragma unroll
        for (int e = 0; e < 4; ++e) u[i][e] = fmaf(w_in[s], x[s][e], u[i][e]);
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) ss = fmaf(u[i][e], u[i][e], ss);
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  float total = 0.f;
  for (int w = 0; w < nt >> 5; ++w) total += red[w];
  const float inv = 1.f / sqrtf(total / static_cast<float>(p.n_true) + p.eps);
#pragma unroll
  for (int i = 0; i < KV; ++i) {
    const int c = (tid + i * nt) * 4;
    if (c < N) {
      float w[4];
      load4(p.w_next + c, w);
#pragma unroll
      for (int e = 0; e < 4; ++e) w[e] = u[i][e] * inv * w[e];
      store4(static_cast<A*>(p.out) + t * p.ld_out + c, w);
    }
  }
}

template <typename A>
__global__ void __launch_bounds__(256) mixture_rows_kernel(const MixtureParts y, float* out, int N) {
  pdl_launch_next();
  pdl_wait_prior();
  const long long t = blockIdx.x;
  const float g = mixture_gate(y, t);
  for (int c = threadIdx.x * 4; c < N; c += blockDim.x * 4) {
    float v[4];
    mixture4<A>(y, t, c, N, g, v);
    store4(out + t * N + c, v);
  }
}

__global__ void __launch_bounds__(256) glu_rows_kernel(const float* g, long long ldg, float* out, long long ldo, int F, GluParams prm) {
  pdl_launch_next();
  pdl_wait_prior();
  const long long t = blockIdx.x;
  for (int c = threadIdx.x; c < F; c += blockDim.x) {
    float a = g[t * ldg + c], b = g[t * ldg + F + c];
    if (prm.limit > 0.f) {
      a = fminf(a, prm.limit);
      b = fminf(fmaxf(b, -prm.limit), prm.limit);
    }
    out[t * ldo + c] = a / (1.f + expf(-prm.slope * a)) * (b + prm.shift);
  }
}

template <typename A, int SM>
cudaError_t pick_width(const StreamArgs& a, cudaStream_t stream, bool pdl) {
  const int pieces = a.N / 4;
  auto threads = [&](int kv) { return dim3(((pieces + kv - 1) / kv + 31) / 32 * 32); };
  if (pieces <= 512) return launch_kernel(stream_rows_kernel<A, 1, SM>, dim3(a.T), threads(1), 0, stream, pdl, 1, a);
  if (pieces <= 1024) return launch_kernel(stream_rows_kernel<A, 2, SM>, dim3(a.T), threads(2), 0, stream, pdl, 1, a);
  if (pieces <= 2048) return launch_kernel(stream_rows_kernel<A, 4, SM>, dim3(a.T), threads(4), 0, stream, pdl, 1, a);
  return launch_kernel(stream_rows_kernel<A, 8, SM>, dim3(a.T), threads(8), 0, stream, pdl, 1, a);
}

template <typename A>
cudaError_t pick_streams(const StreamArgs& a, cudaStream_t stream, bool pdl) {
  if (a.S <= 2) return pick_width<A, 2>(a, stream, pdl);
  if (a.S <= 4) return pick_width<A, 4>(a, stream, pdl);
  if (a.S <= 8) return pick_width<A, 8>(a, stream, pdl);
  return pick_width<A, kMaxStreams>(a, stream, pdl);
}

}  // namespace

const char* stream_rows(const StreamArgs& a, cudaStream_t stream, bool pdl) {
  if (a.T <= 0) return nullptr;
  if (a.N % 8 || a.ld_out % 8 || a.n_true <= 0 || a.n_true > a.N || a.N > 16384) return "stream_rows: bad row width (up to 16384 columns)";
  if (a.S < 1 || a.S > kMaxStreams) return "stream_rows: 1 to 16 streams";
  if (a.w_in == nullptr || a.w_next == nullptr || a.out == nullptr) return "stream_rows: missing weights or output";
  if (a.x_in == nullptr && (a.ids == nullptr || a.table == nullptr || a.vocab < 1)) return "stream_rows: neither streams nor an embedding table";
  if (a.mix != nullptr && a.w_out == nullptr) return "stream_rows: an update needs both of its weights";
  if (a.mix != nullptr && a.y.delta == nullptr && a.y.choice == nullptr) return "stream_rows: an update needs a sublayer's output";
  if (const char* err = bad_mixture(a.y)) return err;
  const cudaError_t e = a.f32 ? pick_streams<float>(a, stream, pdl) : pick_streams<__nv_bfloat16>(a, stream, pdl);
  return e == cudaSuccess ? nullptr : cudaGetErrorString(e);
}

const char* mixture_rows(const MixtureParts& y, float* out, int T, int N, bool f32, cudaStream_t stream, bool pdl) {
  if (T <= 0) return nullptr;
  if (N % 8 || out == nullptr) return "mixture_rows: bad row width";
  if (const char* err = bad_mixture(y)) return err;
  const cudaError_t e = f32 ? launch_kernel(mixture_rows_kernel<float>, dim3(T), dim3(256), 0, stream, pdl, 1, y, out, N)
                            : launch_kernel(mixture_rows_kernel<__nv_bfloat16>, dim3(T), dim3(256), 0, stream, pdl, 1, y, out, N);
  return e == cudaSuccess ? nullptr : cudaGetErrorString(e);
}

const char* glu_rows_f32(const float* g, int64_t ldg, float* out, int64_t ldo, int64_t T, int F, float limit, float slope, float shift,
                         cudaStream_t stream, bool pdl) {
  if (T <= 0 || F <= 0) return nullptr;
  GluParams prm;
  prm.limit = limit; prm.slope = slope; prm.shift = shift;
  const cudaError_t e = launch_kernel(glu_rows_kernel, dim3(static_cast<unsigned>(T)), dim3(256), 0, stream, pdl, 1, g, static_cast<long long>(ldg), out,
                                      static_cast<long long>(ldo), F, prm);
  return e == cudaSuccess ? nullptr : cudaGetErrorString(e);
}

}  // namespace nfb
