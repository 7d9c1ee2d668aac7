// State space over prompt portions, in chunks of 64 tokens on the tensor cores.  With l_t = -rate dt_t and F_t the sum of l over
// the chunk up to t, the recurrence unrolls to
//   y_t = exp(F_t) S_0 C_t + sum_{s <= t} exp(F_t - F_s) dt_s (B_s . C_t) x_s + skip x_t          (every exponent is <= 0)
// Three kernels after the convolution:
//   contrib  one CTA per (chunk, head, 64 channels, 128 state columns): what a chunk adds, U = sum_s exp(F_L - F_s) dt_s x_s B_s^T
//   scan     elementwise over the chunks of a sequence: the state at every chunk's start, kept in fp32 and handed on as bf16
//            hi + lo rows; the sequence's new state and last inputs
//   output   one CTA per (chunk, up to kHeads heads of a group, 64 channels): C . B is the same for all heads of a group and stays
//            in registers while the CTA walks over them
// Weighted x and the state enter the MMAs as hi + lo pairs, so steps, decays and state keep about 17 bits.
#include "ssd.cuh"

#include "../common/launch.h"
#include "../common/mma_sync.cuh"

namespace nfb {

namespace {

using bf16 = __nv_bfloat16;
constexpr int L = kSsdChunk;
constexpr int kVSlice = 64, kNSlice = 128, kHeads = 4;
constexpr int kSmemLimit = 220 * 1024;

struct Work {
  float* c_F = nullptr;      // [NC, H] F at the chunk's end
  float* U = nullptr;        // [NC, H, V, N]
  bf16* Sh = nullptr;        // [NC, H, V, N] state at the chunk's start, high and low part
  bf16* Sl = nullptr;
};

// Chunk slots: those of sequence s start at cu[s] / 64 + s, which leaves room for a ragged last chunk of every sequence.
__device__ __forceinline__ int first_slot(const SsdArgs& p, int s) { return p.cu_seqlens[s] / L + s; }

struct Chunk {
  int seq, t0, len;          // len <= 0: an unused slot
  __device__ __forceinline__ Chunk(const SsdArgs& p, int slot) {
    int lo = 0, hi = p.n_seq - 1;
    while (lo < hi) {
      const int mid = (lo + hi + 1) / 2;
      if (first_slot(p, mid) <= slot) lo = mid; else hi = mid - 1;
    }
    seq = lo;
    t0 = p.cu_seqlens[seq] + (slot - first_slot(p, seq)) * L;
    len = min(L, p.cu_seqlens[seq + 1] - t0);
  }
};

// F and dt of the chunk's tokens of one head, by one warp; tokens past the end have dt = 0 and the F of the last one.
__device__ __forceinline__ void chunk_steps(const SsdArgs& p, const Chunk& ck, int h, float* F, float* dts) {
  const int lane = threadIdx.x & 31;
  const float rate = p.rate[h];
  float l[2];
#pragma unroll
  for (int j = 0; j < 2; ++j) {
    const int i = 2 * lane + j;
    const float dt = i < ck.len ? softplus_of(p.dt[(ck.t0 + i) * p.ld_dt + h]) : 0.f;
    dts[i] = dt;
    l[j] = -rate * dt;
  }
  float sum = l[0] + l[1];
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float y = __shfl_up_sync(0xffffffffu, sum, o);
    if (lane >= o) sum += y;
  }
  F[2 * lane + 1] = sum;
  F[2 * lane] = sum - l[1];
}

// Rows of `width` (a multiple of 8) columns out of a row-major array into shared memory; rows from `rows` on and columns from
// `valid` on become zero.
__device__ __forceinline__ void stage_rows(uint32_t dst, int ld_dst, const bf16* src, long long ld_src, int n_rows, int rows, int width, int valid) {
  const int vecs = width / 8;
  for (int i = threadIdx.x; i < n_rows * vecs; i += blockDim.x) {
    const int r = i / vecs, c = (i % vecs) * 8;
    const bool ok = r < rows && c < valid;
    cp_async16(dst + (r * ld_dst + c) * 2, ok ? src + r * ld_src + c : src, ok);
  }
}

// 8 warps: 16 channels x 64 state columns each.  grid: (chunk slot, head, channel slices x state slices)
__global__ void __launch_bounds__(256) ssd_contrib_kernel(const SsdArgs p, const Work w) {
  constexpr int ldx = kVSlice + 8, ldb = kNSlice + 8;
  extern __shared__ __align__(16) bf16 smem[];
  __shared__ float F[L], dts[L];
  bf16* xh = smem;                 // [L][ldx] weighted x, high part (first as it comes)
  bf16* xl = xh + L * ldx;         // low part
  bf16* bs = xl + L * ldx;         // [L][ldb]
  const int H = p.n_heads, V = p.vdim, N = p.state, h = blockIdx.y, g = h / (H / p.groups);
  const int n_vs = (V + kVSlice - 1) / kVSlice, v0 = (blockIdx.z % n_vs) * kVSlice, n0 = (blockIdx.z / n_vs) * kNSlice;
  const int K = H * V + 2 * p.groups * N;
  pdl_launch_next();
  pdl_wait_prior();
  const Chunk ck(p, blockIdx.x);
  if (ck.len <= 0) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const bf16* u = static_cast<const bf16*>(p.u) + static_cast<long long>(ck.t0) * K;
  stage_rows(smem_u32(xh), ldx, u + h * V + v0, K, L, ck.len, kVSlice, V - v0);
  cp_async_commit();
  stage_rows(smem_u32(bs), ldb, u + H * V + g * N + n0, K, L, ck.len, kNSlice, N - n0);
  cp_async_commit();
  if (warp == 0) chunk_steps(p, ck, h, F, dts);
  cp_async_wait<1>();
  __syncthreads();
  const float end = F[L - 1];
  if (blockIdx.z == 0 && tid == 0) w.c_F[static_cast<long long>(blockIdx.x) * H + h] = end;
  for (int i = tid; i < L * (kVSlice / 8); i += 256) {
    const int s = i / (kVSlice / 8), c = (i % (kVSlice / 8)) * 8;
    const float f = expf(end - F[s]) * dts[s];
    float x[8], hi[8], lo[8];
    load8(xh + s * ldx + c, x);
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      x[j] *= f;
      hi[j] = __bfloat162float(__float2bfloat16(x[j]));
      lo[j] = x[j] - hi[j];
    }
    store8(xh + s * ldx + c, hi);
    store8(xl + s * ldx + c, lo);
  }
  cp_async_wait<0>();
  __syncthreads();
  const int m = (warp & 3) * 16, nn = (warp >> 2) * 64;       // first channel and state column of the warp
  if (v0 + m >= V || n0 + nn >= N) return;
  float acc[8][4];
#pragma unroll
  for (int n = 0; n < 8; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[n][e] = 0.f;
  const int arow = (lane & 7) + (lane >> 4) * 8, acol = ((lane >> 3) & 1) * 8;
#pragma unroll
  for (int k = 0; k < L; k += 16) {
    uint32_t ah[4], al[4];
    ldsm_x4_trans(smem_u32(xh) + ((k + arow) * ldx + m + acol) * 2, ah);
    ldsm_x4_trans(smem_u32(xl) + ((k + arow) * ldx + m + acol) * 2, al);
#pragma unroll
    for (int n = 0; n < 4; ++n) {
      uint32_t b[4];
      ldsm_x4_trans(smem_u32(bs) + ((k + (lane & 15)) * ldb + nn + n * 16 + (lane >> 4) * 8) * 2, b);
      mma_bf16_16816(acc[2 * n], ah, b[0], b[1]);
      mma_bf16_16816(acc[2 * n + 1], ah, b[2], b[3]);
      mma_bf16_16816(acc[2 * n], al, b[0], b[1]);
      mma_bf16_16816(acc[2 * n + 1], al, b[2], b[3]);
    }
  }
  const int v = v0 + m + (lane >> 2), n = n0 + nn + (lane & 3) * 2;
  float* dst = w.U + ((static_cast<long long>(blockIdx.x) * H + h) * V + v) * N + n;
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    if (n + i * 8 < N) {
      *reinterpret_cast<float2*>(dst + i * 8) = make_float2(acc[i][0], acc[i][1]);
      *reinterpret_cast<float2*>(dst + 8LL * N + i * 8) = make_float2(acc[i][2], acc[i][3]);
    }
  }
}

// Four state elements per thread.  grid: (blocks over V x N / 4 and one for the last inputs, head, sequence)
__global__ void __launch_bounds__(256) ssd_scan_kernel(const SsdArgs p, const Work w) {
  pdl_launch_next();
  pdl_wait_prior();
  const int H = p.n_heads, V = p.vdim, N = p.state, h = blockIdx.y, seq = blockIdx.z;
  const int t0 = p.cu_seqlens[seq], t1 = p.cu_seqlens[seq + 1], nc = (t1 - t0 + L - 1) / L;
  const long long slot = p.state_slot[seq];
  if (blockIdx.x == gridDim.x - 1) {
    if (!p.write_state) return;
    const int K = H * V + 2 * p.groups * N, R = H / p.groups;
    float* ring = p.ring + slot * p.taps * K;
    ssd_keep_inputs<bf16>(p, ring, K, t0, t1, h * V, V);
    if (h % R == 0) {
      ssd_keep_inputs<bf16>(p, ring, K, t0, t1, H * V + h / R * N, N);
      ssd_keep_inputs<bf16>(p, ring, K, t0, t1, H * V + (p.groups + h / R) * N, N);
    }
    return;
  }
  const int at = (blockIdx.x * blockDim.x + threadIdx.x) * 4;
  if (at >= V * N) return;
  float* Sg = p.S + (slot * H + h) * V * N + at;
  float4 s = *reinterpret_cast<const float4*>(Sg);
  const long long step = static_cast<long long>(H) * V * N, first = (static_cast<long long>(first_slot(p, seq)) * H + h) * V * N + at;
  const float* cF = w.c_F + static_cast<long long>(first_slot(p, seq)) * H + h;
  constexpr int kAhead = 4;
  for (int c0 = 0; c0 < nc; c0 += kAhead) {
    float4 u[kAhead];
    float f[kAhead];
#pragma unroll
    for (int j = 0; j < kAhead; ++j)
      if (c0 + j < nc) {
        u[j] = __ldcs(reinterpret_cast<const float4*>(w.U + first + (c0 + j) * step));
        f[j] = cF[static_cast<long long>(c0 + j) * H];
      }
#pragma unroll
    for (int j = 0; j < kAhead; ++j)
      if (c0 + j < nc) {
        const float hx = __bfloat162float(__float2bfloat16(s.x)), hy = __bfloat162float(__float2bfloat16(s.y));
        const float hz = __bfloat162float(__float2bfloat16(s.z)), hw = __bfloat162float(__float2bfloat16(s.w));
        const long long o = first + (c0 + j) * step;
        *reinterpret_cast<uint2*>(w.Sh + o) = make_uint2(pack_bf16x2(hx, hy), pack_bf16x2(hz, hw));
        *reinterpret_cast<uint2*>(w.Sl + o) = make_uint2(pack_bf16x2(s.x - hx, s.y - hy), pack_bf16x2(s.z - hz, s.w - hw));
        const float em = expm1f(f[j]);
        s.x = fmaf(em, s.x, s.x + u[j].x);
        s.y = fmaf(em, s.y, s.y + u[j].y);
        s.z = fmaf(em, s.z, s.z + u[j].z);
        s.w = fmaf(em, s.w, s.w + u[j].w);
      }
  }
  if (p.write_state) *reinterpret_cast<float4*>(Sg) = s;
}

// 4 warps: 16 tokens each.  grid: (chunk slot, head blocks of all groups, channel slices)
__global__ void __launch_bounds__(128) ssd_output_kernel(const SsdArgs p, const Work w) {
  constexpr int ldx = kVSlice + 8;
  extern __shared__ __align__(16) bf16 smem[];
  __shared__ float F[L], dts[L];
  const int H = p.n_heads, V = p.vdim, N = p.state, R = H / p.groups, ldn = N + 8;
  bf16* cs = smem;                 // [L][ldn]
  bf16* bs = cs + L * ldn;         // [L][ldn]
  bf16* xs = bs + L * ldn;         // [L][ldx]
  bf16* sh = xs + L * ldx;         // [kVSlice][ldn]
  bf16* sl = sh + kVSlice * ldn;
  const int per = (R + kHeads - 1) / kHeads, g = blockIdx.y / per, h0 = g * R + (blockIdx.y % per) * kHeads, h1 = min(h0 + kHeads, (g + 1) * R);
  const int v0 = blockIdx.z * kVSlice, nv = min(kVSlice, V - v0), K = H * V + 2 * p.groups * N;
  pdl_launch_next();
  pdl_wait_prior();
  const Chunk ck(p, blockIdx.x);
  if (ck.len <= 0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, r4 = lane >> 2, c4 = lane & 3, m = warp * 16;
  const bf16* u = static_cast<const bf16*>(p.u) + static_cast<long long>(ck.t0) * K;
  stage_rows(smem_u32(bs), ldn, u + H * V + g * N, K, L, ck.len, N, N);
  stage_rows(smem_u32(cs), ldn, u + H * V + (p.groups + g) * N, K, L, ck.len, N, N);
  cp_async_commit();
  auto stage_head = [&](int h) {
    const long long at = ((static_cast<long long>(blockIdx.x) * H + h) * V + v0) * N;
    stage_rows(smem_u32(xs), ldx, u + h * V + v0, K, L, ck.len, kVSlice, nv);
    cp_async_commit();
    stage_rows(smem_u32(sh), ldn, w.Sh + at, N, kVSlice, nv, N, N);
    stage_rows(smem_u32(sl), ldn, w.Sl + at, N, kVSlice, nv, N, N);
    cp_async_commit();
  };
  stage_head(h0);
  if (warp == 0) chunk_steps(p, ck, h0, F, dts);
  cp_async_wait<2>();
  __syncthreads();
  // ---- C . B of the warp's 16 tokens and all 64 earlier ones (none after them is used) ----
  const uint32_t ca = smem_u32(cs) + ((m + (lane & 15)) * ldn + (lane >> 4) * 8) * 2;
  const uint32_t brow = ((lane & 7) + (lane >> 4) * 8) * ldn + ((lane >> 3) & 1) * 8;       // rows of a 16-row operand tile
  float cb[8][4];
#pragma unroll
  for (int n = 0; n < 8; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) cb[n][e] = 0.f;
  for (int d = 0; d < N; d += 16) {
    uint32_t a[4];
    ldsm_x4(ca + d * 2, a);
#pragma unroll
    for (int n = 0; n < 4; ++n) {
      if (n <= warp) {
        uint32_t b[4];
        ldsm_x4(smem_u32(bs) + (n * 16 * ldn + brow + d) * 2, b);
        mma_bf16_16816(cb[2 * n], a, b[0], b[1]);
        mma_bf16_16816(cb[2 * n + 1], a, b[2], b[3]);
      }
    }
  }
  for (int h = h0; h < h1; ++h) {
    float o[8][4];
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[n][e] = 0.f;
    cp_async_wait<0>();
    __syncthreads();
    // ---- state at the chunk's start ----
    for (int d = 0; d < N; d += 16) {
      uint32_t a[4];
      ldsm_x4(ca + d * 2, a);
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        if (n * 16 < nv) {
          uint32_t b[4];
          ldsm_x4(smem_u32(sh) + (n * 16 * ldn + brow + d) * 2, b);
          mma_bf16_16816(o[2 * n], a, b[0], b[1]);
          mma_bf16_16816(o[2 * n + 1], a, b[2], b[3]);
          ldsm_x4(smem_u32(sl) + (n * 16 * ldn + brow + d) * 2, b);
          mma_bf16_16816(o[2 * n], a, b[0], b[1]);
          mma_bf16_16816(o[2 * n + 1], a, b[2], b[3]);
        }
      }
    }
    const int i0 = m + r4, i1 = i0 + 8;
    const float F0 = F[i0], F1 = F[i1], e0 = expf(F0), e1 = expf(F1), skip = p.skip[h];
#pragma unroll
    for (int n = 0; n < 8; ++n) {
      o[n][0] *= e0; o[n][1] *= e0; o[n][2] *= e1; o[n][3] *= e1;
    }
    // ---- tokens of the chunk ----
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      if (k <= warp) {
        uint32_t af[4];
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int s = k * 16 + half * 8 + c4 * 2;
          float x[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int sj = s + (e & 1), ti = (e >> 1) ? i1 : i0;
            x[e] = sj <= ti ? cb[2 * k + half][e] * ex2_fast(((e >> 1 ? F1 : F0) - F[sj]) * kLog2e) * dts[sj] : 0.f;
          }
          af[2 * half] = pack_bf16x2(x[0], x[1]);
          af[2 * half + 1] = pack_bf16x2(x[2], x[3]);
        }
#pragma unroll
        for (int n = 0; n < 4; ++n) {
          if (n * 16 < nv) {
            uint32_t b[4];
            ldsm_x4_trans(smem_u32(xs) + ((k * 16 + (lane & 15)) * ldx + n * 16 + (lane >> 4) * 8) * 2, b);
            mma_bf16_16816(o[2 * n], af, b[0], b[1]);
            mma_bf16_16816(o[2 * n + 1], af, b[2], b[3]);
          }
        }
      }
    }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int i = r ? i1 : i0;
      if (i >= ck.len) continue;
      bf16* dst = static_cast<bf16*>(p.out) + (ck.t0 + i) * p.ldo + h * V + v0 + c4 * 2;
#pragma unroll
      for (int n = 0; n < 8; ++n) {
        if (n * 8 < nv) {
          const __nv_bfloat162 x = *reinterpret_cast<const __nv_bfloat162*>(xs + i * ldx + n * 8 + c4 * 2);
          *reinterpret_cast<uint32_t*>(dst + n * 8) = pack_bf16x2(fmaf(skip, __bfloat162float(x.x), o[n][2 * r]),
                                                                  fmaf(skip, __bfloat162float(x.y), o[n][2 * r + 1]));
        }
      }
    }
    if (h + 1 < h1) {
      __syncthreads();
      stage_head(h + 1);
      if (warp == 0) chunk_steps(p, ck, h + 1, F, dts);
    }
  }
}

int64_t align256(int64_t n) { return (n + 255) / 256 * 256; }

// Lays the arrays out at `base` (null: only measures).
int64_t carve(Work* w, char* base, int T, int n_seq, int H, int N, int V) {
  const int64_t nc = T / L + n_seq, states = nc * H * V * N;
  int64_t off = 0;
  auto take = [&](int64_t bytes) {
    char* at = base == nullptr ? nullptr : base + off;
    off += align256(bytes);
    return at;
  };
  Work x;
  x.c_F = reinterpret_cast<float*>(take(nc * H * 4));
  x.U = reinterpret_cast<float*>(take(states * 4));
  x.Sh = reinterpret_cast<bf16*>(take(states * 2));
  x.Sl = reinterpret_cast<bf16*>(take(states * 2));
  if (w != nullptr) *w = x;
  return off;
}

constexpr size_t kContribSmem = sizeof(bf16) * L * (2 * (kVSlice + 8) + kNSlice + 8);
size_t output_smem(int N) { return sizeof(bf16) * (2 * static_cast<size_t>(L + kVSlice) * (N + 8) + L * (kVSlice + 8)); }

template <typename K>
cudaError_t allow_smem(K kern, size_t smem) {
  return smem > 48 * 1024 ? cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)) : cudaSuccess;
}

}  // namespace

bool ssd_chunked_supported(int state, int vdim) {
  return state >= 16 && state % 16 == 0 && vdim >= 16 && vdim % 16 == 0 && output_smem(state) <= kSmemLimit;
}

int64_t ssd_chunked_workspace_bytes(int T, int n_seq, int n_heads, int state, int vdim) {
  return carve(nullptr, nullptr, T, n_seq, n_heads, state, vdim);
}

const char* ssd_chunked(const SsdArgs& a, void* workspace, int64_t workspace_bytes) {
  if (a.T <= 0) return nullptr;
  if (const char* err = ssd_check(a)) return err;
  if (a.f32 || a.u == nullptr || !ssd_chunked_supported(a.state, a.vdim)) return "ssd: chunks are for bf16 and states that fit in shared memory";
  if (a.ldo % 2) return "ssd: misaligned rows";
  Work w;
  if (carve(&w, static_cast<char*>(workspace), a.T, a.n_seq, a.n_heads, a.state, a.vdim) > workspace_bytes) return "ssd: workspace too small";
  const int nc = a.T / L + a.n_seq, n_vs = (a.vdim + kVSlice - 1) / kVSlice, n_ns = (a.state + kNSlice - 1) / kNSlice;
  cudaError_t e = launch_kernel(ssd_contrib_kernel, dim3(nc, a.n_heads, n_vs * n_ns), dim3(256), kContribSmem, a.stream, a.pdl, 1, a, w);
  if (e != cudaSuccess) return cudaGetErrorString(e);
  e = launch_kernel(ssd_scan_kernel, dim3((a.vdim * a.state / 4 + 255) / 256 + 1, a.n_heads, a.n_seq), dim3(256), 0, a.stream, a.pdl, 1, a, w);
  if (e != cudaSuccess) return cudaGetErrorString(e);
  const size_t smem = output_smem(a.state);
  e = allow_smem(ssd_output_kernel, smem);
  if (e != cudaSuccess) return cudaGetErrorString(e);
  const int R = a.n_heads / a.groups, per = (R + kHeads - 1) / kHeads;
  e = launch_kernel(ssd_output_kernel, dim3(nc, a.groups * per, n_vs), dim3(128), smem, a.stream, a.pdl, 1, a, w);
  return e == cudaSuccess ? nullptr : cudaGetErrorString(e);
}

}  // namespace nfb
