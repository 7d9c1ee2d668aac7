// Gated linear recurrence with its convolution and gates in one kernel (bf16, tensor cores).
//
// rglru_decode: one token per sequence.  One CTA = 32 channels of a block x up to 64 tokens: the gates' weights come in before
// the kernel waits for its predecessor, the convolution's outputs of the whole block go to shared memory, a warp multiplies
// eight rows of r and the matching eight of i, so a thread ends with both gates of its channels and updates the state.
//
// rglru_chunked: portions.  Kernel 1 does the same for 64 channels x one query block (up to 64 tokens of a sequence) and runs
// the recurrence inside the block from zero: local states and products of the decays go to the workspace.  Kernel 2 takes
// the state at the block's start out of the blocks before it (their last rows), finishes the states and multiplies with
// the GELU branch.
#include "rglru.cuh"

#include "../common/launch.h"
#include "../common/mma_sync.cuh"

namespace nfb {

namespace {

using bf16 = __nv_bfloat16;
constexpr int kBlock = 64;        // tokens of a query block
constexpr int kSmemLimit = 200 * 1024;

struct Work {
  float* local = nullptr;         // [T, C] states from zero at the block's start
  float* prod = nullptr;          // [T, C] products of a from the block's start
  float* start = nullptr;         // [n_seq, C] state at the step's start
  const int* blk_start = nullptr;
  const int* blk_count = nullptr;
};

template <int NW>
int gate_smem(int width, int mt) {
  const int rows = NW * 16 * (width + 8) * 2;                       // weights
  const int scan = 2 * kBlock * (NW * 8 + 1) * 4 + 2 * 4 * NW * 8 * 4;   // over them
  return (rows > scan ? rows : scan) + mt * 16 * (width + 8) * 2;
}

// NW x WM warps: 8 NW channels; WM groups of warps share the MT tiles of 16 tokens.
template <bool DECODE, int NW, int WM, int MT>
__global__ void __launch_bounds__(NW * WM * 32) rglru_gate_kernel(const RglruArgs p, const Work ws, int slices, int u_off) {
  extern __shared__ __align__(16) uint8_t smem[];
  constexpr int NC = NW * 8, kThreads = NW * WM * 32;
  const int K = p.width, C = p.blocks * K, ld = K + 8, vecs = K / 8;
  const int tid = threadIdx.x, warp = (tid >> 5) % NW, m0 = (tid >> 5) / NW, lane = tid & 31, r4 = lane >> 2, c4 = lane & 3;
  const int block = blockIdx.x / slices, col0 = blockIdx.x % slices * NC, n_cols = min(NC, K - col0);
  bf16* us = reinterpret_cast<bf16*>(smem + u_off);
  const uint32_t w_a = smem_u32(smem), u_a = w_a + u_off;
  // weights: rows 0 .. NC - 1 of r, then of i
  const bf16* gw = static_cast<const bf16*>(p.gate_w) + static_cast<long long>(block) * 2 * K * K;
#pragma unroll
  for (int gate = 0; gate < 2; ++gate) {
    const bf16* src = gw + (static_cast<long long>(gate) * K + col0) * K;
    for (int r = tid >> 5; r < NC; r += kThreads / 32) {
      const bool ok = r < n_cols;
      const bf16* row = ok ? src + r * K : gw;
      const uint32_t dst = w_a + (gate * NC + r) * ld * 2;
      for (int c = lane * 8; c < K; c += 256) cp_async16(dst + c * 2, row + c, ok);
    }
  }
  cp_async_commit();
  pdl_launch_next();
  pdl_wait_prior();
  int t0, n, seq = 0;
  if constexpr (DECODE) {
    t0 = blockIdx.y * (MT * 16);
    n = min(MT * 16, p.T - t0);
  } else {
    t0 = ws.blk_start[blockIdx.y];
    n = ws.blk_count[blockIdx.y];
    seq = p.token_seq[t0];
  }
  const bf16* x = static_cast<const bf16*>(p.proj) + C;
  const int cl = warp * 8 + c4 * 2, cb = col0 + cl, c = block * K + cb;     // the thread's two channels: in the CTA, block, row
  const bool live = cl < n_cols;
  // single tokens: what the thread needs at the end is asked for now
  constexpr int kOwn = DECODE ? MT / WM * 2 : 1;
  float2 own_S[kOwn];
  __nv_bfloat162 own_y[kOwn], own_x[kOwn];
  long long own_slot[kOwn];
  if constexpr (DECODE) {
#pragma unroll
    for (int i = 0; i < kOwn; ++i) {
      const int r = ((i >> 1) * WM + m0) * 16 + r4 + (i & 1) * 8, t = t0 + r;
      own_slot[i] = -1;
      if (live && r < n) {
        own_slot[i] = p.state_slot[p.token_seq[t]];
        own_S[i] = *reinterpret_cast<const float2*>(p.S + own_slot[i] * C + c);
        own_y[i] = *reinterpret_cast<const __nv_bfloat162*>(static_cast<const bf16*>(p.proj) + t * p.ldp + c);
        own_x[i] = *reinterpret_cast<const __nv_bfloat162*>(x + t * p.ldp + c);
      }
    }
  }
  const int first = DECODE ? 0 : p.cu_seqlens[seq];
  // ---- the block's convolution ----
  if constexpr (DECODE) {
#pragma unroll 2
    for (int i = tid; i < MT * 16 * vecs; i += kThreads) {
      const int r = i / vecs, cv = block * K + (i % vecs) * 8;
      float v[8] = {};
      if (r < n) {
        const int t = t0 + r, pos = p.cache_pos[t];
        const float* ring = p.ring + static_cast<long long>(p.state_slot[p.token_seq[t]]) * p.taps * C + cv;
        if (p.taps == 4) {               // all loads at once
          float in[4][8], w[4][8];
          load8(p.conv_b + cv, v);
          load8(x + static_cast<long long>(t) * p.ldp + cv, in[3]);
#pragma unroll
          for (int j = 0; j < 3; ++j) {
            load8(ring + static_cast<long long>((pos + 1 + j) & 3) * C, in[j]);        // of position pos - 3 + j
            if (pos < 3 - j)
#pragma unroll
              for (int e = 0; e < 8; ++e) in[j][e] = 0.f;
          }
#pragma unroll
          for (int j = 0; j < 4; ++j) load8(p.conv_w + static_cast<long long>(j) * C + cv, w[j]);
#pragma unroll
          for (int j = 0; j < 4; ++j)
#pragma unroll
            for (int e = 0; e < 8; ++e) v[e] = fmaf(w[j][e], in[j][e], v[e]);
        } else {
          rglru_conv8(p, x, ring - cv, t, 0, pos, C, cv, v);
        }
      }
      store8(us + r * ld + (i % vecs) * 8, v);
    }
  } else {
    const float* ring = p.ring + static_cast<long long>(p.state_slot[seq]) * p.taps * C;
    const int pos0 = p.cache_pos[t0];
    constexpr int kRun = 8;                       // consecutive tokens of a thread
    for (int i = tid; i < MT * 16 / kRun * vecs; i += kThreads) {
      const int r0 = i / vecs * kRun, cv = (i % vecs) * 8, c = block * K + cv;
      if (p.taps != 4) {
        for (int r = r0; r < r0 + kRun; ++r) {
          float v[8] = {};
          if (r < n) rglru_conv8(p, x, ring, t0 + r, t0 + r - first, pos0 + r, C, c, v);
          store8(us + r * ld + cv, v);
        }
        continue;
      }
      // four taps: the earlier inputs stay in registers
      float w[4][8], b[8], h[3][8];
      load8(p.conv_b + c, b);
#pragma unroll
      for (int j = 0; j < 4; ++j) load8(p.conv_w + static_cast<long long>(j) * C + c, w[j]);
#pragma unroll
      for (int j = 0; j < 3; ++j) {
        const int back = 3 - j, pos = pos0 + r0 - back;
#pragma unroll
        for (int e = 0; e < 8; ++e) h[j][e] = 0.f;
        if (pos >= 0 && r0 < n) {
          if (t0 + r0 - back >= first) load8(x + static_cast<long long>(t0 + r0 - back) * p.ldp + c, h[j]);
          else load8(ring + static_cast<long long>(pos % 4) * C + c, h[j]);
        }
      }
#pragma unroll
      for (int r = 0; r < kRun; ++r) {
        float in[8] = {}, v[8];
        if (r0 + r < n) load8(x + static_cast<long long>(t0 + r0 + r) * p.ldp + c, in);
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          v[e] = fmaf(w[3][e], in[e], fmaf(w[2][e], h[2][e], fmaf(w[1][e], h[1][e], fmaf(w[0][e], h[0][e], b[e]))));
          h[0][e] = h[1][e]; h[1][e] = h[2][e]; h[2][e] = in[e];
        }
        store8(us + (r0 + r) * ld + cv, v);
      }
    }
  }
  cp_async_wait<0>();
  __syncthreads();
  // ---- gates: columns warp * 8 .. of r and of i ----
  float acc[MT][2][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[m][0][e] = acc[m][1][e] = 0.f;
  // matrices of one ldsm: r rows at k and k + 8, i rows at k and k + 8
  const uint32_t b_at = w_a + (((lane >> 4) * NC + warp * 8 + (lane & 7)) * ld + ((lane >> 3) & 1) * 8) * 2;
  const uint32_t a_at = u_a + ((lane & 15) * ld + (lane >> 4) * 8) * 2;
#pragma unroll 4
  for (int k = 0; k < K; k += 16) {
    uint32_t b[4];
    ldsm_x4(b_at + k * 2, b);
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      if (m % WM == m0 && m * 16 < n) {
        uint32_t a[4];
        ldsm_x4(a_at + m * (16 * ld * 2) + k * 2, a);
        mma_bf16_16816(acc[m][0], a, b[0], b[1]);
        mma_bf16_16816(acc[m][1], a, b[2], b[3]);
      }
    }
  }
  float2 rate = make_float2(0.f, 0.f), br = rate, bi = rate;
  if (live) {
    rate = *reinterpret_cast<const float2*>(p.rate + c);
    br = *reinterpret_cast<const float2*>(p.gate_b + static_cast<long long>(block) * 2 * K + cb);
    bi = *reinterpret_cast<const float2*>(p.gate_b + (static_cast<long long>(block) * 2 + 1) * K + cb);
  }
  if constexpr (DECODE) {
#pragma unroll
    for (int i = 0; i < kOwn; ++i) {
      const int m = (i >> 1) * WM + m0, h = i & 1, r = m * 16 + r4 + h * 8, t = t0 + r;
      if (own_slot[i] < 0) continue;
      const float2 u = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(us + r * ld + cb));
      const float2 y = __bfloat1622float2(own_y[i]);
      float raw[4];
#pragma unroll
      for (int mm = 0; mm < MT; ++mm)
        if (mm == m) { raw[0] = acc[mm][0][2 * h]; raw[1] = acc[mm][1][2 * h]; raw[2] = acc[mm][0][2 * h + 1]; raw[3] = acc[mm][1][2 * h + 1]; }
      float2 S = own_S[i];
      float em, in;
      rglru_gates<bf16>(raw[0] + br.x, raw[1] + bi.x, rate.x, u.x, em, in);
      S.x += fmaf(em, S.x, in);
      rglru_gates<bf16>(raw[2] + br.y, raw[3] + bi.y, rate.y, u.y, em, in);
      S.y += fmaf(em, S.y, in);
      *reinterpret_cast<uint32_t*>(static_cast<bf16*>(p.out) + t * p.ldo + c) =
          pack_bf16x2(S.x * gelu_tanh_of<bf16>(y.x), S.y * gelu_tanh_of<bf16>(y.y));
      if (p.write_state) {
        *reinterpret_cast<float2*>(p.S + own_slot[i] * C + c) = S;
        *reinterpret_cast<float2*>(p.ring + (own_slot[i] * p.taps + p.cache_pos[t] % p.taps) * C + c) = __bfloat1622float2(own_x[i]);
      }
    }
    return;
  }
  // ---- recurrence inside the block: four threads per channel, sixteen tokens each ----
  __syncthreads();                                   // the weights are no longer needed
  constexpr int kLd = NC + 1;
  float* em_s = reinterpret_cast<float*>(smem);      // [kBlock][kLd]
  float* in_s = em_s + kBlock * kLd;
  float* end_s = in_s + kBlock * kLd;                // [2][4][NC]: state and product at the end of each run of tokens
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int r = m * 16 + r4 + h * 8;
      float e0 = 0.f, e1 = 0.f, i0 = 0.f, i1 = 0.f;
      if (live && r < n) {
        const float2 u = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(us + r * ld + cb));
        rglru_gates<bf16>(acc[m][0][2 * h] + br.x, acc[m][1][2 * h] + bi.x, rate.x, u.x, e0, i0);
        rglru_gates<bf16>(acc[m][0][2 * h + 1] + br.y, acc[m][1][2 * h + 1] + bi.y, rate.y, u.y, e1, i1);
      }
      em_s[r * kLd + cl] = e0; em_s[r * kLd + cl + 1] = e1;
      in_s[r * kLd + cl] = i0; in_s[r * kLd + cl + 1] = i1;
    }
  __syncthreads();
  static_assert(DECODE || (kThreads == 4 * NC && WM == 1), "four threads per channel");
  constexpr int kRunT = kBlock / 4;
  const int col = tid % NC, run = tid / NC;
  float hs[kRunT], ps[kRunT], h = 0.f, prod = 1.f;
#pragma unroll
  for (int j = 0; j < kRunT; ++j) {
    const int r = run * kRunT + j;
    const float em = em_s[r * kLd + col];
    h += fmaf(em, h, in_s[r * kLd + col]);
    prod = fmaf(em, prod, prod);
    hs[j] = h;
    ps[j] = prod;
  }
  end_s[run * NC + col] = h;
  end_s[(4 + run) * NC + col] = prod;
  __syncthreads();
  float h0 = 0.f, p0 = 1.f;
  for (int q = 0; q < run; ++q) {
    h0 = fmaf(end_s[(4 + q) * NC + col], h0, end_s[q * NC + col]);
    p0 *= end_s[(4 + q) * NC + col];
  }
  if (col >= n_cols) return;
  const long long cg = static_cast<long long>(block) * K + col0 + col;
#pragma unroll
  for (int j = 0; j < kRunT; ++j) {
    const int r = run * kRunT + j;
    if (r < n) {
      ws.local[static_cast<long long>(t0 + r) * C + cg] = fmaf(ps[j], h0, hs[j]);
      ws.prod[static_cast<long long>(t0 + r) * C + cg] = ps[j] * p0;
    }
  }
  if (t0 == first && run == 0) ws.start[static_cast<long long>(seq) * C + cg] = p.S[static_cast<long long>(p.state_slot[seq]) * C + cg];
}

// One CTA = 128 channels of one query block: 32 threads x 4 channels, eight groups of 8 tokens.
constexpr int kOutThreads = 256, kOutGroups = 8, kOutRun = kBlock / kOutGroups;

__global__ void __launch_bounds__(kOutThreads) rglru_out_kernel(const RglruArgs p, const Work ws) {
  __shared__ float4 carry[2][kOutGroups][32];
  pdl_launch_next();
  pdl_wait_prior();
  const int C = p.blocks * p.width, tid = threadIdx.x, q = tid >> 5, lane = tid & 31, c = (blockIdx.x * 32 + lane) * 4;
  const int t0 = ws.blk_start[blockIdx.y], n = ws.blk_count[blockIdx.y], seq = p.token_seq[t0];
  const int first = p.cu_seqlens[seq], before = (t0 - first) / kBlock;      // blocks of the sequence before this one
  const bool live = c < C;
  // state and product of decays over this group's share of the earlier blocks
  float4 h = make_float4(0.f, 0.f, 0.f, 0.f), a = make_float4(1.f, 1.f, 1.f, 1.f);
  if (live) {
    const int per = (before + kOutGroups - 1) / kOutGroups, b1 = min(before, (q + 1) * per);
#pragma unroll 4
    for (int b = q * per; b < b1; ++b) {
      const long long at = static_cast<long long>(first + b * kBlock + kBlock - 1) * C + c;
      const float4 l = *reinterpret_cast<const float4*>(ws.local + at), d = *reinterpret_cast<const float4*>(ws.prod + at);
      h.x = fmaf(d.x, h.x, l.x); h.y = fmaf(d.y, h.y, l.y); h.z = fmaf(d.z, h.z, l.z); h.w = fmaf(d.w, h.w, l.w);
      a.x *= d.x; a.y *= d.y; a.z *= d.z; a.w *= d.w;
    }
  }
  carry[0][q][lane] = h;
  carry[1][q][lane] = a;
  __syncthreads();
  if (!live) return;
  float4 s = *reinterpret_cast<const float4*>(ws.start + static_cast<long long>(seq) * C + c);
#pragma unroll
  for (int k = 0; k < kOutGroups; ++k) {
    const float4 l = carry[0][k][lane], d = carry[1][k][lane];
    s.x = fmaf(d.x, s.x, l.x); s.y = fmaf(d.y, s.y, l.y); s.z = fmaf(d.z, s.z, l.z); s.w = fmaf(d.w, s.w, l.w);
  }
  const int r1 = min(n, (q + 1) * kOutRun);
#pragma unroll 4
  for (int r = q * kOutRun; r < r1; ++r) {
    const long long t = t0 + r, at = t * C + c;
    const float4 l = *reinterpret_cast<const float4*>(ws.local + at), d = *reinterpret_cast<const float4*>(ws.prod + at);
    const uint2 yr = *reinterpret_cast<const uint2*>(static_cast<const bf16*>(p.proj) + t * p.ldp + c);
    const float4 S = make_float4(fmaf(d.x, s.x, l.x), fmaf(d.y, s.y, l.y), fmaf(d.z, s.z, l.z), fmaf(d.w, s.w, l.w));
    const float y0 = __uint_as_float(yr.x << 16), y1 = __uint_as_float(yr.x & 0xffff0000u);
    const float y2 = __uint_as_float(yr.y << 16), y3 = __uint_as_float(yr.y & 0xffff0000u);
    *reinterpret_cast<uint2*>(static_cast<bf16*>(p.out) + t * p.ldo + c) =
        make_uint2(pack_bf16x2(S.x * gelu_tanh_of<bf16>(y0), S.y * gelu_tanh_of<bf16>(y1)),
                   pack_bf16x2(S.z * gelu_tanh_of<bf16>(y2), S.w * gelu_tanh_of<bf16>(y3)));
    if (p.write_state && t + 1 == p.cu_seqlens[seq + 1])
      *reinterpret_cast<float4*>(p.S + static_cast<long long>(p.state_slot[seq]) * C + c) = S;
  }
  if (p.write_state && q == 0 && t0 + n == p.cu_seqlens[seq + 1]) {
    float* ring = p.ring + static_cast<long long>(p.state_slot[seq]) * p.taps * C;
    for (int t = max(first, t0 + n - p.taps); t < t0 + n; ++t) {
      const uint2 xr = *reinterpret_cast<const uint2*>(static_cast<const bf16*>(p.proj) + t * p.ldp + C + c);
      *reinterpret_cast<float4*>(ring + static_cast<long long>(p.cache_pos[t] % p.taps) * C + c) =
          make_float4(__uint_as_float(xr.x << 16), __uint_as_float(xr.x & 0xffff0000u), __uint_as_float(xr.y << 16), __uint_as_float(xr.y & 0xffff0000u));
    }
  }
}

template <bool DECODE, int NW, int WM, int MT>
cudaError_t launch_gates(const RglruArgs& a, const Work& ws, int n_y) {
  auto kern = rglru_gate_kernel<DECODE, NW, WM, MT>;
  const int smem = gate_smem<NW>(a.width, MT), u_off = smem - MT * 16 * (a.width + 8) * 2;
  const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) return e;
  const int slices = (a.width + NW * 8 - 1) / (NW * 8);
  return launch_kernel(kern, dim3(a.blocks * slices, n_y), dim3(NW * WM * 32), smem, a.stream, a.pdl, 1, a, ws, slices, u_off);
}

const char* check_fused(const RglruArgs& a) {
  if (const char* err = rglru_check(a)) return err;
  if (a.f32 || !rglru_fused_supported(a.width)) return "rglru: the fused kernels take bf16 and blocks whose weights fit in shared memory";
  if (a.gate_w == nullptr || a.gate_b == nullptr) return "rglru: missing gates";
  return nullptr;
}

}  // namespace

bool rglru_fused_supported(int width) { return width >= 16 && width % 16 == 0 && gate_smem<8>(width, 4) <= kSmemLimit; }

const char* rglru_decode(const RglruArgs& a) {
  if (a.T <= 0) return nullptr;
  if (const char* err = check_fused(a)) return err;
  if (a.T != a.n_seq) return "rglru: one token per sequence expected";
  cudaError_t e;
  if (a.T <= 16) e = launch_gates<true, 4, 1, 1>(a, Work(), 1);
  else if (a.T <= 32) e = launch_gates<true, 4, 2, 2>(a, Work(), 1);
  else e = launch_gates<true, 4, 2, 4>(a, Work(), (a.T + 63) / 64);
  return e == cudaSuccess ? nullptr : cudaGetErrorString(e);
}

int64_t rglru_chunked_workspace_bytes(int T, int n_seq, int channels) { return (2LL * T + n_seq) * channels * 4; }

const char* rglru_chunked(const RglruArgs& a, const int* blk_start, const int* blk_count, int n_blocks, void* workspace, int64_t bytes) {
  if (a.T <= 0 || n_blocks <= 0) return nullptr;
  if (const char* err = check_fused(a)) return err;
  const int C = a.blocks * a.width;
  if (n_blocks > 65535 || workspace == nullptr || bytes < rglru_chunked_workspace_bytes(a.T, a.n_seq, C)) return "rglru: workspace too small";
  Work ws;
  ws.local = static_cast<float*>(workspace);
  ws.prod = ws.local + static_cast<int64_t>(a.T) * C;
  ws.start = ws.prod + static_cast<int64_t>(a.T) * C;
  ws.blk_start = blk_start;
  ws.blk_count = blk_count;
  cudaError_t e = launch_gates<false, 8, 1, 4>(a, ws, n_blocks);
  if (e == cudaSuccess) e = launch_kernel(rglru_out_kernel, dim3((C + 127) / 128, n_blocks), dim3(kOutThreads), 0, a.stream, a.pdl, 1, a, ws);
  return e == cudaSuccess ? nullptr : cudaGetErrorString(e);
}

}  // namespace nfb
