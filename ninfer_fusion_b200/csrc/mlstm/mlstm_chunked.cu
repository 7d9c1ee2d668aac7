// mLSTM over prompt portions, in chunks of 64 tokens.  With F_t = sum of the log forget gates of the chunk up to t,
// m_0 the running maximum at the chunk's start and S_0, n_0 the state there, the recurrence unrolls to
//   m_t   = F_t + max(m_0, max_{s <= t} (i_s - F_s))
//   S_t^T q = exp(F_t + m_0 - m_t) S_0^T q  +  sum_{s <= t} exp(F_t - F_s + i_s - m_t) (k_s . q) v_s
// and n_t . q is the same with v_s = 1; every exponent is <= 0.  Four kernels:
//   gates    one CTA per (sequence, head): log gates, F, m per token, and m at every chunk boundary
//   contrib  one CTA per (chunk, head, value slice): what a chunk adds to the state, U = sum_s w_s k_s v_s^T
//   scan     elementwise over the chunks of a sequence: the state at every chunk's start, kept in fp32 and handed to
//            the next kernel as bf16 hi + lo pairs (two rows of the state packed per word: an MMA B fragment)
//   output   one CTA per (chunk, head): S_0 and intra-chunk terms on the tensor cores, head norm, output gate
// Weighted keys and the state enter the MMAs as hi + lo pairs, so both keep about 17 bits.
#include "mlstm.h"

#include <math_constants.h>

#include "../common/elem.cuh"
#include "../common/launch.h"
#include "../common/mma_sync.cuh"

namespace nfb {

namespace {

using bf16 = __nv_bfloat16;
constexpr int L = kMlstmChunk;

struct ChunkWs {
  float* F;      // [T, H] inclusive sums of the log forget gate inside the chunk
  float* ig;     // [T, H] log input gate
  float* mt;     // [T, H]
  float* c_m0;   // [NC, H]
  float* c_m1;   // [NC, H]
  float* c_F;    // [NC, H]
  float* c_u;    // [NC, H] max of i_s - F_s
  float* U;      // [NC, H, D, V]
  float* Un;     // [NC, H, D]
  float* Sn;     // [NC, H, D]
  uint32_t* Sh;  // [NC, H, D / 2, V] bf16 pairs (rows 2 r, 2 r + 1)
  uint32_t* Sl;
};

// Chunk slots: the chunks of sequence s start at slot cu[s] / 64 + s (disjoint for any lengths).
__device__ __forceinline__ int chunk_base(const int* cu, int s) { return cu[s] / L + s; }

// Sequence, first token and length of a chunk slot; length 0 = unused slot.
__device__ __forceinline__ void chunk_of(const MlstmArgs& p, int slot, int& seq, int& t0, int& len) {
  int lo = 0, hi = p.n_seq - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (chunk_base(p.cu_seqlens, mid) <= slot) lo = mid; else hi = mid - 1;
  }
  seq = lo;
  t0 = p.cu_seqlens[lo] + (slot - chunk_base(p.cu_seqlens, lo)) * L;
  len = min(L, p.cu_seqlens[lo + 1] - t0);
  if (len < 0 || slot < chunk_base(p.cu_seqlens, lo)) len = 0;
}

__global__ void __launch_bounds__(1024) mlstm_gates_kernel(const MlstmArgs p, const ChunkWs w) {
  pdl_launch_next();
  pdl_wait_prior();
  const int seq = blockIdx.x, h = blockIdx.y, H = p.n_heads;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int tb = p.cu_seqlens[seq], te = p.cu_seqlens[seq + 1];
  const int nc = (te - tb + L - 1) / L, base = chunk_base(p.cu_seqlens, seq);
  const float inv_cap = 1.f / p.gate_cap;
  float* m_state = p.m + static_cast<long long>(p.state_slot[seq]) * H + h;
  for (int c = warp; c < nc; c += static_cast<int>(blockDim.x >> 5)) {
    float f[2], u[2], ig[2];
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int t = tb + c * L + 2 * lane + j;
      f[j] = 0.f;
      ig[j] = -CUDART_INF_F;
      if (t < te) {
        const float fr = p.gate_cap * tanhf(p.gates[t * p.ldg + p.f_off + h] * inv_cap);
        f[j] = fminf(fr, 0.f) - log1pf(expf(-fabsf(fr)));
        ig[j] = p.gate_cap * tanhf(p.gates[t * p.ldg + p.i_off + h] * inv_cap);
      }
    }
    float sum = f[0] + f[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float y = __shfl_up_sync(0xffffffffu, sum, o);
      if (lane >= o) sum += y;
    }
    float F[2];
    F[1] = sum;
    F[0] = sum - f[1];
#pragma unroll
    for (int j = 0; j < 2; ++j) u[j] = ig[j] - F[j];
    float mx = fmaxf(u[0], u[1]);
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float y = __shfl_up_sync(0xffffffffu, mx, o);
      if (lane >= o) mx = fmaxf(mx, y);
    }
    float before = __shfl_up_sync(0xffffffffu, mx, 1);   // prefix maximum of the tokens of lower lanes
    if (lane == 0) before = -CUDART_INF_F;
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int t = tb + c * L + 2 * lane + j;
      if (t < te) {
        w.F[static_cast<long long>(t) * H + h] = F[j];
        w.ig[static_cast<long long>(t) * H + h] = ig[j];
        w.mt[static_cast<long long>(t) * H + h] = j == 0 ? fmaxf(before, u[0]) : mx;
      }
    }
    if (lane == 31) {   // tokens past the end have f = 0 and i = -inf: they change neither
      w.c_F[static_cast<long long>(base + c) * H + h] = F[1];
      w.c_u[static_cast<long long>(base + c) * H + h] = mx;
    }
  }
  __syncthreads();
  if (warp == 0) {
    float m = *m_state;
    for (int c0 = 0; c0 < nc; c0 += 32) {
      const long long at = static_cast<long long>(base + c0 + lane) * H + h;
      const bool ok = c0 + lane < nc;
      const float cF = ok ? w.c_F[at] : 0.f, cu = ok ? w.c_u[at] : -CUDART_INF_F;
      float m0 = 0.f, m1 = 0.f;
      for (int j = 0; j < 32; ++j) {
        const float Fj = __shfl_sync(0xffffffffu, cF, j), uj = __shfl_sync(0xffffffffu, cu, j);
        const float next = Fj + fmaxf(m, uj);
        if (lane == j) { m0 = m; m1 = next; }
        m = next;
      }
      if (ok) { w.c_m0[at] = m0; w.c_m1[at] = m1; }
    }
    if (lane == 0 && p.write_state) *m_state = m;
  }
  __syncthreads();
  for (int t = tb + threadIdx.x; t < te; t += blockDim.x) {
    const long long at = static_cast<long long>(t) * H + h;
    w.mt[at] = w.F[at] + fmaxf(w.c_m0[static_cast<long long>(base + (t - tb) / L) * H + h], w.mt[at]);
  }
}

constexpr int kDBlock = 256;   // state rows per CTA of the contribution kernel
constexpr int kVSlice = 128;   // state columns per CTA

// MT: 16-row tiles per warp.
template <int MT>
__global__ void __launch_bounds__(256) mlstm_contrib_kernel(const MlstmArgs p, const ChunkWs w) {
  extern __shared__ __align__(16) bf16 smem_b[];
  __shared__ float wt[L];
  const int H = p.n_heads, D = p.dim, V = p.vdim;
  const int n_vs = (V + kVSlice - 1) / kVSlice;
  const int slot = blockIdx.x, h = blockIdx.y, v0 = (blockIdx.z % n_vs) * kVSlice, d0 = (blockIdx.z / n_vs) * kDBlock;
  const int nd = min(kDBlock, D - d0), ldk = min(kDBlock, D) + 8;
  constexpr int ldv = kVSlice + 8;
  bf16* kh = smem_b;               // [L][ldk] weighted keys, high part
  bf16* kl = kh + L * ldk;         // low part
  bf16* vs = kl + L * ldk;         // [L][ldv]
  pdl_launch_next();
  pdl_wait_prior();
  int seq, t0, len;
  chunk_of(p, slot, seq, t0, len);
  if (len <= 0) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const long long ch = static_cast<long long>(slot) * H + h;
  if (tid < L)
    wt[tid] = tid < len ? expf(w.c_F[ch] - w.F[static_cast<long long>(t0 + tid) * H + h] +
                               w.ig[static_cast<long long>(t0 + tid) * H + h] - w.c_m1[ch]) : 0.f;
  const bf16* proj = static_cast<const bf16*>(p.proj);
  const uint32_t vs_a = smem_u32(vs);
  for (int i = tid; i < L * (kVSlice / 8); i += 256) {
    const int s = i / (kVSlice / 8), c = (i % (kVSlice / 8)) * 8;
    const bool ok = s < len && v0 + c < V;
    cp_async16(vs_a + (s * ldv + c) * 2, ok ? proj + (t0 + s) * p.ldp + p.v_off + h * V + v0 + c : proj, ok);
  }
  cp_async_commit();
  __syncthreads();
  for (int i = tid; i < L * (nd / 8); i += 256) {
    const int s = i / (nd / 8), c = (i % (nd / 8)) * 8;
    float k[8], hi[8], lo[8];
    if (s < len) load8(proj + (t0 + s) * p.ldp + p.k_off + h * D + d0 + c, k);
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const float x = s < len ? k[j] * wt[s] : 0.f;
      hi[j] = __bfloat162float(__float2bfloat16(x));
      lo[j] = x - hi[j];
    }
    store8(kh + s * ldk + c, hi);
    store8(kl + s * ldk + c, lo);
  }
  if (v0 == 0 && tid < nd) {
    float a = 0.f;
    const bf16* kc = proj + t0 * p.ldp + p.k_off + h * D + d0 + tid;
#pragma unroll 16
    for (int s = 0; s < L; ++s) a = fmaf(wt[s], s < len ? __bfloat162float(kc[s * p.ldp]) : 0.f, a);
    w.Un[ch * D + d0 + tid] = a;
  }
  cp_async_wait<0>();
  __syncthreads();
  const int mt0 = warp * MT;
  if (mt0 * 16 >= nd) return;
  float acc[MT][kVSlice / 8][4];
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int n = 0; n < kVSlice / 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[i][n][e] = 0.f;
  const uint32_t kh_a = smem_u32(kh), kl_a = smem_u32(kl);
  const int arow = (lane & 7) + ((lane >> 4) & 1) * 8, acol = ((lane >> 3) & 1) * 8;
#pragma unroll
  for (int kk = 0; kk < L / 16; ++kk) {
    uint32_t ah[MT][4], al[MT][4];
#pragma unroll
    for (int i = 0; i < MT; ++i) {
      const int m = min((mt0 + i) * 16, nd - 16);
      const uint32_t at = ((kk * 16 + arow) * ldk + m + acol) * 2;
      ldsm_x4_trans(kh_a + at, ah[i]);
      ldsm_x4_trans(kl_a + at, al[i]);
    }
#pragma unroll
    for (int n = 0; n < kVSlice / 16; ++n) {
      if (v0 + n * 16 < V) {
        uint32_t b[4];
        ldsm_x4_trans(vs_a + ((kk * 16 + (lane & 15)) * ldv + n * 16 + (lane >> 4) * 8) * 2, b);
#pragma unroll
        for (int i = 0; i < MT; ++i) {
          mma_bf16_16816(acc[i][2 * n], ah[i], b[0], b[1]);
          mma_bf16_16816(acc[i][2 * n + 1], ah[i], b[2], b[3]);
          mma_bf16_16816(acc[i][2 * n], al[i], b[0], b[1]);
          mma_bf16_16816(acc[i][2 * n + 1], al[i], b[2], b[3]);
        }
      }
    }
  }
#pragma unroll
  for (int i = 0; i < MT; ++i) {
    const int d = (mt0 + i) * 16 + (lane >> 2);
    if ((mt0 + i) * 16 >= nd) break;
    float* dst = w.U + (ch * D + d0 + d) * V + v0 + (lane & 3) * 2;
#pragma unroll
    for (int n = 0; n < kVSlice / 8; ++n) {
      if (v0 + n * 8 < V) {
        *reinterpret_cast<float2*>(dst + n * 8) = make_float2(acc[i][n][0], acc[i][n][1]);
        *reinterpret_cast<float2*>(dst + static_cast<long long>(8) * V + n * 8) = make_float2(acc[i][n][2], acc[i][n][3]);
      }
    }
  }
}

// grid: (blocks over D / 2 x V elements and one more for n, head, sequence)
__global__ void __launch_bounds__(256) mlstm_scan_kernel(const MlstmArgs p, const ChunkWs w) {
  pdl_launch_next();
  pdl_wait_prior();
  const int H = p.n_heads, D = p.dim, V = p.vdim, h = blockIdx.y, seq = blockIdx.z;
  const int tb = p.cu_seqlens[seq], te = p.cu_seqlens[seq + 1];
  const int nc = (te - tb + L - 1) / L, base = chunk_base(p.cu_seqlens, seq);
  const long long sh = static_cast<long long>(p.state_slot[seq]) * H + h;
  if (blockIdx.x == gridDim.x - 1) {
    for (int d = threadIdx.x; d < D; d += blockDim.x) {
      float n = p.n[sh * D + d];
      for (int c = 0; c < nc; ++c) {
        const long long ch = static_cast<long long>(base + c) * H + h;
        w.Sn[ch * D + d] = n;
        n = fmaf(expf(w.c_F[ch] + w.c_m0[ch] - w.c_m1[ch]), n, w.Un[ch * D + d]);
      }
      if (p.write_state) p.n[sh * D + d] = n;
    }
    return;
  }
  const int e = blockIdx.x * blockDim.x + threadIdx.x;
  if (e >= (D / 2) * V) return;
  const int r = e / V, v = e % V;
  float* s_state = p.S + (sh * D + 2 * r) * V + v;
  float s0 = s_state[0], s1 = s_state[V];
  const long long u_step = static_cast<long long>(H) * D * V, p_step = u_step / 2;
  const float* u = w.U + ((static_cast<long long>(base) * H + h) * D + 2 * r) * V + v;
  uint32_t* oh = w.Sh + ((static_cast<long long>(base) * H + h) * (D / 2) + r) * V + v;
  uint32_t* ol = w.Sl + ((static_cast<long long>(base) * H + h) * (D / 2) + r) * V + v;
  constexpr int kAhead = 4;
  for (int c0 = 0; c0 < nc; c0 += kAhead) {
    float u0[kAhead], u1[kAhead], a[kAhead];
#pragma unroll
    for (int j = 0; j < kAhead; ++j) {
      if (c0 + j < nc) {
        const long long ch = static_cast<long long>(base + c0 + j) * H + h;
        u0[j] = __ldcs(u + (c0 + j) * u_step);
        u1[j] = __ldcs(u + (c0 + j) * u_step + V);
        a[j] = w.c_F[ch] + w.c_m0[ch] - w.c_m1[ch];
      }
    }
#pragma unroll
    for (int j = 0; j < kAhead; ++j) {
      if (c0 + j < nc) {
        const float h0 = __bfloat162float(__float2bfloat16(s0)), h1 = __bfloat162float(__float2bfloat16(s1));
        oh[(c0 + j) * p_step] = pack_bf16x2(h0, h1);
        ol[(c0 + j) * p_step] = pack_bf16x2(s0 - h0, s1 - h1);
        const float f = expf(a[j]);
        s0 = fmaf(f, s0, u0[j]);
        s1 = fmaf(f, s1, u1[j]);
      }
    }
  }
  if (p.write_state) {
    s_state[0] = s0;
    s_state[V] = s1;
  }
}

// NW warps, NT: 8-wide value tiles per warp (NW warps cover V).  grid: (chunk slot, head)
template <int NW, int NT>
__global__ void __launch_bounds__(NW * 32, NW == 8 ? 2 : 1) mlstm_output_kernel(const MlstmArgs p, const ChunkWs w) {
  extern __shared__ __align__(16) bf16 smem_b[];
  __shared__ float Fs[L], us[L], ms[L], inter[L], den_s[NW / 4][L], den_state[L], ss_s[NW][L];
  constexpr int kThreads = NW * 32;
  constexpr int kKn = L / (NW / 4) / 8;    // 8-key tiles per warp of the intra-chunk weights
  const int H = p.n_heads, D = p.dim, V = p.vdim;
  const int ldq = D + 8, ldv = V + 8;
  constexpr int ldp = L + 8;
  bf16* qs = smem_b;              // [L][ldq]
  bf16* ks = qs + L * ldq;        // [L][ldq]
  bf16* vs = ks + L * ldq;        // [L][ldv]
  bf16* ps = vs + L * ldv;        // [L][ldp]
  pdl_launch_next();
  pdl_wait_prior();
  const int slot = blockIdx.x, h = blockIdx.y;
  int seq, t0, len;
  chunk_of(p, slot, seq, t0, len);
  if (len <= 0) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, r4 = lane >> 2, c4 = lane & 3;
  const long long ch = static_cast<long long>(slot) * H + h;
  const bf16* proj = static_cast<const bf16*>(p.proj);
  const uint32_t qs_a = smem_u32(qs), ks_a = smem_u32(ks), vs_a = smem_u32(vs), ps_a = smem_u32(ps);
  for (int i = tid; i < L * (D / 8); i += kThreads) {
    const int s = i / (D / 8), c = (i % (D / 8)) * 8;
    const bool ok = s < len;
    const bf16* row = proj + (t0 + (ok ? s : 0)) * p.ldp + h * D + c;
    cp_async16(qs_a + (s * ldq + c) * 2, row + p.q_off, ok);
    cp_async16(ks_a + (s * ldq + c) * 2, row + p.k_off, ok);
  }
  cp_async_commit();
  for (int i = tid; i < L * (V / 8); i += kThreads) {
    const int s = i / (V / 8), c = (i % (V / 8)) * 8;
    const bool ok = s < len;
    cp_async16(vs_a + (s * ldv + c) * 2, proj + (t0 + (ok ? s : 0)) * p.ldp + p.v_off + h * V + c, ok);
  }
  cp_async_commit();
  if (tid < L) {
    const bool ok = tid < len;
    const long long at = static_cast<long long>(t0 + (ok ? tid : 0)) * H + h;
    Fs[tid] = w.F[at];
    us[tid] = ok ? w.ig[at] - w.F[at] : -CUDART_INF_F;
    ms[tid] = w.mt[at];
    inter[tid] = p.q_scale * expf(w.F[at] + w.c_m0[ch] - w.mt[at]);
  }
  cp_async_wait<1>();
  __syncthreads();
  // ---- intra-chunk weights: warp = 16 queries x 8 kKn keys ----
  {
    const int mt = warp & 3, nh = warp >> 2;
    float c[kKn][4] = {};
    if (nh * (kKn * 8) <= mt * 16 + 15) {   // not entirely above the diagonal
      for (int d = 0; d < D; d += 16) {
        uint32_t a[4];
        ldsm_x4(qs_a + ((mt * 16 + (lane & 15)) * ldq + d + (lane >> 4) * 8) * 2, a);
#pragma unroll
        for (int n = 0; n < kKn / 2; ++n) {
          uint32_t b[4];
          ldsm_x4(ks_a + ((nh * (kKn * 8) + n * 16 + (lane & 7) + (lane >> 4) * 8) * ldq + d + ((lane >> 3) & 1) * 8) * 2, b);
          mma_bf16_16816(c[2 * n], a, b[0], b[1]);
          mma_bf16_16816(c[2 * n + 1], a, b[2], b[3]);
        }
      }
    }
    float sum[2] = {0.f, 0.f};
#pragma unroll
    for (int n = 0; n < kKn; ++n) {
      float x[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int t = mt * 16 + r4 + (e >> 1) * 8, s = nh * (kKn * 8) + n * 8 + c4 * 2 + (e & 1);
        x[e] = s <= t ? c[n][e] * p.q_scale * expf(Fs[t] + us[s] - ms[t]) : 0.f;
        sum[e >> 1] += x[e];
      }
#pragma unroll
      for (int r = 0; r < 2; ++r)
        *reinterpret_cast<uint32_t*>(ps + (mt * 16 + r4 + r * 8) * ldp + nh * (kKn * 8) + n * 8 + c4 * 2) =
            pack_bf16x2(x[2 * r], x[2 * r + 1]);
    }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      sum[r] += __shfl_xor_sync(0xffffffffu, sum[r], 1);
      sum[r] += __shfl_xor_sync(0xffffffffu, sum[r], 2);
      if (c4 == 0) den_s[nh][mt * 16 + r4 + r * 8] = sum[r];
    }
  }
  // ---- n_0 . q: warp = L / NW queries ----
  for (int j = 0; j < L / NW; ++j) {
    const int t = warp * (L / NW) + j;
    float d = 0.f;
    for (int i = lane * 8; i < D; i += 256) {
      float q[8], n[8];
      load8(qs + t * ldq + i, q);
      load8(w.Sn + ch * D + i, n);
#pragma unroll
      for (int e = 0; e < 8; ++e) d = fmaf(q[e], n[e], d);
    }
    d = warp_sum(d);
    if (lane == 0) den_state[t] = d;
  }
  // ---- S_0^T q: all 64 queries x this warp's value tiles, S_0 fragments straight from global memory ----
  float acc[4][NT][4];
#pragma unroll
  for (int m = 0; m < 4; ++m)
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[m][n][e] = 0.f;
  const int vt0 = warp * NT;
  const int n_live = min(NT, V / 8 - vt0);
  if (n_live > 0) {
    const uint32_t* sh = w.Sh + (ch * (D / 2) + c4) * V + vt0 * 8 + r4;
    const uint32_t* sl = w.Sl + (ch * (D / 2) + c4) * V + vt0 * 8 + r4;
    for (int d = 0; d < D; d += 16) {
      uint32_t bh[NT][2], bl[NT][2];
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        if (n < n_live) {
          const long long at = static_cast<long long>(d / 2) * V + n * 8;
          bh[n][0] = sh[at]; bh[n][1] = sh[at + 4LL * V];
          bl[n][0] = sl[at]; bl[n][1] = sl[at + 4LL * V];
        } else {
          bh[n][0] = bh[n][1] = bl[n][0] = bl[n][1] = 0u;
        }
      }
#pragma unroll
      for (int m = 0; m < 4; ++m) {
        uint32_t a[4];
        ldsm_x4(qs_a + ((m * 16 + (lane & 15)) * ldq + d + (lane >> 4) * 8) * 2, a);
#pragma unroll
        for (int n = 0; n < NT; ++n) {
          mma_bf16_16816(acc[m][n], a, bh[n][0], bh[n][1]);
          mma_bf16_16816(acc[m][n], a, bl[n][0], bl[n][1]);
        }
      }
    }
#pragma unroll
    for (int m = 0; m < 4; ++m) {
      const float f0 = inter[m * 16 + r4], f1 = inter[m * 16 + r4 + 8];
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        acc[m][n][0] *= f0; acc[m][n][1] *= f0; acc[m][n][2] *= f1; acc[m][n][3] *= f1;
      }
    }
  }
  cp_async_wait<0>();
  __syncthreads();
  // ---- + weights x values ----
  if (n_live > 0) {
#pragma unroll
    for (int kk = 0; kk < L / 16; ++kk) {
      uint32_t b[NT][2];
#pragma unroll
      for (int n = 0; n < NT; n += 2) {
        uint32_t r[4];
        const int col = min((vt0 + n) * 8, V - 16);            // V is a multiple of 16
        const int sh8 = (vt0 + n) * 8 - col;                   // 8 when a single last tile is read from its pair
        ldsm_x4_trans(vs_a + ((kk * 16 + (lane & 15)) * ldv + col + (lane >> 4) * 8) * 2, r);
        b[n][0] = sh8 ? r[2] : r[0];
        b[n][1] = sh8 ? r[3] : r[1];
        if (n + 1 < NT) { b[n + 1][0] = r[2]; b[n + 1][1] = r[3]; }
      }
#pragma unroll
      for (int m = 0; m < 4; ++m) {
        if (kk > m) continue;   // keys after every query of the tile
        uint32_t a[4];
        ldsm_x4(ps_a + ((m * 16 + (lane & 15)) * ldp + kk * 16 + (lane >> 4) * 8) * 2, a);
#pragma unroll
        for (int n = 0; n < NT; ++n) mma_bf16_16816(acc[m][n], a, b[n][0], b[n][1]);
      }
    }
  }
  // ---- denominator, head norm, gate ----
#pragma unroll
  for (int m = 0; m < 4; ++m) {
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int t = m * 16 + r4 + r * 8;
      float den = inter[t] * den_state[t];
#pragma unroll
      for (int i = 0; i < NW / 4; ++i) den += den_s[i][t];
      const float inv = 1.f / (fmaxf(fabsf(den), expf(-ms[t])) + 1e-6f);
      float sq = 0.f;
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        if (n < n_live) {
          acc[m][n][2 * r] *= inv;
          acc[m][n][2 * r + 1] *= inv;
          sq += acc[m][n][2 * r] * acc[m][n][2 * r] + acc[m][n][2 * r + 1] * acc[m][n][2 * r + 1];
        }
      }
      sq += __shfl_xor_sync(0xffffffffu, sq, 1);
      sq += __shfl_xor_sync(0xffffffffu, sq, 2);
      if (c4 == 0) ss_s[warp][t] = sq;
    }
  }
  __syncthreads();
#pragma unroll
  for (int m = 0; m < 4; ++m) {
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int t = m * 16 + r4 + r * 8;
      if (t >= len) continue;
      float tot = 0.f;
#pragma unroll
      for (int i = 0; i < NW; ++i) tot += ss_s[i][t];
      const float inv = 1.f / sqrtf(tot / static_cast<float>(p.vdim_true) + p.eps);
      const bf16* gr = proj + (t0 + t) * p.ldp + p.g_off + h * V;
      bf16* dst = static_cast<bf16*>(p.out) + (t0 + t) * p.ldo + h * V;
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        if (n < n_live) {
          const int v = (vt0 + n) * 8 + c4 * 2;
          const __nv_bfloat162 g2 = *reinterpret_cast<const __nv_bfloat162*>(gr + v);
          const float2 nw = *reinterpret_cast<const float2*>(p.norm + h * V + v);
          *reinterpret_cast<uint32_t*>(dst + v) =
              pack_bf16x2(acc[m][n][2 * r] * inv * nw.x * sigmoid_of<bf16>(__bfloat162float(g2.x)),
                          acc[m][n][2 * r + 1] * inv * nw.y * sigmoid_of<bf16>(__bfloat162float(g2.y)));
        }
      }
    }
  }
}

int64_t align256(int64_t n) { return (n + 255) & ~static_cast<int64_t>(255); }

// Lays the arrays out at `base` (null: only measures).
int64_t carve(ChunkWs* w, char* base, int T, int n_seq, int H, int D, int V) {
  const int64_t nc = T / L + n_seq;
  int64_t off = 0;
  auto take = [&](int64_t elems) {
    char* at = base == nullptr ? nullptr : base + off;
    off += align256(elems * 4);
    return at;
  };
  ChunkWs x;
  x.F = reinterpret_cast<float*>(take(static_cast<int64_t>(T) * H));
  x.ig = reinterpret_cast<float*>(take(static_cast<int64_t>(T) * H));
  x.mt = reinterpret_cast<float*>(take(static_cast<int64_t>(T) * H));
  x.c_m0 = reinterpret_cast<float*>(take(nc * H));
  x.c_m1 = reinterpret_cast<float*>(take(nc * H));
  x.c_F = reinterpret_cast<float*>(take(nc * H));
  x.c_u = reinterpret_cast<float*>(take(nc * H));
  x.U = reinterpret_cast<float*>(take(nc * H * D * V));
  x.Un = reinterpret_cast<float*>(take(nc * H * D));
  x.Sn = reinterpret_cast<float*>(take(nc * H * D));
  x.Sh = reinterpret_cast<uint32_t*>(take(nc * H * (D / 2) * V));
  x.Sl = reinterpret_cast<uint32_t*>(take(nc * H * (D / 2) * V));
  if (w != nullptr) *w = x;
  return off;
}

size_t output_smem(int D, int V) {
  return sizeof(bf16) * (2 * static_cast<size_t>(L) * (D + 8) + static_cast<size_t>(L) * (V + 8) + L * (L + 8));
}

template <typename K>
cudaError_t allow_smem(K kern, size_t smem) {
  return smem > 48 * 1024 ? cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem))
                          : cudaSuccess;
}

template <int NW, int NT>
cudaError_t launch_output(const MlstmArgs& a, const ChunkWs& w, int nc) {
  const size_t smem = output_smem(a.dim, a.vdim);
  const cudaError_t e = allow_smem(mlstm_output_kernel<NW, NT>, smem);
  if (e != cudaSuccess) return e;
  return launch_kernel(mlstm_output_kernel<NW, NT>, dim3(nc, a.n_heads), dim3(NW * 32), smem, a.stream, a.pdl, 1, a, w);
}

template <int MT>
cudaError_t launch_contrib(const MlstmArgs& a, const ChunkWs& w, int nc) {
  const int dk = a.dim < kDBlock ? a.dim : kDBlock;
  const size_t smem = sizeof(bf16) * (2 * static_cast<size_t>(L) * (dk + 8) + L * (kVSlice + 8));
  const cudaError_t e = allow_smem(mlstm_contrib_kernel<MT>, smem);
  if (e != cudaSuccess) return e;
  const int z = ((a.vdim + kVSlice - 1) / kVSlice) * ((a.dim + kDBlock - 1) / kDBlock);
  return launch_kernel(mlstm_contrib_kernel<MT>, dim3(nc, a.n_heads, z), dim3(256), smem, a.stream, a.pdl, 1, a, w);
}

}  // namespace

int64_t mlstm_chunked_workspace_bytes(int T, int n_seq, int n_heads, int dim, int vdim) {
  return carve(nullptr, nullptr, T, n_seq, n_heads, dim, vdim);
}

bool mlstm_chunked_supported(int dim, int vdim) {
  return dim % 16 == 0 && vdim % 16 == 0 && dim <= 512 && vdim <= 512 && output_smem(dim, vdim) <= 220 * 1024;
}

const char* mlstm_chunked(const MlstmArgs& a, void* workspace, int64_t workspace_bytes) {
  if (a.T <= 0 || a.n_seq <= 0) return nullptr;
  if (a.f32) return "mlstm_chunked: bf16 only";
  if (!mlstm_chunked_supported(a.dim, a.vdim)) return "mlstm_chunked: head widths must be multiples of 16 up to 512";
  if (a.ldp % 8 || a.ldo % 2 || a.q_off % 8 || a.k_off % 8 || a.v_off % 8 || a.g_off % 2) return "mlstm_chunked: misaligned rows";
  if (!(a.gate_cap > 0.f)) return "mlstm_chunked: the gate cap must be positive";
  if (a.n_seq > 65535 || a.n_heads > 65535) return "mlstm_chunked: too many sequences or heads";
  ChunkWs w;
  if (carve(&w, static_cast<char*>(workspace), a.T, a.n_seq, a.n_heads, a.dim, a.vdim) > workspace_bytes)
    return "mlstm_chunked: workspace too small";
  const int nc = a.T / L + a.n_seq;
  cudaError_t e = launch_kernel(mlstm_gates_kernel, dim3(a.n_seq, a.n_heads), dim3(a.T >= 8 * L * a.n_seq ? 1024 : 256), 0, a.stream, a.pdl, 1, a, w);
  if (e != cudaSuccess) return cudaGetErrorString(e);
  e = a.dim <= 128 ? launch_contrib<1>(a, w, nc) : launch_contrib<2>(a, w, nc);
  if (e != cudaSuccess) return cudaGetErrorString(e);
  const int blocks = ((a.dim / 2) * a.vdim + 255) / 256 + 1;
  e = launch_kernel(mlstm_scan_kernel, dim3(blocks, a.n_heads, a.n_seq), dim3(256), 0, a.stream, a.pdl, 1, a, w);
  if (e != cudaSuccess) return cudaGetErrorString(e);
  const int nt = (a.vdim / 8 + 7) / 8;
  if (nt <= 1) e = launch_output<8, 1>(a, w, nc);
  else if (nt <= 2) e = launch_output<8, 2>(a, w, nc);
  else if (nt <= 4) e = launch_output<16, 2>(a, w, nc);
  else e = launch_output<16, 4>(a, w, nc);
  return e == cudaSuccess ? nullptr : cudaGetErrorString(e);
}

}  // namespace nfb
