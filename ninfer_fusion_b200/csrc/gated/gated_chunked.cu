// Gated linear memory over prompt portions, in chunks of 64 tokens.  Unrolled over a chunk with the state S_0 at its start:
//   S_t^T q_t = (q_t * f_1 .. f_t)^T S_0  +  sum_{s <= t} [ sum_d q_t k_s f_{s+1} .. f_t ] v_s
// Decay products only ever cover consecutive tokens, so they are formed by multiplication (each factor is at most one, an
// underflow is a true zero); nothing is divided by a decay.  Three kernels:
//   contrib  one CTA per (chunk, head, value slice): what a chunk adds to the state, U = sum_s (k_s f_{s+1} .. f_64) v_s^T,
//            and the chunk's decay per channel
//   scan     elementwise over the chunks of a sequence: the state at every chunk's start, kept in fp32 and handed to the
//            next kernel as bf16 hi + lo pairs (two rows of the state packed per word: an MMA B fragment)
//   output   one CTA per (chunk, head): the bracket between blocks of 16 tokens on the tensor cores (queries decayed from
//            their block's start, keys to their block's end, whole blocks in between), inside a block pair by pair in
//            fp32; then values, S_0, head norm
// Decayed queries and keys, the state and the weights of the values enter the MMAs as hi + lo pairs (about 17 bits).
#include "gated.h"

#include "../common/elem.cuh"
#include "../common/launch.h"
#include "../common/mma_sync.cuh"

namespace nfb {

namespace {

using bf16 = __nv_bfloat16;
constexpr int L = kGatedChunk;
constexpr int B = 16;          // tokens per block
constexpr int NB = L / B;
constexpr int DB = 64;         // channels per pass
constexpr int kThreads = NB * DB;
constexpr int kVSlice = 128;   // state columns per CTA of the contribution kernel

struct Ws {
  float* U;       // [NC, H, D, V]
  float* decay;   // [NC, H, D]
  uint32_t* Sh;   // [NC, H, D / 2, V] bf16 pairs (rows 2 r, 2 r + 1)
  uint32_t* Sl;
};

// Chunk slots: the chunks of sequence s start at slot cu[s] / 64 + s (disjoint for any lengths).
__device__ __forceinline__ int chunk_base(const int* cu, int s) { return cu[s] / L + s; }

// Sequence, first token and length of a chunk slot; length 0 = unused slot.
__device__ __forceinline__ void chunk_of(const GatedArgs& p, int slot, int& t0, int& len) {
  int lo = 0, hi = p.n_seq - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (chunk_base(p.cu_seqlens, mid) <= slot) lo = mid; else hi = mid - 1;
  }
  const int k = slot - chunk_base(p.cu_seqlens, lo);
  t0 = p.cu_seqlens[lo] + k * L;
  len = k < 0 ? 0 : max(0, min(L, p.cu_seqlens[lo + 1] - t0));
}

__device__ __forceinline__ void split2(float x, float& hi, float& lo) {
  hi = __bfloat162float(__float2bfloat16(x));
  lo = x - hi;
}

// Thread (block i, channel): 16 tokens' keys decayed to the chunk's end.  DB channels per CTA.
__global__ void __launch_bounds__(kThreads) gated_contrib_kernel(const GatedArgs p, const Ws w) {
  extern __shared__ __align__(16) uint8_t smem[];
  __shared__ float tot[NB][DB];
  constexpr int ldk = DB + 8, ldv = kVSlice + 8;
  bf16* kh = reinterpret_cast<bf16*>(smem);   // [L][ldk]
  bf16* kl = kh + L * ldk;
  bf16* vs = kl + L * ldk;       // [L][ldv]
  const int H = p.n_heads, D = p.dim, V = p.vdim, n_vs = (V + kVSlice - 1) / kVSlice;
  const int slot = blockIdx.x, h = blockIdx.y, v0 = (blockIdx.z % n_vs) * kVSlice, d0 = (blockIdx.z / n_vs) * DB;
  pdl_launch_next();
  pdl_wait_prior();
  int t0, len;
  chunk_of(p, slot, t0, len);
  if (len <= 0) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, nd = min(DB, D - d0);
  const long long ch = static_cast<long long>(slot) * H + h;
  const bf16* proj = static_cast<const bf16*>(p.proj);
  const uint32_t vs_a = smem_u32(vs);
  for (int i = tid; i < L * (kVSlice / 8); i += kThreads) {
    const int s = i / (kVSlice / 8), c = (i % (kVSlice / 8)) * 8;
    const bool ok = s < len && v0 + c < V;
    cp_async16(vs_a + (s * ldv + c) * 2, ok ? proj + (t0 + s) * p.ldp + p.v_off + h * V + v0 + c : proj, ok);
  }
  cp_async_commit();
  const int blk = tid / DB, d = tid % DB;
  float k[B], prod = 1.f;
  {
    const float lower = d < nd ? p.lower[h * D + d0 + d] : 1.f;
    const float* g = p.gates + static_cast<long long>(t0 + blk * B) * p.ldg + h * D + d0 + d;
    const int n = d < nd ? min(B, len - blk * B) : 0;    // tokens of the block that exist
    float f[B], raw[B];
#pragma unroll
    for (int j = 0; j < B; ++j) raw[j] = j < n ? __ldg(g + j * p.ldg) : 0.f;
#pragma unroll
    for (int j = 0; j < B; ++j) {
      gated_forget(raw[j], lower, f[j], k[j]);
      f[j] = j < n ? f[j] : 1.f;
      k[j] = j < n ? k[j] : 0.f;
    }
#pragma unroll
    for (int j = B - 1; j >= 0; --j) {
      k[j] *= prod;
      prod *= f[j];
    }
  }
  tot[blk][d] = prod;
  __syncthreads();
  float after = 1.f;
#pragma unroll
  for (int i = NB - 1; i > 0; --i)
    if (i > blk) after *= tot[i][d];
#pragma unroll
  for (int j = 0; j < B; ++j) {
    float hi, lo;
    split2(k[j] * after, hi, lo);
    kh[(blk * B + j) * ldk + d] = __float2bfloat16(hi);
    kl[(blk * B + j) * ldk + d] = __float2bfloat16(lo);
  }
  if (blk == 0 && v0 == 0 && d < nd) w.decay[ch * D + d0 + d] = prod * after;
  cp_async_wait<0>();
  __syncthreads();
  const int mt = warp & 3, c0 = (warp >> 2) * (kVSlice / 2);   // 16 channels x 64 columns
  if (mt * 16 >= nd || v0 + c0 >= V) return;
  float acc[kVSlice / 16][4];
#pragma unroll
  for (int n = 0; n < kVSlice / 16; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[n][e] = 0.f;
  const uint32_t kh_a = smem_u32(kh), kl_a = smem_u32(kl);
  const int arow = (lane & 7) + ((lane >> 4) & 1) * 8, acol = ((lane >> 3) & 1) * 8;
#pragma unroll
  for (int kk = 0; kk < L / 16; ++kk) {
    uint32_t ah[4], al[4];
    const uint32_t at = ((kk * 16 + arow) * ldk + mt * 16 + acol) * 2;
    ldsm_x4_trans(kh_a + at, ah);
    ldsm_x4_trans(kl_a + at, al);
#pragma unroll
    for (int n = 0; n < kVSlice / 32; ++n) {
      if (v0 + c0 + n * 16 < V) {
        uint32_t b[4];
        ldsm_x4_trans(vs_a + ((kk * 16 + (lane & 15)) * ldv + c0 + n * 16 + (lane >> 4) * 8) * 2, b);
        mma_bf16_16816(acc[2 * n], ah, b[0], b[1]);
        mma_bf16_16816(acc[2 * n + 1], ah, b[2], b[3]);
        mma_bf16_16816(acc[2 * n], al, b[0], b[1]);
        mma_bf16_16816(acc[2 * n + 1], al, b[2], b[3]);
      }
    }
  }
  float* dst = w.U + (ch * D + d0 + mt * 16 + (lane >> 2)) * V + v0 + c0 + (lane & 3) * 2;
#pragma unroll
  for (int n = 0; n < kVSlice / 16; ++n) {
    if (v0 + c0 + n * 8 < V) {
      *reinterpret_cast<float2*>(dst + n * 8) = make_float2(acc[n][0], acc[n][1]);
      *reinterpret_cast<float2*>(dst + 8LL * V + n * 8) = make_float2(acc[n][2], acc[n][3]);
    }
  }
}

// grid: (blocks over D / 2 x V elements, head, sequence)
__global__ void __launch_bounds__(256) gated_scan_kernel(const GatedArgs p, const Ws w) {
  pdl_launch_next();
  pdl_wait_prior();
  const int H = p.n_heads, D = p.dim, V = p.vdim, h = blockIdx.y, seq = blockIdx.z;
  const int tb = p.cu_seqlens[seq], te = p.cu_seqlens[seq + 1];
  const int nc = (te - tb + L - 1) / L, base = chunk_base(p.cu_seqlens, seq);
  const int e = blockIdx.x * blockDim.x + threadIdx.x;
  if (e >= (D / 2) * V) return;
  const int r = e / V, v = e % V;
  float* s_state = p.S + ((static_cast<long long>(p.state_slot[seq]) * H + h) * D + 2 * r) * V + v;
  float s0 = s_state[0], s1 = s_state[V];
  const long long u_step = static_cast<long long>(H) * D * V, p_step = u_step / 2, d_step = static_cast<long long>(H) * D;
  const long long ch = static_cast<long long>(base) * H + h;
  const float* u = w.U + (ch * D + 2 * r) * V + v;
  const float2* dec = reinterpret_cast<const float2*>(w.decay + ch * D + 2 * r);
  uint32_t* oh = w.Sh + (ch * (D / 2) + r) * V + v;
  uint32_t* ol = w.Sl + (ch * (D / 2) + r) * V + v;
  constexpr int kAhead = 4;
  for (int c0 = 0; c0 < nc; c0 += kAhead) {
    float u0[kAhead], u1[kAhead];
    float2 f[kAhead];
#pragma unroll
    for (int j = 0; j < kAhead; ++j) {
      if (c0 + j < nc) {
        u0[j] = __ldcs(u + (c0 + j) * u_step);
        u1[j] = __ldcs(u + (c0 + j) * u_step + V);
        f[j] = dec[(c0 + j) * (d_step / 2)];
      }
    }
#pragma unroll
    for (int j = 0; j < kAhead; ++j) {
      if (c0 + j < nc) {
        float h0, l0, h1, l1;
        split2(s0, h0, l0);
        split2(s1, h1, l1);
        oh[(c0 + j) * p_step] = pack_bf16x2(h0, h1);
        ol[(c0 + j) * p_step] = pack_bf16x2(l0, l1);
        s0 = fmaf(f[j].x, s0, u0[j]);
        s1 = fmaf(f[j].y, s1, u1[j]);
      }
    }
  }
  if (p.write_state) {
    s_state[0] = s0;
    s_state[V] = s1;
  }
}

// Shared memory of the output kernel, in bytes.  The value weights reuse the pair operands' room, the values that of the
// decayed queries and keys (wider heads have room of their own).
struct OutPlan {
  static constexpr int ldq = DB + 8, ldf = DB + 4, ldp = L + 8;
  static constexpr int q = 0;                              // float [L][ldf] queries (pairs inside a block)
  static constexpr int k = q + L * ldf * 4;                // float [L][ldf] keys
  static constexpr int g = k + L * ldf * 4;                // float [L][ldf] log2 of the decay from the block's start
  static constexpr int wh = q;                             // bf16 [L][ldp] x 2: weights of the values, hi and lo
  static constexpr int wl = wh + L * ldp * 2;
  static constexpr int qb = g + L * ldf * 4;               // bf16 [L][ldq] x 2: queries decayed from their block's start
  static constexpr int kb = qb + 2 * L * ldq * 2;          // bf16 [L][ldq] x 2: keys decayed to their block's end
  static constexpr int qc = kb + 2 * L * ldq * 2;          // bf16 [L][ldq] x 2: queries decayed from the chunk's start
  static constexpr int tot = qc + 2 * L * ldq * 2;         // float [NB][DB] decay of whole blocks
  static constexpr int ss = tot + NB * DB * 4;             // float [8][L]
  static constexpr int end = ss + 8 * L * 4;
  static_assert(wl + L * ldp * 2 <= qb, "the weights fit into the pair operands' room");
  __host__ __device__ static int v(int V) { return L * (V + 8) * 2 <= qc - qb ? qb : end; }    // bf16 [L][V + 8]
  static int bytes(int V) { return v(V) == qb ? end : end + L * (V + 8) * 2; }
};

// NT: 8-wide value tiles per warp (8 warps cover V).  grid: (chunk slot, head)
template <int NT>
__global__ void __launch_bounds__(kThreads, NT <= 2 ? 2 : 1) gated_output_kernel(const GatedArgs p, const Ws w) {
  extern __shared__ __align__(16) uint8_t smem[];
  constexpr int ldq = OutPlan::ldq, ldf = OutPlan::ldf, ldp = OutPlan::ldp;
  float* q_s = reinterpret_cast<float*>(smem + OutPlan::q);
  float* k_s = reinterpret_cast<float*>(smem + OutPlan::k);
  float* g_s = reinterpret_cast<float*>(smem + OutPlan::g);
  bf16* wh_s = reinterpret_cast<bf16*>(smem + OutPlan::wh);
  bf16* wl_s = reinterpret_cast<bf16*>(smem + OutPlan::wl);
  float* tot = reinterpret_cast<float*>(smem + OutPlan::tot);
  float* ss = reinterpret_cast<float*>(smem + OutPlan::ss);
  const int H = p.n_heads, D = p.dim, V = p.vdim, ldv = V + 8;
  pdl_launch_next();
  pdl_wait_prior();
  const int slot = blockIdx.x, h = blockIdx.y;
  int t0, len;
  chunk_of(p, slot, t0, len);
  if (len <= 0) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, r4 = lane >> 2, c4 = lane & 3;
  const long long ch = static_cast<long long>(slot) * H + h;
  const bf16* proj = static_cast<const bf16*>(p.proj);
  const uint32_t base = smem_u32(smem), vs_a = base + OutPlan::v(p.vdim);
  constexpr int lo_q = L * ldq;                 // elements from a hi array to its lo array
  const int vt0 = warp * NT, n_live = min(NT, V / 8 - vt0);
  float acc[NB][NT][4];
#pragma unroll
  for (int m = 0; m < NB; ++m)
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[m][n][e] = 0.f;
  const int mi = warp & 3, nh = warp >> 2;      // query block and key half of the warp's weights between blocks
  float cb[NB - 1][4];
#pragma unroll
  for (int j = 0; j < NB - 1; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) cb[j][e] = 0.f;
  // pairs inside a block: NB * 136, thread i has pairs i, i + 256, i + 512
  constexpr int kPairs = B * (B + 1) / 2, kPer = (NB * kPairs + kThreads - 1) / kThreads;
  int pt[kPer], ps[kPer];
  float pa[kPer];
#pragma unroll
  for (int i = 0; i < kPer; ++i) {
    const int n = tid + i * kThreads, blk = n / kPairs, r = n % kPairs;
    int t = static_cast<int>((sqrtf(8.f * r + 1.f) - 1.f) * 0.5f);
    if ((t + 1) * (t + 2) / 2 <= r) ++t;
    if (t * (t + 1) / 2 > r) --t;
    pt[i] = n < NB * kPairs ? blk * B + t : -1;
    ps[i] = blk * B + r - t * (t + 1) / 2;
    pa[i] = 0.f;
  }
  for (int d0 = 0; d0 < D; d0 += DB) {
    const int nd = min(DB, D - d0);
    // ---- gates of 64 tokens x DB channels: thread = (block, channel) ----
    const int blk = tid / DB, d = tid % DB;
    float q[B], f[B], k[B], prod = 1.f, glog = 0.f;
    {
      const float lower = d < nd ? p.lower[h * D + d0 + d] : 1.f;
      const float* g = p.gates + static_cast<long long>(t0 + blk * B) * p.ldg + h * D + d0 + d;
      const bf16* qr = proj + static_cast<long long>(t0 + blk * B) * p.ldp + p.q_off + h * D + d0 + d;
      const int n = d < nd ? min(B, len - blk * B) : 0;    // tokens of the block that exist
#pragma unroll
      for (int j = 0; j < B; ++j) {
        f[j] = j < n ? __ldg(g + j * p.ldg) : 0.f;
        q[j] = j < n ? __bfloat162float(qr[j * p.ldp]) : 0.f;
      }
#pragma unroll
      for (int j = 0; j < B; ++j) {
        const float raw = f[j];
        gated_forget(raw, lower, f[j], k[j]);
        f[j] = j < n ? f[j] : 1.f;
        k[j] = j < n ? k[j] : 0.f;
        q[j] = q[j] * sigmoid_of<bf16>(q[j]);
      }
    }
    __syncthreads();            // the last pass is done with the arrays
#pragma unroll
    for (int j = 0; j < B; ++j) {
      const int at = blk * B + j;
      prod *= f[j];
      // log2 f without cancellation near one; f may underflow
      glog += k[j] < 0.5f ? log1pf(-k[j]) * kLog2e : log2f(fmaxf(f[j], 1e-37f));
      float hi, lo;
      split2(q[j] * prod, hi, lo);
      bf16* dst = reinterpret_cast<bf16*>(smem + OutPlan::qb) + at * ldq + d;
      dst[0] = __float2bfloat16(hi);
      dst[lo_q] = __float2bfloat16(lo);
      q_s[at * ldf + d] = q[j];
      k_s[at * ldf + d] = k[j];
      g_s[at * ldf + d] = glog;
      q[j] *= prod;
    }
    tot[blk * DB + d] = prod;
    float suffix = 1.f;
#pragma unroll
    for (int j = B - 1; j >= 0; --j) {
      float hi, lo;
      split2(k[j] * suffix, hi, lo);
      bf16* dst = reinterpret_cast<bf16*>(smem + OutPlan::kb) + (blk * B + j) * ldq + d;
      dst[0] = __float2bfloat16(hi);
      dst[lo_q] = __float2bfloat16(lo);
      suffix *= f[j];
    }
    __syncthreads();
    float before = 1.f;
#pragma unroll
    for (int i = 0; i < NB - 1; ++i)
      if (i < blk) before *= tot[i * DB + d];
#pragma unroll
    for (int j = 0; j < B; ++j) {
      float hi, lo;
      split2(q[j] * before, hi, lo);
      bf16* dst = reinterpret_cast<bf16*>(smem + OutPlan::qc) + (blk * B + j) * ldq + d;
      dst[0] = __float2bfloat16(hi);
      dst[lo_q] = __float2bfloat16(lo);
    }
    // ---- weights between blocks: 16 queries x 8 keys of every earlier block ----
    if (mi > 0) {
      for (int kk = 0; kk < nd; kk += 16) {
        uint32_t a[4], al[4];
        const uint32_t qa = base + OutPlan::qb + ((mi * 16 + (lane & 15)) * ldq + kk + (lane >> 4) * 8) * 2;
        ldsm_x4(qa, a);
        ldsm_x4(qa + lo_q * 2, al);
#pragma unroll
        for (int j = NB - 2; j >= 0; --j) {
          if (j >= mi) continue;
          if (j < mi - 1) {     // over the whole block j + 1
            const float* f1 = tot + (j + 1) * DB + kk + c4 * 2;
#pragma unroll
            for (int e = 0; e < 4; ++e) {          // e & 2: columns + 8
              const float x0 = __uint_as_float(a[e] << 16) + __uint_as_float(al[e] << 16);
              const float x1 = __uint_as_float(a[e] & 0xffff0000u) + __uint_as_float(al[e] & 0xffff0000u);
              float h0, l0, h1, l1;
              split2(x0 * f1[(e & 2) * 4], h0, l0);
              split2(x1 * f1[(e & 2) * 4 + 1], h1, l1);
              a[e] = pack_bf16x2(h0, h1);
              al[e] = pack_bf16x2(l0, l1);
            }
          }
          // keys 16 j + 8 nh .. + 7: hi of both 8-channel halves, then lo
          uint32_t b[4];
          ldsm_x4(base + OutPlan::kb + (lane >> 4) * (lo_q * 2) + ((j * 16 + nh * 8 + (lane & 7)) * ldq + kk + ((lane >> 3) & 1) * 8) * 2, b);
          mma_bf16_16816(cb[j], a, b[0], b[1]);
          mma_bf16_16816(cb[j], al, b[0], b[1]);
          mma_bf16_16816(cb[j], a, b[2], b[3]);
        }
      }
    }
    // ---- pairs inside a block ----
#pragma unroll
    for (int i = 0; i < kPer; ++i) {
      if (pt[i] < 0) continue;
      const float* qr = q_s + pt[i] * ldf;
      const float* kr = k_s + ps[i] * ldf;
      const float* gt = g_s + pt[i] * ldf;
      const float* gs = g_s + ps[i] * ldf;
      float s = pa[i];
#pragma unroll 4
      for (int c = 0; c < DB; c += 4) {
        const float4 qv = *reinterpret_cast<const float4*>(qr + c), kv = *reinterpret_cast<const float4*>(kr + c),
                     a = *reinterpret_cast<const float4*>(gt + c), b = *reinterpret_cast<const float4*>(gs + c);
        s = fmaf(qv.x * kv.x, ex2_fast(a.x - b.x), s);
        s = fmaf(qv.y * kv.y, ex2_fast(a.y - b.y), s);
        s = fmaf(qv.z * kv.z, ex2_fast(a.z - b.z), s);
        s = fmaf(qv.w * kv.w, ex2_fast(a.w - b.w), s);
      }
      pa[i] = s;
    }
    __syncthreads();            // the decayed queries are complete
    if (d0 + DB >= D) {         // the values, in place of the operands between blocks
      for (int i = tid; i < L * (V / 8); i += kThreads) {
        const int s = i / (V / 8), c = (i % (V / 8)) * 8;
        const bool ok = s < len;
        cp_async16(vs_a + (s * ldv + c) * 2, proj + (t0 + (ok ? s : 0)) * p.ldp + p.v_off + h * V + c, ok);
      }
      cp_async_commit();
    }
    // ---- S_0: all 64 queries x this warp's value tiles, its fragments straight from global memory ----
    if (n_live > 0) {
      const uint32_t* sh = w.Sh + (ch * (D / 2) + d0 / 2 + c4) * V + vt0 * 8 + r4;
      const uint32_t* sl = w.Sl + (ch * (D / 2) + d0 / 2 + c4) * V + vt0 * 8 + r4;
      for (int kk = 0; kk < nd; kk += 16) {
        uint32_t bh[NT][2], bl[NT][2];
#pragma unroll
        for (int n = 0; n < NT; ++n) {
          bh[n][0] = bh[n][1] = bl[n][0] = bl[n][1] = 0u;
          if (n < n_live) {
            const long long at = static_cast<long long>(kk / 2) * V + n * 8;
            bh[n][0] = sh[at]; bh[n][1] = sh[at + 4LL * V];
            bl[n][0] = sl[at]; bl[n][1] = sl[at + 4LL * V];
          }
        }
#pragma unroll
        for (int m = 0; m < NB; ++m) {
          uint32_t a[4], al[4];
          const uint32_t qa = base + OutPlan::qc + ((m * 16 + (lane & 15)) * ldq + kk + (lane >> 4) * 8) * 2;
          ldsm_x4(qa, a);
          ldsm_x4(qa + lo_q * 2, al);
#pragma unroll
          for (int n = 0; n < NT; ++n) {
            mma_bf16_16816(acc[m][n], a, bh[n][0], bh[n][1]);
            mma_bf16_16816(acc[m][n], al, bh[n][0], bh[n][1]);
            mma_bf16_16816(acc[m][n], a, bl[n][0], bl[n][1]);
          }
        }
      }
    }
  }
  // ---- weights of the values ----
  auto put = [&](int t, int s, float x) {
    float hi, lo;
    split2(x, hi, lo);
    wh_s[t * ldp + s] = __float2bfloat16(hi);
    wl_s[t * ldp + s] = __float2bfloat16(lo);
  };
  for (int i = tid; i < L * B; i += kThreads) {      // keys after their query, inside a block
    const int t = i / B, s = i % B;
    if (s > t % B) put(t, t / B * B + s, 0.f);
  }
#pragma unroll
  for (int i = 0; i < kPer; ++i)
    if (pt[i] >= 0) put(pt[i], ps[i], pa[i]);
#pragma unroll
  for (int j = 0; j < NB - 1; ++j) {
    if (j < mi) {
#pragma unroll
      for (int e = 0; e < 4; ++e) put(mi * 16 + r4 + (e >> 1) * 8, j * 16 + nh * 8 + c4 * 2 + (e & 1), cb[j][e]);
    }
  }
  cp_async_wait<0>();
  __syncthreads();
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
      for (int m = kk; m < NB; ++m) {                          // (keys after every query of the tile are left out)
        uint32_t a[4], al[4];
        const int at = ((m * 16 + (lane & 15)) * ldp + kk * 16 + (lane >> 4) * 8) * 2;
        ldsm_x4(base + OutPlan::wh + at, a);
        ldsm_x4(base + OutPlan::wl + at, al);
#pragma unroll
        for (int n = 0; n < NT; ++n) {
          mma_bf16_16816(acc[m][n], a, b[n][0], b[n][1]);
          mma_bf16_16816(acc[m][n], al, b[n][0], b[n][1]);
        }
      }
    }
  }
  // ---- head norm ----
#pragma unroll
  for (int m = 0; m < NB; ++m) {
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      float sq = 0.f;
#pragma unroll
      for (int n = 0; n < NT; ++n)
        if (n < n_live) sq += acc[m][n][2 * r] * acc[m][n][2 * r] + acc[m][n][2 * r + 1] * acc[m][n][2 * r + 1];
      sq += __shfl_xor_sync(0xffffffffu, sq, 1);
      sq += __shfl_xor_sync(0xffffffffu, sq, 2);
      if (c4 == 0) ss[warp * L + m * 16 + r4 + r * 8] = sq;
    }
  }
  __syncthreads();
#pragma unroll
  for (int m = 0; m < NB; ++m) {
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int t = m * 16 + r4 + r * 8;
      if (t >= len) continue;
      float sum = 0.f;
#pragma unroll
      for (int i = 0; i < kThreads / 32; ++i) sum += ss[i * L + t];
      const float inv = 1.f / sqrtf(sum / static_cast<float>(p.vdim_true) + p.eps);
      bf16* dst = static_cast<bf16*>(p.out) + (t0 + t) * p.ldo + h * V;
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        if (n < n_live) {
          const int v = (vt0 + n) * 8 + c4 * 2;
          const float2 nw = *reinterpret_cast<const float2*>(p.norm + v);
          *reinterpret_cast<uint32_t*>(dst + v) = pack_bf16x2(acc[m][n][2 * r] * inv * nw.x, acc[m][n][2 * r + 1] * inv * nw.y);
        }
      }
    }
  }
}

int64_t align256(int64_t n) { return (n + 255) & ~static_cast<int64_t>(255); }

// Lays the arrays out at `base` (null: only measures).
int64_t carve(Ws* w, char* base, int T, int n_seq, int H, int D, int V) {
  const int64_t nc = T / L + n_seq;
  int64_t off = 0;
  auto take = [&](int64_t elems) {
    char* at = base == nullptr ? nullptr : base + off;
    off += align256(elems * 4);
    return at;
  };
  Ws x;
  x.U = reinterpret_cast<float*>(take(nc * H * D * V));
  x.decay = reinterpret_cast<float*>(take(nc * H * D));
  x.Sh = reinterpret_cast<uint32_t*>(take(nc * H * (D / 2) * V));
  x.Sl = reinterpret_cast<uint32_t*>(take(nc * H * (D / 2) * V));
  if (w != nullptr) *w = x;
  return off;
}

template <typename K>
cudaError_t allow_smem(K kern, int smem) {
  return smem > 48 * 1024 ? cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) : cudaSuccess;
}

template <int NT>
cudaError_t launch_output(const GatedArgs& a, const Ws& w, int nc) {
  const int smem = OutPlan::bytes(a.vdim);
  const cudaError_t e = allow_smem(gated_output_kernel<NT>, smem);
  if (e != cudaSuccess) return e;
  return launch_kernel(gated_output_kernel<NT>, dim3(nc, a.n_heads), dim3(kThreads), smem, a.stream, a.pdl, 1, a, w);
}

}  // namespace

int64_t gated_chunked_workspace_bytes(int T, int n_seq, int n_heads, int dim, int vdim) {
  return carve(nullptr, nullptr, T, n_seq, n_heads, dim, vdim);
}

bool gated_chunked_supported(int dim, int vdim) {
  return dim % 16 == 0 && vdim % 16 == 0 && dim > 0 && vdim > 0 && dim <= 512 && vdim <= 512 && OutPlan::bytes(vdim) <= 225 * 1024;
}

const char* gated_chunked(const GatedArgs& a, void* workspace, int64_t workspace_bytes) {
  if (a.T <= 0 || a.n_seq <= 0) return nullptr;
  if (a.f32) return "gated_chunked: bf16 only";
  if (!gated_chunked_supported(a.dim, a.vdim)) return "gated_chunked: head widths must be multiples of 16 up to 512";
  if (a.ldp % 8 || a.ldo % 2 || a.q_off % 8 || a.v_off % 8) return "gated_chunked: misaligned rows";
  if (a.n_seq > 65535 || a.n_heads > 65535) return "gated_chunked: too many sequences or heads";
  Ws w;
  if (carve(&w, static_cast<char*>(workspace), a.T, a.n_seq, a.n_heads, a.dim, a.vdim) > workspace_bytes)
    return "gated_chunked: workspace too small";
  const int nc = a.T / L + a.n_seq;
  constexpr int smem = (2 * L * (DB + 8) + L * (kVSlice + 8)) * 2;
  cudaError_t e = allow_smem(gated_contrib_kernel, smem);
  if (e != cudaSuccess) return cudaGetErrorString(e);
  const int z = ((a.vdim + kVSlice - 1) / kVSlice) * ((a.dim + DB - 1) / DB);
  e = launch_kernel(gated_contrib_kernel, dim3(nc, a.n_heads, z), dim3(kThreads), smem, a.stream, a.pdl, 1, a, w);
  if (e != cudaSuccess) return cudaGetErrorString(e);
  e = launch_kernel(gated_scan_kernel, dim3(((a.dim / 2) * a.vdim + 255) / 256, a.n_heads, a.n_seq), dim3(256), 0, a.stream, a.pdl, 1, a, w);
  if (e != cudaSuccess) return cudaGetErrorString(e);
  const int nt = (a.vdim / 8 + 7) / 8;
  if (nt <= 1) e = launch_output<1>(a, w, nc);
  else if (nt <= 2) e = launch_output<2>(a, w, nc);
  else if (nt <= 4) e = launch_output<4>(a, w, nc);
  else e = launch_output<8>(a, w, nc);
  return e == cudaSuccess ? nullptr : cudaGetErrorString(e);
}

}  // namespace nfb
