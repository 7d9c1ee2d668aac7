// Grouped-query attention over paged rows on the tensor cores (bf16): scores are scaled dot products, masks are causal with an
// optional window or chunk, sinks only count in the denominator.
//
// Prefill: one CTA = (query head, block of 64 queries), a warp owns 16 queries; key and value tiles of 64 positions come
// through a two-stage cp.async ring, scores, weights and running sums stay in registers.  Tiles start at multiples of 64
// positions, so that with pages of 64 k tokens a tile lies in one page.
//
// Decode: one CTA = (token, kv head, split of the keys).  The rows of the MMA are the query heads of the group.  Each of the
// four warps streams every fourth 16-key tile through a ring of its own and keeps its own running softmax; no barrier
// until the four meet at the end.
#include "head_mix.h"

#include <math_constants.h>

#include "../common/elem.cuh"
#include "../common/launch.h"
#include "../common/mma_sync.cuh"

namespace nfb {

namespace {

using bf16 = __nv_bfloat16;
constexpr int KT = 64, QT = kHeadMixBlock, kThreads = 128;
constexpr int kSmemLimit = 225 * 1024;

// DT / VT: upper bounds of dim / 16 and vdim / 8.  ALIGNED: page_size % 64 == 0.
template <int DT, int VT, bool ALIGNED>
__global__ void __launch_bounds__(kThreads) group_prefill_kernel(const HeadMixArgs p, const int* __restrict__ blk_start,
                                                                  const int* __restrict__ blk_count) {
  extern __shared__ __align__(16) bf16 smem_b[];
  constexpr bool kQReg = DT <= 8;
  const int D = p.dim, V = p.vdim, G = p.n_kv, P = p.page_size;
  const int ldk = D + 8, ldv = V + 8, stage = KT * (ldk + ldv);
  bf16* qs = smem_b;                       // [QT][ldk]
  const uint32_t qs_a = smem_u32(qs), ring_a = qs_a + QT * ldk * 2;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, r4 = lane >> 2, c4 = lane & 3;
  pdl_launch_next();
  pdl_wait_prior();
  const int h = blockIdx.x, g = h / (p.n_heads / G), blk = static_cast<int>(gridDim.y) - 1 - static_cast<int>(blockIdx.y);
  const int t0 = blk_start[blk], count = blk_count[blk];
  const int first_len = p.kv_len[t0], len = first_len + count - 1;
  const int k_lo = first_visible(first_len, p.window, p.chunk), k_begin = k_lo / KT * KT;
  const int n_tiles = (len - k_begin + KT - 1) / KT;
  const int* table = p.block_table + static_cast<long long>(p.table_row[t0]) * p.table_ld;
  const bf16* kp = static_cast<const bf16*>(p.k_pages);
  const bf16* vp = static_cast<const bf16*>(p.v_pages);
  const int d8 = D / 8, v8 = V / 8;
  // 16 threads walk a row; a thread's rows of a tile are lr, lr + 8, ..., its 16-byte pieces lc, lc + 16, ...
  const int lr = tid >> 4, lc = tid & 15;
  auto load = [&](int tile) {
    const int k0 = k_begin + tile * KT, left = len - k0;
    const uint32_t dk = ring_a + (tile & 1) * stage * 2 + lr * ldk * 2, dv = ring_a + ((tile & 1) * stage + KT * ldk + lr * ldv) * 2;
    if constexpr (ALIGNED) {
      const int page = table[k0 / P];
      const long long row = (static_cast<long long>(max(page, 0)) * G + g) * P + k0 % P + lr;
      const int n = page < 0 ? 0 : left;
      for (int c = lc; c < d8; c += 16) {
        const bf16* src = kp + row * D + c * 8;
#pragma unroll
        for (int j = 0; j < KT / 8; ++j) {
          const bool ok = lr + j * 8 < n;
          cp_async16(dk + c * 16 + j * (8 * ldk * 2), ok ? src + j * 8 * D : kp, ok);
        }
      }
      for (int c = lc; c < v8; c += 16) {
        const bf16* src = vp + row * V + c * 8;
#pragma unroll
        for (int j = 0; j < KT / 8; ++j) {
          const bool ok = lr + j * 8 < n;
          cp_async16(dv + c * 16 + j * (8 * ldv * 2), ok ? src + j * 8 * V : vp, ok);
        }
      }
    } else {
      for (int j = 0; j < KT / 8; ++j) {
        const int r = lr + j * 8;
        const int page = r < left ? table[(k0 + r) / P] : -1;
        const bool ok = page >= 0;
        const long long row = (static_cast<long long>(ok ? page : 0) * G + g) * P + (ok ? (k0 + r) % P : 0);
        for (int c = lc; c < d8; c += 16) cp_async16(dk + c * 16 + j * (8 * ldk * 2), kp + row * D + c * 8, ok);
        for (int c = lc; c < v8; c += 16) cp_async16(dv + c * 16 + j * (8 * ldv * 2), vp + row * V + c * 8, ok);
      }
    }
  };
  load(0);
  cp_async_commit();
  for (int i = tid; i < QT * d8; i += kThreads) {
    const int r = i / d8, c = (i % d8) * 8;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (r < count) v = *reinterpret_cast<const uint4*>(static_cast<const bf16*>(p.q) + (t0 + r) * p.ldq + static_cast<long long>(h) * D + c);
    *reinterpret_cast<uint4*>(qs + r * ldk + c) = v;
  }
  const int row0 = warp * 16;
  const uint32_t qa = qs_a + ((row0 + (lane & 15)) * ldk + (lane >> 4) * 8) * 2;
  uint32_t qf[kQReg ? DT : 1][4];
  if constexpr (kQReg) {
    __syncthreads();
#pragma unroll
    for (int d = 0; d < DT; ++d)
      if (d * 16 < D) ldsm_x4(qa + d * 32, qf[d]);
  }
  float o[VT][4];
#pragma unroll
  for (int n = 0; n < VT; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[n][e] = 0.f;
  float m[2] = {-CUDART_INF_F, -CUDART_INF_F}, l[2] = {0.f, 0.f};
  int rlen[2], rlo[2];
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int row = row0 + r4 + r * 8;
    rlen[r] = row < count ? first_len + row : 0;
    rlo[r] = row < count ? first_visible(first_len + row, p.window, p.chunk) : 0;
  }
  const int last_lo = first_visible(len, p.window, p.chunk);     // every query of the block sees keys [last_lo, first_len)
  const float scale2 = p.scale * kLog2e;
  for (int tile = 0; tile < n_tiles; ++tile) {
    cp_async_wait<0>();
    __syncthreads();
    if (tile + 1 < n_tiles) load(tile + 1);
    cp_async_commit();
    const uint32_t kt = ring_a + (tile & 1) * stage * 2, vt = kt + KT * ldk * 2;
    float s[KT / 8][4];
#pragma unroll
    for (int n = 0; n < KT / 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[n][e] = 0.f;
    const uint32_t ka = kt + (((lane & 7) + (lane >> 4) * 8) * ldk + ((lane >> 3) & 1) * 8) * 2;
    auto step = [&](int d, const uint32_t* a) {
#pragma unroll
      for (int n = 0; n < KT / 16; ++n) {
        uint32_t k[4];
        ldsm_x4(ka + n * (16 * ldk * 2) + d * 32, k);
        mma_bf16_16816(s[2 * n], a, k[0], k[1]);
        mma_bf16_16816(s[2 * n + 1], a, k[2], k[3]);
      }
    };
    if constexpr (kQReg) {
#pragma unroll
      for (int d = 0; d < DT; ++d)
        if (d * 16 < D) step(d, qf[d]);
    } else {
#pragma unroll 2
      for (int d = 0; d < D / 16; ++d) {
        uint32_t a[4];
        ldsm_x4(qa + d * 32, a);
        step(d, a);
      }
    }
    const int k0 = k_begin + tile * KT;
    if (k0 + KT > first_len || k0 < last_lo) {       // some query of the block does not see all of the tile
#pragma unroll
      for (int n = 0; n < KT / 8; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int key = k0 + n * 8 + c4 * 2 + (e & 1);
          if (key >= rlen[e >> 1] || key < rlo[e >> 1]) s[n][e] = -CUDART_INF_F;
        }
    }
    float mt[2] = {m[0], m[1]};
#pragma unroll
    for (int n = 0; n < KT / 8; ++n) {
      mt[0] = fmaxf(mt[0], fmaxf(s[n][0], s[n][1]) * scale2);
      mt[1] = fmaxf(mt[1], fmaxf(s[n][2], s[n][3]) * scale2);
    }
    float f[2], off[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      mt[r] = fmaxf(mt[r], __shfl_xor_sync(0xffffffffu, mt[r], 1));
      mt[r] = fmaxf(mt[r], __shfl_xor_sync(0xffffffffu, mt[r], 2));
      off[r] = mt[r] > -CUDART_INF_F ? mt[r] : 0.f;
      f[r] = ex2_fast(m[r] - off[r]);
      m[r] = mt[r];
      l[r] *= f[r];
    }
#pragma unroll
    for (int n = 0; n < KT / 8; ++n) {
      s[n][0] = ex2_fast(fmaf(s[n][0], scale2, -off[0])); s[n][1] = ex2_fast(fmaf(s[n][1], scale2, -off[0]));
      s[n][2] = ex2_fast(fmaf(s[n][2], scale2, -off[1])); s[n][3] = ex2_fast(fmaf(s[n][3], scale2, -off[1]));
      l[0] += s[n][0] + s[n][1];
      l[1] += s[n][2] + s[n][3];
    }
#pragma unroll
    for (int n = 0; n < VT; ++n) { o[n][0] *= f[0]; o[n][1] *= f[0]; o[n][2] *= f[1]; o[n][3] *= f[1]; }
#pragma unroll
    for (int kk = 0; kk < KT / 16; ++kk) {
      const uint32_t a[4] = {pack_bf16x2(s[2 * kk][0], s[2 * kk][1]), pack_bf16x2(s[2 * kk][2], s[2 * kk][3]),
                             pack_bf16x2(s[2 * kk + 1][0], s[2 * kk + 1][1]), pack_bf16x2(s[2 * kk + 1][2], s[2 * kk + 1][3])};
#pragma unroll
      for (int n = 0; n < VT; n += 2) {
        if (n * 8 < V) {
          uint32_t v[4];
          ldsm_x4_trans(vt + ((kk * 16 + (lane & 15)) * ldv + n * 8 + (lane >> 4) * 8) * 2, v);
          mma_bf16_16816(o[n], a, v[0], v[1]);
          mma_bf16_16816(o[n + 1], a, v[2], v[3]);
        }
      }
    }
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
    const int row = row0 + r4 + r * 8;
    if (row >= count) continue;
    const float inv = head_mix_finish(m[r] * (1.f / kLog2e), l[r], p.sink, p.sinks, h);
    bf16* dst = static_cast<bf16*>(p.out) + (t0 + row) * p.ldo + static_cast<long long>(h) * V;
#pragma unroll
    for (int n = 0; n < VT; ++n)
      if (n * 8 < V) *reinterpret_cast<uint32_t*>(dst + n * 8 + c4 * 2) = pack_bf16x2(o[n][2 * r] * inv, o[n][2 * r + 1] * inv);
  }
}

// ---------------------------------------------------------------------------------------------------------- decode
constexpr int NW = 4, DK = 16;    // warps, keys per tile of a warp

struct DecodePlan {
  int ldk, ldv, stage, ring, meet, total;     // bytes, from the start of shared memory
  __host__ __device__ DecodePlan(int D, int V, int stages) {
    ldk = D + 8;
    ldv = V + 8;
    stage = DK * (ldk + ldv) * 2;
    ring = DK * ldk * 2;                       // behind the query heads [16][ldk]
    const int rings = ring + NW * stages * stage;
    meet = NW * 16 * (V + 2) * 4;              // the warps' sums, maxima and partial outputs, over the rings
    total = rings > ring + meet ? rings : ring + meet;
  }
};

template <int DT, int VT, int S>
__global__ void __launch_bounds__(kThreads) group_decode_kernel(const HeadMixArgs p, int split_keys, int n_splits, float* __restrict__ part_o,
                                                                 float* __restrict__ part_ml) {
  extern __shared__ __align__(16) uint8_t smem[];
  constexpr bool kQReg = DT <= 8;
  const int H = p.n_heads, G = p.n_kv, R = H / G, D = p.dim, V = p.vdim, P = p.page_size;
  const int row_tiles = (R + 15) / 16;
  const DecodePlan plan(D, V, S);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, r4 = lane >> 2, c4 = lane & 3;
  pdl_launch_next();
  pdl_wait_prior();
  const int t = blockIdx.x, g = blockIdx.y / row_tiles, h0 = g * R + blockIdx.y % row_tiles * 16, split = blockIdx.z;
  const int n_rows = min(16, (g + 1) * R - h0);
  const int len = p.kv_len[t], lo = first_visible(len, p.window, p.chunk);
  const int k_begin = lo + split * split_keys, k_end = min(len, k_begin + split_keys);
  const int n_tiles = k_end > k_begin ? (k_end - k_begin + DK - 1) / DK : 0;
  const int mine = n_tiles > warp ? (n_tiles - warp + NW - 1) / NW : 0;
  const int* table = p.block_table + static_cast<long long>(p.table_row[t]) * p.table_ld;
  const bf16* kp = static_cast<const bf16*>(p.k_pages);
  const bf16* vp = static_cast<const bf16*>(p.v_pages);
  const uint32_t q_a = smem_u32(smem), ring_a = q_a + plan.ring + warp * S * plan.stage;
  const int ldk = plan.ldk, ldv = plan.ldv;
  auto key_row = [&](int i) {          // row of key lane & 15 of the warp's tile i, -1: past the end or not mapped
    const int key = k_begin + (warp + i * NW) * DK + (lane & 15);
    if (i >= mine || key >= k_end) return -1;
    const int page = table[key / P];
    return page < 0 ? -1 : (page * G + g) * P + key % P;
  };
  // four lanes walk a row, 64 bytes at a time; a lane's rows are lane / 4 and lane / 4 + 8
  auto load = [&](int row, int i) {
    const uint32_t dst = ring_a + (i % S) * plan.stage + (lane & 3) * 16;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int key = (lane >> 2) + half * 8, r = __shfl_sync(0xffffffffu, row, key);
      const bool ok = r >= 0;
      const bf16* ks = kp + static_cast<long long>(ok ? r : 0) * D + (lane & 3) * 8;
      const bf16* vs = vp + static_cast<long long>(ok ? r : 0) * V + (lane & 3) * 8;
      const uint32_t dk = dst + key * ldk * 2, dv = dst + (DK * ldk + key * ldv) * 2;
#pragma unroll
      for (int c = 0; c < DT * 16; c += 32)
        if (c + (lane & 3) * 8 < D) cp_async16(dk + c * 2, ks + c, ok);
#pragma unroll
      for (int c = 0; c < VT * 8; c += 32)
        if (c + (lane & 3) * 8 < V) cp_async16(dv + c * 2, vs + c, ok);
    }
  };
#pragma unroll
  for (int s = 0; s < S - 1; ++s) {
    const int row = key_row(s);
    if (s < mine) load(row, s);
    cp_async_commit();
  }
  int next_row = key_row(S - 1);
  bf16* qs = reinterpret_cast<bf16*>(smem);
  for (int i = tid; i < 16 * (D / 8); i += kThreads) {
    const int r = i / (D / 8), c = (i % (D / 8)) * 8;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (r < n_rows) v = *reinterpret_cast<const uint4*>(static_cast<const bf16*>(p.q) + t * p.ldq + static_cast<long long>(h0 + r) * D + c);
    *reinterpret_cast<uint4*>(qs + r * ldk + c) = v;
  }
  __syncthreads();
  const uint32_t qa = q_a + ((lane & 15) * ldk + (lane >> 4) * 8) * 2;
  uint32_t qf[kQReg ? DT : 1][4];
  if constexpr (kQReg) {
#pragma unroll
    for (int d = 0; d < DT; ++d)
      if (d * 16 < D) ldsm_x4(qa + d * 32, qf[d]);
  }
  float o[VT][4];
#pragma unroll
  for (int n = 0; n < VT; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[n][e] = 0.f;
  float m[2] = {-CUDART_INF_F, -CUDART_INF_F}, l[2] = {0.f, 0.f};
  const float scale2 = p.scale * kLog2e;
  for (int i = 0; i < mine; ++i) {
    cp_async_wait<S - 2>();
    __syncwarp();
    if (i + S - 1 < mine) load(next_row, i + S - 1);
    cp_async_commit();
    next_row = key_row(i + S);
    const uint32_t kt = ring_a + (i % S) * plan.stage, vt = kt + DK * ldk * 2;
    const uint32_t ka = kt + (((lane & 7) + (lane >> 4) * 8) * ldk + ((lane >> 3) & 1) * 8) * 2;
    float c[2][4] = {};
    auto step = [&](int d, const uint32_t* a) {
      uint32_t k[4];
      ldsm_x4(ka + d * 32, k);
      mma_bf16_16816(c[0], a, k[0], k[1]);
      mma_bf16_16816(c[1], a, k[2], k[3]);
    };
    if constexpr (kQReg) {
#pragma unroll
      for (int d = 0; d < DT; ++d)
        if (d * 16 < D) step(d, qf[d]);
    } else {
#pragma unroll 4
      for (int d = 0; d < D / 16; ++d) {
        uint32_t a[4];
        ldsm_x4(qa + d * 32, a);
        step(d, a);
      }
    }
    const int key0 = k_begin + (warp + i * NW) * DK;
    if (key0 + DK > k_end) {
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (key0 + n * 8 + c4 * 2 + (e & 1) >= k_end) c[n][e] = -CUDART_INF_F;
    }
    float f[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      float mx = fmaxf(fmaxf(c[0][2 * r], c[0][2 * r + 1]), fmaxf(c[1][2 * r], c[1][2 * r + 1])) * scale2;
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
      mx = fmaxf(mx, m[r]);                 // (every tile has a key: mx is finite)
      f[r] = ex2_fast(m[r] - mx);
      m[r] = mx;
      l[r] *= f[r];
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 2 * r; e < 2 * r + 2; ++e) {
          c[n][e] = ex2_fast(fmaf(c[n][e], scale2, -mx));
          l[r] += c[n][e];
        }
    }
    const uint32_t af[4] = {pack_bf16x2(c[0][0], c[0][1]), pack_bf16x2(c[0][2], c[0][3]), pack_bf16x2(c[1][0], c[1][1]),
                            pack_bf16x2(c[1][2], c[1][3])};
#pragma unroll
    for (int n = 0; n < VT; n += 2) {
      if (n * 8 < V) {
        uint32_t b[4];
        ldsm_x4_trans(vt + ((lane & 15) * ldv + n * 8 + (lane >> 4) * 8) * 2, b);
#pragma unroll
        for (int u = 0; u < 2; ++u) {
          o[n + u][0] *= f[0]; o[n + u][1] *= f[0];
          o[n + u][2] *= f[1]; o[n + u][3] *= f[1];
          mma_bf16_16816(o[n + u], af, b[2 * u], b[2 * u + 1]);
        }
      }
    }
    __syncwarp();
  }
  cp_async_wait<0>();
  __syncthreads();
  // ---- the warps meet ----
  float* sums = reinterpret_cast<float*>(smem + plan.ring);       // [NW][16][V], then [NW][16][2]
  float* ml = sums + NW * 16 * V;
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
    const int row = warp * 16 + r4 + r * 8;
    if (c4 == 0) {
      ml[row * 2] = m[r];
      ml[row * 2 + 1] = l[r];
    }
#pragma unroll
    for (int n = 0; n < VT; ++n)
      if (n * 8 < V) *reinterpret_cast<float2*>(sums + row * V + n * 8 + c4 * 2) = make_float2(o[n][2 * r], o[n][2 * r + 1]);
  }
  __syncthreads();
  const int v4 = V / 4;
  for (int i = tid; i < n_rows * v4; i += kThreads) {
    const int r = i / v4, col = (i % v4) * 4, h = h0 + r;
    float mx = -CUDART_INF_F;
#pragma unroll
    for (int w = 0; w < NW; ++w) mx = fmaxf(mx, ml[(w * 16 + r) * 2]);
    float sum = 0.f, x[4] = {};
#pragma unroll
    for (int w = 0; w < NW; ++w) {
      const float mw = ml[(w * 16 + r) * 2];
      const float e = mw > -CUDART_INF_F ? ex2_fast(mw - mx) : 0.f;
      sum = fmaf(e, ml[(w * 16 + r) * 2 + 1], sum);
      const float4 v = *reinterpret_cast<const float4*>(sums + (w * 16 + r) * V + col);
      x[0] = fmaf(e, v.x, x[0]); x[1] = fmaf(e, v.y, x[1]); x[2] = fmaf(e, v.z, x[2]); x[3] = fmaf(e, v.w, x[3]);
    }
    const float m_e = mx > -CUDART_INF_F ? mx * (1.f / kLog2e) : -CUDART_INF_F;      // the merge works with natural exponents
    if (n_splits > 1) {
      const long long at = (static_cast<long long>(t) * n_splits + split) * H + h;
      *reinterpret_cast<float4*>(part_o + at * V + col) = make_float4(x[0], x[1], x[2], x[3]);
      if (col == 0) {
        part_ml[at * 2] = m_e;
        part_ml[at * 2 + 1] = sum;
      }
    } else {
      const float f = head_mix_finish(m_e, sum, p.sink, p.sinks, h);
      *reinterpret_cast<uint2*>(static_cast<bf16*>(p.out) + t * p.ldo + static_cast<long long>(h) * V + col) =
          make_uint2(pack_bf16x2(x[0] * f, x[1] * f), pack_bf16x2(x[2] * f, x[3] * f));
    }
  }
}

template <int DT, int VT, int S>
cudaError_t launch_decode(const HeadMixArgs& a, int split_keys, int n_splits, float* part_o, float* part_ml) {
  auto kern = group_decode_kernel<DT, VT, S>;
  const int smem = DecodePlan(a.dim, a.vdim, S).total;
  const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) return e;
  const int row_tiles = (a.n_heads / a.n_kv + 15) / 16;
  return launch_kernel(kern, dim3(a.T, a.n_kv * row_tiles, n_splits), dim3(kThreads), smem, a.stream, a.pdl, 1, a, split_keys, n_splits,
                       part_o, part_ml);
}

int prefill_smem(int D, int V) { return (QT * (D + 8) + 2 * KT * (D + 8 + V + 8)) * 2; }

template <int DT, int VT>
cudaError_t launch_prefill(const HeadMixArgs& a, const int* start, const int* count, int n) {
  auto kern = a.page_size % KT == 0 ? group_prefill_kernel<DT, VT, true> : group_prefill_kernel<DT, VT, false>;
  const int smem = prefill_smem(a.dim, a.vdim);
  const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) return e;
  return launch_kernel(kern, dim3(a.n_heads, n), dim3(kThreads), smem, a.stream, a.pdl, 1, a, start, count);
}

}  // namespace

bool group_attention_supported(const HeadMixArgs& a) {
  return !a.f32 && !a.sigmoid && a.mix == nullptr && a.slope == nullptr && a.gate == nullptr && a.softcap == 0.f && a.dim % 16 == 0 && a.vdim % 16 == 0 &&
         a.dim <= 256 && a.vdim <= 256 && a.n_kv > 0 && a.n_heads % a.n_kv == 0 && a.ldq % 8 == 0 && a.ldo % 8 == 0 &&
         a.n_kv * ((a.n_heads / a.n_kv + 15) / 16) <= 65535 && prefill_smem(a.dim, a.vdim) <= kSmemLimit;
}

const char* group_decode(const HeadMixArgs& a, int split_keys, int n_splits, float* part_o, float* part_ml) {
  if (a.T <= 0) return nullptr;
  if (!group_attention_supported(a)) return "group attention: unsupported head geometry or scores";
  if (split_keys <= 0 || n_splits <= 0 || n_splits > 65535 || (n_splits > 1 && (part_o == nullptr || part_ml == nullptr)))
    return "group attention: bad split";
  cudaError_t e;
  if (a.dim <= 64 && a.vdim <= 64) e = launch_decode<4, 8, 4>(a, split_keys, n_splits, part_o, part_ml);
  else if (a.dim <= 128 && a.vdim <= 128) e = launch_decode<8, 16, 3>(a, split_keys, n_splits, part_o, part_ml);
  else e = launch_decode<16, 32, 2>(a, split_keys, n_splits, part_o, part_ml);
  return e == cudaSuccess ? nullptr : cudaGetErrorString(e);
}

const char* group_prefill(const HeadMixArgs& a, const int* blk_start, const int* blk_count, int n_blocks) {
  if (a.T <= 0 || n_blocks <= 0) return nullptr;
  if (!group_attention_supported(a) || n_blocks > 65535) return "group attention: unsupported head geometry or scores";
  cudaError_t e;
  if (a.dim <= 64 && a.vdim <= 64) e = launch_prefill<4, 8>(a, blk_start, blk_count, n_blocks);
  else if (a.dim <= 128 && a.vdim <= 128) e = launch_prefill<8, 16>(a, blk_start, blk_count, n_blocks);
  else e = launch_prefill<16, 32>(a, blk_start, blk_count, n_blocks);
  return e == cudaSuccess ? nullptr : cudaGetErrorString(e);
}

}  // namespace nfb
