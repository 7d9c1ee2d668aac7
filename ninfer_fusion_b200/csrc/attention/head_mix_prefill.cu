// Head-mixing attention for prompt portions (bf16 operands, tensor cores).  A mixed score needs every head's score of
// the same (query, key), while the weighted sum over values is per head, so the work is cut in two kernels that meet in
// a scratch of fp32 scores:
//
//   scores   one warp = 16 queries x 8 NT keys x ALL heads (two kernels: query heads resident in shared memory, or, for
//            head counts and widths that do not fit there, every operand from global memory).  The scores of one head come out of mma.sync in registers,
//            are soft-capped there and added into the mixed scores of every head, acc[h] += mix[h, g] * c_g (outer
//            product form: no score ever crosses a thread).  Distance bias and mask are applied to the finished sums,
//            which are stored in accumulator-fragment order.  Query and key fragments are read straight from global /
//            L1: the k index of an MMA may be permuted freely as long as both operands agree, so each lane takes four
//            consecutive values per 16-wide step.
//   values   one CTA = (64 queries, head): flash-style running softmax over score fragments read back in the same
//            order (they are exactly the A operand of the value MMA), V tiles staged with cp.async.
//
// Sigmoid weights stand by themselves, so they are made before the mix: the first kernel leaves mixed WEIGHTS as bf16 pairs,
// half the scratch, and the second one only multiplies them with the values.
//
// Query blocks are processed as many at a time as the scratch holds.
#include "head_mix.h"

#include <math_constants.h>

#include "../common/elem.cuh"
#include "../common/launch.h"
#include "../common/mma_sync.cuh"

namespace nfb {

namespace {

using bf16 = __nv_bfloat16;

struct PrefillParams {
  HeadMixArgs a;
  const int* blk_start;
  const int* blk_count;
  int blk0;            // first query block of this launch
  int n_tiles;         // 8-key tiles reserved per query block
  float4* scratch;     // [block][tile][q tile 0..3][head][lane]; sigmoid: uint2, weights of rows r4 and r4 + 8 as bf16 pairs
};

// Sigmoid weights of the accumulators c[NT][4] of one head.  `base` is the distance of element 0 of tile 0: tiles lie 8 keys
// apart and the two rows of a thread 8 queries, so 2 (NT + 1) logarithms do for 4 NT elements.
template <int NT>
__device__ __forceinline__ void sigmoid_tile(float (*c)[4], const SigmoidHead& hd, float base) {
  float b[NT + 1][2];
#pragma unroll
  for (int m = 0; m <= NT; ++m)
#pragma unroll
    for (int e = 0; e < 2; ++e) b[m][e] = hd.bias_fast(base + static_cast<float>(8 - 8 * m - e));
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) c[n][e] = hd.weight_fast(c[n][e], b[n + 1 - (e >> 1)][e & 1]);
}

// Key range of a query block and of one of its 16-query tiles, in 8-key tiles counted from the block's first key.
struct BlockRange {
  int t0, cnt, row, pos0, last, lo, k0;
  __device__ __forceinline__ BlockRange(const PrefillParams& p, int blk) {
    t0 = p.blk_start[blk];
    cnt = p.blk_count[blk];
    row = p.a.table_row[t0];
    pos0 = p.a.kv_len[t0] - 1;
    last = pos0 + cnt - 1;
    lo = p.a.window > 0 ? max(0, pos0 - p.a.window + 1) : 0;
    k0 = lo & ~7;
  }
  __device__ __forceinline__ int first_query(int qt) const { return pos0 + qt * 16; }
  __device__ __forceinline__ int last_query(int qt) const { return min(pos0 + qt * 16 + 15, last); }
  __device__ __forceinline__ int first_tile(int qt, int window) const {
    const int f = window > 0 ? max(0, first_query(qt) - window + 1) : 0;
    return (f - k0) >> 3;
  }
  __device__ __forceinline__ int last_tile(int qt) const { return (last_query(qt) - k0) >> 3; }
};

// HMAX: heads rounded up (mixed scores of all of them are live in registers); NT: 8-key tiles per warp.
// blockDim 256: 8 warps = 4 query tiles x 2 key groups.  grid: (query block, key group pair, group of HMAX output heads)
template <int HMAX, int NT, bool SIG>
__global__ void __launch_bounds__(256) head_mix_scores_kernel(const PrefillParams p) {
  extern __shared__ __align__(16) float mix_s[];   // [H][HMAX]: mix_s[g][h] = mix[h0 + h, g]
  const HeadMixArgs& a = p.a;
  const int H = a.n_heads, G = a.n_kv, R = H / G, D = a.dim, P = a.page_size, W = a.window;
  const int h0 = blockIdx.z * HMAX;
  for (int i = threadIdx.x; i < H * HMAX; i += blockDim.x) {
    const int g = i / HMAX, h = h0 + i % HMAX;
    mix_s[i] = h < H ? (a.mix != nullptr ? a.mix[h * H + g] : (h == g ? 1.f : 0.f)) : 0.f;
  }
  pdl_launch_next();
  pdl_wait_prior();
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int qt = warp & 3;
  const BlockRange br(p, p.blk0 + blockIdx.x);
  if (qt * 16 >= br.cnt) return;
  const int tile0 = (blockIdx.y * 2 + (warp >> 2)) * NT;
  if (tile0 > br.last_tile(qt) || tile0 + NT <= br.first_tile(qt, W)) return;
  const int r4 = lane >> 2, c4 = lane & 3;

  // query rows (A fragment rows r4, r4 + 8), clamped to the block
  const bf16* qrow0;
  const bf16* qrow1;
  {
    const int i0 = min(qt * 16 + r4, br.cnt - 1), i1 = min(qt * 16 + r4 + 8, br.cnt - 1);
    qrow0 = static_cast<const bf16*>(a.q) + (br.t0 + i0) * a.ldq + c4 * 4;
    qrow1 = static_cast<const bf16*>(a.q) + (br.t0 + i1) * a.ldq + c4 * 4;
  }
  // key rows (B fragment column r4 of each tile), clamped to mapped positions; the mask below removes the others
  const bf16* krow[NT];
#pragma unroll
  for (int n = 0; n < NT; ++n) {
    const int key = min(max(br.k0 + (tile0 + n) * 8 + r4, br.lo), br.last);
    const int page = max(a.block_table[static_cast<long long>(br.row) * a.table_ld + key / P], 0);
    krow[n] = static_cast<const bf16*>(a.k_pages) + (static_cast<long long>(page) * G * P + key % P) * D + c4 * 4;
  }
  float acc[HMAX][NT * 4];
#pragma unroll
  for (int h = 0; h < HMAX; ++h)
#pragma unroll
    for (int j = 0; j < NT * 4; ++j) acc[h][j] = 0.f;
  const float cap_k = a.softcap > 0.f ? 2.f * kLog2e * a.scale / a.softcap : 0.f;
  for (int g = 0; g < H; ++g) {
    float c[NT * 4];
#pragma unroll
    for (int j = 0; j < NT * 4; ++j) c[j] = 0.f;
    const long long kofs = static_cast<long long>(g / R) * P * D;
    const bf16* q0 = qrow0 + g * D;
    const bf16* q1 = qrow1 + g * D;
#pragma unroll 4
    for (int d = 0; d < D; d += 16) {
      const uint2 x0 = *reinterpret_cast<const uint2*>(q0 + d);
      const uint2 x1 = *reinterpret_cast<const uint2*>(q1 + d);
      const uint32_t af[4] = {x0.x, x1.x, x0.y, x1.y};
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        const uint2 y = *reinterpret_cast<const uint2*>(krow[n] + kofs + d);
        mma_bf16_16816(c + 4 * n, af, y.x, y.y);
      }
    }
    if constexpr (SIG) {
      sigmoid_tile<NT>(reinterpret_cast<float(*)[4]>(c), SigmoidHead(a, g, true),
                       static_cast<float>(br.first_query(qt) + r4 - (br.k0 + tile0 * 8 + c4 * 2)));
    } else if (a.softcap > 0.f) {
#pragma unroll
      for (int j = 0; j < NT * 4; ++j) c[j] = softcap_fast(c[j], cap_k, a.softcap);
    } else {
#pragma unroll
      for (int j = 0; j < NT * 4; ++j) c[j] *= a.scale;
    }
    const float4* mg = reinterpret_cast<const float4*>(mix_s + g * HMAX);
#pragma unroll
    for (int h = 0; h < HMAX; h += 4) {
      const float4 m = mg[h / 4];
#pragma unroll
      for (int j = 0; j < NT * 4; ++j) {
        acc[h][j] = fmaf(m.x, c[j], acc[h][j]);
        acc[h + 1][j] = fmaf(m.y, c[j], acc[h + 1][j]);
        acc[h + 2][j] = fmaf(m.z, c[j], acc[h + 2][j]);
        acc[h + 3][j] = fmaf(m.w, c[j], acc[h + 3][j]);
      }
    }
  }
#pragma unroll
  for (int n = 0; n < NT; ++n) {
    const int tile = tile0 + n;
    if (tile >= p.n_tiles) break;
    const int j0 = br.k0 + tile * 8 + c4 * 2;             // key of accumulator columns 0, 1
    const int i0 = br.first_query(qt) + r4;               // query of rows 0, 1 (i0, i0 + 8)
    float dist[4];
    bool vis[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int d = (i0 + (e >> 1) * 8) - (j0 + (e & 1));
      dist[e] = static_cast<float>(d);
      vis[e] = d >= 0 && (W <= 0 || d < W);
    }
    float4* dst = p.scratch + ((static_cast<long long>(blockIdx.x) * p.n_tiles + tile) * 4 + qt) * H * 32 + lane;
    if constexpr (SIG) {
      uint2* pairs = reinterpret_cast<uint2*>(p.scratch) + ((static_cast<long long>(blockIdx.x) * p.n_tiles + tile) * 4 + qt) * H * 32 + lane;
#pragma unroll
      for (int h = 0; h < HMAX; ++h)
        if (h0 + h < H)
          pairs[(h0 + h) * 32] = make_uint2(pack_bf16x2(vis[0] ? acc[h][4 * n] : 0.f, vis[1] ? acc[h][4 * n + 1] : 0.f),
                                            pack_bf16x2(vis[2] ? acc[h][4 * n + 2] : 0.f, vis[3] ? acc[h][4 * n + 3] : 0.f));
      continue;
    }
#pragma unroll
    for (int h = 0; h < HMAX; ++h) {
      if (h0 + h < H) {
        const float sl = a.slope != nullptr ? a.slope[h0 + h] : 0.f;
        float4 o;
        o.x = vis[0] ? acc[h][4 * n] - sl * dist[0] : -CUDART_INF_F;
        o.y = vis[1] ? acc[h][4 * n + 1] - sl * dist[1] : -CUDART_INF_F;
        o.z = vis[2] ? acc[h][4 * n + 2] - sl * dist[2] : -CUDART_INF_F;
        o.w = vis[3] ? acc[h][4 * n + 3] - sl * dist[3] : -CUDART_INF_F;
        dst[(h0 + h) * 32] = o;
      }
    }
  }
}

// The same tile of work with the query heads of its 16 queries resident in shared memory: one CTA = 16 queries, eight
// warps side by side along the keys, each walking `iters` groups of 8 NT keys.  Key fragments are private to a warp, so
// they go straight from global memory to registers, one kv head ahead of their use; query fragments come through
// ldmatrix.  The mixing multiply-adds run as packed pairs.
__device__ __forceinline__ void fma2(unsigned long long& acc, unsigned long long a, unsigned long long b) {
  asm("fma.rn.f32x2 %0, %1, %2, %0;" : "+l"(acc) : "l"(a), "l"(b));
}
__device__ __forceinline__ unsigned long long pack2(float x, float y) {
  unsigned long long r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(x), "f"(y));
  return r;
}
__device__ __forceinline__ void unpack2(unsigned long long v, float& x, float& y) {
  asm("mov.b64 {%0, %1}, %2;" : "=f"(x), "=f"(y) : "l"(v));
}

// KS: dim / 16 (EXACT) or an upper bound of it.
template <int HMAX, int NT, int KS, bool EXACT, bool SIG>
__global__ void __launch_bounds__(256) head_mix_scores_resident_kernel(const PrefillParams p, int iters) {
  extern __shared__ __align__(16) uint8_t smem_raw[];
  const HeadMixArgs& a = p.a;
  const int H = a.n_heads, G = a.n_kv, R = H / G, D = a.dim, P = a.page_size, W = a.window;
  const int ldq = (EXACT ? KS * 16 : D) + 8, steps = EXACT ? KS : D / 16;
  float2* mix_s = reinterpret_cast<float2*>(smem_raw);                             // [H][HMAX]: (mix[h, g], mix[h, g])
  SigmoidHead* sig_s = reinterpret_cast<SigmoidHead*>(smem_raw + sizeof(float2) * H * HMAX);     // [H], sigmoid weights only
  bf16* q_s = reinterpret_cast<bf16*>(sig_s + (SIG ? H : 0));                      // [H][16][ldq], k order of the fragments
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, r4 = lane >> 2, c4 = lane & 3;
  for (int i = tid; i < H * HMAX; i += 256) {
    const int g = i / HMAX, h = i % HMAX;
    const float m = h < H ? (a.mix != nullptr ? a.mix[h * H + g] : (h == g ? 1.f : 0.f)) : 0.f;
    mix_s[i] = make_float2(m, m);
  }
  if constexpr (SIG)
    for (int h = tid; h < H; h += 256) sig_s[h] = SigmoidHead(a, h, true);
  pdl_launch_next();
  pdl_wait_prior();
  const int qt = blockIdx.x & 3;
  const BlockRange br(p, p.blk0 + (blockIdx.x >> 2));
  if (qt * 16 >= br.cnt) return;
  const int first = br.first_tile(qt, W), last = br.last_tile(qt);
  const int span = 8 * NT;                                   // tiles per iteration of the CTA
  const int cta0 = blockIdx.y * iters * span;
  if (cta0 > last || cta0 + iters * span <= first) return;
  {
    const int vecs = D / 8;
    for (int i = tid; i < H * 16 * vecs; i += 256) {
      const int v = i % vecs, row = (i / vecs) & 15, h = i / (vecs * 16);
      const int qi = min(qt * 16 + row, br.cnt - 1);
      const uint4 x = *reinterpret_cast<const uint4*>(static_cast<const bf16*>(a.q) + (br.t0 + qi) * a.ldq + h * D + v * 8);
      uint32_t* dst = reinterpret_cast<uint32_t*>(q_s + (h * 16 + row) * ldq);
      const int d = v * 8, b32 = d & ~31;
      if (b32 + 32 <= D) {            // a lane's fragment words of two 16-wide steps are eight consecutive values
        const int c = (d & 31) >> 3;
        dst[(b32 + 2 * c) / 2] = x.x;
        dst[(b32 + 8 + 2 * c) / 2] = x.y;
        dst[(b32 + 16 + 2 * c) / 2] = x.z;
        dst[(b32 + 24 + 2 * c) / 2] = x.w;
      } else {                        // last single step: four consecutive values per lane
        const int c = (d & 15) >> 2;
        dst[(b32 + 2 * c) / 2] = x.x;
        dst[(b32 + 8 + 2 * c) / 2] = x.y;
        dst[(b32 + 2 * c + 2) / 2] = x.z;
        dst[(b32 + 8 + 2 * c + 2) / 2] = x.w;
      }
    }
  }
  __syncthreads();
  const uint32_t q_a = smem_u32(q_s) + ((lane & 15) * ldq + (lane >> 4) * 8) * 2;
  const float cap_k = a.softcap > 0.f ? 2.f * kLog2e * a.scale / a.softcap : 0.f;
  const long long k_head = static_cast<long long>(P) * D;
  for (int it = 0; it < iters; ++it) {
    const int tile0 = cta0 + it * span + warp * NT;
    if (tile0 > last || tile0 + NT <= first) continue;
    const bf16* krow[NT];
#pragma unroll
    for (int n = 0; n < NT; ++n) {
      const int key = min(max(br.k0 + (tile0 + n) * 8 + r4, br.lo), br.last);
      const int page = max(a.block_table[static_cast<long long>(br.row) * a.table_ld + key / P], 0);
      krow[n] = static_cast<const bf16*>(a.k_pages) + (static_cast<long long>(page) * G * P + key % P) * D;
    }
    auto load_k = [&](int g, uint32_t (*k)[KS][2]) {
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        const bf16* kr = krow[n] + g * k_head;
#pragma unroll
        for (int s = 0; s < KS; s += 2) {
          if (s + 1 < steps) {
            const uint4 x = *reinterpret_cast<const uint4*>(kr + s * 16 + c4 * 8);
            k[n][s][0] = x.x; k[n][s][1] = x.y;
            if (s + 1 < KS) { k[n][s + 1][0] = x.z; k[n][s + 1][1] = x.w; }
          } else if (s < steps) {
            const uint2 x = *reinterpret_cast<const uint2*>(kr + s * 16 + c4 * 4);
            k[n][s][0] = x.x; k[n][s][1] = x.y;
          }
        }
      }
    };
    unsigned long long acc[HMAX][NT * 2];
#pragma unroll
    for (int h = 0; h < HMAX; ++h)
#pragma unroll
      for (int j = 0; j < NT * 2; ++j) acc[h][j] = 0ull;
    const float base = static_cast<float>(br.first_query(qt) + r4 - (br.k0 + tile0 * 8 + c4 * 2));
    uint32_t kf[NT][KS][2], kn[NT][KS][2];
    load_k(0, kf);
    for (int g = 0; g < G; ++g) {
      if (g + 1 < G) load_k(g + 1, kn);
#pragma unroll 2
      for (int r = 0; r < R; ++r) {
        const int hq = g * R + r;
        const uint32_t qa = q_a + hq * 16 * ldq * 2;
        float c[NT][4], c2[NT][4];   // two accumulation chains
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) c[n][e] = c2[n][e] = 0.f;
#pragma unroll
        for (int s = 0; s < KS; ++s) {
          if (s < steps) {
            uint32_t af[4];
            ldsm_x4(qa + s * 32, af);
#pragma unroll
            for (int n = 0; n < NT; ++n) mma_bf16_16816((s & 1) ? c2[n] : c[n], af, kf[n][s][0], kf[n][s][1]);
          }
        }
        unsigned long long cp[NT * 2];
#pragma unroll
        for (int n = 0; n < NT; ++n) {
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            c[n][e] += c2[n][e];
            if constexpr (!SIG) c[n][e] = a.softcap > 0.f ? softcap_fast(c[n][e], cap_k, a.softcap) : c[n][e] * a.scale;
          }
        }
        if constexpr (SIG) sigmoid_tile<NT>(c, sig_s[hq], base);
#pragma unroll
        for (int n = 0; n < NT; ++n) {
          cp[2 * n] = pack2(c[n][0], c[n][1]);
          cp[2 * n + 1] = pack2(c[n][2], c[n][3]);
        }
        const ulonglong2* mg = reinterpret_cast<const ulonglong2*>(mix_s + hq * HMAX);
#pragma unroll
        for (int h = 0; h < HMAX; h += 2) {
          const ulonglong2 m = mg[h / 2];
#pragma unroll
          for (int j = 0; j < NT * 2; ++j) {
            fma2(acc[h][j], m.x, cp[j]);
            fma2(acc[h + 1][j], m.y, cp[j]);
          }
        }
      }
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int s = 0; s < KS; ++s) { kf[n][s][0] = kn[n][s][0]; kf[n][s][1] = kn[n][s][1]; }
    }
#pragma unroll
    for (int n = 0; n < NT; ++n) {
      const int tile = tile0 + n;
      if (tile >= p.n_tiles) break;
      const int j0 = br.k0 + tile * 8 + c4 * 2, i0 = br.first_query(qt) + r4;
      float dist[4];
      bool vis[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int d = (i0 + (e >> 1) * 8) - (j0 + (e & 1));
        dist[e] = static_cast<float>(d);
        vis[e] = d >= 0 && (W <= 0 || d < W);
      }
      float4* dst = p.scratch + ((static_cast<long long>(blockIdx.x >> 2) * p.n_tiles + tile) * 4 + qt) * H * 32 + lane;
      if constexpr (SIG) {
        uint2* pairs = reinterpret_cast<uint2*>(p.scratch) + ((static_cast<long long>(blockIdx.x >> 2) * p.n_tiles + tile) * 4 + qt) * H * 32 + lane;
#pragma unroll
        for (int h = 0; h < HMAX; ++h) {
          if (h < H) {
            float4 o;
            unpack2(acc[h][2 * n], o.x, o.y);
            unpack2(acc[h][2 * n + 1], o.z, o.w);
            pairs[h * 32] = make_uint2(pack_bf16x2(vis[0] ? o.x : 0.f, vis[1] ? o.y : 0.f), pack_bf16x2(vis[2] ? o.z : 0.f, vis[3] ? o.w : 0.f));
          }
        }
        continue;
      }
#pragma unroll
      for (int h = 0; h < HMAX; ++h) {
        if (h < H) {
          const float sl = a.slope != nullptr ? a.slope[h] : 0.f;
          float4 o;
          unpack2(acc[h][2 * n], o.x, o.y);
          unpack2(acc[h][2 * n + 1], o.z, o.w);
          o.x = vis[0] ? o.x - sl * dist[0] : -CUDART_INF_F;
          o.y = vis[1] ? o.y - sl * dist[1] : -CUDART_INF_F;
          o.z = vis[2] ? o.z - sl * dist[2] : -CUDART_INF_F;
          o.w = vis[3] ? o.w - sl * dist[3] : -CUDART_INF_F;
          dst[h * 32] = o;
        }
      }
    }
  }
}

constexpr int kVTile = 64;   // keys per V tile

// VT: 16-wide value column tiles per CTA.  blockDim 128: warp = query tile.  grid: (head, query block, value chunk)
template <int VT, bool SIG>
__global__ void __launch_bounds__(128, VT <= 8 ? 4 : 2) head_mix_values_kernel(const PrefillParams p) {
  constexpr int kLd = VT * 16 + 8;
  extern __shared__ __align__(16) bf16 v_s[];   // [2][kVTile][kLd]
  const HeadMixArgs& a = p.a;
  const int H = a.n_heads, G = a.n_kv, V = a.vdim, P = a.page_size, W = a.window;
  const int h = blockIdx.x, g = h / (H / G), v0 = blockIdx.z * VT * 16;
  pdl_launch_next();
  pdl_wait_prior();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int qt = warp;
  const int blk = gridDim.y - 1 - blockIdx.y;   // later blocks of a sequence see more keys: longest first
  const BlockRange br(p, p.blk0 + blk);
  const bool live = qt * 16 < br.cnt;
  const int first = live ? br.first_tile(qt, W) : 1, last = live ? br.last_tile(qt) : 0;
  const int r4 = lane >> 2, c4 = lane & 3;
  const int n_vt = (br.last - br.k0) / kVTile + 1;
  const int* table = a.block_table + static_cast<long long>(br.row) * a.table_ld;
  const bf16* vp = static_cast<const bf16*>(a.v_pages) + static_cast<long long>(g) * P * V;
  const uint32_t vs_base = smem_u32(v_s);
  // a warp stages 16 rows of every V tile, kRows at a time; lane L < 16 looks up the page of row L / kRows * 4 kRows +
  // warp * kRows + L % kRows once
  constexpr int kRows = 32 / (VT * 2);
  const int col = (lane % (VT * 2)) * 8;
  const bool col_ok = v0 + col < V;
  auto stage = [&](int vt) {
    int row = -1;
    {
      const int L = lane & 15, key = br.k0 + vt * kVTile + L / kRows * (4 * kRows) + warp * kRows + L % kRows;
      if (key >= br.lo && key <= br.last) {
        const int page = table[key / P];
        row = page < 0 ? -1 : page * G * P + key % P;
      }
    }
    const uint32_t dst = vs_base + (vt & 1) * (kVTile * kLd * 2) + ((warp * kRows + lane / (VT * 2)) * kLd + col) * 2;
#pragma unroll
    for (int i = 0; i < 16 / kRows; ++i) {
      const int r = __shfl_sync(0xffffffffu, row, i * kRows + lane / (VT * 2));
      const bool ok = r >= 0 && col_ok;
      cp_async16(dst + i * (4 * kRows * kLd * 2), ok ? vp + static_cast<long long>(r) * V + v0 + col : vp, ok);
    }
    cp_async_commit();
  };
  float o[VT * 2][4];
#pragma unroll
  for (int n = 0; n < VT * 2; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[n][e] = 0.f;
  float m[2] = {-CUDART_INF_F, -CUDART_INF_F}, l[2] = {0.f, 0.f};
  const float4* sc = p.scratch + ((static_cast<long long>(blk) * p.n_tiles) * 4 + qt) * H * 32 + h * 32 + lane;
  const long long sc_tile = static_cast<long long>(4) * H * 32;
  const uint2* wt = reinterpret_cast<const uint2*>(p.scratch) + ((static_cast<long long>(blk) * p.n_tiles) * 4 + qt) * H * 32 + h * 32 + lane;
  // weights of half a V tile, likewise
  auto fetch_w = [&](int half, uint2* s) {
#pragma unroll
    for (int n = 0; n < 4; ++n) {
      const int tile = half * 4 + n;
      s[n] = (tile >= first && tile <= last) ? __ldcs(wt + tile * sc_tile) : make_uint2(0u, 0u);
    }
  };
  // scores of half a V tile, fetched one half ahead of their use
  auto fetch = [&](int half, float4* s) {
    if (half * 4 > last || half * 4 + 3 < first) return;
#pragma unroll
    for (int n = 0; n < 4; ++n) {
      const int tile = half * 4 + n;
      s[n] = (tile >= first && tile <= last) ? __ldcs(sc + tile * sc_tile)
                                             : make_float4(-CUDART_INF_F, -CUDART_INF_F, -CUDART_INF_F, -CUDART_INF_F);
    }
  };
  float4 nxt[4];
  uint2 nxt_w[4];
  if constexpr (SIG) fetch_w(0, nxt_w); else fetch(0, nxt);
  stage(0);
  for (int vt = 0; vt < n_vt; ++vt) {
    if (vt + 1 < n_vt) { stage(vt + 1); cp_async_wait<1>(); } else { cp_async_wait<0>(); }
    __syncthreads();
    const uint32_t tile_base = vs_base + (vt & 1) * (kVTile * kLd * 2) + ((lane & 15) * kLd + (lane >> 4) * 8) * 2;
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      const int half = vt * 2 + hf;
      if constexpr (SIG) {
        uint2 w[4];
#pragma unroll
        for (int n = 0; n < 4; ++n) w[n] = nxt_w[n];
        fetch_w(half + 1, nxt_w);
        if (half * 4 > last || half * 4 + 3 < first) continue;
#pragma unroll
        for (int kk = 0; kk < 2; ++kk) {
          const uint32_t af[4] = {w[2 * kk].x, w[2 * kk].y, w[2 * kk + 1].x, w[2 * kk + 1].y};
#pragma unroll
          for (int n = 0; n < VT; ++n) {
            uint32_t b[4];
            ldsm_x4_trans(tile_base + ((hf * 32 + kk * 16) * kLd + n * 16) * 2, b);
            mma_bf16_16816(o[2 * n], af, b[0], b[1]);
            mma_bf16_16816(o[2 * n + 1], af, b[2], b[3]);
          }
        }
        continue;
      }
      float4 s[4];
#pragma unroll
      for (int n = 0; n < 4; ++n)     // scaled for 2^x
        s[n] = make_float4(nxt[n].x * kLog2e, nxt[n].y * kLog2e, nxt[n].z * kLog2e, nxt[n].w * kLog2e);
      fetch(half + 1, nxt);
      if (half * 4 > last || half * 4 + 3 < first) continue;
      float mx0 = m[0], mx1 = m[1];
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        mx0 = fmaxf(mx0, fmaxf(s[n].x, s[n].y));
        mx1 = fmaxf(mx1, fmaxf(s[n].z, s[n].w));
      }
#pragma unroll
      for (int d = 1; d < 4; d <<= 1) {
        mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, d));
        mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, d));
      }
      // a row without a visible key so far keeps maximum -inf; its weights are 2^(-inf - 0) = 0
      const float b0 = mx0 == -CUDART_INF_F ? 0.f : mx0, b1 = mx1 == -CUDART_INF_F ? 0.f : mx1;
      if (__any_sync(0xffffffffu, mx0 > m[0] || mx1 > m[1])) {   // some row has a new maximum
        const float cr0 = ex2_fast(m[0] - b0), cr1 = ex2_fast(m[1] - b1);
        m[0] = mx0;
        m[1] = mx1;
        l[0] *= cr0;
        l[1] *= cr1;
#pragma unroll
        for (int n = 0; n < VT * 2; ++n) {
          o[n][0] *= cr0; o[n][1] *= cr0; o[n][2] *= cr1; o[n][3] *= cr1;
        }
      }
#pragma unroll
      for (int kk = 0; kk < 2; ++kk) {
        float w[8];
#pragma unroll
        for (int u = 0; u < 2; ++u) {
          const float4 x = s[2 * kk + u];
          w[4 * u] = ex2_fast(x.x - b0); w[4 * u + 1] = ex2_fast(x.y - b0);
          w[4 * u + 2] = ex2_fast(x.z - b1); w[4 * u + 3] = ex2_fast(x.w - b1);
          l[0] += w[4 * u] + w[4 * u + 1];
          l[1] += w[4 * u + 2] + w[4 * u + 3];
        }
        const uint32_t af[4] = {pack_bf16x2(w[0], w[1]), pack_bf16x2(w[2], w[3]), pack_bf16x2(w[4], w[5]), pack_bf16x2(w[6], w[7])};
#pragma unroll
        for (int n = 0; n < VT; ++n) {
          uint32_t b[4];
          ldsm_x4_trans(tile_base + ((hf * 32 + kk * 16) * kLd + n * 16) * 2, b);
          mma_bf16_16816(o[2 * n], af, b[0], b[1]);
          mma_bf16_16816(o[2 * n + 1], af, b[2], b[3]);
        }
      }
    }
    __syncthreads();
  }
  if (!live) return;
#pragma unroll
  for (int d = 1; d < 4; d <<= 1) {
    l[0] += __shfl_xor_sync(0xffffffffu, l[0], d);
    l[1] += __shfl_xor_sync(0xffffffffu, l[1], d);
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int i = qt * 16 + r4 + r * 8;
    if (i >= br.cnt) continue;
    const long long t = br.t0 + i;
    float f = SIG ? 1.f : head_mix_finish(m[r] * (1.f / kLog2e), l[r], a.sink, a.sinks, h);
    if (a.gate != nullptr) f *= sigmoid_of<bf16>(a.gate[t * a.ld_gate + h]);
    bf16* dst = static_cast<bf16*>(a.out) + t * a.ldo + static_cast<long long>(h) * V + v0 + c4 * 2;
#pragma unroll
    for (int n = 0; n < VT * 2; ++n)
      if (v0 + n * 8 < V) *reinterpret_cast<uint32_t*>(dst + n * 8) = pack_bf16x2(o[n][2 * r] * f, o[n][2 * r + 1] * f);
  }
}

int tiles_for(int max_keys, int window) {
  // 8-key tiles of the widest query block: its first query reaches window - 1 keys back, the start is rounded down
  int keys = max_keys;
  if (window > 0 && window + kHeadMixBlock - 1 < keys) keys = window + kHeadMixBlock - 1;
  return (keys + 7 + 7) / 8;
}

template <int HMAX, int NT, bool SIG>
cudaError_t launch_scores(const PrefillParams& p, int n_blocks) {
  auto kern = head_mix_scores_kernel<HMAX, NT, SIG>;
  const size_t smem = sizeof(float) * static_cast<size_t>(p.a.n_heads) * HMAX;
  const int groups = (p.n_tiles + 2 * NT - 1) / (2 * NT);
  const dim3 grid(n_blocks, groups, (p.a.n_heads + HMAX - 1) / HMAX);
  if (smem > 48 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return e;
  }
  return launch_kernel(kern, grid, dim3(256), smem, p.a.stream, p.a.pdl, 1, p);
}

constexpr size_t kResidentSmem = 200 * 1024;
size_t resident_smem(int H, int hmax, int D) {
  return (sizeof(float2) * hmax + sizeof(SigmoidHead)) * static_cast<size_t>(H) + sizeof(bf16) * static_cast<size_t>(H) * 16 * (D + 8);
}

template <int HMAX, int NT, int KS, bool EXACT, bool SIG>
cudaError_t launch_resident(const PrefillParams& p, int n_blocks) {
  auto kern = head_mix_scores_resident_kernel<HMAX, NT, KS, EXACT, SIG>;
  const size_t smem = resident_smem(p.a.n_heads, HMAX, p.a.dim);
  if (smem > 48 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return e;
  }
  constexpr int span = 8 * NT;
  const int groups = (p.n_tiles + span - 1) / span;
  // several key groups per CTA amortise the staging of the queries, as long as the grid still fills the GPU
  int iters = 4;
  while (iters > 1 && static_cast<long long>(n_blocks) * 4 * ((groups + iters - 1) / iters) < 4 * 148) iters >>= 1;
  const dim3 grid(n_blocks * 4, (groups + iters - 1) / iters);
  return launch_kernel(kern, grid, dim3(256), smem, p.a.stream, p.a.pdl, 1, p, iters);
}

template <int HMAX, int NT, bool SIG>
cudaError_t launch_resident_dim(const PrefillParams& p, int n_blocks) {
  if (p.a.dim == 64) return launch_resident<HMAX, NT, 4, true, SIG>(p, n_blocks);
  if (p.a.dim == 128) return launch_resident<HMAX, NT, 8, true, SIG>(p, n_blocks);
  if (p.a.dim < 64) return launch_resident<HMAX, NT, 4, false, SIG>(p, n_blocks);
  return launch_resident<HMAX, NT, 8, false, SIG>(p, n_blocks);
}

template <int VT, bool SIG>
cudaError_t launch_values(const PrefillParams& p, int n_blocks) {
  auto kern = head_mix_values_kernel<VT, SIG>;
  constexpr int smem = 2 * kVTile * (VT * 16 + 8) * 2;
  static bool attr_set = false;
  if (smem > 48 * 1024 && !attr_set) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return e;
    attr_set = true;
  }
  const dim3 grid(p.a.n_heads, n_blocks, (p.a.vdim + VT * 16 - 1) / (VT * 16));
  return launch_kernel(kern, grid, dim3(128), smem, p.a.stream, p.a.pdl, 1, p);
}

// Both kernels of `n` query blocks.
template <bool SIG>
cudaError_t launch_both(const PrefillParams& p, int n, bool resident) {
  const int H = p.a.n_heads, V = p.a.vdim;
  cudaError_t e;
  if (resident && H <= 8) e = launch_resident_dim<8, 2, SIG>(p, n);
  else if (resident && H <= 16) e = launch_resident_dim<16, 2, SIG>(p, n);
  else if (resident) e = launch_resident_dim<32, 1, SIG>(p, n);
  else if (H <= 4) e = launch_scores<4, 4, SIG>(p, n);
  else if (H <= 8) e = launch_scores<8, 2, SIG>(p, n);
  else if (H <= 16) e = launch_scores<16, 2, SIG>(p, n);
  else e = launch_scores<32, 1, SIG>(p, n);
  if (e != cudaSuccess) return e;
  if (V <= 32) return launch_values<2, SIG>(p, n);
  if (V <= 64) return launch_values<4, SIG>(p, n);
  if (V <= 128) return launch_values<8, SIG>(p, n);
  return launch_values<16, SIG>(p, n);
}

}  // namespace

int64_t head_mix_prefill_scratch(int n_heads, int max_keys, int window, int blocks, bool sigmoid) {
  return static_cast<int64_t>(blocks) * tiles_for(max_keys, window) * 4 * n_heads * 32 * (sigmoid ? 8 : 16);
}

const char* head_mix_prefill(const HeadMixArgs& a, const int* blk_start, const int* blk_count, int n_blocks, int max_keys,
                             void* scratch, int64_t scratch_bytes) {
  if (a.T <= 0 || n_blocks <= 0) return nullptr;
  if (a.f32 || a.chunk > 0) return "head_mix_prefill: bf16 without chunks only";
  if (a.dim % 16 || a.vdim % 16 || a.n_kv <= 0 || a.n_heads % a.n_kv) return "head_mix_prefill: bad head geometry";
  if (a.n_heads > 512 || n_blocks > 65535) return "head_mix_prefill: too many heads or query blocks";
  if (a.ldq % 4 || a.ldo % 2) return "head_mix_prefill: misaligned rows";
  PrefillParams p;
  p.a = a;
  p.blk_start = blk_start;
  p.blk_count = blk_count;
  p.scratch = static_cast<float4*>(scratch);
  p.n_tiles = tiles_for(max_keys, a.window);
  const int64_t per_block = head_mix_prefill_scratch(a.n_heads, max_keys, a.window, 1, a.sigmoid);
  const int fit = static_cast<int>(scratch_bytes / per_block < n_blocks ? scratch_bytes / per_block : n_blocks);
  if (fit < 1) return "head_mix_prefill: the scratch does not hold one query block";
  const int launches = (n_blocks + fit - 1) / fit, at_once = (n_blocks + launches - 1) / launches;   // equal shares
  for (p.blk0 = 0; p.blk0 < n_blocks; p.blk0 += at_once) {
    const int n = n_blocks - p.blk0 < at_once ? n_blocks - p.blk0 : at_once;
    cudaError_t e;
    const bool resident = a.n_heads <= 32 && a.dim <= 128 && a.ldq % 8 == 0 && resident_smem(a.n_heads, 32, a.dim) <= kResidentSmem;
    e = a.sigmoid ? launch_both<true>(p, n, resident) : launch_both<false>(p, n, resident);
    if (e != cudaSuccess) return cudaGetErrorString(e);
  }
  return nullptr;
}

}  // namespace nfb
