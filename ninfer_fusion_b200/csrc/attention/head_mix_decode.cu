// Head-mixing attention of single query tokens on the tensor cores (bf16): one CTA = (token, split of its keys), all
// heads.  A warp owns one or two kv heads: it streams their key and value rows through rings of its own (cp.async, no
// block barrier on the loads) and multiplies them against all query heads of the group at once, the query heads being
// the rows of the MMA.  Scores meet in shared memory once per 16-key tile for the mix:
//   scores(t) | barrier | mix(t) | barrier | softmax + values(t), scores(t + 1) | barrier | ...
// Sigmoid weights are made where the scores are, and the mixed ones go straight to the values.
#include "head_mix.h"

#include <math_constants.h>

#include "../common/elem.cuh"
#include "../common/launch.h"
#include "../common/mma_sync.cuh"

namespace nfb {

namespace {

using bf16 = __nv_bfloat16;
constexpr int KT = 16;        // keys per tile
constexpr int kLdS = KT + 2;  // floats per row of the score arrays

struct SmemPlan {
  int hp;            // heads rounded up to 2
  int mix, q, cs, ss, ring, stage_k, stage_v, total;   // byte offsets / sizes
  __host__ __device__ SmemPlan(int H, int G, int D, int V, int stages) {
    hp = (H + 1) & ~1;
    mix = 0;                                     // [H][hp] float, mix[g][h]
    q = mix + (H * hp * 4 + 15) / 16 * 16;       // [H][D + 8] bf16
    cs = q + H * (D + 8) * 2;                    // [H][kLdS] float
    ss = cs + (H * kLdS * 4 + 15) / 16 * 16;     // [hp][kLdS] float
    ring = ss + (hp * kLdS * 4 + 15) / 16 * 16;
    stage_k = KT * (D + 8) * 2;
    stage_v = KT * (V + 8) * 2;
    total = ring + G * stages * (stage_k + stage_v);
  }
};

// NW warps, WG kv heads per warp, VT: upper bound of vdim / 16, S: ring stages.
template <int NW, int WG, int VT, int S, bool SIG>
__global__ void __launch_bounds__(NW * 32) head_mix_decode_kernel(const HeadMixArgs p, int split_keys, int n_splits,
                                                                   float* __restrict__ part_o, float* __restrict__ part_ml) {
  extern __shared__ __align__(16) uint8_t smem[];
  const int H = p.n_heads, G = p.n_kv, R = H / G, D = p.dim, V = p.vdim, P = p.page_size;
  const SmemPlan plan(H, G, D, V, S);
  float* mix_s = reinterpret_cast<float*>(smem + plan.mix);
  bf16* q_s = reinterpret_cast<bf16*>(smem + plan.q);
  float* cs = reinterpret_cast<float*>(smem + plan.cs);
  float* ss = reinterpret_cast<float*>(smem + plan.ss);
  const int t = blockIdx.y, split = blockIdx.x;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, r4 = lane >> 2, c4 = lane & 3;
  for (int i = tid; i < H * plan.hp; i += NW * 32) {
    const int g = i / plan.hp, h = i % plan.hp;
    mix_s[i] = h < H ? (p.mix != nullptr ? p.mix[h * H + g] : (h == g ? 1.f : 0.f)) : 0.f;
  }
  pdl_launch_next();
  pdl_wait_prior();
  const int len = p.kv_len[t], qpos = len - 1;
  const int lo = first_visible(len, p.window, p.chunk);
  const int k_begin = lo + split * split_keys, k_end = min(len, k_begin + split_keys);
  const int n_tiles = k_end > k_begin ? (k_end - k_begin + KT - 1) / KT : 0;
  const int* table = p.block_table + static_cast<long long>(p.table_row[t]) * p.table_ld;
  const bf16* kp = static_cast<const bf16*>(p.k_pages);
  const bf16* vp = static_cast<const bf16*>(p.v_pages);
  const uint32_t ring = smem_u32(smem) + plan.ring;

  // row of key k_begin + tile * KT + (lane & 15) in a kv head's page plane, -1 past the end or unmapped
  auto key_row = [&](int tile) {
    const int key = k_begin + tile * KT + (lane & 15);
    if (key >= k_end) return -1;
    const int page = table[key / P];
    return page < 0 ? -1 : page * G * P + key % P;
  };
  auto load = [&](int row, int tile, bool values) {
    const int width = values ? V : D, vecs = width / 8;
    const int slot = tile % S;
#pragma unroll
    for (int j = 0; j < WG; ++j) {
      const int g = warp + j * NW;
      if (g >= G) break;
      const uint32_t dst = ring + (g * S + slot) * (plan.stage_k + plan.stage_v) + (values ? plan.stage_k : 0);
      const bf16* base = (values ? vp : kp) + static_cast<long long>(g) * P * width;
      for (int i = lane; i < KT * vecs; i += 32) {      // (KT * vecs is a multiple of 32: no lane leaves the loop early)
        const int key = i / vecs, c = (i % vecs) * 8;
        const int r = __shfl_sync(0xffffffffu, row, key);
        cp_async16(dst + (key * (width + 8) + c) * 2, r >= 0 ? base + static_cast<long long>(r) * width + c : base, r >= 0);
      }
    }
    cp_async_commit();
  };
#pragma unroll
  for (int s = 0; s < S; ++s) {
    if (s < n_tiles) {
      const int row = key_row(s);
      load(row, s, false);
      load(row, s, true);
    } else {
      cp_async_commit();
      cp_async_commit();
    }
  }
  {
    const bf16* q = static_cast<const bf16*>(p.q) + t * p.ldq;
    const int vecs = D / 8;
    for (int i = tid; i < H * vecs; i += NW * 32)
      *reinterpret_cast<uint4*>(q_s + (i / vecs) * (D + 8) + (i % vecs) * 8) = *reinterpret_cast<const uint4*>(q + i * 8);
  }
  float o[WG][VT * 2][4];
  float m[WG][2], l[WG][2];
#pragma unroll
  for (int j = 0; j < WG; ++j) {
    m[j][0] = m[j][1] = -CUDART_INF_F;
    l[j][0] = l[j][1] = 0.f;
#pragma unroll
    for (int n = 0; n < VT * 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[j][n][e] = 0.f;
  }
  const float cap_k = p.softcap > 0.f ? 2.f * kLog2e * p.scale / p.softcap : 0.f;
  SigmoidHead sig[WG][2];       // of the two query heads of each group that this thread's accumulator rows belong to
  if constexpr (SIG) {
#pragma unroll
    for (int j = 0; j < WG; ++j)
#pragma unroll
      for (int r = 0; r < 2; ++r)
        if (warp + j * NW < G && r4 + r * 8 < R) sig[j][r] = SigmoidHead(p, (warp + j * NW) * R + r4 + r * 8, true);
  }
  const uint32_t q_a = smem_u32(q_s);
  __syncthreads();

  for (int tile = 0; tile < n_tiles; ++tile) {
    const int slot = tile % S;
    const int next_row = tile + S < n_tiles ? key_row(tile + S) : -1;
    // ---- scores of this tile ----
    cp_async_wait<2 * S - 1>();
    __syncwarp();
#pragma unroll
    for (int j = 0; j < WG; ++j) {
      const int g = warp + j * NW;
      if (g >= G) break;
      const uint32_t ks = ring + (g * S + slot) * (plan.stage_k + plan.stage_v);
      const uint32_t qa = q_a + ((g * R + min(lane & 15, R - 1)) * (D + 8) + (lane >> 4) * 8) * 2;
      const uint32_t ka = ks + (((lane & 7) + (lane >> 4) * 8) * (D + 8) + ((lane >> 3) & 1) * 8) * 2;
      float c[2][4] = {};
#pragma unroll 4
      for (int d = 0; d < D; d += 16) {
        uint32_t a[4], b[4];
        ldsm_x4(qa + d * 2, a);
        ldsm_x4(ka + d * 2, b);
        mma_bf16_16816(c[0], a, b[0], b[1]);
        mma_bf16_16816(c[1], a, b[2], b[3]);
      }
#pragma unroll
      for (int n = 0; n < 2; ++n) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int r = r4 + (e >> 1) * 8;
          if (r < R) {
            float s = c[n][e];
            if constexpr (SIG) {
              const SigmoidHead& hd = sig[j][e >> 1];
              s = hd.weight_fast(s, hd.bias_fast(static_cast<float>(qpos - (k_begin + tile * KT + n * 8 + c4 * 2 + (e & 1)))));
            } else {
              s = p.softcap > 0.f ? softcap_fast(s, cap_k, p.softcap) : s * p.scale;
            }
            cs[(g * R + r) * kLdS + n * 8 + c4 * 2 + (e & 1)] = s;
          }
        }
      }
    }
    __syncwarp();
    if (tile + S < n_tiles) load(next_row, tile + S, false); else cp_async_commit();
    __syncthreads();
    // ---- mix across heads, bias, end of the range: two heads x one key per item ----
    for (int i = tid; i < plan.hp / 2 * KT; i += NW * 32) {
      const int key = i % KT, h = i / KT * 2;
      const float* c = cs + key;
      const float2* mg = reinterpret_cast<const float2*>(mix_s + h);
      float s0 = 0.f, s1 = 0.f;
#pragma unroll 8
      for (int g = 0; g < H; ++g) {
        const float x = c[g * kLdS];
        const float2 w = mg[g * (plan.hp / 2)];
        s0 = fmaf(w.x, x, s0);
        s1 = fmaf(w.y, x, s1);
      }
      const int kpos = k_begin + tile * KT + key;
      const float d = static_cast<float>(qpos - kpos);
      if (p.slope != nullptr) {
        s0 -= p.slope[h] * d;
        if (h + 1 < H) s1 -= p.slope[h + 1] * d;
      }
      const bool in = kpos < k_end;
      ss[h * kLdS + key] = in ? s0 : (SIG ? 0.f : -CUDART_INF_F);
      ss[(h + 1) * kLdS + key] = in ? s1 : (SIG ? 0.f : -CUDART_INF_F);
    }
    cp_async_wait<2 * S - 1>();
    __syncthreads();
    // ---- running softmax and values ----
#pragma unroll
    for (int j = 0; j < WG; ++j) {
      const int g = warp + j * NW;
      if (g >= G) break;
      const uint32_t va = ring + (g * S + slot) * (plan.stage_k + plan.stage_v) + plan.stage_k +
                          ((lane & 15) * (V + 8) + (lane >> 4) * 8) * 2;
      float w[2][4], corr[2];
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int row = r4 + r * 8;
        if (row < R) {
          const float2* sp = reinterpret_cast<const float2*>(ss + (g * R + row) * kLdS + c4 * 2);
          const float2 x = sp[0], y = sp[4];
          w[r][0] = x.x; w[r][1] = x.y; w[r][2] = y.x; w[r][3] = y.y;
        } else {
#pragma unroll
          for (int e = 0; e < 4; ++e) w[r][e] = SIG ? 0.f : -CUDART_INF_F;
        }
        if constexpr (SIG) continue;
        float mx = fmaxf(fmaxf(w[r][0], w[r][1]), fmaxf(w[r][2], w[r][3]));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
        mx = fmaxf(mx, m[j][r]);
        const float base = mx == -CUDART_INF_F ? 0.f : mx;
        corr[r] = __expf(m[j][r] - base);
        m[j][r] = mx;
        l[j][r] *= corr[r];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          w[r][e] = __expf(w[r][e] - base);
          l[j][r] += w[r][e];
        }
      }
      const uint32_t af[4] = {pack_bf16x2(w[0][0], w[0][1]), pack_bf16x2(w[1][0], w[1][1]), pack_bf16x2(w[0][2], w[0][3]),
                              pack_bf16x2(w[1][2], w[1][3])};
#pragma unroll
      for (int n = 0; n < VT; ++n) {
        if (n * 16 < V) {
          uint32_t b[4];
          ldsm_x4_trans(va + n * 32, b);
#pragma unroll
          for (int u = 0; u < 2; ++u) {
            if constexpr (!SIG) {
              o[j][2 * n + u][0] *= corr[0]; o[j][2 * n + u][1] *= corr[0];
              o[j][2 * n + u][2] *= corr[1]; o[j][2 * n + u][3] *= corr[1];
            }
            mma_bf16_16816(o[j][2 * n + u], af, b[2 * u], b[2 * u + 1]);
          }
        }
      }
    }
    __syncwarp();
    if (tile + S < n_tiles) load(next_row, tile + S, true); else cp_async_commit();
  }
  cp_async_wait<0>();
#pragma unroll
  for (int j = 0; j < WG; ++j) {
    const int g = warp + j * NW;
    if (g >= G) break;
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      float sum = l[j][r];
      sum += __shfl_xor_sync(0xffffffffu, sum, 1);
      sum += __shfl_xor_sync(0xffffffffu, sum, 2);
      const int row = r4 + r * 8;
      if (row >= R) continue;
      const int h = g * R + row;
      if (n_splits > 1) {
        const long long at = (static_cast<long long>(t) * n_splits + split) * H + h;
        float* dst = part_o + at * V + c4 * 2;
#pragma unroll
        for (int n = 0; n < VT * 2; ++n)
          if (n * 8 < V) *reinterpret_cast<float2*>(dst + n * 8) = make_float2(o[j][n][2 * r], o[j][n][2 * r + 1]);
        if (c4 == 0) {
          part_ml[at * 2] = SIG ? 0.f : m[j][r];
          part_ml[at * 2 + 1] = SIG ? 1.f : sum;
        }
      } else {
        float f = SIG ? 1.f : head_mix_finish(m[j][r], sum, p.sink, p.sinks, h);
        if (p.gate != nullptr) f *= sigmoid_of<bf16>(p.gate[t * p.ld_gate + h]);
        bf16* dst = static_cast<bf16*>(p.out) + t * p.ldo + static_cast<long long>(h) * V + c4 * 2;
#pragma unroll
        for (int n = 0; n < VT * 2; ++n)
          if (n * 8 < V) *reinterpret_cast<uint32_t*>(dst + n * 8) = pack_bf16x2(o[j][n][2 * r] * f, o[j][n][2 * r + 1] * f);
      }
    }
  }
}

template <int NW, int WG, int VT, int S, bool SIG>
const char* launch(const HeadMixArgs& a, int split_keys, int n_splits, float* part_o, float* part_ml) {
  const int smem = SmemPlan(a.n_heads, a.n_kv, a.dim, a.vdim, S).total;
  auto kern = head_mix_decode_kernel<NW, WG, VT, S, SIG>;
  if (smem > 48 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return cudaGetErrorString(e);
  }
  const cudaError_t e = launch_kernel(kern, dim3(n_splits, a.T), dim3(NW * 32), smem, a.stream, a.pdl, 1, a, split_keys, n_splits,
                                      part_o, part_ml);
  return e == cudaSuccess ? nullptr : cudaGetErrorString(e);
}

constexpr int kMaxSmem = 220 * 1024;

template <bool SIG, int NW, int WG, int VT>
const char* launch_stages(const HeadMixArgs& a, int split_keys, int n_splits, float* part_o, float* part_ml) {
  // two CTAs per SM hide each other's barriers better than a deeper ring; the ring takes what is left
  auto fits = [&](int s, int limit) { return SmemPlan(a.n_heads, a.n_kv, a.dim, a.vdim, s).total <= limit; };
  if (fits(4, kMaxSmem / 2)) return launch<NW, WG, VT, 4, SIG>(a, split_keys, n_splits, part_o, part_ml);
  if (fits(2, kMaxSmem / 2) || !fits(1, kMaxSmem / 2)) {
    if (fits(2, kMaxSmem)) return launch<NW, WG, VT, 2, SIG>(a, split_keys, n_splits, part_o, part_ml);
  }
  return launch<NW, WG, VT, 1, SIG>(a, split_keys, n_splits, part_o, part_ml);
}

}  // namespace

bool head_mix_decode_supported(const HeadMixArgs& a) {
  if (a.f32 || a.n_heads / a.n_kv > 16 || a.ldq % 8 || a.T > 65535 || SmemPlan(a.n_heads, a.n_kv, a.dim, a.vdim, 1).total > kMaxSmem) return false;
  if (a.vdim <= 64) return a.n_kv <= 32;
  if (a.vdim <= 128) return a.n_kv <= 16;
  return a.vdim <= 256 && a.n_kv <= 8;
}

namespace {
template <bool SIG>
const char* pick_shape(const HeadMixArgs& a, int split_keys, int n_splits, float* part_o, float* part_ml) {
  if (a.vdim <= 64) {
    if (a.n_kv <= 8) return launch_stages<SIG, 8, 1, 4>(a, split_keys, n_splits, part_o, part_ml);
    if (a.n_kv <= 16) return launch_stages<SIG, 16, 1, 4>(a, split_keys, n_splits, part_o, part_ml);
    return launch_stages<SIG, 16, 2, 4>(a, split_keys, n_splits, part_o, part_ml);
  }
  if (a.vdim <= 128) {
    if (a.n_kv <= 8) return launch_stages<SIG, 8, 1, 8>(a, split_keys, n_splits, part_o, part_ml);
    return launch_stages<SIG, 16, 1, 8>(a, split_keys, n_splits, part_o, part_ml);
  }
  return launch_stages<SIG, 8, 1, 16>(a, split_keys, n_splits, part_o, part_ml);
}
}  // namespace

const char* head_mix_decode(const HeadMixArgs& a, int split_keys, int n_splits, float* part_o, float* part_ml) {
  return a.sigmoid ? pick_shape<true>(a, split_keys, n_splits, part_o, part_ml) : pick_shape<false>(a, split_keys, n_splits, part_o, part_ml);
}

}  // namespace nfb
