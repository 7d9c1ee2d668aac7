// Absorbed latent attention on the tensor cores (bf16): rows of the MMA are (token, head) pairs of one query block, so a
// cached row is read once for all of them.  One CTA = (split of the keys, up to 16 MT rows, query block), NW = 8 or 16
// warps.  Per tile of 4 NW keys, which live in a cp.async ring:
//   scores   a warp owns sixteen keys and a quarter of the width, for all rows
//   softmax  a warp owns 16 MT / NW rows, a lane one or two keys; weights go to shared memory in bf16, with the rows' rescale
//            factors
//   values   a warp owns 8 NT columns of the latent for all rows; the key tile is its own value tile
// Sixteen warps serve the few rows of a decode step (three barriers per tile, so larger tiles and more warps hide more);
// eight warps keep the 64 rows of a short portion in registers.
#include "latent.h"

#include <math_constants.h>

#include "../common/elem.cuh"
#include "../common/launch.h"
#include "../common/mma_sync.cuh"

namespace nfb {

namespace {

using bf16 = __nv_bfloat16;

struct Plan {
  int ldk, q, ring, stage, s, p, alpha, len, total;
  __host__ __device__ Plan(int rows, int width, int stages, int keys) {
    ldk = width + 8;
    q = 0;
    ring = q + rows * ldk * 2;
    stage = keys * ldk * 2;
    s = ring + stages * stage;
    p = s + 4 * rows * (keys + 4) * 4;            // one score array per quarter of the width
    alpha = p + rows * (keys + 8) * 2;
    len = alpha + rows * 2 * 4;                  // two floats per row: rescale factor / maximum and sum at the end
    total = len + rows * 4;
  }
};

template <int NW, int MT, int NT, int S>
__global__ void __launch_bounds__(NW * 32) latent_absorbed_kernel(const LatentArgs p, const LatentBlocks b, int split_keys, int n_splits,
                                                                    float* __restrict__ part_o, float* __restrict__ part_ml) {
  constexpr int KT = 4 * NW, kThreads = NW * 32, kLdS = KT + 4, kLdP = KT + 8;
  constexpr int M = 16 * MT, kRows = M / NW, kPer = KT / 32, kLoad = KT / NW;
  extern __shared__ __align__(16) uint8_t smem[];
  const int H = p.n_heads, W = p.rank + p.rot, P = p.page_size;
  const Plan plan(M, W, S, KT);
  bf16* qs = reinterpret_cast<bf16*>(smem + plan.q);
  float* ss = reinterpret_cast<float*>(smem + plan.s);
  bf16* ps = reinterpret_cast<bf16*>(smem + plan.p);
  float* alpha = reinterpret_cast<float*>(smem + plan.alpha);
  int* row_len = reinterpret_cast<int*>(smem + plan.len);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, r4 = lane >> 2, c4 = lane & 3;
  pdl_launch_next();
  pdl_wait_prior();
  const int split = blockIdx.x, t0 = b.start[blockIdx.z], count = b.count[blockIdx.z];
  const int r0 = blockIdx.y * M, n_rows = min(M, count * H - r0);
  if (n_rows <= 0) return;
  if (b.max_tokens > 0) {
    const int seq = b.token_seq[t0];
    if (b.cu_seqlens[seq + 1] - b.cu_seqlens[seq] >= b.max_tokens) return;
  }
  const int max_len = p.kv_len[t0 + (r0 + n_rows - 1) / H];
  const int lo = latent_first(p.kv_len[t0 + r0 / H], p.window);       // of the CTA's first row
  const int k_begin = lo + split * split_keys, k_end = min(max_len, k_begin + split_keys);
  const int n_tiles = k_end > k_begin ? (k_end - k_begin + KT - 1) / KT : 0;
  const int* table = p.block_table + static_cast<long long>(p.table_row[t0]) * p.table_ld;
  const bf16* pages = static_cast<const bf16*>(p.pages);
  const uint32_t qs_a = smem_u32(qs), ps_a = smem_u32(ps), ring_a = smem_u32(smem) + plan.ring;
  const int ldk = plan.ldk, vecs = W / 8;

  int row_at[kLoad];          // page * P + place of the warp's rows of the tile to load next, -1: none
  auto look_up = [&](int tile) {
#pragma unroll
    for (int j = 0; j < kLoad; ++j) {
      const int key = k_begin + tile * KT + j * NW + warp;
      const int page = key < k_end ? table[key / P] : -1;
      row_at[j] = page < 0 ? -1 : page * P + key % P;
    }
  };
  auto load = [&](int tile) {
    const uint32_t dst = ring_a + (tile % S) * plan.stage;
#pragma unroll
    for (int j = 0; j < kLoad; ++j) {
      const bool ok = row_at[j] >= 0;
      const bf16* src = pages + static_cast<long long>(ok ? row_at[j] : 0) * W;
      for (int c = lane; c < vecs; c += 32) cp_async16(dst + ((j * NW + warp) * ldk + c * 8) * 2, src + c * 8, ok);
    }
  };
#pragma unroll
  for (int s = 0; s < S - 1; ++s) {
    if (s < n_tiles) {
      look_up(s);
      load(s);
    }
    cp_async_commit();
  }
  look_up(S - 1);
  // queries: absorbed part as it is, rotated part turned here
  for (int i = tid; i < M * (p.rank / 8); i += kThreads) {
    const int r = i / (p.rank / 8), c = (i % (p.rank / 8)) * 8;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (r < n_rows) {
      const int t = t0 + (r0 + r) / H, h = (r0 + r) % H;
      v = *reinterpret_cast<const uint4*>(static_cast<const bf16*>(p.q_latent) + t * p.ldl + static_cast<long long>(h) * p.rank + c);
    }
    *reinterpret_cast<uint4*>(qs + r * ldk + c) = v;
  }
  for (int i = tid; i < M * (p.rot / 2); i += kThreads) {
    const int r = i / (p.rot / 2), e = i % (p.rot / 2);
    float u = 0.f, v = 0.f;
    if (r < n_rows && 2 * e < p.rot_true) {
      const int t = t0 + (r0 + r) / H, h = (r0 + r) % H;
      const bf16* q = static_cast<const bf16*>(p.q) + t * p.ldq + static_cast<long long>(h) * (p.dim + p.rot) + p.dim + 2 * e;
      float c, s;
      rotary_angle(p.kv_len[t] - 1, p.freq[e], c, s);
      const float x = __bfloat162float(q[0]), y = __bfloat162float(q[1]);
      u = x * c - y * s;
      v = y * c + x * s;
    }
    *reinterpret_cast<uint32_t*>(qs + r * ldk + p.rank + 2 * e) = pack_bf16x2(u, v);
  }
  if (tid < M) row_len[tid] = tid < n_rows ? p.kv_len[t0 + (r0 + tid) / H] : 0;

  float o[MT][NT][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[m][n][e] = 0.f;
  float mx[kRows], l[kRows];   // of rows warp * kRows + i, the same in every lane
#pragma unroll
  for (int i = 0; i < kRows; ++i) { mx[i] = -CUDART_INF_F; l[i] = 0.f; }
  const float scale2 = p.scale * kLog2e;
  const int n_steps = W / 16, col0 = warp * NT * 8;
  const int kg = warp % (KT / 16), quarter = warp / (KT / 16), q_steps = (n_steps + 3) / 4;
  const int ks0 = quarter * q_steps, ks1 = min(n_steps, ks0 + q_steps);

  for (int tile = 0; tile < n_tiles; ++tile) {
    cp_async_wait<S - 2>();
    __syncthreads();
    if (tile + S - 1 < n_tiles) load(tile + S - 1);
    cp_async_commit();
    look_up(tile + S);
    const uint32_t kt = ring_a + (tile % S) * plan.stage;
    // ---- scores ----
    float c[MT][2][4];
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) c[i][0][e] = c[i][1][e] = 0.f;
    const uint32_t b_at = kt + ((kg * 16 + (lane & 7) + (lane >> 4) * 8) * ldk + ((lane >> 3) & 1) * 8) * 2;
    const uint32_t a_at = qs_a + ((lane & 15) * ldk + (lane >> 4) * 8) * 2;
#pragma unroll 3
    for (int ks = ks0; ks < ks1; ++ks) {
      uint32_t bk[4];
      ldsm_x4(b_at + ks * 32, bk);
#pragma unroll
      for (int i = 0; i < MT; ++i) {
        uint32_t a[4];
        ldsm_x4(a_at + i * (16 * ldk * 2) + ks * 32, a);
        mma_bf16_16816(c[i][0], a, bk[0], bk[1]);
        mma_bf16_16816(c[i][1], a, bk[2], bk[3]);
      }
    }
#pragma unroll
    for (int i = 0; i < MT; ++i) {
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        float* dst = ss + (quarter * M + i * 16 + r4) * kLdS + kg * 16 + n * 8 + c4 * 2;
        *reinterpret_cast<float2*>(dst) = make_float2(c[i][n][0], c[i][n][1]);
        *reinterpret_cast<float2*>(dst + 8 * kLdS) = make_float2(c[i][n][2], c[i][n][3]);
      }
    }
    __syncthreads();
    // ---- softmax ----
    const int key = k_begin + tile * KT + lane;
#pragma unroll
    for (int i = 0; i < kRows; ++i) {
      const int row = warp * kRows + i, limit = min(row_len[row], k_end), first = latent_first(row_len[row], p.window);
      float v[kPer], t = -CUDART_INF_F;
#pragma unroll
      for (int j = 0; j < kPer; ++j) {
        const float* sp = ss + row * kLdS + lane + 32 * j;
        v[j] = (sp[0] + sp[M * kLdS]) + (sp[2 * M * kLdS] + sp[3 * M * kLdS]);
        v[j] = key + 32 * j < limit && key + 32 * j >= first ? v[j] * scale2 : -CUDART_INF_F;
        t = fmaxf(t, v[j]);
      }
#pragma unroll
      for (int off = 16; off > 0; off >>= 1) t = fmaxf(t, __shfl_xor_sync(0xffffffffu, t, off));
      const float m_new = fmaxf(mx[i], t);
      const bool any = m_new > -CUDART_INF_F;
      const float f = any ? ex2_fast(mx[i] - m_new) : 1.f;
      float sum = 0.f;
#pragma unroll
      for (int j = 0; j < kPer; ++j) {
        const float w = any ? ex2_fast(v[j] - m_new) : 0.f;
        sum += w;
        ps[row * kLdP + lane + 32 * j] = __float2bfloat16(w);
      }
      l[i] = l[i] * f + warp_sum(sum);
      mx[i] = m_new;
      if (lane == 0) alpha[row] = f;
    }
    __syncthreads();
    // ---- values ----
    if (col0 < p.rank) {
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        const float f0 = alpha[m * 16 + r4], f1 = alpha[m * 16 + r4 + 8];
#pragma unroll
        for (int n = 0; n < NT; ++n) { o[m][n][0] *= f0; o[m][n][1] *= f0; o[m][n][2] *= f1; o[m][n][3] *= f1; }
      }
#pragma unroll
      for (int kk = 0; kk < KT / 16; ++kk) {
        uint32_t a[MT][4];
#pragma unroll
        for (int m = 0; m < MT; ++m) ldsm_x4(ps_a + ((m * 16 + (lane & 15)) * kLdP + kk * 16 + (lane >> 4) * 8) * 2, a[m]);
#pragma unroll
        for (int n = 0; n < NT; n += 2) {
          if (col0 + n * 8 < p.rank) {
            uint32_t v[4];
            ldsm_x4_trans(kt + ((kk * 16 + (lane & 15)) * ldk + col0 + n * 8 + (lane >> 4) * 8) * 2, v);
#pragma unroll
            for (int m = 0; m < MT; ++m) {
              mma_bf16_16816(o[m][n], a[m], v[0], v[1]);
              mma_bf16_16816(o[m][n + 1], a[m], v[2], v[3]);
            }
          }
        }
      }
    }
  }
  cp_async_wait<0>();
  __syncthreads();
  // ---- store: alpha holds [factor] per row, or the row's maximum and sum go out as they are ----
#pragma unroll
  for (int i = 0; i < kRows; ++i) {
    const int row = warp * kRows + i;
    if (lane == 0 && row < n_rows) {
      const long long at = static_cast<long long>(t0) * H + r0 + row;
      if (n_splits > 1) {
        part_ml[(at * n_splits + split) * 2] = mx[i];
        part_ml[(at * n_splits + split) * 2 + 1] = l[i];
      } else {
        const float sink = p.sink != nullptr ? p.sink[(r0 + row) % H] * kLog2e : -CUDART_INF_F;
        const float top = fmaxf(mx[i], sink);
        const float e = mx[i] > -CUDART_INF_F ? exp2f(mx[i] - top) : 0.f;
        const float den = e * l[i] + (p.sink != nullptr ? exp2f(sink - top) : 0.f);
        alpha[row] = den > 0.f ? e / den : 0.f;
      }
    }
  }
  __syncthreads();
#pragma unroll
  for (int m = 0; m < MT; ++m) {
#pragma unroll
    for (int half_row = 0; half_row < 2; ++half_row) {
      const int row = m * 16 + r4 + half_row * 8;
      if (row >= n_rows) continue;
      const long long at = static_cast<long long>(t0) * H + r0 + row;
      const float f = n_splits > 1 ? 1.f : alpha[row];
      const int t = t0 + (r0 + row) / H, h = (r0 + row) % H;
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        const int col = col0 + n * 8 + c4 * 2;
        if (col < p.rank) {
          const float x = o[m][n][half_row * 2], y = o[m][n][half_row * 2 + 1];
          if (n_splits > 1)
            *reinterpret_cast<float2*>(part_o + (at * n_splits + split) * p.rank + col) = make_float2(x, y);
          else
            *reinterpret_cast<uint32_t*>(static_cast<bf16*>(p.out) + t * p.ldo + static_cast<long long>(h) * p.rank + col) = pack_bf16x2(x * f, y * f);
        }
      }
    }
  }
}

// One CTA per (token, head) row: the splits' sums on a common maximum, the sink, the quotient.
__global__ void __launch_bounds__(128) latent_merge_kernel(const LatentArgs p, const LatentBlocks b, int n_splits,
                                                            const float* __restrict__ part_o, const float* __restrict__ part_ml) {
  pdl_launch_next();
  pdl_wait_prior();
  const int t = blockIdx.x, h = blockIdx.y;
  if (b.max_tokens > 0) {
    const int seq = b.token_seq[t];
    if (b.cu_seqlens[seq + 1] - b.cu_seqlens[seq] >= b.max_tokens) return;
  }
  const long long at = (static_cast<long long>(t) * p.n_heads + h) * n_splits;
  const float sink = p.sink != nullptr ? p.sink[h] * kLog2e : -CUDART_INF_F;
  float top = sink;
  for (int s = 0; s < n_splits; ++s) top = fmaxf(top, part_ml[(at + s) * 2]);
  float den = p.sink != nullptr && top > -CUDART_INF_F ? exp2f(sink - top) : 0.f;
  float o[4] = {0.f, 0.f, 0.f, 0.f};
  const int c0 = threadIdx.x * 4;
  for (int s = 0; s < n_splits; ++s) {
    const float m = part_ml[(at + s) * 2];
    const float e = m > -CUDART_INF_F ? exp2f(m - top) : 0.f;
    den += e * part_ml[(at + s) * 2 + 1];
    if (c0 < p.rank && e > 0.f) {
      const float4 v = *reinterpret_cast<const float4*>(part_o + (at + s) * p.rank + c0);
      o[0] = fmaf(e, v.x, o[0]); o[1] = fmaf(e, v.y, o[1]); o[2] = fmaf(e, v.z, o[2]); o[3] = fmaf(e, v.w, o[3]);
    }
  }
  const float inv = den > 0.f ? 1.f / den : 0.f;
  bf16* out = static_cast<bf16*>(p.out) + t * p.ldo + static_cast<long long>(h) * p.rank;
  if (c0 < p.rank)
    *reinterpret_cast<uint2*>(out + c0) = make_uint2(pack_bf16x2(o[0] * inv, o[1] * inv), pack_bf16x2(o[2] * inv, o[3] * inv));
}

constexpr int kSmemLimit = 225 * 1024;

template <int NW, int MT, int NT, int S>
cudaError_t launch(const LatentArgs& a, const LatentBlocks& b, int split_keys, int n_splits, float* part_o, float* part_ml) {
  const Plan plan(16 * MT, a.rank + a.rot, S, 4 * NW);
  auto kern = latent_absorbed_kernel<NW, MT, NT, S>;
  const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, plan.total);
  if (e != cudaSuccess) return e;
  const int row_blocks = (b.max_count * a.n_heads + 16 * MT - 1) / (16 * MT);
  return launch_kernel(kern, dim3(n_splits, row_blocks, b.n), dim3(NW * 32), plan.total, a.stream, a.pdl, 1, a, b, split_keys, n_splits,
                       part_o, part_ml);
}

template <int NW, int MT, int NT>
cudaError_t pick_stages(const LatentArgs& a, const LatentBlocks& b, int split_keys, int n_splits, float* part_o, float* part_ml) {
  if (Plan(16 * MT, a.rank + a.rot, 3, 4 * NW).total <= kSmemLimit)
    return launch<NW, MT, NT, 3>(a, b, split_keys, n_splits, part_o, part_ml);
  return launch<NW, MT, NT, 2>(a, b, split_keys, n_splits, part_o, part_ml);
}

// NT: columns per warp / 8 with sixteen warps; eight warps hold twice as many.
template <int NT>
cudaError_t pick_rows(const LatentArgs& a, const LatentBlocks& b, int split_keys, int n_splits, float* part_o, float* part_ml) {
  const int rows = b.max_count * a.n_heads;
  if (rows <= 16) return pick_stages<16, 1, NT>(a, b, split_keys, n_splits, part_o, part_ml);
  if (rows <= 32) return pick_stages<16, 2, NT>(a, b, split_keys, n_splits, part_o, part_ml);
  return pick_stages<8, 4, 2 * NT>(a, b, split_keys, n_splits, part_o, part_ml);
}

}  // namespace

bool latent_absorbed_supported(int rank, int rot) {
  return rank % 16 == 0 && rot % 16 == 0 && rank > 0 && rank <= 512 && Plan(64, rank + rot, 2, 32).total <= kSmemLimit &&
         Plan(32, rank + rot, 2, 64).total <= kSmemLimit;
}

const char* latent_absorbed_attention(const LatentArgs& a, const LatentBlocks& b, int split_keys, int n_splits, float* part_o,
                                      float* part_ml) {
  if (a.T <= 0 || b.n <= 0) return nullptr;
  if (a.f32) return "latent_absorbed_attention: bf16 only";
  if (!latent_absorbed_supported(a.rank, a.rot) || a.rot_true > a.rot || a.rot_true % 2)
    return "latent_absorbed_attention: widths must be multiples of 16, the latent at most 512 wide";
  if (a.ldl % 8 || a.ldq % 2 || a.ldo % 4) return "latent_absorbed_attention: misaligned rows";
  if (b.max_count < 1 || b.max_count > kLatentBlock || b.n > 65535 || n_splits < 1 || n_splits > 1024 || split_keys < 1)
    return "latent_absorbed_attention: bad blocks or splits";
  if (a.n_heads > 4096) return "latent_absorbed_attention: too many heads";
  if (n_splits > 1 && (part_o == nullptr || part_ml == nullptr)) return "latent_absorbed_attention: splits need their workspace";
  cudaError_t e;
  if (a.rank <= 256) e = pick_rows<2>(a, b, split_keys, n_splits, part_o, part_ml);
  else e = pick_rows<4>(a, b, split_keys, n_splits, part_o, part_ml);
  if (e == cudaSuccess && n_splits > 1)
    e = launch_kernel(latent_merge_kernel, dim3(a.T, a.n_heads), dim3(128), 0, a.stream, a.pdl, 1, a, b, n_splits, const_cast<const float*>(part_o),
                      const_cast<const float*>(part_ml));
  return e == cudaSuccess ? nullptr : cudaGetErrorString(e);
}

}  // namespace nfb
