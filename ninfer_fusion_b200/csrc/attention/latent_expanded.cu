// Expanded latent attention (bf16): for sequences that bring a long portion, the cached rows of all visible positions are
// gathered into one contiguous array, a GEMM makes every head's keys and values out of their latents, and a flash kernel
// attends to them as ordinary heads.  The rotated key part stays shared: it is read from the gathered rows.
// Flash kernel: one CTA = (head, block of 64 queries), a warp owns 16 queries; key and value tiles of 64 positions come
// through a two-stage cp.async ring, scores, weights and the running sums stay in registers.
#include "latent.h"

#include <math_constants.h>

#include "../common/elem.cuh"
#include "../common/launch.h"
#include "../common/mma_sync.cuh"

namespace nfb {

namespace {

using bf16 = __nv_bfloat16;
constexpr int KT = 64, QT = kLatentBlock, kThreads = 128;

// grid: (blocks of 8 positions, sequence)
__global__ void __launch_bounds__(256) latent_gather_kernel(const LatentArgs p, const LatentExpand x) {
  pdl_launch_next();
  pdl_wait_prior();
  const int* s = x.seqs + blockIdx.y * 4;
  const int at = blockIdx.x * 8 + (threadIdx.x >> 5), W = p.rank + p.rot;
  if (at >= s[3]) return;
  const int pos = s[2] + at;
  const int page = p.block_table[static_cast<long long>(s[0]) * p.table_ld + pos / p.page_size];
  const uint4* src = reinterpret_cast<const uint4*>(static_cast<const bf16*>(p.pages) + (static_cast<long long>(max(page, 0)) * p.page_size + pos % p.page_size) * W);
  uint4* dst = reinterpret_cast<uint4*>(static_cast<bf16*>(x.rows) + static_cast<long long>(s[1] + at) * W);
  for (int c = threadIdx.x & 31; c < W / 8; c += 32) dst[c] = page < 0 ? make_uint4(0u, 0u, 0u, 0u) : src[c];
}

// VT: 8-wide value tiles (at least vdim / 8).
template <int VT>
__global__ void __launch_bounds__(kThreads) latent_flash_kernel(const LatentArgs p, const LatentBlocks b, const LatentExpand x) {
  extern __shared__ __align__(16) bf16 smem_b[];
  const int D = p.dim, R = p.rot, W = D + R, V = x.vdim, H = p.n_heads;
  const int ldk = W + 8, ldv = V + 8, stage = KT * (ldk + ldv);
  bf16* qs = smem_b;                       // [QT][ldk]
  const uint32_t qs_a = smem_u32(qs), ring_a = qs_a + QT * ldk * 2;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, r4 = lane >> 2, c4 = lane & 3;
  pdl_launch_next();
  pdl_wait_prior();
  const int h = blockIdx.x, blk = static_cast<int>(gridDim.y) - 1 - static_cast<int>(blockIdx.y);   // later (longer) blocks first
  const int t0 = b.start[blk], count = b.count[blk], seq = b.token_seq[t0];
  const int row_of_first = x.seq_base[seq * 2];
  if (row_of_first < 0) return;
  const int len = p.kv_len[t0 + count - 1], first_len = p.kv_len[t0];
  const int k_begin = latent_first(first_len, p.window);             // the block's keys: positions k_begin .. len - 1
  const int n_tiles = (len - k_begin + KT - 1) / KT;
  const long long base = static_cast<long long>(row_of_first) + k_begin - x.seq_base[seq * 2 + 1];   // row of position k_begin
  const long long ldx = static_cast<long long>(H) * (D + V);
  const bf16* keys = static_cast<const bf16*>(x.kv) + base * ldx + static_cast<long long>(h) * D;
  const bf16* vals = static_cast<const bf16*>(x.kv) + base * ldx + static_cast<long long>(H) * D + static_cast<long long>(h) * V;
  const bf16* rots = static_cast<const bf16*>(x.rows) + base * (p.rank + R) + p.rank;
  const int kv8 = W / 8, d8 = D / 8, v8 = V / 8;
  // 16 threads walk a row; a thread's rows of a tile are lr, lr + 8, ..., its 16-byte pieces lc, lc + 16, ...
  const int lr = tid >> 4, lc = tid & 15;
  auto copy = [&](uint32_t dst, int ld_dst, const bf16* src, long long ld_src, int left) {   // one piece of the tile's rows
    if (left >= KT) {
#pragma unroll
      for (int j = 0; j < KT / 8; ++j) {
        cp_async16(dst + j * (8 * ld_dst * 2), src, true);
        src += 8 * ld_src;
      }
    } else {
#pragma unroll
      for (int j = 0; j < KT / 8; ++j) {
        const bool ok = lr + j * 8 < left;
        cp_async16(dst + j * (8 * ld_dst * 2), ok ? src : keys, ok);
        src += 8 * ld_src;
      }
    }
  };
  auto load = [&](int tile) {
    const uint32_t dk = ring_a + (tile & 1) * stage * 2 + lr * ldk * 2, dv = ring_a + ((tile & 1) * stage + KT * ldk + lr * ldv) * 2;
    const int left = len - k_begin - tile * KT;
    const long long first = static_cast<long long>(tile) * KT + lr;
    const long long ldr = p.rank + R;
    for (int c = lc; c < kv8; c += 16)
      copy(dk + c * 16, ldk, c < d8 ? keys + first * ldx + c * 8 : rots + first * ldr + (c - d8) * 8, c < d8 ? ldx : ldr, left);
    for (int c = lc; c < v8; c += 16) copy(dv + c * 16, ldv, vals + first * ldx + c * 8, ldx, left);
  };
  load(0);
  cp_async_commit();
  for (int i = tid; i < QT * d8; i += kThreads) {
    const int r = i / d8, c = (i % d8) * 8;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (r < count) v = *reinterpret_cast<const uint4*>(static_cast<const bf16*>(p.q) + (t0 + r) * p.ldq + static_cast<long long>(h) * W + c);
    *reinterpret_cast<uint4*>(qs + r * ldk + c) = v;
  }
  for (int i = tid; i < QT * (R / 2); i += kThreads) {
    const int r = i / (R / 2), e = i % (R / 2);
    float u = 0.f, v = 0.f;
    if (r < count && 2 * e < p.rot_true) {
      const bf16* q = static_cast<const bf16*>(p.q) + (t0 + r) * p.ldq + static_cast<long long>(h) * W + D + 2 * e;
      float c, s;
      rotary_angle(p.kv_len[t0 + r] - 1, p.freq[e], c, s);
      const float a = __bfloat162float(q[0]), bb = __bfloat162float(q[1]);
      u = a * c - bb * s;
      v = bb * c + a * s;
    }
    *reinterpret_cast<uint32_t*>(qs + r * ldk + D + 2 * e) = pack_bf16x2(u, v);
  }
  float o[VT][4];
#pragma unroll
  for (int n = 0; n < VT; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[n][e] = 0.f;
  float m[2] = {-CUDART_INF_F, -CUDART_INF_F}, l[2] = {0.f, 0.f};
  const int row0 = warp * 16;
  const int rlen[2] = {row0 + r4 < count ? p.kv_len[t0 + row0 + r4] : 0, row0 + r4 + 8 < count ? p.kv_len[t0 + row0 + r4 + 8] : 0};
  const int rlo[2] = {latent_first(rlen[0], p.window), latent_first(rlen[1], p.window)}, last_lo = latent_first(len, p.window);
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
#pragma unroll 2
    for (int d = 0; d < W; d += 16) {
      uint32_t a[4];
      ldsm_x4(qs_a + ((row0 + (lane & 15)) * ldk + d + (lane >> 4) * 8) * 2, a);
#pragma unroll
      for (int n = 0; n < KT / 16; ++n) {
        uint32_t k[4];
        ldsm_x4(kt + ((n * 16 + (lane & 7) + (lane >> 4) * 8) * ldk + d + ((lane >> 3) & 1) * 8) * 2, k);
        mma_bf16_16816(s[2 * n], a, k[0], k[1]);
        mma_bf16_16816(s[2 * n + 1], a, k[2], k[3]);
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
  const float sink = p.sink != nullptr ? p.sink[h] * kLog2e : -CUDART_INF_F;
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
    const int row = row0 + r4 + r * 8;
    if (row >= count) continue;
    const float top = fmaxf(m[r], sink);
    const float e = exp2f(m[r] - top);
    const float inv = e / (e * l[r] + (p.sink != nullptr ? exp2f(sink - top) : 0.f));
    bf16* dst = static_cast<bf16*>(p.out) + (t0 + row) * p.ldo + static_cast<long long>(h) * V;
#pragma unroll
    for (int n = 0; n < VT; ++n)
      if (n * 8 < V) *reinterpret_cast<uint32_t*>(dst + n * 8 + c4 * 2) = pack_bf16x2(o[n][2 * r] * inv, o[n][2 * r + 1] * inv);
  }
}

int flash_smem(int dim, int rot, int vdim) { return (QT * (dim + rot + 8) + 2 * KT * (dim + rot + 8 + vdim + 8)) * 2; }

template <int VT>
cudaError_t launch(const LatentArgs& a, const LatentBlocks& b, const LatentExpand& x) {
  const int smem = flash_smem(a.dim, a.rot, x.vdim);
  const cudaError_t e = cudaFuncSetAttribute(latent_flash_kernel<VT>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) return e;
  return launch_kernel(latent_flash_kernel<VT>, dim3(a.n_heads, b.n), dim3(kThreads), smem, a.stream, a.pdl, 1, a, b, x);
}

}  // namespace

bool latent_expanded_supported(int dim, int rot, int vdim) {
  return dim % 16 == 0 && rot % 16 == 0 && vdim % 16 == 0 && dim > 0 && vdim > 0 && vdim <= 256 && flash_smem(dim, rot, vdim) <= 225 * 1024;
}

const char* latent_gather(const LatentArgs& a, const LatentExpand& x) {
  if (x.n_seqs <= 0 || x.max_len <= 0) return nullptr;
  if (a.f32 || x.n_seqs > 65535 || (a.rank + a.rot) % 8) return "latent_gather: bf16 rows only";
  const cudaError_t e = launch_kernel(latent_gather_kernel, dim3((x.max_len + 7) / 8, x.n_seqs), dim3(256), 0, a.stream, a.pdl, 1, a, x);
  return e == cudaSuccess ? nullptr : cudaGetErrorString(e);
}

const char* latent_expanded_attention(const LatentArgs& a, const LatentBlocks& b, const LatentExpand& x) {
  if (a.T <= 0 || b.n <= 0) return nullptr;
  if (a.f32) return "latent_expanded_attention: bf16 only";
  if (!latent_expanded_supported(a.dim, a.rot, x.vdim) || a.rot_true > a.rot || a.rot_true % 2)
    return "latent_expanded_attention: head widths must be multiples of 16 that fit the shared memory of a block";
  if (a.ldq % 8 || a.ldo % 2) return "latent_expanded_attention: misaligned rows";
  if (b.max_count < 1 || b.max_count > kLatentBlock || b.n > 65535) return "latent_expanded_attention: bad blocks";
  cudaError_t e;
  if (x.vdim <= 32) e = launch<4>(a, b, x);
  else if (x.vdim <= 64) e = launch<8>(a, b, x);
  else if (x.vdim <= 128) e = launch<16>(a, b, x);
  else e = launch<32>(a, b, x);
  return e == cudaSuccess ? nullptr : cudaGetErrorString(e);
}

}  // namespace nfb
