// Head-mixing attention, one query token per CTA, on the FP32 pipes (every size, bf16 or 32-bit; bf16 head geometries
// that suit the tensor cores take head_mix_decode.cu, or group_attention.cu for plain scores, instead): the CTA holds ALL heads of its token, because a mixed score needs every head's score of the same key.  Keys are walked in blocks of 32:
//   scores   eight lanes per (key, kv head): 16-byte loads along the key row, reduced by shuffles, soft-capped
//   mix      one thread per (head, key): the row of the mixing matrix times the column of scores, bias, mask
//   softmax  one warp per head, lane = key: running maximum and sum (sigmoid weights need none: they are made before the mix)
//   values   one thread per (head, eight value columns): 16-byte loads along the value row
// Splits of the key range are merged by a second kernel (fp32 partial outputs with their maximum and sum).
#include "head_mix.h"

#include <math_constants.h>

#include "../common/elem.cuh"
#include "../common/launch.h"

namespace nfb {

namespace {

constexpr int kThreads = 256;
constexpr int kKeys = 32;
constexpr int kMaxItems = 8;   // (head, 8 value columns) items per thread and pass

template <typename A, int NI, bool SIG>
__global__ void __launch_bounds__(kThreads) head_mix_token_kernel(const HeadMixArgs p, int split_keys, int n_splits,
                                                                   float* __restrict__ part_o, float* __restrict__ part_ml) {
  extern __shared__ __align__(16) float smem[];
  const int H = p.n_heads, G = p.n_kv, R = H / G, D = p.dim, V = p.vdim, P = p.page_size;
  const int Hp = (H + 3) & ~3;
  float* qs = smem;                       // [H][D]
  float* mixs = qs + H * D;               // [H][Hp]
  float* cs = mixs + H * Hp;              // [H][kKeys] scores, later weights
  float* ss = cs + H * kKeys;             // [H][kKeys] mixed scores
  float* ms = ss + H * kKeys;             // [H] running max
  float* ls = ms + H;                     // [H] running sum
  float* corr = ls + H;                   // [H]
  int* pages = reinterpret_cast<int*>(corr + H);   // [kKeys] row of the key in a kv head's page plane, -1 = none
  const int t = blockIdx.y, split = blockIdx.x;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;

  if (p.mix != nullptr)
    for (int i = tid; i < H * H; i += kThreads) mixs[(i / H) * Hp + i % H] = p.mix[i];
  pdl_launch_next();
  pdl_wait_prior();
  const int len = p.kv_len[t];
  const int qpos = len - 1;
  const int lo = first_visible(len, p.window, p.chunk);
  const int k_begin = lo + split * split_keys;
  const int k_end = min(len, k_begin + split_keys);
  const int* table = p.block_table + static_cast<long long>(p.table_row[t]) * p.table_ld;
  const A* q = static_cast<const A*>(p.q) + t * p.ldq;
  for (int i = tid * 8; i < H * D; i += kThreads * 8) load8(q + i, qs + i);
  for (int h = tid; h < H; h += kThreads) { ms[h] = -CUDART_INF_F; ls[h] = 0.f; }
  const int vecs = V / 8, items = H * vecs;
  const float inv_cap = p.softcap > 0.f ? 1.f / p.softcap : 0.f;
  const A* kp = static_cast<const A*>(p.k_pages);
  const A* vp = static_cast<const A*>(p.v_pages);
  float acc[NI][8];
#pragma unroll
  for (int i = 0; i < NI; ++i)
#pragma unroll
    for (int j = 0; j < 8; ++j) acc[i][j] = 0.f;

  for (int k0 = k_begin; k0 < k_end; k0 += kKeys) {
    const int nk = min(kKeys, k_end - k0);
    if (tid < kKeys) {
      int row = -1;
      if (tid < nk) {
        const int page = table[(k0 + tid) / P];
        if (page >= 0) row = page * G * P + (k0 + tid) % P;
      }
      pages[tid] = row;
    }
    __syncthreads();
    // ---- scores: group of eight lanes = (key, kv head) ----
    {
      const int grp = tid >> 3, l8 = tid & 7;
      for (int task = grp; task < kKeys * G; task += kThreads / 8) {
        const int key = task % kKeys, g = task / kKeys;
        const int row = pages[key];
        const A* kr = kp + (static_cast<long long>(row) + static_cast<long long>(g) * P) * D;
        for (int r = 0; r < R; ++r) {
          const float* qh = qs + (g * R + r) * D;
          float d = 0.f;
          if (row >= 0) {
            for (int c = l8 * 8; c < D; c += 64) {
              float kv[8];
              load8(kr + c, kv);
#pragma unroll
              for (int j = 0; j < 8; ++j) d = fmaf(kv[j], qh[c + j], d);
            }
          }
          d += __shfl_xor_sync(0xffffffffu, d, 4);
          d += __shfl_xor_sync(0xffffffffu, d, 2);
          d += __shfl_xor_sync(0xffffffffu, d, 1);
          if (l8 == 0) {
            if constexpr (SIG) {
              const SigmoidHead hd(p, g * R + r, sizeof(A) == 2);
              const float dist = static_cast<float>(qpos - (k0 + key));
              d = sizeof(A) == 2 ? hd.weight_fast(d, hd.bias_fast(dist)) : hd.weight(d, dist);
            } else {
              d *= p.scale;
              if (p.softcap > 0.f) d = p.softcap * tanh_of<A>(d * inv_cap);
            }
            cs[(g * R + r) * kKeys + key] = d;
          }
        }
      }
    }
    __syncthreads();
    // ---- mix across heads, distance bias, mask ----
    for (int i = tid; i < H * kKeys; i += kThreads) {
      const int h = i / kKeys, key = i % kKeys;
      float s;
      if (p.mix != nullptr) {
        s = 0.f;
        for (int g = 0; g < H; ++g) s = fmaf(mixs[h * Hp + g], cs[g * kKeys + key], s);
      } else {
        s = cs[i];
      }
      if (p.slope != nullptr) s -= p.slope[h] * static_cast<float>(qpos - (k0 + key));
      ss[i] = (key < nk && pages[key] >= 0) ? s : (SIG ? 0.f : -CUDART_INF_F);
    }
    __syncthreads();
    // ---- running softmax: warp = head, lane = key ----
    for (int h = warp; !SIG && h < H; h += kThreads / 32) {
      const float s = ss[h * kKeys + lane];
      const float m_old = ms[h];
      const float m_new = fmaxf(m_old, warp_max(s));
      const float e = m_new == -CUDART_INF_F ? 0.f : exp_of<A>(s - m_new);
      const float sum = warp_sum(e);
      cs[h * kKeys + lane] = e;
      if (lane == 0) {
        const float c = m_old == -CUDART_INF_F ? 0.f : exp_of<A>(m_old - m_new);
        corr[h] = c;
        ls[h] = ls[h] * c + sum;
        ms[h] = m_new;
      }
    }
    if constexpr (!SIG) __syncthreads();
    const float* wgt = SIG ? ss : cs;
    // ---- values ----
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int it = tid + i * kThreads;
      if (it < items) {
        const int h = it / vecs, c = (it % vecs) * 8, g = h / R;
        if constexpr (!SIG) {
          const float cr = corr[h];
#pragma unroll
          for (int j = 0; j < 8; ++j) acc[i][j] *= cr;
        }
        const A* vb = vp + static_cast<long long>(g) * P * V + c;
#pragma unroll 8
        for (int key = 0; key < nk; ++key) {
          const int row = pages[key];
          if (row >= 0) {
            float vv[8];
            load8(vb + static_cast<long long>(row) * V, vv);
            const float w = wgt[h * kKeys + key];
#pragma unroll
            for (int j = 0; j < 8; ++j) acc[i][j] = fmaf(w, vv[j], acc[i][j]);
          }
        }
      }
    }
    __syncthreads();
  }
  __syncthreads();
  if (n_splits > 1) {
    const long long base = static_cast<long long>(t) * n_splits + split;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int it = tid + i * kThreads;
      if (it < items) store8(part_o + base * H * V + it * 8, acc[i]);
    }
    for (int h = tid; h < H; h += kThreads) {
      part_ml[(base * H + h) * 2] = SIG ? 0.f : ms[h];
      part_ml[(base * H + h) * 2 + 1] = SIG ? 1.f : ls[h];
    }
    return;
  }
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int it = tid + i * kThreads;
    if (it < items) {
      const int h = it / vecs;
      float f = SIG ? 1.f : head_mix_finish(ms[h], ls[h], p.sink, p.sinks, h);
      if (p.gate != nullptr) f *= sigmoid_of<A>(p.gate[t * p.ld_gate + h]);
#pragma unroll
      for (int j = 0; j < 8; ++j) acc[i][j] *= f;
      store8(static_cast<A*>(p.out) + t * p.ldo + it * 8, acc[i]);
    }
  }
}

template <typename A>
__global__ void __launch_bounds__(128) head_mix_merge_kernel(const HeadMixArgs p, int n_splits,
                                                             const float* __restrict__ part_o,
                                                             const float* __restrict__ part_ml) {
  pdl_launch_next();
  pdl_wait_prior();
  const int H = p.n_heads, V = p.vdim, vecs = V / 8;
  const int t = blockIdx.y;
  const int it = blockIdx.x * blockDim.x + threadIdx.x;
  if (it >= H * vecs) return;
  const int h = it / vecs;
  const float* ml = part_ml + (static_cast<long long>(t) * n_splits * H + h) * 2;
  float m = -CUDART_INF_F;
  for (int s = 0; s < n_splits; ++s) m = fmaxf(m, ml[static_cast<long long>(s) * H * 2]);
  float l = 0.f, o[8] = {};
  for (int s = 0; s < n_splits; ++s) {
    const float ms = ml[static_cast<long long>(s) * H * 2];
    if (ms == -CUDART_INF_F) continue;
    const float e = exp_of<A>(ms - m);
    l = fmaf(e, ml[static_cast<long long>(s) * H * 2 + 1], l);
    float v[8];
    load8(part_o + (static_cast<long long>(t) * n_splits + s) * H * V + it * 8, v);
#pragma unroll
    for (int j = 0; j < 8; ++j) o[j] = fmaf(e, v[j], o[j]);
  }
  float f = p.sigmoid ? 1.f : head_mix_finish(m, l, p.sink, p.sinks, h);
  if (p.gate != nullptr) f *= sigmoid_of<A>(p.gate[t * p.ld_gate + h]);
#pragma unroll
  for (int j = 0; j < 8; ++j) o[j] *= f;
  store8(static_cast<A*>(p.out) + t * p.ldo + it * 8, o);
}

template <typename A>
const char* merge_splits(const HeadMixArgs& a, int n_splits, const float* part_o, const float* part_ml) {
  if (n_splits <= 1) return nullptr;
  const int items = a.n_heads * a.vdim / 8;
  const cudaError_t e = launch_kernel(head_mix_merge_kernel<A>, dim3((items + 127) / 128, a.T), dim3(128), 0, a.stream, a.pdl, 1, a,
                                      n_splits, part_o, part_ml);
  return e == cudaSuccess ? nullptr : cudaGetErrorString(e);
}

template <typename A, int NI, bool SIG>
const char* launch_token(const HeadMixArgs& a, int split_keys, int n_splits, float* part_o, float* part_ml) {
  const int H = a.n_heads, Hp = (H + 3) & ~3;
  const size_t smem = sizeof(float) * (static_cast<size_t>(H) * a.dim + static_cast<size_t>(H) * Hp + 2u * H * kKeys + 3u * H) +
                      sizeof(int) * kKeys;
  if (smem > 227 * 1024) return "head_mix attention: the heads of one token do not fit in shared memory";
  auto kern = head_mix_token_kernel<A, NI, SIG>;
  static size_t granted = 48 * 1024;
  if (smem > granted) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return cudaGetErrorString(e);
    granted = smem;
  }
  for (int t0 = 0; t0 < a.T; t0 += 65535) {   // grid.y limit
    HeadMixArgs b = a;
    const size_t es = a.f32 ? 4 : 2;
    b.T = a.T - t0 < 65535 ? a.T - t0 : 65535;
    b.q = static_cast<const char*>(a.q) + es * t0 * a.ldq;
    b.out = static_cast<char*>(a.out) + es * t0 * a.ldo;
    b.table_row = a.table_row + t0;
    b.kv_len = a.kv_len + t0;
    if (a.gate != nullptr) b.gate = a.gate + t0 * a.ld_gate;
    float* po = part_o == nullptr ? nullptr : part_o + static_cast<int64_t>(t0) * n_splits * H * a.vdim;
    float* pm = part_ml == nullptr ? nullptr : part_ml + static_cast<int64_t>(t0) * n_splits * H * 2;
    const cudaError_t e = launch_kernel(kern, dim3(n_splits, b.T), dim3(kThreads), smem, a.stream, a.pdl, 1, b, split_keys, n_splits, po, pm);
    if (e != cudaSuccess) return cudaGetErrorString(e);
    if (const char* err = merge_splits<A>(b, n_splits, po, pm)) return err;
  }
  return nullptr;
}

template <typename A, bool SIG>
const char* launch_items(const HeadMixArgs& a, int split_keys, int n_splits, float* part_o, float* part_ml) {
  const int per = (a.n_heads * (a.vdim / 8) + kThreads - 1) / kThreads;
  if (per <= 1) return launch_token<A, 1, SIG>(a, split_keys, n_splits, part_o, part_ml);
  if (per <= 2) return launch_token<A, 2, SIG>(a, split_keys, n_splits, part_o, part_ml);
  if (per <= 4) return launch_token<A, 4, SIG>(a, split_keys, n_splits, part_o, part_ml);
  if (per <= kMaxItems) return launch_token<A, kMaxItems, SIG>(a, split_keys, n_splits, part_o, part_ml);
  return "head_mix attention: heads x value width above 16384 is not supported";
}

}  // namespace

const char* head_mix_token_attention(const HeadMixArgs& a, int split_keys, int n_splits, float* part_o, float* part_ml) {
  if (a.T <= 0) return nullptr;
  if (a.dim % 16 || a.vdim % 16 || a.n_kv <= 0 || a.n_heads % a.n_kv) return "head_mix attention: bad head geometry";
  const int align = a.f32 ? 4 : 8;
  if (a.ldq % align || a.ldo % align) return "head_mix attention: misaligned rows";
  if (split_keys <= 0 || n_splits <= 0 || (n_splits > 1 && (part_o == nullptr || part_ml == nullptr)))
    return "head_mix attention: bad split";
  if (group_attention_supported(a)) {
    if (const char* err = group_decode(a, split_keys, n_splits, part_o, part_ml)) return err;
    return merge_splits<__nv_bfloat16>(a, n_splits, part_o, part_ml);
  }
  if (head_mix_decode_supported(a)) {
    if (const char* err = head_mix_decode(a, split_keys, n_splits, part_o, part_ml)) return err;
    return merge_splits<__nv_bfloat16>(a, n_splits, part_o, part_ml);
  }
  if (a.sigmoid)
    return a.f32 ? launch_items<float, true>(a, split_keys, n_splits, part_o, part_ml)
                 : launch_items<__nv_bfloat16, true>(a, split_keys, n_splits, part_o, part_ml);
  return a.f32 ? launch_items<float, false>(a, split_keys, n_splits, part_o, part_ml)
               : launch_items<__nv_bfloat16, false>(a, split_keys, n_splits, part_o, part_ml);
}

}  // namespace nfb
