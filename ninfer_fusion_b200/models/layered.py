"""Decoders described as a list of layers (`models/layered_config.py`): weight packing and the forward pass on the
native kernels.

A layer is a mixer (head-mixing attention, latent attention, matrix memory or gated linear memory) and an optional
feed-forward on a 32-bit residual stream.  A sublayer meets the stream in one of two ways: the norm after the sum,
``x <- rms_norm(alpha x + f(x)) * gain``, or norms around it, ``x <- x + mult * norm(f(norm(x)))``, with an optional
causal convolution in front of every mixer.  Layers can run several times with the same weights; cache and state belong
to layer runs.  Every size and constant is a field of the description, so a design is a mapping onto these fields
(`models/kuzanex.py`, `models/tebivik.py`) and not a model file of its own.

The engine side is the hybrid runtime's: one ragged token batch per step (`runtime/batch.py`), K / V or latent rows in the
paged cache (one geometry per run), recurrent state in per-sequence slots, preallocated buffers so that a decode step can
be captured in a CUDA graph.  Activations are bf16 (tcgen05 GEMMs, tensor-core prefill kernels) or, for exact runs, fp32.
Head widths are padded to multiples of 16 and the model width to a multiple of 8 when the weights are packed: zero rows
and columns change no product, and every norm divides by the true width.
"""
from __future__ import annotations

from typing import Dict, List, Tuple

import torch

from .._lib import StatusWord, load_native
from .hybrid import EPI_STORE, LaunchCounter, StepBatch
from .layered_config import (ATTENTION_KINDS, AttentionMixer, GatedMemoryMixer, LatentAttentionMixer, LayeredConfig,
                             MatrixMemoryMixer, pad_to)

ACTIVATIONS = {"xielu": 3, "relu2": 4}     # csrc/gemm/gemm.h GemmActivation
BLOCK_TOKENS = 64          # query tokens per attention block of a step (kHeadMixBlock, kLatentBlock)
PREFILL_MIN_TOKENS = 8     # shorter portions take the token-by-token kernels
EXPAND_BYTES = 4 << 30     # keys and values of expanded latents in flight
SCORE_SCRATCH_BYTES = 1 << 30    # fp32 scores in flight between the two prefill attention kernels


# ---------------------------------------------------------------------------------------------- weight packing
def _pad2(w: torch.Tensor, rows: int, cols: int) -> torch.Tensor:
    out = torch.zeros((rows, cols), dtype=w.dtype, device=w.device)
    out[: w.shape[0], : w.shape[1]] = w
    return out


def _pad_head_rows(w: torch.Tensor, heads: int, width: int, width_p: int, cols: int) -> torch.Tensor:
    out = torch.zeros((heads, width_p, cols), dtype=w.dtype, device=w.device)
    out[:, :width, : w.shape[1]] = w.reshape(heads, width, w.shape[1])
    return out.reshape(heads * width_p, cols)


def _pad_head_vec(v: torch.Tensor, heads: int, width: int, width_p: int) -> torch.Tensor:
    out = torch.zeros((heads, width_p), dtype=torch.float32, device=v.device)
    out[:, :width] = v.float().reshape(heads, width)
    return out.reshape(-1)


def _pad_head_cols(w: torch.Tensor, heads: int, width: int, width_p: int, rows: int) -> torch.Tensor:
    out = torch.zeros((rows, heads, width_p), dtype=w.dtype, device=w.device)
    out[: w.shape[0], :, :width] = w.reshape(w.shape[0], heads, width)
    return out.reshape(rows, heads * width_p)


def distance_slopes(heads: int) -> torch.Tensor:
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)], dtype=torch.float64)


def check_tensor_shapes(expected, shape_of) -> None:
    """Every (name, shape) of `expected` is there; `shape_of(name)` returns None for a missing tensor."""
    for name, shape in expected:
        have = shape_of(name)
        if have is None:
            raise ValueError(f"checkpoint has no tensor '{name}'")
        if tuple(have) != shape:
            raise ValueError(f"tensor '{name}' has shape {list(have)}, the configuration asks for {list(shape)}")


def _pack_attention(w, p, m: AttentionMixer, get, n_out: int, hp: int, device):
    H, G, D, V, Dp, Vp = m.heads, m.kv_heads, m.dim, m.vdim, m.dim_p, m.vdim_p
    rows = [_pad_head_rows(get("q"), H, D, Dp, hp), _pad_head_rows(get("k"), G, D, Dp, hp), _pad_head_rows(get("v"), G, V, Vp, hp)]
    bias = torch.zeros(n_out, dtype=torch.float32, device=device)
    if m.head_gate:
        rows.append(_pad2(get("g"), H, hp))
    if m.bias:
        b = torch.cat([_pad_head_vec(get("q_bias"), H, D, Dp), _pad_head_vec(get("k_bias"), G, D, Dp),
                       _pad_head_vec(get("v_bias"), G, V, Vp)])
        bias[: b.numel()] = b
    if m.qk_norm:
        w[f"{p}/mix/q_norm"] = _pad_head_vec(get("q_norm"), 1, D, Dp)
        w[f"{p}/mix/k_norm"] = _pad_head_vec(get("k_norm"), 1, D, Dp)
    mix = get("talk").double() if m.head_mixing else torch.eye(H, dtype=torch.float64, device=device)
    if m.head_mixing:
        w[f"{p}/mix/heads"] = mix.float().contiguous()
    if m.distance_bias:
        # mixing is linear: the bias taken off before it is (mix @ slope) taken off after it
        w[f"{p}/mix/slope"] = (mix @ distance_slopes(H).to(device)).float().contiguous()
    w[f"{p}/mix/in_bias"] = bias
    return rows


def _pack_matrix_memory(w, p, m: MatrixMemoryMixer, get, n_out: int, hp: int, device):
    H, D, V, Dp, Vp = m.heads, m.dim, m.vdim, m.dim_p, m.vdim_p
    bias = torch.zeros(n_out, dtype=torch.float32, device=device)
    bias[m.main_cols: m.main_cols + H] = get("i_bias").float()
    bias[m.main_cols + H: m.main_cols + 2 * H] = get("f_bias").float()
    w[f"{p}/mix/in_bias"] = bias
    w[f"{p}/mix/norm"] = _pad_head_vec(get("norm"), H, V, Vp)
    return [_pad_head_rows(get("q"), H, D, Dp, hp), _pad_head_rows(get("k"), H, D, Dp, hp), _pad_head_rows(get("v"), H, V, Vp, hp),
            _pad_head_rows(get("g"), H, V, Vp, hp), _pad2(get("i"), H, hp), _pad2(get("f"), H, hp)]


def _pack_gated_memory(w, p, m: GatedMemoryMixer, get, n_out: int, hp: int, device):
    H, D, V, Dp, Vp = m.heads, m.dim, m.vdim, m.dim_p, m.vdim_p
    bias = torch.zeros(n_out, dtype=torch.float32, device=device)
    bias[m.main_cols: m.main_cols + H * Dp] = _pad_head_vec(get("f_bias"), H, D, Dp)
    lower = torch.ones((H, Dp), dtype=torch.float32, device=device)       # padded channels forget nothing and take nothing in
    lower[:, :D] = get("lower").float().reshape(H, D)
    w[f"{p}/mix/in_bias"] = bias
    w[f"{p}/mix/lower"] = lower.reshape(-1)
    w[f"{p}/mix/norm"] = _pad_head_vec(get("norm"), 1, V, Vp)
    return [_pad_head_rows(get("q"), H, D, Dp, hp), _pad_head_rows(get("v"), H, V, Vp, hp), _pad_head_rows(get("f"), H, D, Dp, hp)]


def _pack_latent(w, p, m: LatentAttentionMixer, get, hp: int, dtype, device):
    H, D, R, V, Q, C = m.heads, m.dim, m.rot_dim, m.vdim, m.q_rank, m.kv_rank
    Dp, Rp, Vp, Qp, Cp = m.dim_p, m.rot_p, m.vdim_p, m.q_rank_p, m.kv_rank_p
    uq = get("uq").reshape(H, D + R, Q)
    q = torch.zeros((H, Dp + Rp, Qp), dtype=uq.dtype, device=device)
    q[:, :D, :Q] = uq[:, :D]
    q[:, Dp: Dp + R, :Q] = uq[:, D:]
    w[f"{p}/mix/uq"] = q.reshape(H * (Dp + Rp), Qp).to(dtype)
    k, v = _pad_head_rows(get("uk"), H, D, Dp, Cp), _pad_head_rows(get("uv"), H, V, Vp, Cp)
    w[f"{p}/mix/ukv"] = torch.cat([k, v]).to(dtype)                        # rows: keys of all heads, values of all heads
    w[f"{p}/mix/uv"] = w[f"{p}/mix/ukv"][H * Dp:].view(H, Vp, Cp)
    w[f"{p}/mix/uk_t"] = k.reshape(H, Dp, Cp).transpose(1, 2).contiguous().to(dtype)   # takes a query to the latent space
    w[f"{p}/mix/q_norm"] = _pad_head_vec(get("dq_norm"), 1, Q, Qp)
    w[f"{p}/mix/kv_norm"] = _pad_head_vec(get("dkv_norm"), 1, C, Cp)
    w[f"{p}/mix/freq"] = torch.tensor([m.rot_base ** (-2.0 * i / R) for i in range(R // 2)], dtype=torch.float64, device=device)
    if m.sink:
        w[f"{p}/mix/sink"] = get("sink").float().contiguous()
    dkv = get("dkv")
    return [_pad2(get("dq"), Qp, hp), _pad2(dkv[:C], Cp, hp), _pad2(dkv[C:], Rp, hp)]


def pack_weights(cfg: LayeredConfig, get, dtype: torch.dtype = torch.bfloat16, device="cpu") -> Dict[str, torch.Tensor]:
    """Fused, padded weights of the forward pass.  `get(layer, name)` returns a design's tensor by its role (layer -1:
    the model's own): embed, head, final_norm, loop_in, loop_step; norm1, norm1b, norm2, norm2b, conv; the mixers' (see
    the _pack functions) and o; up, up_bias, down, down_bias, act."""
    hp, wide = cfg.hidden_p, cfg.residual == "sandwich"
    w: Dict[str, torch.Tensor] = {}

    def g(layer, name):
        return get(layer, name).to(device)

    def norm(layer, name):
        return _pad_head_vec(g(layer, name), 1, cfg.hidden, hp) if wide else g(layer, name).float().contiguous().reshape(1)
    if cfg.tie_head:
        w["text/embed"] = w["text/lm_head"] = _pad2(g(-1, "embed"), cfg.vocab_p, hp).to(dtype)
    else:
        w["text/embed"] = _pad2(g(-1, "embed"), cfg.vocab, hp).to(dtype)
        w["text/lm_head"] = _pad2(g(-1, "head"), cfg.vocab_p, hp).to(dtype)
    w["text/final_norm"] = norm(-1, "final_norm")
    if cfg.loop is not None:
        w["text/loop/in_proj"] = _pad_head_cols(g(-1, "loop_in"), 2, cfg.hidden, hp, hp).to(dtype)
        w["text/loop/step"] = torch.stack([_pad_head_vec(v, 1, cfg.hidden, hp) for v in g(-1, "loop_step")])
    for i, spec in enumerate(cfg.layers):
        m, p = spec.mixer, f"text/layers/{i}"

        def mix(name, i=i):
            return g(i, name)
        w[f"{p}/norm1"] = norm(i, "norm1")
        if wide:
            w[f"{p}/norm1b"] = norm(i, "norm1b")
        if cfg.conv_taps:
            w[f"{p}/conv"] = torch.stack([_pad_head_vec(v, 1, cfg.hidden, hp) for v in g(i, "conv").t()])      # [taps, width]
        n_out = pad_to(m.main_cols + m.gate_cols, 2)
        if m.kind == "attention":
            rows = _pack_attention(w, p, m, mix, n_out, hp, device)
        elif m.kind == "latent_attention":
            rows = _pack_latent(w, p, m, mix, hp, dtype, device)
        elif m.kind == "hgrn2":
            rows = _pack_gated_memory(w, p, m, mix, n_out, hp, device)
        else:
            rows = _pack_matrix_memory(w, p, m, mix, n_out, hp, device)
        w[f"{p}/mix/in_proj"] = _pad2(torch.cat(rows), n_out, hp).to(dtype)
        w[f"{p}/mix/out_proj"] = _pad_head_cols(g(i, "o"), m.heads, m.vdim, m.vdim_p, hp).to(dtype)
        if spec.mlp is not None:
            fp = pad_to(spec.mlp.ff, 8)
            w[f"{p}/norm2"] = norm(i, "norm2")
            if wide:
                w[f"{p}/norm2b"] = norm(i, "norm2b")
            w[f"{p}/mlp/up"] = _pad2(g(i, "up"), fp, hp).to(dtype)
            w[f"{p}/mlp/down"] = _pad2(g(i, "down"), hp, fp).to(dtype)
            if spec.mlp.bias:
                w[f"{p}/mlp/up_bias"] = _pad_head_vec(g(i, "up_bias"), 1, spec.mlp.ff, fp)
                w[f"{p}/mlp/down_bias"] = _pad_head_vec(g(i, "down_bias"), 1, cfg.hidden, hp)
            if spec.mlp.activation not in ACTIVATIONS:
                raise ValueError(f"layer {i}: unknown feed-forward activation '{spec.mlp.activation}'")
            if spec.mlp.activation == "xielu":
                a = torch.nn.functional.softplus(g(i, "act").double())
                w[f"{p}/mlp/act"] = torch.stack([a[0], 0.5 + a[1]]).float().contiguous()
    return w


# ---------------------------------------------------------------------------------------------- runtime
class LayeredWorkspace:
    """Activation buffers for up to `max_tokens` tokens; addresses are stable across steps."""

    def __init__(self, cfg: LayeredConfig, max_tokens: int, max_logit_rows: int, device, dtype: torch.dtype,
                 split_rows: int = 1024):
        T, dev, f32 = max_tokens, device, torch.float32
        mixers = [l.mixer for l in cfg.layers]
        attn = [m for m in mixers if m.kind == "attention"]
        latent = [m for m in mixers if m.kind == "latent_attention"]

        def rows(cols, dt=dtype):
            return torch.zeros((T, cols), dtype=dt, device=dev)

        def widest(values, default, mult=64):
            return pad_to(max(values, default=default), mult)
        self.max_tokens, self.max_logit_rows = T, max_logit_rows
        self.x = rows(cfg.hidden_p, f32)           # residual stream
        self.x2 = rows(cfg.hidden_p, f32) if cfg.conv_taps else self.x     # its other copy: a convolution reads rows that its step replaces
        self.xa = rows(cfg.hidden_p)               # what the next GEMM reads, in the activation type
        self.pair = rows(2 * cfg.hidden_p) if cfg.loop is not None else None   # [x, embedding output] of a pass's entry
        self.delta = rows(cfg.hidden_p, f32)       # output of the running sublayer
        self.proj = rows(widest((m.main_cols for m in mixers), 64))
        self.gates = rows(widest((m.gate_cols for m in mixers), 2, 4), f32)
        self.mix = rows(widest((m.out_cols for m in mixers), 64))
        self.q = rows(max([m.heads * m.dim_p for m in attn] + [m.q_cols for m in latent], default=16))
        self.act = rows(widest((l.mlp.ff for l in cfg.layers if l.mlp is not None), 8))
        if latent:
            self.q_latent = rows(max(m.q_rank_p for m in latent))
            self.q_abs = rows(max(m.heads * m.kv_rank_p for m in latent))     # absorbed queries, head by head
            self.o_latent = rows(max(m.heads * m.kv_rank_p for m in latent))  # attended latents
        # split-KV partials: (query token x split) rows of decode-sized steps
        self.split_rows = split_rows
        self.part_o = torch.empty(split_rows * max([m.out_cols for m in attn] + [m.heads * m.kv_rank_p for m in latent], default=0),
                                  dtype=f32, device=dev)
        self.part_ml = torch.empty(split_rows * max((m.heads for m in attn + latent), default=0) * 2, dtype=f32, device=dev)
        self.logits = torch.zeros((max_logit_rows, cfg.vocab_p), dtype=f32, device=dev)
        self.head_in = torch.zeros((max_logit_rows, cfg.hidden_p), dtype=dtype, device=dev)
        self.next_ids = torch.zeros((max_logit_rows,), dtype=torch.int32, device=dev)


def native_subset(cfg: LayeredConfig) -> str:
    """The stand-alone library (see `_build.SUBSETS`) that has the mixers of this configuration."""
    kinds = {l.mixer.kind for l in cfg.layers}
    for name, have in (("head_mix", {"attention", "mlstm"}), ("latent", {"latent_attention", "hgrn2"})):
        if kinds <= have:
            return name
    return "layered"


class LayeredModel:
    """Forward pass of a `LayeredConfig` over the ragged step batch; the interface is `models.hybrid.HybridModel`'s."""

    def __init__(self, cfg: LayeredConfig, weights: Dict[str, torch.Tensor], device, pdl: bool = False):
        self.cfg, self.w = cfg, weights
        self.device = torch.device(device)
        self._raw_ops = load_native(subset=native_subset(cfg))
        self.ops = LaunchCounter(self._raw_ops)
        self.status = StatusWord(self.device)
        self.dtype = weights["text/embed"].dtype
        if self.dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("weights must be bf16 or fp32")
        self.f32 = self.dtype == torch.float32
        self.pdl = pdl
        self.comm = None
        self.k_row_scale: Dict[int, torch.Tensor] = {}
        self.l2_prefetch = True
        self.prefill_kernels = True     # False: the token-by-token kernels for every size (tests)
        self.layer_hook = None          # called as hook(layer, x[:T]) after every layer run (tests, debugging)
        self._runs = cfg.runs
        self._attn_idx = {r: i for i, r in enumerate(cfg.attn_layers)}
        self._state_idx = {r: i for i, r in enumerate(cfg.state_layers)}
        self._scratch: Dict[str, torch.Tensor] = {}
        self._keep: List[torch.Tensor] = []

    def _grown(self, name: str, n_bytes: int) -> torch.Tensor:
        """Byte scratch of at least `n_bytes` (earlier buffers stay alive: a captured graph may point at them)."""
        cur = self._scratch.get(name)
        if cur is None or cur.numel() < n_bytes:
            cur = torch.empty(n_bytes, dtype=torch.uint8, device=self.device)
            self._keep.append(cur)
            self._scratch[name] = cur
        return cur

    # ------------------------------------------------------------------ GEMM
    def _gemm(self, x, w, bias, out=None, out32=None, out32_from=0, act=0, act_params=None, prefetch=None):
        if self.f32:
            self.ops.gemm_f32(x, w, out, bias, act, act_params, out32, out32_from)
            return
        T, (N, K) = x.shape[0], w.shape
        splits = int(self.ops.gemm_pick_splits(T, N, K, EPI_STORE))
        if not (self.l2_prefetch and T <= 64):
            prefetch = None
        self.ops.gemm_bf16(x, w, out, EPI_STORE, None, bias, None, splits, self.status.tensor, self.pdl, act, None, None, None,
                           None, prefetch, out32, out32_from, act_params)

    def _in_proj(self, ws, T, p, m):
        """Fused input projection: [T, main_cols] in the activation type and [T, gate_cols] in fp32."""
        proj = ws.proj[:T, : m.main_cols]
        gates = ws.gates[:T] if m.gate_cols else None
        self._gemm(ws.xa[:T], self.w[f"{p}/mix/in_proj"], self.w.get(f"{p}/mix/in_bias"), proj, gates, m.main_cols if gates is not None else 0,
                   prefetch=self.w[f"{p}/mix/out_proj"])
        return proj, gates

    # ------------------------------------------------------------------ mixers
    def _attention(self, ws, b: StepBatch, kv, run: int, T: int, p: str, m: AttentionMixer):
        ops, w = self.ops, self.w
        proj, gates = self._in_proj(ws, T, p, m)
        planes = kv.layers[self._attn_idx[run]]
        k_pages, v_pages = planes.typed(self.dtype)
        H, G, Dp, Vp = m.heads, m.kv_heads, m.dim_p, m.vdim_p
        q = ws.q[:T, : H * Dp]
        ops.qkv_append(proj, 0, H * Dp, (H + G) * Dp, H, G, m.dim, w.get(f"{p}/mix/q_norm"), w.get(f"{p}/mix/k_norm"),
                       self.cfg.rms_eps, b.table_row, b.cache_pos, kv.table, q, k_pages, v_pages, kv.page_size, self.pdl)
        out = ws.mix[:T, : H * Vp]
        shape = (m.window, m.scale, m.softcap, m.sink, w.get(f"{p}/mix/heads"), w.get(f"{p}/mix/slope"),
                 gates if m.head_gate else None, out)
        if not self.f32 and self.prefill_kernels and b.max_seq_tokens >= PREFILL_MIN_TOKENS:
            one = int(ops.head_mix_prefill_scratch(H, b.max_kv_len, m.window, 1))
            nb = b.qblk_start.numel()
            scratch = self._grown("scores", max(one, min(one * nb, SCORE_SCRATCH_BYTES)))
            ops.head_mix_prefill(q, k_pages, v_pages, kv.table, b.table_row, b.kv_len, *shape, b.qblk_start, b.qblk_count,
                                 b.max_kv_len, scratch, self.pdl)
            return out
        split, n = self.pick_split(ws, T, b.max_kv_len, m.window)
        ops.head_mix_attention(q, k_pages, v_pages, kv.table, b.table_row, b.kv_len, *shape, split, n,
                               ws.part_o if n > 1 else None, ws.part_ml if n > 1 else None, self.pdl)
        return out

    @staticmethod
    def pick_split(ws, T: int, max_kv_len: int, window: int, sm_count: int = 148) -> Tuple[int, int]:
        """Keys per split (a multiple of 32) and splits per token: two CTAs per SM when the step is small."""
        keys = min(max_kv_len, window) if window > 0 else max_kv_len
        want = max(1, min(2 * sm_count // T, ws.split_rows // T, 64))
        split = max(64, pad_to(-(-keys // want), 32))
        return split, -(-keys // split)

    @staticmethod
    def pick_latent_split(ws, b: StepBatch, m: LatentAttentionMixer, sm_count: int = 148) -> Tuple[int, int]:
        """Keys per split (a multiple of 32) and splits per query block: about one CTA per SM when the step is small."""
        rows = min(b.max_seq_tokens, BLOCK_TOKENS) * m.heads
        ctas = b.qblk_start.numel() * max(1, -(-rows // 64))
        want = max(1, min(sm_count // ctas, ws.split_rows // b.n_tokens, 64))
        split = max(128, pad_to(-(-b.max_kv_len // want), 32))
        return split, -(-b.max_kv_len // split)

    def _head_gemm(self, x: torch.Tensor, x_step: int, w: torch.Tensor, out: torch.Tensor, b: StepBatch, max_tokens: int) -> None:
        """out[t, h * N + n] = sum_k w[h, n, k] x[t, h * x_step + k]; tokens of sequences with `max_tokens` or more may be left out"""
        if not self.f32:
            self.ops.head_gemm(x, x_step, w, out, b.token_seq, b.cu_seqlens, max_tokens, self.pdl)
            return
        H, N, K = w.shape
        for h in range(H):
            self._gemm(x[:, h * x_step: h * x_step + K], w[h], None, out[:, h * N: (h + 1) * N])

    @staticmethod
    def expand_tokens(m: LatentAttentionMixer) -> int:
        """Portion length from which making the keys and values of all visible positions takes fewer multiply-adds than
        attending in the latent space; 0: never."""
        wide, heads = 2 * m.kv_rank_p, m.dim_p + m.vdim_p
        return max(16, -(-m.kv_rank_p * heads // (wide - heads))) if wide > heads else 0

    def _expand_plan(self, b: StepBatch, m: LatentAttentionMixer):
        """Which sequences of the step take the expanded form: (threshold, [n, 3] of block-table row / first gathered row /
        positions, first row per sequence or -1, total rows, longest, whether the others are left) or None."""
        least = self.expand_tokens(m)
        if (self.f32 or not self.prefill_kernels or b.seq_host is None or not least or b.max_seq_tokens < least
                or not self._raw_ops.latent_expanded_supported(m.dim_p, m.rot_p, m.vdim_p)):
            return None
        key = (least, m.heads * (m.dim_p + m.vdim_p))
        if key not in b.plans:
            seqs, base, total = [], [], 0
            for row, n, end in b.seq_host:
                base.append(total if n >= least else -1)
                if n >= least:
                    seqs.append((row, total, end))
                    total += end
            plan = None
            if total * key[1] * 2 <= EXPAND_BYTES:
                host = torch.tensor(base + [v for s in seqs for v in s], dtype=torch.int32)
                dev = (host.pin_memory() if self.device.type == "cuda" else host).to(self.device, non_blocking=True)
                plan = (least, dev[len(base):].view(-1, 3), dev[: len(base)], total, max(s[2] for s in seqs), len(seqs) < len(base))
            b.plans[key] = plan
        return b.plans[key]

    def _latent_attention(self, ws, b: StepBatch, kv, run: int, T: int, p: str, m: LatentAttentionMixer):
        ops, w, eps = self.ops, self.w, self.cfg.rms_eps
        proj, _ = self._in_proj(ws, T, p, m)
        pages, _ = kv.layers[self._attn_idx[run]].typed(self.dtype)
        c_q, q = ws.q_latent[:T, : m.q_rank_p], ws.q[:T, : m.q_cols]
        freq, sink = w[f"{p}/mix/freq"], w.get(f"{p}/mix/sink")
        ops.latent_prep(proj, m.q_rank, m.kv_rank, m.rot_dim, w[f"{p}/mix/q_norm"], w[f"{p}/mix/kv_norm"], eps, freq, b.table_row,
                        b.cache_pos, kv.table, c_q, pages, self.pdl)
        self._gemm(c_q, w[f"{p}/mix/uq"], None, q, prefetch=w[f"{p}/mix/uk_t"])
        out = ws.mix[:T, : m.out_cols]
        plan, blocks = self._expand_plan(b, m), (b.qblk_start, b.qblk_count, min(b.max_seq_tokens, BLOCK_TOKENS))
        if plan is None or plan[-1]:
            skip = 0 if plan is None else plan[0]
            q_abs, o_latent = ws.q_abs[:T, : m.heads * m.kv_rank_p], ws.o_latent[:T, : m.heads * m.kv_rank_p]
            self._head_gemm(q, m.dim_p + m.rot_p, w[f"{p}/mix/uk_t"], q_abs, b, skip)
            args = (q_abs, q, pages, kv.table, b.table_row, b.kv_len, m.heads, m.rot_dim, m.scale, freq, sink, o_latent)
            if self.f32 or not self._raw_ops.latent_absorbed_supported(m.kv_rank_p, m.rot_p):
                ops.latent_token_attention(*args, self.pdl)
            else:
                split, n = self.pick_latent_split(ws, b, m)
                ops.latent_absorbed_attention(*args, *blocks, b.token_seq, b.cu_seqlens, skip, split, n,
                                              ws.part_o if n > 1 else None, ws.part_ml if n > 1 else None, self.pdl)
            self._head_gemm(o_latent, m.kv_rank_p, w[f"{p}/mix/uv"], out, b, skip)
        if plan is not None:
            _, seqs, base, total, longest, _ = plan
            ukv = w[f"{p}/mix/ukv"]
            rows = self._grown("latent rows", total * m.row_cols * 2)[: total * m.row_cols * 2].view(self.dtype).view(total, m.row_cols)
            wide = self._grown("latent keys", total * ukv.shape[0] * 2)[: total * ukv.shape[0] * 2].view(self.dtype).view(total, ukv.shape[0])
            ops.latent_gather(pages, kv.table, seqs, longest, rows, self.pdl)
            self._gemm(rows[:, : m.kv_rank_p], ukv, None, wide)
            ops.latent_expanded_attention(q, rows, wide, b.kv_len, m.heads, m.kv_rank_p, m.rot_dim, m.scale, freq, sink, out, *blocks,
                                          b.token_seq, base, self.pdl)
        return out

    def _chunk_workspace(self, b: StepBatch, T: int, kind: str, m) -> "torch.Tensor | None":
        """Scratch of a memory's chunked prefill kernels; None when the step takes the token-by-token kernel."""
        supported, size = getattr(self._raw_ops, f"{kind}_chunked_supported"), getattr(self._raw_ops, f"{kind}_chunked_workspace_bytes")
        if self.f32 or not self.prefill_kernels or b.max_seq_tokens < PREFILL_MIN_TOKENS or not supported(m.dim_p, m.vdim_p):
            return None
        return self._grown("chunks", int(size(T, b.n_seqs, m.heads, m.dim_p, m.vdim_p)))

    def _matrix_memory(self, ws, b: StepBatch, states, run: int, T: int, p: str, m: MatrixMemoryMixer, write_state: bool):
        proj, gates = self._in_proj(ws, T, p, m)
        S, n, mx = states.layers[self._state_idx[run]][-3:]
        H, Dp, Vp = m.heads, m.dim_p, m.vdim_p
        chunk_ws = self._chunk_workspace(b, T, "mlstm", m)
        self.ops.count += 3 if chunk_ws is not None else 0
        out = ws.mix[:T, : H * Vp]
        self.ops.mlstm(proj, 0, H * Dp, 2 * H * Dp, H * (2 * Dp + Vp), gates, 0, H, m.vdim, m.dim ** -0.5, m.gate_cap,
                       self.cfg.rms_eps, self.w[f"{p}/mix/norm"], b.cu_seqlens, b.state_slot, S, n, mx, out, write_state,
                       chunk_ws, self.pdl, b.one_token_per_seq)
        return out

    def _gated_memory(self, ws, b: StepBatch, states, run: int, T: int, p: str, m: GatedMemoryMixer, write_state: bool):
        proj, gates = self._in_proj(ws, T, p, m)
        S = states.layers[self._state_idx[run]][-1]
        chunk_ws = self._chunk_workspace(b, T, "gated", m)
        self.ops.count += 2 if chunk_ws is not None else 0
        out = ws.mix[:T, : m.out_cols]
        self.ops.gated_memory(proj, 0, m.heads * m.dim_p, gates, self.w[f"{p}/mix/lower"], m.vdim, self.cfg.rms_eps,
                              self.w[f"{p}/mix/norm"], b.cu_seqlens, b.state_slot, S, out, write_state, chunk_ws, self.pdl,
                              b.one_token_per_seq)
        return out

    def _mixer(self, ws, b: StepBatch, kv, states, run: int, T: int, p: str, m, write_state: bool) -> torch.Tensor:
        if m.kind in ATTENTION_KINDS:
            fn = self._attention if m.kind == "attention" else self._latent_attention
            return fn(ws, b, kv, run, T, p, m)
        fn = self._gated_memory if m.kind == "hgrn2" else self._matrix_memory
        return fn(ws, b, states, run, T, p, m, write_state)

    def _feed_forward(self, ws, T: int, p: str, spec, prefetch) -> None:
        w, up, down = self.w, self.w[f"{p}/mlp/up"], self.w[f"{p}/mlp/down"]
        act = ws.act[:T, : up.shape[0]]
        self._gemm(ws.xa[:T], up, w.get(f"{p}/mlp/up_bias"), act, act=ACTIVATIONS[spec.activation], act_params=w.get(f"{p}/mlp/act"),
                   prefetch=down)
        self._gemm(act, down, w.get(f"{p}/mlp/down_bias"), out32=ws.delta[:T], prefetch=prefetch)

    # ------------------------------------------------------------------ forward
    def forward_hidden(self, ws: LayeredWorkspace, b: StepBatch, kv, states, write_state: bool = True) -> torch.Tensor:
        """Runs all layers; returns the final-normed hidden states [T, hidden (padded)]."""
        if b.n_tokens > ws.max_tokens:
            raise ValueError(f"step of {b.n_tokens} tokens exceeds the workspace ({ws.max_tokens})")
        run = self._forward_sandwich if self.cfg.residual == "sandwich" else self._forward_post_sum
        return run(ws, b, kv, states, write_state)

    def _next_weights(self, run: int):
        """What the GEMM after the last one of `run` reads (an L2 hint)."""
        if run + 1 == len(self._runs):
            return self.w["text/lm_head"]
        layer, opens = self._runs[run + 1]
        return self.w["text/loop/in_proj"] if opens >= 0 else self.w[f"text/layers/{layer}/mix/in_proj"]

    def _forward_post_sum(self, ws, b: StepBatch, kv, states, write_state: bool) -> torch.Tensor:
        cfg, ops, w, T = self.cfg, self.ops, self.w, b.n_tokens
        x, xa, delta = ws.x[:T], ws.xa[:T], ws.delta[:T]
        ops.embed_rows32(b.ids, w["text/embed"], x, xa, cfg.embed_scale, self.pdl)
        for run, (layer, _) in enumerate(self._runs):
            spec, p = cfg.layers[layer], f"text/layers/{layer}"
            mix = self._mixer(ws, b, kv, states, run, T, p, spec.mixer, write_state)
            last, nxt = w["text/final_norm"] if run + 1 == len(self._runs) else None, self._next_weights(run)
            self._gemm(mix, w[f"{p}/mix/out_proj"], None, out32=delta, prefetch=w.get(f"{p}/mlp/up", nxt))
            ops.post_norm_rows(x, delta, xa, cfg.hidden, cfg.residual_alpha, cfg.rms_eps, w[f"{p}/norm1"],
                               last if spec.mlp is None else None, self.pdl)
            if spec.mlp is not None:
                self._feed_forward(ws, T, p, spec.mlp, nxt)
                ops.post_norm_rows(x, delta, xa, cfg.hidden, cfg.residual_alpha, cfg.rms_eps, w[f"{p}/norm2"], last, self.pdl)
            if self.layer_hook is not None:
                self.layer_hook(run, x[:, : cfg.hidden])
        return xa

    def _forward_sandwich(self, ws, b: StepBatch, kv, states, write_state: bool) -> torch.Tensor:
        """The residual update of a sublayer waits for the row step in front of the next one (`sandwich_rows`)."""
        cfg, ops, w, T, hp = self.cfg, self.ops, self.w, b.n_tokens, self.cfg.hidden_p
        x, other, xa, delta = ws.x[:T], ws.x2[:T], ws.xa[:T], ws.delta[:T]
        post = None                   # weights of the norm of the sublayer output that waits in `delta`

        def rows(w_next, out, conv_run=-1, layer=0):
            nonlocal x, other, post
            conv = (None, None, None, None)
            if conv_run >= 0 and cfg.conv_taps:
                state = states.layers[self._state_idx[conv_run]][0] if cfg.conv_taps > 1 else None
                conv = (w[f"text/layers/{layer}/conv"], state, b.cu_seqlens, b.state_slot)
            dst = other if conv[0] is not None and post is not None and b.max_seq_tokens > 1 else x
            ops.sandwich_rows(x, dst, None if post is None else delta, post, w_next, out, cfg.hidden, cfg.norm_groups, cfg.residual_mult,
                              cfg.rms_eps, *conv, b.max_seq_tokens, write_state, self.pdl)
            if dst is other:
                x, other = other, x
            post = None
        ops.embed_rows32(b.ids, w["text/embed"], x, ws.pair[:T, hp:] if cfg.loop is not None else xa, cfg.embed_scale, self.pdl)
        for run, (layer, opens) in enumerate(self._runs):
            spec, p = cfg.layers[layer], f"text/layers/{layer}"
            if opens >= 0:
                rows(None, ws.pair[:T, :hp])
                self._gemm(ws.pair[:T], w["text/loop/in_proj"], w["text/loop/step"][opens], out32=x, prefetch=w[f"{p}/mix/in_proj"])
            rows(w[f"{p}/norm1"], xa, run, layer)
            mix = self._mixer(ws, b, kv, states, run, T, p, spec.mixer, write_state)
            nxt = self._next_weights(run)
            self._gemm(mix, w[f"{p}/mix/out_proj"], None, out32=delta, prefetch=w.get(f"{p}/mlp/up", nxt))
            post = w[f"{p}/norm1b"]
            if spec.mlp is not None:
                rows(w[f"{p}/norm2"], xa)
                self._feed_forward(ws, T, p, spec.mlp, nxt)
                post = w[f"{p}/norm2b"]
            if self.layer_hook is not None:
                rows(None, xa)
                self.layer_hook(run, x[:, : cfg.hidden])
        rows(w["text/final_norm"], xa)
        return xa

    def head(self, ws: LayeredWorkspace, head_in: torch.Tensor) -> torch.Tensor:
        """fp32 logits [rows, vocab] of final-normed hidden states (at most `max_logit_rows`)."""
        out = ws.logits[: head_in.shape[0]]
        self._gemm(head_in, self.w["text/lm_head"], None, out32=out)
        return out[:, : self.cfg.vocab]

    def logits(self, ws: LayeredWorkspace, b: StepBatch, hidden: torch.Tensor) -> torch.Tensor:
        R = b.logit_rows.numel()
        if R == hidden.shape[0]:
            return self.head(ws, hidden)       # decode: every row is a logit row, in order
        head_in = ws.head_in[:R]
        torch.index_select(hidden, 0, b.logit_rows.long(), out=head_in)
        return self.head(ws, head_in)

    def forward_greedy(self, ws: LayeredWorkspace, b: StepBatch, kv, states) -> torch.Tensor:
        """One step ending in arg-max token ids for `b.logit_rows` (int32 [R], ws.next_ids)."""
        start = self.ops.count
        hidden = self.forward_hidden(ws, b, kv, states)
        if b.logit_rows.numel() == 0:
            return ws.next_ids[:0]
        lg = self.logits(ws, b, hidden)
        out = ws.next_ids[: lg.shape[0]]
        self.ops.argmax_rows(lg, out, self.pdl)
        self.ops.launches_last_forward = self.ops.count - start
        return out
