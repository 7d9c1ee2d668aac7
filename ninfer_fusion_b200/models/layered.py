"""Decoders described as a list of layers (`models/layered_config.py`): weight packing and the forward pass on the
native kernels.

A layer is a mixer (head-mixing attention or matrix memory) and an optional feed-forward, each followed by the
norm-after-the-sum step ``x <- rms_norm(alpha x + f(x)) * gain`` on a 32-bit residual stream.  Every size and constant
is a field of the layer's description; which mechanisms a mixer has (biases, query / key norm, soft cap, distance bias,
mixing across heads, sink, window, head gate) is too, so a design is a mapping onto these fields
(`models/kuzanex.py`) and not a model file of its own.

The engine side is the hybrid runtime's: one ragged token batch per step (`runtime/batch.py`), K / V rows in the paged
cache (one geometry per layer), recurrent state in per-sequence slots, preallocated buffers so that a decode step can be
captured in a CUDA graph.  Activations are bf16 (tcgen05 GEMMs, tensor-core prefill kernels) or, for exact runs, fp32.
Head widths are padded to multiples of 16 and the model width to a multiple of 8 when the weights are packed: zero rows
and columns change no product, and every norm divides by the true width.
"""
from __future__ import annotations

from typing import Dict, List, Tuple

import torch

from .._lib import StatusWord, load_native
from .hybrid import EPI_STORE, LaunchCounter, StepBatch
from .layered_config import AttentionMixer, LayeredConfig, MatrixMemoryMixer, pad_to

ACT_XIELU = 3              # csrc/gemm/gemm.h GemmActivation
PREFILL_MIN_TOKENS = 8     # shorter portions take the token-by-token kernels
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


def pack_weights(cfg: LayeredConfig, get, dtype: torch.dtype = torch.bfloat16, device="cpu") -> Dict[str, torch.Tensor]:
    """Fused, padded weights of the forward pass.  `get(layer, name)` returns a design's tensor by its role (layer -1:
    the model's own): embed, head, final_norm; norm1, norm2; q, k, v, o, g, q_bias, k_bias, v_bias, q_norm, k_norm,
    talk; i, f, i_bias, f_bias, norm; up, up_bias, down, down_bias, act."""
    hp = cfg.hidden_p
    w: Dict[str, torch.Tensor] = {}

    def g(layer, name):
        return get(layer, name).to(device)

    def f32(layer, name):
        return g(layer, name).float().contiguous()
    w["text/embed"] = _pad2(g(-1, "embed"), cfg.vocab, hp).to(dtype)
    w["text/lm_head"] = _pad2(g(-1, "head"), cfg.vocab_p, hp).to(dtype)
    w["text/final_norm"] = f32(-1, "final_norm").reshape(1)
    for i, spec in enumerate(cfg.layers):
        m, p = spec.mixer, f"text/layers/{i}"
        D, V, Dp, Vp, H = m.dim, m.vdim, m.dim_p, m.vdim_p, m.heads
        w[f"{p}/norm1"] = f32(i, "norm1").reshape(1)
        n_out = pad_to(m.main_cols + m.gate_cols, 2)
        bias = torch.zeros(n_out, dtype=torch.float32, device=device)
        if m.kind == "attention":
            G = m.kv_heads
            rows = [_pad_head_rows(g(i, "q"), H, D, Dp, hp), _pad_head_rows(g(i, "k"), G, D, Dp, hp),
                    _pad_head_rows(g(i, "v"), G, V, Vp, hp)]
            if m.head_gate:
                rows.append(_pad2(g(i, "g"), H, hp))
            if m.bias:
                b = torch.cat([_pad_head_vec(g(i, "q_bias"), H, D, Dp), _pad_head_vec(g(i, "k_bias"), G, D, Dp),
                               _pad_head_vec(g(i, "v_bias"), G, V, Vp)])
                bias[: b.numel()] = b
            if m.qk_norm:
                w[f"{p}/mix/q_norm"] = _pad_head_vec(g(i, "q_norm"), 1, D, Dp)
                w[f"{p}/mix/k_norm"] = _pad_head_vec(g(i, "k_norm"), 1, D, Dp)
            mix = g(i, "talk").double() if m.head_mixing else torch.eye(H, dtype=torch.float64, device=device)
            if m.head_mixing:
                w[f"{p}/mix/heads"] = mix.float().contiguous()
            if m.distance_bias:
                # mixing is linear: the bias taken off before it is (mix @ slope) taken off after it
                w[f"{p}/mix/slope"] = (mix @ distance_slopes(H).to(device)).float().contiguous()
        else:
            rows = [_pad_head_rows(g(i, "q"), H, D, Dp, hp), _pad_head_rows(g(i, "k"), H, D, Dp, hp),
                    _pad_head_rows(g(i, "v"), H, V, Vp, hp), _pad_head_rows(g(i, "g"), H, V, Vp, hp),
                    _pad2(g(i, "i"), H, hp), _pad2(g(i, "f"), H, hp)]
            bias[m.main_cols: m.main_cols + H] = g(i, "i_bias").float()
            bias[m.main_cols + H: m.main_cols + 2 * H] = g(i, "f_bias").float()
            w[f"{p}/mix/norm"] = _pad_head_vec(g(i, "norm"), H, V, Vp)
        w[f"{p}/mix/in_proj"] = _pad2(torch.cat(rows), n_out, hp).to(dtype)
        w[f"{p}/mix/in_bias"] = bias
        w[f"{p}/mix/out_proj"] = _pad_head_cols(g(i, "o"), H, V, Vp, hp).to(dtype)
        if spec.mlp is not None:
            fp = pad_to(spec.mlp.ff, 8)
            w[f"{p}/norm2"] = f32(i, "norm2").reshape(1)
            w[f"{p}/mlp/up"] = _pad2(g(i, "up"), fp, hp).to(dtype)
            w[f"{p}/mlp/down"] = _pad2(g(i, "down"), hp, fp).to(dtype)
            if spec.mlp.bias:
                w[f"{p}/mlp/up_bias"] = _pad_head_vec(g(i, "up_bias"), 1, spec.mlp.ff, fp)
                w[f"{p}/mlp/down_bias"] = _pad_head_vec(g(i, "down_bias"), 1, cfg.hidden, hp)
            if spec.mlp.activation != "xielu":
                raise ValueError(f"layer {i}: unknown feed-forward activation '{spec.mlp.activation}'")
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
        self.max_tokens, self.max_logit_rows = T, max_logit_rows
        self.x = torch.zeros((T, cfg.hidden_p), dtype=f32, device=dev)      # residual stream
        self.xa = torch.zeros((T, cfg.hidden_p), dtype=dtype, device=dev)   # its copy in the activation type
        self.delta = torch.zeros((T, cfg.hidden_p), dtype=f32, device=dev)  # output of the running sublayer
        self.proj = torch.zeros((T, pad_to(max(m.main_cols for m in mixers), 64)), dtype=dtype, device=dev)
        self.gates = torch.zeros((T, pad_to(max(2, max(m.gate_cols for m in mixers)), 4)), dtype=f32, device=dev)
        self.mix = torch.zeros((T, pad_to(max(m.out_cols for m in mixers), 64)), dtype=dtype, device=dev)
        self.q = torch.zeros((T, max((m.heads * m.dim_p for m in attn), default=16)), dtype=dtype, device=dev)
        self.act = torch.zeros((T, pad_to(max((l.mlp.ff for l in cfg.layers if l.mlp is not None), default=8), 64)),
                               dtype=dtype, device=dev)
        # split-KV partials: (query token x split) rows of decode-sized steps
        self.split_rows = split_rows
        self.part_o = torch.empty(split_rows * max((m.out_cols for m in attn), default=0), dtype=f32, device=dev)
        self.part_ml = torch.empty(split_rows * max((m.heads for m in attn), default=0) * 2, dtype=f32, device=dev)
        self.logits = torch.zeros((max_logit_rows, cfg.vocab_p), dtype=f32, device=dev)
        self.head_in = torch.zeros((max_logit_rows, cfg.hidden_p), dtype=dtype, device=dev)
        self.next_ids = torch.zeros((max_logit_rows,), dtype=torch.int32, device=dev)


class LayeredModel:
    """Forward pass of a `LayeredConfig` over the ragged step batch; the interface is `models.hybrid.HybridModel`'s."""

    def __init__(self, cfg: LayeredConfig, weights: Dict[str, torch.Tensor], device, pdl: bool = False):
        self.cfg, self.w = cfg, weights
        self.device = torch.device(device)
        self._raw_ops = load_native(subset="layered")
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
        self.layer_hook = None          # called as hook(layer, x[:T]) after every layer (tests, debugging)
        self._attn_idx = {l: i for i, l in enumerate(cfg.attn_layers)}
        self._state_idx = {l: i for i, l in enumerate(cfg.state_layers)}
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
        self._gemm(ws.xa[:T], self.w[f"{p}/mix/in_proj"], self.w[f"{p}/mix/in_bias"], proj, gates, m.main_cols,
                   prefetch=self.w[f"{p}/mix/out_proj"])
        return proj, gates

    # ------------------------------------------------------------------ mixers
    def _attention(self, ws, b: StepBatch, kv, layer: int, T: int, p: str, m: AttentionMixer):
        ops, w = self.ops, self.w
        proj, gates = self._in_proj(ws, T, p, m)
        planes = kv.layers[self._attn_idx[layer]]
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

    def _matrix_memory(self, ws, b: StepBatch, states, layer: int, T: int, p: str, m: MatrixMemoryMixer,
                       write_state: bool):
        proj, gates = self._in_proj(ws, T, p, m)
        S, n, mx = states.layers[self._state_idx[layer]]
        H, Dp, Vp = m.heads, m.dim_p, m.vdim_p
        chunk_ws = None
        if (not self.f32 and self.prefill_kernels and b.max_seq_tokens >= PREFILL_MIN_TOKENS
                and self._raw_ops.mlstm_chunked_supported(Dp, Vp)):
            chunk_ws = self._grown("chunks", int(self._raw_ops.mlstm_chunked_workspace_bytes(T, b.n_seqs, H, Dp, Vp)))
            self.ops.count += 3
        out = ws.mix[:T, : H * Vp]
        self.ops.mlstm(proj, 0, H * Dp, 2 * H * Dp, H * (2 * Dp + Vp), gates, 0, H, m.vdim, m.dim ** -0.5, m.gate_cap,
                       self.cfg.rms_eps, self.w[f"{p}/mix/norm"], b.cu_seqlens, b.state_slot, S, n, mx, out, write_state,
                       chunk_ws, self.pdl, b.one_token_per_seq)
        return out

    # ------------------------------------------------------------------ forward
    def forward_hidden(self, ws: LayeredWorkspace, b: StepBatch, kv, states, write_state: bool = True) -> torch.Tensor:
        """Runs all layers; returns the final-normed hidden states [T, hidden (padded)]."""
        cfg, ops, w = self.cfg, self.ops, self.w
        T = b.n_tokens
        if T > ws.max_tokens:
            raise ValueError(f"step of {T} tokens exceeds the workspace ({ws.max_tokens})")
        x, xa, delta = ws.x[:T], ws.xa[:T], ws.delta[:T]
        ops.embed_rows32(b.ids, w["text/embed"], x, xa, self.pdl)
        for layer, spec in enumerate(cfg.layers):
            p, m = f"text/layers/{layer}", spec.mixer
            mix = (self._attention(ws, b, kv, layer, T, p, m) if m.kind == "attention" else
                   self._matrix_memory(ws, b, states, layer, T, p, m, write_state))
            last = w["text/final_norm"] if layer + 1 == cfg.n_layers else None
            nxt = w.get(f"text/layers/{layer + 1}/mix/in_proj", w["text/lm_head"])
            self._gemm(mix, w[f"{p}/mix/out_proj"], None, out32=delta, prefetch=w.get(f"{p}/mlp/up", nxt))
            ops.post_norm_rows(x, delta, xa, cfg.hidden, cfg.residual_alpha, cfg.rms_eps, w[f"{p}/norm1"],
                               last if spec.mlp is None else None, self.pdl)
            if spec.mlp is not None:
                up, down = w[f"{p}/mlp/up"], w[f"{p}/mlp/down"]
                act = ws.act[:T, : up.shape[0]]
                self._gemm(xa, up, w.get(f"{p}/mlp/up_bias"), act, act=ACT_XIELU, act_params=w[f"{p}/mlp/act"], prefetch=down)
                self._gemm(act, down, w.get(f"{p}/mlp/down_bias"), out32=delta, prefetch=nxt)
                ops.post_norm_rows(x, delta, xa, cfg.hidden, cfg.residual_alpha, cfg.rms_eps, w[f"{p}/norm2"], last, self.pdl)
            if self.layer_hook is not None:
                self.layer_hook(layer, x[:, : cfg.hidden])
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
