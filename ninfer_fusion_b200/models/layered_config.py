"""Description of decoders given as a list of layers (read by `models/layered.py`, which runs them).

A layer is a mixer (attention with shaped or plain scores, latent attention, matrix memory, gated linear memory, gated
linear recurrence, a selective state space, or two of them side by side) and an optional feed-forward (dense or a mixture of
experts); every size and constant is a field, and so is which mechanisms a mixer has.  The model's own fields say how a sublayer meets the residual stream (or streams), what
precedes a mixer, and which layers run several times.  Cache and state belong
to layer RUNS: a layer that runs twice has two of each.  No torch here: the package table and the host diagnostics read
these descriptions too."""
from __future__ import annotations

import math
from dataclasses import dataclass, replace
from typing import List, Optional, Tuple, Union


def pad_to(n: int, m: int) -> int:
    return (n + m - 1) // m * m


@dataclass(frozen=True)
class RotaryScaling:
    """Frequencies whose wavelength is beyond `original` / `low` positions are divided by `factor`, those within `original` /
    `high` stay, and in between the two are mixed linearly in `original` / wavelength."""
    factor: float
    low: float
    high: float
    original: float


@dataclass(frozen=True)
class Rotary:
    """The first `dims` values of a head, neighbours (2i, 2i + 1), turned by position * frequency i."""
    base: float
    dims: int
    scaling: Optional[RotaryScaling] = None

    def frequencies(self) -> List[float]:
        out = []
        for i in range(self.dims // 2):
            f, s = self.base ** (-2.0 * i / self.dims), self.scaling
            if s is not None:
                turns = s.original * f / (2.0 * math.pi)          # original / wavelength
                if turns < s.low:
                    f /= s.factor
                elif turns <= s.high:
                    keep = (turns - s.low) / (s.high - s.low)
                    f = (1.0 - keep) * f / s.factor + keep * f
            out.append(f)
        return out


@dataclass(frozen=True)
class AttentionMixer:
    heads: int
    kv_heads: int
    dim: int                      # query / key width per head
    vdim: int                     # value width per head
    scale: float
    softcap: float = 0.0          # 0: scores are not capped
    window: int = 0               # keys a query sees, itself included; 0: all of the past
    bias: bool = False            # q, k and v projections have biases
    qk_norm: bool = False         # RMS norm of every query and key head, weight of size dim shared by the heads
    distance_bias: bool = False   # slope_h * (i - j) taken off the scores, slope_h = 2^(-8 (h + 1) / heads)
    head_mixing: bool = False     # scores are mixed across heads by a [heads, heads] matrix before the softmax
    sink: float = 0.0             # added to the softmax denominator
    head_gate: bool = False       # sigmoid gate per head on the output
    chunk: int = 0                # keys of the query's own chunk of this many positions only (counted from 0); 0: no chunks
    head_sink: bool = False       # one learned score per head in the softmax denominator
    rotary: Optional[Rotary] = None   # after the norm, on q and k
    qk_unit: bool = False         # RMS norm of every query and key head without a weight
    sigmoid: bool = False         # weight sigmoid(score + a learned number per head) instead of a softmax; mixed instead of the scores
    log_bias: bool = False        # r1_h ln(1 + r2_h (i - j)) taken off the scores, two learned numbers per head (sigmoid weights)
    value_mix: bool = False       # v <- (1 - l) v + l v_first, l learned, v_first the values of the first such layer (which keeps its own)

    kind = "attention"

    @property
    def plain_scores(self) -> bool:
        """Scaled dot products and nothing else: no cap, bias, mix, gate or sigmoid."""
        return not (self.softcap or self.distance_bias or self.head_mixing or self.head_gate or self.sigmoid)

    @property
    def look_back(self) -> int:
        """Keys that a query can still look at, itself included; 0: all of the past."""
        return min(n for n in (self.window, self.chunk) if n) if self.window or self.chunk else 0

    @property
    def dim_p(self) -> int:
        return pad_to(self.dim, 16)

    @property
    def vdim_p(self) -> int:
        return pad_to(self.vdim, 16)

    @property
    def main_cols(self) -> int:
        """Columns of the fused input projection in the activation type: [q, k, v]."""
        return (self.heads + self.kv_heads) * self.dim_p + self.kv_heads * self.vdim_p

    @property
    def gate_cols(self) -> int:
        """Columns behind them that stay fp32: the head gate."""
        return self.heads if self.head_gate else 0

    @property
    def out_cols(self) -> int:
        return self.heads * self.vdim_p


@dataclass(frozen=True)
class MatrixMemoryMixer:
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    kind = "mlstm"

    @property
    def dim_p(self) -> int:
        return pad_to(self.dim, 16)

    @property
    def vdim_p(self) -> int:
        return pad_to(self.vdim, 16)

    @property
    def main_cols(self) -> int:
        """[q, k, v, output gate]"""
        return 2 * self.heads * (self.dim_p + self.vdim_p)

    @property
    def gate_cols(self) -> int:
        """[input gate, forget gate], fp32"""
        return 2 * self.heads

    @property
    def out_cols(self) -> int:
        return self.heads * self.vdim_p


@dataclass(frozen=True)
class LatentAttentionMixer:
    """Queries through a normed latent, or straight from the input (q_rank 0); keys and values out of one normed latent row
    per token, plus one rotated key part that all heads share (rot_dim 0: none).  The cache keeps one row per token:
    [latent, rotated part]."""
    heads: int
    dim: int                      # query / key width per head without rotation
    rot_dim: int                  # rotated query / key width per head
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot_base: float
    sink: bool = True             # one learned score per head in the softmax denominator
    window: int = 0               # keys a query sees, itself included; 0: all of the past

    kind = "latent_attention"
    kv_heads = 1

    @property
    def look_back(self) -> int:
        return self.window

    @property
    def dim_p(self) -> int:
        return pad_to(self.dim, 16)

    @property
    def rot_p(self) -> int:
        return pad_to(self.rot_dim, 16)

    @property
    def vdim_p(self) -> int:
        return pad_to(self.vdim, 16)

    @property
    def q_rank_p(self) -> int:
        return pad_to(self.q_rank, 16)

    @property
    def kv_rank_p(self) -> int:
        return pad_to(self.kv_rank, 16)

    @property
    def row_cols(self) -> int:
        """Width of a cached row."""
        return self.kv_rank_p + self.rot_p

    @property
    def main_cols(self) -> int:
        """Columns of the fused input projection: [query latent or queries, key / value latent, rotated key part]."""
        return (self.q_rank_p if self.q_rank else self.q_cols) + self.row_cols

    gate_cols = 0

    @property
    def q_cols(self) -> int:
        """Query columns, head by head [unrotated, rotated]."""
        return self.heads * (self.dim_p + self.rot_p)

    @property
    def out_cols(self) -> int:
        return self.heads * self.vdim_p


@dataclass(frozen=True)
class GatedMemoryMixer:
    """Linear attention with a forget gate per head and channel, f = lower + (1 - lower) sigmoid(raw), whose complement
    takes the place of the key (HGRN2)."""
    heads: int
    dim: int
    vdim: int

    kind = "hgrn2"

    @property
    def dim_p(self) -> int:
        return pad_to(self.dim, 16)

    @property
    def vdim_p(self) -> int:
        return pad_to(self.vdim, 16)

    @property
    def main_cols(self) -> int:
        """[q, v]"""
        return self.heads * (self.dim_p + self.vdim_p)

    @property
    def gate_cols(self) -> int:
        """Raw forget gates, fp32."""
        return self.heads * self.dim_p

    @property
    def out_cols(self) -> int:
        return self.heads * self.vdim_p


@dataclass(frozen=True)
class GatedRecurrenceMixer:
    """Griffin's recurrent block: a causal convolution in front of a diagonal linear recurrence whose decay and input gates
    are block-diagonal maps of its input, times a GELU branch."""
    width: int
    blocks: int                   # equal parts of the width, each with gate matrices of its own
    taps: int                     # of the convolution

    kind = "rglru"

    @property
    def vdim(self) -> int:
        return self.width // self.blocks

    @property
    def vdim_p(self) -> int:
        return pad_to(self.vdim, 16)

    @property
    def heads(self) -> int:
        return self.blocks

    @property
    def main_cols(self) -> int:
        """[GELU branch, recurrent branch]"""
        return 2 * self.out_cols

    gate_cols = 0

    @property
    def out_cols(self) -> int:
        return self.blocks * self.vdim_p


@dataclass(frozen=True)
class StateSpaceMixer:
    """Selective state space with one decay per head (Mamba-2): a causal convolution with SiLU in front of
    S <- exp(-rate dt) S + dt x B^T, y = S C + skip x; then y silu(z), normed in equal parts."""
    heads: int
    vdim: int                     # channels per head
    state: int                    # state columns per channel
    groups: int                   # of heads that share B and C
    taps: int                     # of the convolution
    norm_groups: int = 1

    kind = "ssd"

    @property
    def vdim_p(self) -> int:
        return pad_to(self.vdim, 16)

    @property
    def state_p(self) -> int:
        return pad_to(self.state, 16)

    @property
    def conv_cols(self) -> int:
        """Convolved channels: [x, B, C]"""
        return self.out_cols + 2 * self.groups * self.state_p

    @property
    def main_cols(self) -> int:
        """[z, x, B, C]"""
        return self.out_cols + self.conv_cols

    @property
    def gate_cols(self) -> int:
        """Raw step sizes, fp32."""
        return self.heads

    @property
    def out_cols(self) -> int:
        return self.heads * self.vdim_p


@dataclass(frozen=True)
class ParallelMixer:
    """Attention and a state space side by side on the same input; the layer's output is the mean of the two, each normed by
    itself first.  One fused input projection: the left columns, the right ones, then the right gates."""
    left: AttentionMixer
    right: StateSpaceMixer

    kind = "parallel"

    @property
    def main_cols(self) -> int:
        return self.left.main_cols + self.right.main_cols

    @property
    def gate_cols(self) -> int:
        return self.right.gate_cols

    @property
    def out_cols(self) -> int:
        return self.left.out_cols + self.right.out_cols


@dataclass(frozen=True)
class DenseMlp:
    ff: int
    activation: str = "xielu"     # xielu (two learned numbers per layer) | relu2 (square of relu)
    bias: bool = False

    kind = "dense"


@dataclass(frozen=True)
class GatedUnit:
    """down( g sigmoid(slope g) (u + shift) ) with g = min(gate h, limit), u = clamp(up h, +- limit); limit 0: no bounds.
    An expert, or a layer's dense feed-forward."""
    ff: int
    limit: float = 0.0
    slope: float = 1.0
    shift: float = 0.0

    kind = "glu"
    activation = "swiglu"
    bias = False

    @property
    def ff_p(self) -> int:
        return pad_to(self.ff, 64)

    def params(self, h: int) -> int:
        return 3 * h * self.ff


@dataclass(frozen=True)
class ExpertMlp:
    """Mixture of experts: scores are the softmax over all router outputs or the sigmoid of each; the `top` largest scores
    (with a learned correction added for the choice only) times `scale`, or divided by their sum, weigh the chosen experts.
    With `groups` (equal runs of neighbours) only experts of the `keep` best groups can be chosen, a group's score being the
    sum of its two largest corrected scores.  The last `identity` outputs stand for the input itself.  A shared expert runs for
    every token, under a sigmoid gate or as it is."""
    experts: int
    top: int
    expert: GatedUnit
    identity: int = 0
    scale: float = 1.0
    shared: Optional[GatedUnit] = None
    shared_gate: bool = True
    sigmoid: bool = False
    renormalise: bool = False
    groups: int = 0
    keep: int = 0

    kind = "moe"

    @property
    def choices(self) -> int:
        return self.experts + self.identity

    @property
    def router_cols(self) -> int:
        """Router outputs and the shared expert's gate."""
        return pad_to(self.choices + (1 if self.shared and self.shared_gate else 0), 8)

    @property
    def slots(self) -> int:
        """Most experts with weights of their own that one token uses."""
        return min(self.top, self.experts)


@dataclass(frozen=True)
class LayerSpec:
    mixer: Union[AttentionMixer, LatentAttentionMixer, MatrixMemoryMixer, GatedMemoryMixer, GatedRecurrenceMixer, StateSpaceMixer,
                 ParallelMixer]
    mlp: Optional[Union[DenseMlp, GatedUnit, ExpertMlp]] = None


@dataclass(frozen=True)
class LoopSpec:
    """Layers start .. stop - 1 run `times` times in a row.  Every pass opens with x <- in_proj [x; x0] + step[pass], x0
    the embedding output."""
    start: int
    stop: int
    times: int


ATTENTION_KINDS = ("attention", "latent_attention")


def attention_part(m):
    """The mixer that owns cache rows, or None."""
    return m.left if m.kind == "parallel" else (m if m.kind in ATTENTION_KINDS else None)


def memory_part(m):
    """The mixer that owns recurrent state, or None."""
    return m.right if m.kind == "parallel" else (None if m.kind in ATTENTION_KINDS else m)


def mixer_parts(m) -> tuple:
    return (m.left, m.right) if m.kind == "parallel" else (m,)


@dataclass(frozen=True)
class LayeredConfig:
    name: str
    hidden: int
    vocab: int
    layers: Tuple[LayerSpec, ...]
    rms_eps: float
    residual_alpha: float         # post_sum: x <- norm(residual_alpha * x + f(x))
    max_context: int = 131072
    architecture: str = ""        # name of the design that maps checkpoints onto this description
    # post_sum | sandwich: x <- x + residual_mult * norm(f(norm(x))) | streams: `streams` copies of the embedding output; a
    # sublayer reads a weighted sum of them, u = sum_s in[s] x_s, and x_t <- sum_s mix[s, t] x_s + out[t] f(norm(u)) |
    # branch: x <- x + norm(f(x))
    residual: str = "post_sum"
    residual_mult: float = 1.0    # sandwich
    norm_groups: int = 1          # sandwich: equal parts of a row that are normed by themselves, one weight per column
    conv_taps: int = 0            # h <- h + causal convolution of h before every mixer, this many taps (0: none)
    embed_scale: float = 1.0
    tie_head: bool = False        # logits from the embedding table (without its scale)
    loop: Optional[LoopSpec] = None
    streams: int = 1
    norm_offset: float = 0.0      # added to the stored weights of the sublayers' and the final norm
    logit_softcap: float = 0.0    # logits <- cap tanh(logits / cap); 0: as they are
    logit_scale: float = 1.0
    learned_positions: int = 0    # rows of a table of position vectors that are added to the embedding: as many positions a
                                  # sequence can have; 0: no table

    moe = None
    mtp_layers = 0

    # ---- what the engine, the cache and the capacity arithmetic ask of a configuration
    @property
    def n_layers(self) -> int:
        return len(self.layers)

    @property
    def hidden_p(self) -> int:
        return pad_to(self.hidden, 8)

    @property
    def vocab_p(self) -> int:
        return pad_to(self.vocab, 8)

    @property
    def runs(self) -> List[Tuple[int, int]]:
        """Layer runs in order: (layer, pass it opens or -1)."""
        lp, n = self.loop, len(self.layers)
        if lp is None:
            return [(i, -1) for i in range(n)]
        looped = [(i, t if i == lp.start else -1) for t in range(lp.times) for i in range(lp.start, lp.stop)]
        return [(i, -1) for i in range(lp.start)] + looped + [(i, -1) for i in range(lp.stop, n)]

    def mixer_of(self, run: int):
        return self.layers[self.runs[run][0]].mixer

    @property
    def attn_layers(self) -> List[int]:
        """Layer runs that have a cache (without a loop a run is a layer)."""
        return [r for r, (i, _) in enumerate(self.runs) if attention_part(self.layers[i].mixer) is not None]

    @property
    def state_layers(self) -> List[int]:
        """Layer runs that have recurrent state: a memory, or the inputs that a convolution looks back on."""
        return [r for r, (i, _) in enumerate(self.runs)
                if self.conv_taps > 1 or memory_part(self.layers[i].mixer) is not None]

    def attention_of(self, run: int):
        return attention_part(self.mixer_of(run))

    @property
    def value_runs(self) -> List[int]:
        """Layer runs whose values are mixed with those of the first of them."""
        return [r for r in self.attn_layers if getattr(self.attention_of(r), "value_mix", False)]

    @property
    def position_limit(self) -> int:
        """Most positions that a sequence can have; 0: no limit of the model's own."""
        return self.learned_positions

    @property
    def n_kv_heads(self) -> int:
        return max((self.attention_of(r).kv_heads for r in self.attn_layers), default=0)

    @property
    def head_dim(self) -> int:
        return max((self.attention_of(r).dim for r in self.attn_layers), default=0)

    @property
    def kv_geometry(self) -> List[Tuple[int, int, int]]:
        """Per attention run: kv heads, key width, value width of a cache row (padded).  A latent row has no separate
        values."""
        ms = [self.attention_of(r) for r in self.attn_layers]
        return [(1, m.row_cols, 0) if m.kind == "latent_attention" else (m.kv_heads, m.dim_p, m.vdim_p) for m in ms]

    @property
    def cache_window(self) -> int:
        """Keys that any layer still looks back on: the widest window, 0 when some layer sees all of the past."""
        w = [self.attention_of(r).look_back for r in self.attn_layers]
        return max(w) if w and min(w) > 0 else 0

    def state_shapes(self) -> List[List[tuple]]:
        """Per run in `state_layers`: shapes (without the slot) of its fp32 state arrays: the convolution's last inputs
        (oldest first) when there are any, then the memory: S, n, m (matrix memory), S (gated memory), or the inputs of
        the last `taps` positions (row position mod taps) and S (gated recurrence, state space)."""
        out = []
        for r in self.state_layers:
            m, arrays = memory_part(self.mixer_of(r)), []
            if self.conv_taps > 1:
                arrays.append((self.conv_taps - 1, self.hidden_p))
            if m is None:
                pass
            elif m.kind == "rglru":
                arrays += [(m.taps, m.out_cols), (m.out_cols,)]
            elif m.kind == "ssd":
                arrays += [(m.taps, m.conv_cols), (m.heads, m.vdim_p, m.state_p)]
            else:
                arrays.append((m.heads, m.dim_p, m.vdim_p))
            if m is not None and m.kind == "mlstm":
                arrays += [(m.heads, m.dim_p), (m.heads,)]
            out.append(arrays)
        return out

    def state_bytes_per_slot(self) -> int:
        return sum(4 * math.prod(shape) for layer in self.state_shapes() for shape in layer)

    def param_count(self) -> int:
        h, wide = self.hidden, self.residual == "sandwich"
        norm = 1 if self.residual == "post_sum" else h                      # weights of one norm
        hyper = self.streams * (self.streams + 2) if self.residual == "streams" else 0
        n = (1 if self.tie_head else 2) * self.vocab * h + norm + self.learned_positions * h
        if self.loop is not None:
            n += 2 * h * h + self.loop.times * h
        for l in self.layers:
            n += (2 if wide else 1) * norm + hyper + self.conv_taps * h + sum(self._mixer_params(m) for m in mixer_parts(l.mixer))
            n += 2 * h if l.mixer.kind == "parallel" else 0
            if l.mlp is not None:
                n += (2 * norm if wide else norm) + hyper
            if l.mlp is not None and l.mlp.kind == "moe":
                n += l.mlp.choices * (h + 1) + l.mlp.experts * l.mlp.expert.params(h)
                n += l.mlp.shared.params(h) + (h if l.mlp.shared_gate else 0) if l.mlp.shared else 0
            elif l.mlp is not None and l.mlp.kind == "glu":
                n += l.mlp.params(h)
            elif l.mlp is not None:
                n += 2 * h * l.mlp.ff
                n += 2 if l.mlp.activation == "xielu" else (l.mlp.ff + h if l.mlp.bias else 0)
        return n

    def _mixer_params(self, m) -> int:
        h = self.hidden
        n = h * m.heads * m.vdim
        if m.kind == "attention":
            cols = (m.heads + m.kv_heads) * m.dim + m.kv_heads * m.vdim
            n += (cols + (m.heads if m.head_gate else 0)) * h
            n += (m.heads * m.heads if m.head_mixing else 0) + (2 * m.dim if m.qk_norm else 0) + (1 if m.value_mix else 0)
            n += m.heads * (int(m.head_sink) + int(m.sigmoid) + 2 * int(m.log_bias))
        elif m.kind == "latent_attention":
            n += (m.q_rank + m.kv_rank + m.rot_dim) * h + m.q_rank + m.kv_rank + (m.heads if m.sink else 0)
            n += m.heads * (m.dim + m.rot_dim) * (m.q_rank or h) + m.heads * (m.dim + m.vdim) * m.kv_rank
        elif m.kind == "rglru":
            n += 2 * m.width * (h + 1) + m.width * (m.taps + 1) + 2 * m.width * (m.vdim + 1) + m.width
        elif m.kind == "ssd":
            inner, conv = m.heads * m.vdim, m.heads * m.vdim + 2 * m.groups * m.state
            n += (inner + conv + m.heads) * h + conv * (m.taps + 1) + 3 * m.heads + inner
        elif m.kind == "hgrn2":
            n += (2 * m.heads * m.dim + m.heads * m.vdim) * h + 2 * m.heads * m.dim + m.vdim
        else:
            n += (2 * m.heads * (m.dim + m.vdim) + 2 * m.heads) * h + m.heads * m.vdim + 2 * m.heads
        return n

    def shrink(self, n_layers: int) -> "LayeredConfig":
        """The first `n_layers` layers; a loop keeps what is left of it."""
        lp = self.loop
        if lp is not None:
            lp = None if lp.start >= n_layers else replace(lp, stop=min(lp.stop, n_layers))
        return replace(self, name=f"{self.name}-{n_layers}L", layers=self.layers[:n_layers], loop=lp)
