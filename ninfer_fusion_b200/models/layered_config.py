"""Description of decoders given as a list of layers (read by `models/layered.py`, which runs them).

A layer is a mixer (head-mixing attention or matrix memory) and an optional feed-forward; every size and constant is a
field, and so is which mechanisms a mixer has.  No torch here: the package table and the host diagnostics read these
descriptions too."""
from __future__ import annotations

import math
from dataclasses import dataclass, replace
from typing import List, Optional, Tuple, Union


def pad_to(n: int, m: int) -> int:
    return (n + m - 1) // m * m


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

    kind = "attention"

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
class DenseMlp:
    ff: int
    activation: str = "xielu"     # two learned numbers per layer
    bias: bool = False


@dataclass(frozen=True)
class LayerSpec:
    mixer: Union[AttentionMixer, MatrixMemoryMixer]
    mlp: Optional[DenseMlp] = None


@dataclass(frozen=True)
class LayeredConfig:
    name: str
    hidden: int
    vocab: int
    layers: Tuple[LayerSpec, ...]
    rms_eps: float
    residual_alpha: float         # x <- norm(residual_alpha * x + f(x))
    max_context: int = 131072
    architecture: str = ""        # name of the design that maps checkpoints onto this description

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
    def attn_layers(self) -> List[int]:
        return [i for i, l in enumerate(self.layers) if l.mixer.kind == "attention"]

    @property
    def state_layers(self) -> List[int]:
        return [i for i, l in enumerate(self.layers) if l.mixer.kind == "mlstm"]

    @property
    def n_kv_heads(self) -> int:
        return max((self.layers[i].mixer.kv_heads for i in self.attn_layers), default=0)

    @property
    def head_dim(self) -> int:
        return max((self.layers[i].mixer.dim for i in self.attn_layers), default=0)

    @property
    def kv_geometry(self) -> List[Tuple[int, int, int]]:
        """Per attention layer: kv heads, key width, value width of a cache row (padded)."""
        return [(m.kv_heads, m.dim_p, m.vdim_p) for m in (self.layers[i].mixer for i in self.attn_layers)]

    @property
    def cache_window(self) -> int:
        """Keys that any layer still looks back on: the widest window, 0 when some layer sees all of the past."""
        w = [self.layers[i].mixer.window for i in self.attn_layers]
        return max(w) if w and min(w) > 0 else 0

    def state_shapes(self) -> List[List[tuple]]:
        """Per recurrent layer: shapes (without the slot) of its fp32 state arrays: S, n, m."""
        out = []
        for i in self.state_layers:
            m = self.layers[i].mixer
            out.append([(m.heads, m.dim_p, m.vdim_p), (m.heads, m.dim_p), (m.heads,)])
        return out

    def state_bytes_per_slot(self) -> int:
        return sum(4 * math.prod(shape) for layer in self.state_shapes() for shape in layer)

    def param_count(self) -> int:
        n = 2 * self.vocab * self.hidden + 1
        for l in self.layers:
            m = l.mixer
            if m.kind == "attention":
                rows = (m.heads + m.kv_heads) * m.dim + m.kv_heads * m.vdim + (m.heads if m.head_gate else 0)
                n += rows * self.hidden + self.hidden * m.heads * m.vdim + 1
                n += (m.heads * m.heads if m.head_mixing else 0) + (2 * m.dim if m.qk_norm else 0)
            else:
                n += (2 * m.heads * (m.dim + m.vdim) + 2 * m.heads) * self.hidden + self.hidden * m.heads * m.vdim
                n += m.heads * m.vdim + 2 * m.heads + 1
            if l.mlp is not None:
                n += 2 * self.hidden * l.mlp.ff + 3
        return n

    def shrink(self, n_layers: int) -> "LayeredConfig":
        return replace(self, name=f"{self.name}-{n_layers}L", layers=self.layers[:n_layers])
