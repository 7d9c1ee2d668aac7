"""Kuzanex: how its config.json and checkpoint tensors map onto the layer-list decoder (`models/layered.py`).

The design fixes: soft-capped scores with a per-head distance bias and a learned mix across heads, a sink of score 0,
one output gate per head, query / key norm and q / k / v biases in its attention; biases and xIELU in its feed-forward;
a norm with one gain after every residual sum.  Sizes, windows, scales, caps and the order of layers come from the
configuration."""
from __future__ import annotations

from typing import Dict, Iterator, Tuple

from .layered_config import AttentionMixer, DenseMlp, LayeredConfig, LayerSpec, MatrixMemoryMixer

ARCHITECTURE = "Kuzanex"
SINK = 1.0


def _attention(c: dict) -> AttentionMixer:
    m = AttentionMixer(heads=int(c["heads"]), kv_heads=int(c["kv_heads"]), dim=int(c["dim"]), vdim=int(c["vdim"]),
                       scale=float(c["scale"]), softcap=float(c["softcap"]), window=int(c["mask"]["size"]), bias=True,
                       qk_norm=True, distance_bias=True, head_mixing=True, sink=SINK, head_gate=True)
    if m.heads % m.kv_heads or m.window < 1:
        raise ValueError("attention: heads must be a multiple of kv_heads and the window at least 1")
    return m


def _mlstm(c: dict) -> MatrixMemoryMixer:
    return MatrixMemoryMixer(heads=int(c["heads"]), dim=int(c["dim"]), vdim=int(c["vdim"]), gate_cap=float(c["gate_cap"]))


_MIXERS = {"attention": _attention, "mlstm": _mlstm}


def parse_config(c: dict, name: str = "kuzanex") -> LayeredConfig:
    layers = []
    for i, l in enumerate(c["layers"]):
        if l["type"] not in _MIXERS:
            raise ValueError(f"layer {i}: unknown mixer '{l['type']}'")
        mlp = l.get("mlp")
        if mlp is not None:
            if mlp.get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward '{mlp['kind']}'")
            mlp = DenseMlp(int(mlp["ff"]), "xielu", bias=True)
        layers.append(LayerSpec(_MIXERS[l["type"]](l["mixer"]), mlp))
    return LayeredConfig(name=name, hidden=int(c["width"]), vocab=int(c["vocab"]), layers=tuple(layers),
                         rms_eps=float(c["norm"]["eps"]), residual_alpha=float(c["postln_alpha"]), architecture=ARCHITECTURE)


def config_dict(cfg: LayeredConfig) -> dict:
    """The config.json of a configuration of this design."""
    layers = []
    for l in cfg.layers:
        m = l.mixer
        if m.kind == "attention":
            mixer = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale,
                     "softcap": m.softcap, "mask": {"size": m.window}}
        else:
            mixer = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "gate_cap": m.gate_cap}
        layers.append({"type": m.kind, "mixer": mixer, "mlp": None if l.mlp is None else {"kind": "dense", "ff": l.mlp.ff}})
    return {"architecture": ARCHITECTURE, "width": cfg.hidden, "vocab": cfg.vocab, "norm": {"eps": cfg.rms_eps},
            "postln_alpha": cfg.residual_alpha, "layers": layers}


# role (layered.pack_weights) -> checkpoint name
_MODEL = {"embed": "embed", "head": "head", "final_norm": "final.norm"}
_LAYER = {"norm1": "norm1", "norm2": "norm2"}
_LAYER.update({r: f"mix.{r}" for r in ("q", "k", "v", "o", "g", "i", "f", "norm", "talk")})
_LAYER.update({"q_bias": "mix.q.b", "k_bias": "mix.k.b", "v_bias": "mix.v.b", "q_norm": "mix.q.norm", "k_norm": "mix.k.norm",
               "i_bias": "mix.i.b", "f_bias": "mix.f.b", "up": "mlp.up", "up_bias": "mlp.up.b", "down": "mlp.down",
               "down_bias": "mlp.down.b", "act": "mlp.act"})


def tensor_name(layer: int, role: str) -> str:
    return _MODEL[role] if layer < 0 else f"l{layer}.{_LAYER[role]}"


def tensor_shapes(cfg: LayeredConfig) -> Iterator[Tuple[str, tuple]]:
    """Names and shapes of a checkpoint of this configuration."""
    h = cfg.hidden
    yield "embed", (cfg.vocab, h)
    for i, l in enumerate(cfg.layers):
        m, H = l.mixer, l.mixer.heads
        roles: Dict[str, tuple] = {"norm1": (), "q": (H * m.dim, h), "o": (h, H * m.vdim)}
        if m.kind == "attention":
            G = m.kv_heads
            roles.update(k=(G * m.dim, h), v=(G * m.vdim, h), q_bias=(H * m.dim,), k_bias=(G * m.dim,), v_bias=(G * m.vdim,),
                         q_norm=(m.dim,), k_norm=(m.dim,), talk=(H, H), g=(H, h))
        else:
            roles.update(k=(H * m.dim, h), v=(H * m.vdim, h), g=(H * m.vdim, h), norm=(H * m.vdim,), i=(H, h), f=(H, h),
                         i_bias=(H,), f_bias=(H,))
        if l.mlp is not None:
            ff = l.mlp.ff
            roles.update(norm2=(), up=(ff, h), up_bias=(ff,), down=(h, ff), down_bias=(h,), act=(2,))
        for role, shape in roles.items():
            yield tensor_name(i, role), shape
    yield "final.norm", ()
    yield "head", (cfg.vocab, h)


def check_tensors(cfg: LayeredConfig, shape_of) -> None:
    """Every tensor of the configuration is there in its shape; `shape_of(name)` returns None for a missing one."""
    from .layered import check_tensor_shapes
    check_tensor_shapes(tensor_shapes(cfg), shape_of)


def pack(cfg: LayeredConfig, tensors, dtype, device="cpu") -> dict:
    """Packed weights from checkpoint tensors (`tensors(name)`)."""
    from .layered import pack_weights
    return pack_weights(cfg, lambda layer, role: tensors(tensor_name(layer, role)), dtype, device)


def random_tensors(cfg: LayeredConfig, seed: int = 0, std: float = 0.0, device="cpu") -> dict:
    """Random bf16 checkpoint tensors (matrices of deviation `std`, default 1 / sqrt(columns))."""
    import torch
    gen = torch.Generator(device=device)
    gen.manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg):
        t = torch.empty(shape, dtype=torch.float32, device=device)
        if name.endswith("norm") or name.endswith(("norm1", "norm2")):
            t.normal_(1.0, 0.1, generator=gen)
        elif name.endswith("mix.talk"):
            t.normal_(0.0, 0.15, generator=gen).add_(torch.eye(shape[0], device=device))
        elif name.endswith("mix.f.b"):
            t.normal_(3.0, 1.0, generator=gen)       # long memory
        elif name.endswith((".b", "mlp.act")):
            t.normal_(0.0, 0.1, generator=gen)
        else:
            t.normal_(0.0, std or (0.5 if name == "embed" else shape[-1] ** -0.5), generator=gen)
        out[name] = t.to(torch.bfloat16)
    return out


def _design(name: str, hidden: int, vocab: int, pattern: str, attn: dict, mem: dict, ff: int, max_context: int = 131072) -> LayeredConfig:
    """pattern: one letter per layer, 'm' matrix memory, 'a' attention."""
    full = {"m": LayerSpec(_mlstm(mem), DenseMlp(ff, "xielu", True)), "a": LayerSpec(_attention(attn), DenseMlp(ff, "xielu", True))}
    return LayeredConfig(name=name, hidden=hidden, vocab=vocab, layers=tuple(full[c] for c in pattern), rms_eps=1e-6,
                         residual_alpha=2.0, max_context=max_context, architecture=ARCHITECTURE)


# Geometries for random-init runs: a small one, and two whose layers have the widths of real models.
TINY = _design("kuzanex-tiny", 160, 1024, "maam", dict(heads=6, kv_heads=2, dim=32, vdim=48, scale=0.2, softcap=30.0, mask={"size": 24}),
               dict(heads=3, dim=32, vdim=64, gate_cap=10.0), 352, 4096)
K1B = _design("kuzanex-1b", 2048, 65536, "mmma" * 4, dict(heads=16, kv_heads=4, dim=128, vdim=128, scale=0.0884, softcap=50.0, mask={"size": 1024}),
              dict(heads=4, dim=256, vdim=512, gate_cap=15.0), 8192)
K7B = _design("kuzanex-7b", 4096, 131072, "mmma" * 8, dict(heads=32, kv_heads=8, dim=128, vdim=128, scale=0.0884, softcap=50.0, mask={"size": 2048}),
              dict(heads=8, dim=256, vdim=512, gate_cap=15.0), 12288)
CONFIGS = {c.name: c for c in (TINY, K1B, K7B)}
