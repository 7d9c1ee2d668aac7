"""Tuzupel: how its config.json and checkpoint tensors map onto the layer-list decoder (`models/layered.py`).

The design fixes: several residual streams that every sublayer reads from and mixes, one norm in front of it with weights
stored around zero, chunked attention with query / key norm, interleaved rotation and a learned sink per head, latent
attention without positions in a sliding window, gated linear recurrences, and experts with bounded gated units beside
identity experts and a gated shared one.  Sizes, constants and the order of layers come from the configuration."""
from __future__ import annotations

from typing import Dict, Iterator, Optional, Tuple

from .layered_config import (AttentionMixer, ExpertMlp, GatedRecurrenceMixer, GatedUnit, LatentAttentionMixer, LayeredConfig,
                             LayerSpec, Rotary, RotaryScaling)

ARCHITECTURE = "Tuzupel"
SLOPE, SHIFT = 1.702, 1.0        # of the experts' gated units
NORM_OFFSET = 1.0


def _mask(c: dict) -> int:
    if c.get("mask") is None:
        return 0
    size = int(c["mask"]["size"])
    if size < 1:
        raise ValueError("the mask must leave a query its own key")
    return size


def _rotary(c: Optional[dict]) -> Optional[Rotary]:
    if c is None or int(c["dims"]) == 0:
        return None
    s = c.get("scaling")
    scaling = None if s is None else RotaryScaling(*(float(s[k]) for k in ("factor", "low", "high", "original")))
    return Rotary(float(c["base"]), int(c["dims"]), scaling)


def _attention(c: dict) -> AttentionMixer:
    m = AttentionMixer(heads=int(c["heads"]), kv_heads=int(c["kv_heads"]), dim=int(c["dim"]), vdim=int(c["vdim"]),
                       scale=float(c["scale"]), qk_norm=True, chunk=_mask(c), head_sink=True, rotary=_rotary(c.get("rot")))
    if m.heads % m.kv_heads:
        raise ValueError("attention: heads must be a multiple of kv_heads")
    if m.rotary is not None and (m.rotary.dims % 2 or m.rotary.dims > m.dim):
        raise ValueError("attention: the rotated part must be of even width within the head")
    return m


def _latent(c: dict) -> LatentAttentionMixer:
    return LatentAttentionMixer(heads=int(c["heads"]), dim=int(c["dim"]), rot_dim=0, vdim=int(c["vdim"]), q_rank=0,
                                kv_rank=int(c["kv_rank"]), scale=float(c["scale"]), rot_base=0.0, sink=False, window=_mask(c))


def _rglru(c: dict) -> GatedRecurrenceMixer:
    m = GatedRecurrenceMixer(width=int(c["width"]), blocks=int(c["blocks"]), taps=int(c["conv"]))
    if m.blocks < 1 or m.width % m.blocks:
        raise ValueError(f"rglru: a width of {m.width} has no {m.blocks} equal parts")
    if m.taps < 1:
        raise ValueError("rglru: the convolution needs at least one tap")
    return m


_MIXERS = {"attention": _attention, "latent_attention": _latent, "rglru": _rglru}


def _unit(c: Optional[dict]) -> Optional[GatedUnit]:
    return None if c is None else GatedUnit(int(c["ff"]), float(c["limit"]), SLOPE, SHIFT)


def _experts(c: dict) -> ExpertMlp:
    r = c["router"]
    m = ExpertMlp(experts=int(r["experts"]), top=int(r["top"]), expert=_unit(c["expert"]), identity=int(r.get("identity", 0)),
                  scale=float(r["scale"]), shared=_unit(c.get("shared")))
    if m.experts < 1 or not 1 <= m.top <= m.choices:
        raise ValueError(f"router: {m.top} of {m.choices} experts")
    return m


def parse_config(c: dict, name: str = "tuzupel") -> LayeredConfig:
    layers = []
    for i, l in enumerate(c["layers"]):
        if l["type"] not in _MIXERS:
            raise ValueError(f"layer {i}: unknown mixer '{l['type']}'")
        mlp = l.get("mlp")
        if mlp is not None:
            if mlp.get("kind", "moe") != "moe":
                raise ValueError(f"layer {i}: unknown feed-forward '{mlp['kind']}'")
            mlp = _experts(mlp)
        layers.append(LayerSpec(_MIXERS[l["type"]](l["mixer"]), mlp))
    cfg = LayeredConfig(name=name, hidden=int(c["width"]), vocab=int(c["vocab"]), layers=tuple(layers),
                        rms_eps=float(c["norm"]["eps"]), residual_alpha=1.0, architecture=ARCHITECTURE, residual="streams",
                        streams=int(c["streams"]), norm_offset=NORM_OFFSET, logit_softcap=float(c.get("logit_softcap") or 0.0))
    if cfg.streams < 1:
        raise ValueError("the residual needs at least one stream")
    return cfg


def config_dict(cfg: LayeredConfig) -> dict:
    """The config.json of a configuration of this design."""
    layers = []
    for l in cfg.layers:
        m, f = l.mixer, l.mlp
        if m.kind == "rglru":
            mixer = {"width": m.width, "blocks": m.blocks, "conv": m.taps}
        else:
            mixer = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale}
            if m.look_back:
                mixer["mask"] = {"size": m.look_back}
        if m.kind == "latent_attention":
            mixer["kv_rank"] = m.kv_rank
        if m.kind == "attention":
            mixer["kv_heads"] = m.kv_heads
            if m.rotary is not None:
                mixer["rot"] = {"base": m.rotary.base, "dims": m.rotary.dims}
                if m.rotary.scaling is not None:
                    mixer["rot"]["scaling"] = dict(vars(m.rotary.scaling))
        mlp = None
        if f is not None:
            mlp = {"kind": "moe", "expert": {"ff": f.expert.ff, "limit": f.expert.limit},
                   "router": {"experts": f.experts, "identity": f.identity, "top": f.top, "scale": f.scale}}
            if f.shared is not None:
                mlp["shared"] = {"ff": f.shared.ff, "limit": f.shared.limit}
        layers.append({"type": m.kind, "mixer": mixer, "mlp": mlp})
    out = {"architecture": ARCHITECTURE, "width": cfg.hidden, "vocab": cfg.vocab, "norm": {"eps": cfg.rms_eps},
           "streams": cfg.streams, "layers": layers}
    if cfg.logit_softcap:
        out["logit_softcap"] = cfg.logit_softcap
    return out


# role (layered.pack_weights) -> checkpoint name; the experts' units are "e<number>.gate" and so on
_MODEL = {"embed": "embed", "head": "head", "final_norm": "final.norm"}
_LAYER = {"norm1": "norm1", "norm2": "norm2"}
_LAYER.update({f"hc{q}_{r}": f"hc{q}.{r}" for q in (1, 2) for r in ("in", "out", "mix")})
_LAYER.update({r: f"mix.{r}" for r in ("q", "k", "v", "o", "sink", "dkv", "uk", "uv", "y", "x", "conv", "ra", "ri", "lam")})
_LAYER.update({"q_norm": "mix.q.norm", "k_norm": "mix.k.norm", "dkv_norm": "mix.dkv.norm"})
_LAYER.update({f"{r}_bias": f"mix.{r}.b" for r in ("y", "x", "conv", "ra", "ri")})
_LAYER.update({"router": "mlp.router", "correction": "mlp.correction", "shared_gate": "mlp.shared.sg"})


def tensor_name(layer: int, role: str) -> str:
    if layer < 0:
        return _MODEL[role]
    return f"l{layer}.{_LAYER[role]}" if role in _LAYER else f"l{layer}.mlp.{role}"


def tensor_shapes(cfg: LayeredConfig) -> Iterator[Tuple[str, tuple]]:
    """Names and shapes of a checkpoint of this configuration."""
    h, S = cfg.hidden, cfg.streams
    yield "embed", (cfg.vocab, h)
    for i, l in enumerate(cfg.layers):
        m, f = l.mixer, l.mlp
        roles: Dict[str, tuple] = {"norm1": (h,), "hc1_in": (S,), "hc1_out": (S,), "hc1_mix": (S, S)}
        if m.kind == "rglru":
            n, per = m.width, (m.blocks, m.vdim)
            roles.update(y=(n, h), y_bias=(n,), x=(n, h), x_bias=(n,), conv=(n, m.taps), conv_bias=(n,), ra=per + (m.vdim,),
                         ra_bias=per, ri=per + (m.vdim,), ri_bias=per, lam=(n,), o=(h, n))
        else:
            H = m.heads
            roles.update(q=(H * m.dim, h), o=(h, H * m.vdim))
            if m.kind == "attention":
                roles.update(k=(m.kv_heads * m.dim, h), v=(m.kv_heads * m.vdim, h), q_norm=(m.dim,), k_norm=(m.dim,), sink=(H,))
            else:
                roles.update(dkv=(m.kv_rank, h), dkv_norm=(m.kv_rank,), uk=(H * m.dim, m.kv_rank), uv=(H * m.vdim, m.kv_rank))
        if f is not None:
            roles.update(norm2=(h,), hc2_in=(S,), hc2_out=(S,), hc2_mix=(S, S), router=(f.choices, h), correction=(f.choices,))
            units = {f"e{e}": f.expert for e in range(f.experts)}
            if f.shared is not None:
                units["shared"] = f.shared
                roles["shared_gate"] = (1, h)
            for u, spec in units.items():
                roles.update({f"{u}.gate": (spec.ff, h), f"{u}.up": (spec.ff, h), f"{u}.down": (h, spec.ff)})
        for role, shape in roles.items():
            yield tensor_name(i, role), shape
    yield "final.norm", (h,)
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
        if name.endswith(("norm1", "norm2", "final.norm")):
            t.normal_(0.0, 0.1, generator=gen)                  # around zero
        elif name.endswith(".norm"):
            t.normal_(1.0, 0.1, generator=gen)
        elif ".hc" in name and name.endswith("mix"):
            t.normal_(0.0, 0.1, generator=gen).add_(0.8 * torch.eye(shape[0], device=device))
        elif ".hc" in name:
            t.normal_(0.5, 0.3, generator=gen)
        elif name.endswith("mix.lam"):
            t.uniform_(-6.0, -1.0, generator=gen)               # from almost never forgetting to a few tokens
        elif name.endswith("mix.sink"):
            t.normal_(1.0, 1.0, generator=gen)
        elif name.endswith("mlp.correction"):
            t.normal_(0.0, 0.02, generator=gen)
        elif name.endswith("mix.conv"):
            t.normal_(0.0, shape[-1] ** -0.5, generator=gen)
        elif name.endswith(".b"):
            t.normal_(0.0, 0.2, generator=gen)
        else:
            t.normal_(0.0, std or (1.0 if name == "embed" else shape[-1] ** -0.5), generator=gen)
        out[name] = t.to(torch.bfloat16)
    return out


def _design(name: str, hidden: int, vocab: int, pattern: str, attn: dict, latent: dict, rec: dict, mlp: dict, streams: int = 4,
            max_context: int = 131072) -> LayeredConfig:
    """pattern: one letter per layer, 'a' attention, 'l' latent attention, 'r' recurrence; every layer has experts."""
    kinds = {"a": ("attention", attn), "l": ("latent_attention", latent), "r": ("rglru", rec)}
    c = {"width": hidden, "vocab": vocab, "norm": {"eps": 1e-6}, "streams": streams, "logit_softcap": 30.0,
         "layers": [{"type": kinds[k][0], "mixer": kinds[k][1], "mlp": dict(mlp, kind="moe")} for k in pattern]}
    return LayeredConfig(**dict(vars(parse_config(c, name)), max_context=max_context))


def _moe(experts: int, top: int, ff: int, shared: int, identity: int) -> dict:
    return {"expert": {"ff": ff, "limit": 7.0}, "shared": {"ff": shared, "limit": 7.0},
            "router": {"experts": experts, "top": top, "identity": identity, "scale": 2.0}}


# Geometries for random-init runs: a small one, and two whose layers have the widths of real models.
TINY = _design("tuzupel-tiny", 208, 1024, "rlar", dict(heads=6, kv_heads=3, dim=48, vdim=32, scale=0.2, mask={"size": 40}, rot={"base": 1e4, "dims": 32}),
               dict(heads=5, dim=48, vdim=32, kv_rank=80, scale=0.15, mask={"size": 56}), dict(width=240, blocks=5, conv=4),
               _moe(6, 3, 96, 112, 1), 3, 4096)
_ROT = {"base": 5e5, "dims": 64, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}
T1B = _design("tuzupel-1b", 2048, 65536, "rral" * 4, dict(heads=16, kv_heads=4, dim=128, vdim=128, scale=0.0884, mask={"size": 8192}, rot=_ROT),
              dict(heads=16, dim=128, vdim=128, kv_rank=512, scale=0.0884, mask={"size": 1024}), dict(width=2560, blocks=10, conv=4),
              _moe(32, 4, 1024, 1024, 4))
T7B = _design("tuzupel-7b", 4096, 131072, "rral" * 8, dict(heads=32, kv_heads=8, dim=128, vdim=128, scale=0.0884, mask={"size": 8192}, rot=_ROT),
              dict(heads=32, dim=128, vdim=128, kv_rank=512, scale=0.0884, mask={"size": 2048}), dict(width=4096, blocks=16, conv=4),
              _moe(64, 6, 1536, 3072, 8))
CONFIGS = {c.name: c for c in (TINY, T1B, T7B)}
