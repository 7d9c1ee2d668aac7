"""Ratilorn: how its config.json and checkpoint tensors map onto the layer-list decoder (`models/layered.py`).

The design fixes: a table of position vectors, a norm on every sublayer's output only (weights stored around zero), attention
with sigmoid weights that are mixed across heads, a logarithmic distance bias and values mixed with those of the first such
layer, softmax attention and a Mamba-2 state space side by side, SwiGLU feed-forwards and experts that are chosen by
sigmoid scores inside the best groups, logits from the embedding table.  Sizes, constants and the order of layers come from the
configuration."""
from __future__ import annotations

from typing import Dict, Iterator, Optional, Tuple

from .layered_config import AttentionMixer, ExpertMlp, GatedUnit, LayeredConfig, LayerSpec, ParallelMixer, StateSpaceMixer

ARCHITECTURE = "Ratilorn"
NORM_OFFSET = 1.0


def _heads(c: dict) -> dict:
    out = {k: int(c[k]) for k in ("heads", "kv_heads", "dim", "vdim")}
    if out["kv_heads"] < 1 or out["heads"] % out["kv_heads"]:
        raise ValueError("attention: heads must be a multiple of kv_heads")
    return dict(out, scale=float(c["scale"]))


def _attention(c: dict) -> AttentionMixer:
    return AttentionMixer(**_heads(c), bias=True, qk_unit=True, head_mixing=True, sigmoid=True, log_bias=True,
                          value_mix=bool(c.get("v_mix", False)))


def _state_space(c: dict) -> StateSpaceMixer:
    m = StateSpaceMixer(heads=int(c["heads"]), vdim=int(c["vdim"]), state=int(c["state"]), groups=int(c["groups"]), taps=int(c["conv"]),
                        norm_groups=int(c["norm_groups"]))
    if m.groups < 1 or m.heads % m.groups:
        raise ValueError("state space: heads must be a multiple of groups")
    if m.norm_groups < 1 or m.heads * m.vdim % m.norm_groups:
        raise ValueError(f"state space: {m.heads * m.vdim} channels have no {m.norm_groups} equal parts")
    if m.taps < 1:
        raise ValueError("state space: the convolution needs at least one tap")
    return m


def _parallel(c: dict) -> ParallelMixer:
    return ParallelMixer(left=AttentionMixer(**_heads(c["left"]), bias=True, qk_norm=True), right=_state_space(c["right"]))


_MIXERS = {"attention": _attention, "parallel": _parallel}


def _unit(c: Optional[dict]) -> Optional[GatedUnit]:
    return None if c is None else GatedUnit(int(c["ff"]))


def _experts(c: dict) -> ExpertMlp:
    r, g = c["router"], c["router"].get("groups") or {}
    m = ExpertMlp(experts=int(r["experts"]), top=int(r["top"]), expert=_unit(c["expert"]), shared=_unit(c.get("shared")), shared_gate=False,
                  sigmoid=True, renormalise=True, groups=int(g.get("count", 0)), keep=int(g.get("keep", 0)))
    if m.experts < 1 or not 1 <= m.top <= m.experts:
        raise ValueError(f"router: {m.top} of {m.experts} experts")
    if g and (m.groups < 1 or m.experts % m.groups or not 1 <= m.keep <= m.groups or m.experts // m.groups * m.keep < m.top):
        raise ValueError(f"router: {m.experts} experts in {m.groups} groups, {m.keep} of them kept, leave no choice of {m.top}")
    return m


def _mlp(c: Optional[dict], layer: int):
    if c is None:
        return None
    kind = c.get("kind", "dense")
    if kind not in ("dense", "moe"):
        raise ValueError(f"layer {layer}: unknown feed-forward '{kind}'")
    return _experts(c) if kind == "moe" else _unit(c)


def parse_config(c: dict, name: str = "ratilorn") -> LayeredConfig:
    layers = []
    for i, l in enumerate(c["layers"]):
        if l["type"] not in _MIXERS:
            raise ValueError(f"layer {i}: unknown mixer '{l['type']}'")
        layers.append(LayerSpec(_MIXERS[l["type"]](l["mixer"]), _mlp(l.get("mlp"), i)))
    places = int(c["max_positions"])
    cfg = LayeredConfig(name=name, hidden=int(c["width"]), vocab=int(c["vocab"]), layers=tuple(layers), rms_eps=float(c["norm"]["eps"]),
                        residual_alpha=1.0, max_context=places, architecture=ARCHITECTURE, residual="branch", tie_head=True,
                        norm_offset=NORM_OFFSET, logit_scale=float(c["logit_scale"]), learned_positions=places)
    if places < 1:
        raise ValueError("max_positions must be positive")
    if len({(m.kv_heads, m.vdim) for m in map(cfg.attention_of, cfg.value_runs)}) > 1:
        raise ValueError("layers that mix their values must have the same value heads")
    return cfg


def config_dict(cfg: LayeredConfig) -> dict:
    """The config.json of a configuration of this design."""
    def heads(m):
        return {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale}
    layers = []
    for l in cfg.layers:
        m, f, mlp = l.mixer, l.mlp, None
        if m.kind == "parallel":
            r = m.right
            mixer = {"left": heads(m.left), "right": {"heads": r.heads, "vdim": r.vdim, "state": r.state, "groups": r.groups, "conv": r.taps,
                                                      "norm_groups": r.norm_groups}}
        else:
            mixer = dict(heads(m), v_mix=m.value_mix)
        if f is not None and f.kind == "moe":
            mlp = {"kind": "moe", "expert": {"ff": f.expert.ff}, "router": {"experts": f.experts, "top": f.top}}
            if f.groups:
                mlp["router"]["groups"] = {"count": f.groups, "keep": f.keep}
            if f.shared is not None:
                mlp["shared"] = {"ff": f.shared.ff}
        elif f is not None:
            mlp = {"kind": "dense", "ff": f.ff}
        layers.append({"type": m.kind, "mixer": mixer, "mlp": mlp})
    return {"architecture": ARCHITECTURE, "width": cfg.hidden, "vocab": cfg.vocab, "max_positions": cfg.learned_positions,
            "norm": {"eps": cfg.rms_eps}, "logit_scale": cfg.logit_scale, "layers": layers}


# role (layered.pack_weights) -> checkpoint name; the feed-forward's units are "gate", "e<number>.gate", "shared.gate" and so on
_MODEL = {"embed": "embed", "positions": "pos", "final_norm": "final.norm"}
_HEADS = {r: r for r in ("q", "k", "v", "o")}
_HEADS.update({f"{r}_bias": f"{r}.b" for r in ("q", "k", "v")})
_LAYER = {"norm1": "norm1", "norm2": "norm2"}
_LAYER.update({r: f"mix.{n}" for r, n in _HEADS.items()})
_LAYER.update({"log_rate": "mix.r1", "log_step": "mix.r2", "offset": "mix.pb", "talk": "mix.talk", "v_lambda": "mix.vmix"})
_LAYER.update({f"left.{r}": f"mix.left.{n}" for r, n in _HEADS.items()})
_LAYER.update({"left.q_norm": "mix.left.q.norm", "left.k_norm": "mix.left.k.norm"})
_LAYER.update({f"right.{r}": f"mix.right.{r}" for r in ("in", "conv", "dt_bias", "norm", "o")})
_LAYER.update({"right.conv_bias": "mix.right.conv.b", "right.a_log": "mix.right.A_log", "right.skip": "mix.right.D"})
_LAYER.update({f"{side}.out": f"mix.{side}.out" for side in ("left", "right")})


def tensor_name(layer: int, role: str) -> str:
    if layer < 0:
        return _MODEL[role]
    return f"l{layer}.{_LAYER[role]}" if role in _LAYER else f"l{layer}.mlp.{role}"


def _head_shapes(m: AttentionMixer, h: int) -> Dict[str, tuple]:
    q, k, v = m.heads * m.dim, m.kv_heads * m.dim, m.kv_heads * m.vdim
    return {"q": (q, h), "k": (k, h), "v": (v, h), "q_bias": (q,), "k_bias": (k,), "v_bias": (v,), "o": (h, m.heads * m.vdim)}


def tensor_shapes(cfg: LayeredConfig) -> Iterator[Tuple[str, tuple]]:
    """Names and shapes of a checkpoint of this configuration."""
    h = cfg.hidden
    yield "embed", (cfg.vocab, h)
    yield "pos", (cfg.learned_positions, h)
    for i, l in enumerate(cfg.layers):
        m, f = l.mixer, l.mlp
        roles: Dict[str, tuple] = {"norm1": (h,)}
        if m.kind == "parallel":
            r = m.right
            inner, channels = r.heads * r.vdim, r.heads * r.vdim + 2 * r.groups * r.state
            roles.update({f"left.{n}": s for n, s in _head_shapes(m.left, h).items()})
            roles.update({"left.q_norm": (m.left.dim,), "left.k_norm": (m.left.dim,), "right.in": (inner + channels + r.heads, h),
                          "right.conv": (channels, r.taps), "right.conv_bias": (channels,), "right.dt_bias": (r.heads,),
                          "right.a_log": (r.heads,), "right.skip": (r.heads,), "right.norm": (inner,), "right.o": (h, inner),
                          "left.out": (h,), "right.out": (h,)})
        else:
            roles.update(_head_shapes(m, h), log_rate=(m.heads,), log_step=(m.heads,), talk=(m.heads, m.heads), offset=(m.heads,))
            if m.value_mix:
                roles["v_lambda"] = ()
        if f is not None:
            roles["norm2"] = (h,)
            units = {"": f} if f.kind == "glu" else {f"e{e}.": f.expert for e in range(f.experts)}
            if f.kind == "moe":
                roles.update(router=(f.experts, h), correction=(f.experts,))
                if f.shared is not None:
                    units["shared."] = f.shared
            for u, spec in units.items():
                roles.update({f"{u}gate": (spec.ff, h), f"{u}up": (spec.ff, h), f"{u}down": (h, spec.ff)})
        for role, shape in roles.items():
            yield tensor_name(i, role), shape
    yield "final.norm", (h,)


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
        elif name.endswith((".norm", ".out")):
            t.normal_(1.0, 0.1, generator=gen)
        elif name.endswith("mix.talk"):
            t.normal_(0.0, 0.15, generator=gen).add_(torch.eye(shape[0], device=device))
        elif name.endswith(("mix.r1", "mix.r2", "mix.vmix")):
            t.uniform_(0.1, 0.9, generator=gen)
        elif name.endswith("mix.pb"):
            t.normal_(-3.0, 0.5, generator=gen)                 # weights of about 1 / 20 before the scores speak
        elif name.endswith("A_log"):
            t.uniform_(-0.5, 1.5, generator=gen)
        elif name.endswith("dt_bias"):
            t.uniform_(-6.0, -1.0, generator=gen)               # from almost never forgetting to a few tokens
        elif name.endswith("right.D"):
            t.normal_(1.0, 0.3, generator=gen)
        elif name.endswith("mlp.correction"):
            t.normal_(0.0, 0.05, generator=gen)
        elif name.endswith("right.conv"):
            t.normal_(0.0, shape[-1] ** -0.5, generator=gen)
        elif name.endswith(".b"):
            t.normal_(0.0, 0.2, generator=gen)
        elif name == "pos":
            t.normal_(0.0, 0.5, generator=gen)
        else:
            t.normal_(0.0, std or (1.0 if name == "embed" else shape[-1] ** -0.5), generator=gen)
        out[name] = t.to(torch.bfloat16)
    return out


def _design(name: str, hidden: int, vocab: int, pattern: str, attn: dict, left: dict, right: dict, mlp: dict, ff: int,
            max_positions: int = 131072, logit_scale: float = 0.05) -> LayeredConfig:
    """pattern: one letter per layer, 'a' sigmoid attention, 'p' the two mixers side by side; every layer but the first has
    experts, the first a dense feed-forward."""
    kinds = {"a": ("attention", attn), "p": ("parallel", {"left": left, "right": right})}
    c = {"width": hidden, "vocab": vocab, "max_positions": max_positions, "norm": {"eps": 1e-6}, "logit_scale": logit_scale,
         "layers": [{"type": kinds[k][0], "mixer": kinds[k][1], "mlp": dict(mlp, kind="moe") if i else {"kind": "dense", "ff": ff}}
                    for i, k in enumerate(pattern)]}
    return parse_config(c, name)


def _moe(experts: int, top: int, ff: int, shared: int, groups: int, keep: int) -> dict:
    return {"expert": {"ff": ff}, "shared": {"ff": shared}, "router": {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep}}}


# Geometries for random-init runs: a small one, and two whose layers have the widths of real models.
TINY = _design("ratilorn-tiny", 208, 1024, "pappa", dict(heads=6, kv_heads=3, dim=48, vdim=32, scale=0.2, v_mix=True),
               dict(heads=4, kv_heads=2, dim=32, vdim=48, scale=0.18), dict(heads=5, vdim=32, state=48, groups=1, conv=4, norm_groups=1),
               _moe(8, 3, 96, 112, 4, 2), 256, 4096)
R1B = _design("ratilorn-1b", 2048, 65536, "pppa" * 4, dict(heads=16, kv_heads=4, dim=128, vdim=128, scale=0.0884, v_mix=True),
              dict(heads=16, kv_heads=4, dim=128, vdim=128, scale=0.0884), dict(heads=32, vdim=64, state=128, groups=1, conv=4, norm_groups=1),
              _moe(32, 4, 1024, 1024, 4, 2), 8192)
R7B = _design("ratilorn-7b", 4096, 131072, "pppa" * 8, dict(heads=32, kv_heads=8, dim=128, vdim=128, scale=0.0884, v_mix=True),
              dict(heads=32, kv_heads=8, dim=128, vdim=128, scale=0.0884), dict(heads=64, vdim=64, state=128, groups=8, conv=4, norm_groups=8),
              _moe(64, 6, 1536, 3072, 8, 4), 14336)
CONFIGS = {c.name: c for c in (TINY, R1B, R7B)}
