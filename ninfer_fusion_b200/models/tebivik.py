"""Tebivik: how its config.json and checkpoint tensors map onto the layer-list decoder (`models/layered.py`).

The design fixes: a grouped norm before and after every sublayer, a short causal convolution in front of every mixer,
gated linear memories and latent attention with a learned sink per head and interleaved rotation, biased feed-forwards
with the square of relu, one stretch of layers that runs several times with the embedding output fed back in, and logits
from the embedding table.  Sizes, constants and the order of layers come from the configuration."""
from __future__ import annotations

from typing import Dict, Iterator, Tuple

from .layered_config import DenseMlp, GatedMemoryMixer, LatentAttentionMixer, LayeredConfig, LayerSpec, LoopSpec

ARCHITECTURE = "Tebivik"
ACTIVATION = "relu2"


def _latent(c: dict) -> LatentAttentionMixer:
    m = LatentAttentionMixer(heads=int(c["heads"]), dim=int(c["dim"]), rot_dim=int(c["rot_dim"]), vdim=int(c["vdim"]),
                             q_rank=int(c["q_rank"]), kv_rank=int(c["kv_rank"]), scale=float(c["scale"]),
                             rot_base=float(c["rot"]["base"]))
    if m.rot_dim % 2 or int(c["rot"].get("dims", m.rot_dim)) != m.rot_dim:
        raise ValueError("latent attention: the rotated part must be of even width and rotated as a whole")
    return m


def _hgrn2(c: dict) -> GatedMemoryMixer:
    return GatedMemoryMixer(heads=int(c["heads"]), dim=int(c["dim"]), vdim=int(c["vdim"]))


_MIXERS = {"latent_attention": _latent, "hgrn2": _hgrn2}


def parse_config(c: dict, name: str = "tebivik") -> LayeredConfig:
    layers = []
    for i, l in enumerate(c["layers"]):
        if l["type"] not in _MIXERS:
            raise ValueError(f"layer {i}: unknown mixer '{l['type']}'")
        mlp = l.get("mlp")
        if mlp is not None:
            if mlp.get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward '{mlp['kind']}'")
            mlp = DenseMlp(int(mlp["ff"]), ACTIVATION, bias=True)
        layers.append(LayerSpec(_MIXERS[l["type"]](l["mixer"]), mlp))
    loop = c.get("loop")
    if loop is not None:
        loop = LoopSpec(int(loop["start"]), int(loop["stop"]), int(loop["times"]))
        if not (0 <= loop.start < loop.stop <= len(layers)) or loop.times < 1:
            raise ValueError(f"loop: layers {loop.start} .. {loop.stop} run {loop.times} times, of {len(layers)} layers")
    cfg = LayeredConfig(name=name, hidden=int(c["width"]), vocab=int(c["vocab"]), layers=tuple(layers),
                        rms_eps=float(c["norm"]["eps"]), residual_alpha=1.0, architecture=ARCHITECTURE, residual="sandwich",
                        residual_mult=float(c["residual_mult"]), norm_groups=int(c["norm"]["groups"]),
                        conv_taps=int(c["canon"]["taps"]), embed_scale=float(c["embedding"]["scale"]), tie_head=True, loop=loop)
    if cfg.norm_groups < 1 or cfg.hidden % cfg.norm_groups:
        raise ValueError(f"norm: a width of {cfg.hidden} has no {cfg.norm_groups} equal parts")
    if cfg.conv_taps < 1:
        raise ValueError("the input convolution needs at least one tap")
    return cfg


def config_dict(cfg: LayeredConfig) -> dict:
    """The config.json of a configuration of this design."""
    layers = []
    for l in cfg.layers:
        m = l.mixer
        mixer = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim}
        if m.kind == "latent_attention":
            mixer.update(q_rank=m.q_rank, kv_rank=m.kv_rank, rot_dim=m.rot_dim, scale=m.scale,
                         rot={"base": m.rot_base, "dims": m.rot_dim})
        layers.append({"type": m.kind, "mixer": mixer, "mlp": None if l.mlp is None else {"kind": "dense", "ff": l.mlp.ff}})
    out = {"architecture": ARCHITECTURE, "width": cfg.hidden, "vocab": cfg.vocab,
           "norm": {"eps": cfg.rms_eps, "groups": cfg.norm_groups}, "residual_mult": cfg.residual_mult,
           "canon": {"taps": cfg.conv_taps}, "embedding": {"scale": cfg.embed_scale}, "layers": layers}
    if cfg.loop is not None:
        out["loop"] = {"start": cfg.loop.start, "stop": cfg.loop.stop, "times": cfg.loop.times}
    return out


# role (layered.pack_weights) -> checkpoint name
_MODEL = {"embed": "embed", "final_norm": "final.norm", "loop_in": "loop.in", "loop_step": "loop.step"}
_LAYER = {"norm1": "norm1", "norm1b": "norm1b", "norm2": "norm2", "norm2b": "norm2b", "conv": "canon1"}
_LAYER.update({r: f"mix.{r}" for r in ("q", "v", "f", "o", "lower", "norm", "dq", "dkv", "uq", "uk", "uv", "sink")})
_LAYER.update({"f_bias": "mix.f.b", "dq_norm": "mix.dq.norm", "dkv_norm": "mix.dkv.norm", "up": "mlp.up", "up_bias": "mlp.up.b",
               "down": "mlp.down", "down_bias": "mlp.down.b"})


def tensor_name(layer: int, role: str) -> str:
    return _MODEL[role] if layer < 0 else f"l{layer}.{_LAYER[role]}"


def tensor_shapes(cfg: LayeredConfig) -> Iterator[Tuple[str, tuple]]:
    """Names and shapes of a checkpoint of this configuration."""
    h = cfg.hidden
    yield "embed", (cfg.vocab, h)
    if cfg.loop is not None:
        yield "loop.in", (h, 2 * h)
        yield "loop.step", (cfg.loop.times, h)
    for i, l in enumerate(cfg.layers):
        m, H = l.mixer, l.mixer.heads
        roles: Dict[str, tuple] = {"norm1": (h,), "norm1b": (h,), "conv": (h, cfg.conv_taps), "o": (h, H * m.vdim)}
        if m.kind == "latent_attention":
            roles.update(dq=(m.q_rank, h), dq_norm=(m.q_rank,), uq=(H * (m.dim + m.rot_dim), m.q_rank),
                         dkv=(m.kv_rank + m.rot_dim, h), dkv_norm=(m.kv_rank,), uk=(H * m.dim, m.kv_rank),
                         uv=(H * m.vdim, m.kv_rank), sink=(H,))
        else:
            roles.update(q=(H * m.dim, h), f=(H * m.dim, h), f_bias=(H * m.dim,), lower=(H * m.dim,), v=(H * m.vdim, h),
                         norm=(m.vdim,))
        if l.mlp is not None:
            ff = l.mlp.ff
            roles.update(norm2=(h,), norm2b=(h,), up=(ff, h), up_bias=(ff,), down=(h, ff), down_bias=(h,))
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
        if name.endswith(("norm", "norm1", "norm1b", "norm2", "norm2b")):
            t.normal_(1.0, 0.1, generator=gen)
            if name == "final.norm":
                t.mul_(cfg.hidden ** -0.5)           # the head is the embedding table: rows of length about sqrt(width)
        elif name.endswith("mix.f.b"):
            t.normal_(3.0, 1.5, generator=gen)       # long memory
        elif name.endswith("mix.lower"):
            t.uniform_(0.0, 0.9, generator=gen)
        elif name.endswith("mix.sink"):
            t.normal_(1.0, 1.0, generator=gen)
        elif name.endswith((".b", "canon1", "loop.step")):
            t.normal_(0.0, 0.2, generator=gen)
        else:
            t.normal_(0.0, std or (1.0 if name == "embed" else shape[-1] ** -0.5), generator=gen)
        out[name] = t.to(torch.bfloat16)
    return out


def _design(name: str, hidden: int, vocab: int, pattern: str, latent: dict, mem: dict, ff: int, loop: tuple, groups: int,
            taps: int = 4, max_context: int = 131072) -> LayeredConfig:
    """pattern: one letter per layer, 'm' gated memory, 'a' latent attention; every layer has a feed-forward."""
    mlp = DenseMlp(ff, ACTIVATION, True)
    full = {"m": LayerSpec(_hgrn2(mem), mlp), "a": LayerSpec(_latent(latent), mlp)}
    return LayeredConfig(name=name, hidden=hidden, vocab=vocab, layers=tuple(full[c] for c in pattern), rms_eps=1e-6,
                         residual_alpha=1.0, max_context=max_context, architecture=ARCHITECTURE, residual="sandwich",
                         residual_mult=0.7, norm_groups=groups, conv_taps=taps, embed_scale=1.0, tie_head=True, loop=LoopSpec(*loop))


# Geometries for random-init runs: a small one, and two whose layers have the widths of real models.
TINY = _design("tebivik-tiny", 192, 1024, "mamm", dict(heads=5, dim=32, rot_dim=16, vdim=48, q_rank=96, kv_rank=64, scale=0.14,
                                                         rot={"base": 1e4}),
               dict(heads=3, dim=48, vdim=64), 384, (1, 3, 2), 3, 4, 4096)
T1B = _design("tebivik-1b", 2048, 65536, "mmma" * 4, dict(heads=16, dim=128, rot_dim=64, vdim=128, q_rank=768, kv_rank=512,
                                                            scale=0.0722, rot={"base": 1e4}),
              dict(heads=16, dim=128, vdim=128), 8192, (12, 16, 2), 4)
T7B = _design("tebivik-7b", 4096, 131072, "mmma" * 8, dict(heads=32, dim=128, rot_dim=64, vdim=128, q_rank=1536, kv_rank=512,
                                                             scale=0.0722, rot={"base": 1e4}),
              dict(heads=32, dim=128, vdim=128), 12288, (4, 8, 2), 8)
CONFIGS = {c.name: c for c in (TINY, T1B, T7B)}
