"""Small Tebivik configurations of the tests and weights that make faults visible."""
import torch

from ninfer_fusion_b200.models import tebivik


def lat(H, D, R, V, Q, C, scale=0.2, base=1e4, ff=72):
    return {"type": "latent_attention", "mixer": {"heads": H, "dim": D, "vdim": V, "q_rank": Q, "kv_rank": C, "rot_dim": R, "scale": scale,
                                                  "rot": {"base": base, "dims": R}}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def mem(H, D, V, ff=0):
    return {"type": "hgrn2", "mixer": {"heads": H, "dim": D, "vdim": V}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def conf(width, vocab, layers, loop, groups=2, taps=4, m=0.6, scale=1.5, eps=1e-4):
    return {"architecture": "Tebivik", "width": width, "vocab": vocab, "norm": {"eps": eps, "groups": groups}, "residual_mult": m,
            "canon": {"taps": taps}, "embedding": {"scale": scale}, "layers": layers,
            "loop": {"start": loop[0], "stop": loop[1], "times": loop[2]}}


CASES = {
    "mixed": conf(96, 211, [mem(2, 32, 48), lat(3, 32, 16, 32, 48, 80), mem(3, 16, 64, ff=40)], (1, 3, 2), 3, 4),
    # widths that are no multiple of anything, groups of odd width, the whole stack looped three times from the first layer
    "odd": conf(90, 77, [lat(5, 12, 6, 20, 28, 36, scale=0.1, base=500.0, ff=30), mem(1, 24, 40), lat(1, 40, 32, 8, 20, 24, scale=0.05, ff=0), mem(5, 12, 20, ff=26)],
                (0, 4, 3), 6, 3, m=0.4, scale=1.0, eps=1e-2),
    # one pass, one group, a long convolution, a layer after the loop
    "plain": conf(64, 128, [mem(2, 48, 32, ff=50), lat(4, 16, 16, 16, 32, 32), mem(2, 32, 32)], (0, 2, 1), 1, 7, m=1.0),
    "attention_only": conf(64, 128, [lat(2, 48, 32, 64, 64, 128), lat(20, 16, 16, 16, 48, 64, scale=0.4)], (1, 2, 2), 4, 2),
    "memory_only": conf(64, 130, [mem(2, 80, 96), mem(4, 16, 16, ff=64)], (0, 1, 2), 8, 1),
    # the last layers looped; wide heads and a latent wider than the tensor-core kernel's
    "wide": conf(128, 96, [mem(1, 144, 272), lat(2, 64, 64, 160, 96, 528, ff=0)], (1, 2, 2), 2, 5),
}


def build(name, seed=0):
    """(config dict, LayeredConfig, checkpoint tensors bf16, the same as float64 arrays)."""
    c = CASES[name]
    cfg = tebivik.parse_config(c, name)
    t = tebivik.random_tensors(cfg, seed)
    for n in list(t):
        if n.endswith("mix.uq"):
            t[n] = (t[n].float() * 4).to(torch.bfloat16)             # scores that single keys out
        if n.endswith("mix.sink"):
            t[n] = torch.linspace(0.0, 5.0, t[n].numel()).to(torch.bfloat16)
        if n.endswith("mix.lower"):
            t[n][0], t[n][-1] = 0.0, 0.98
        if n.endswith("mix.f.b"):
            t[n] = torch.linspace(-6.0, 9.0, t[n].numel()).to(torch.bfloat16)      # from forgetting at once to almost never
        if n.endswith("canon1"):
            t[n] = (t[n].float() * 2.5).to(torch.bfloat16)
    return c, cfg, t, {n: v.double().numpy() for n, v in t.items()}
