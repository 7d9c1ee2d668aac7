"""Plain, slow Tebivik decoder in float64 numpy: one function per mechanism, whole sequences only, no cache, no code of
the package.  Weights are a dict name -> array, the configuration is the parsed config.json."""
import numpy as np


def rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def sigmoid(z):
    e = np.exp(-np.abs(z))
    return np.where(z >= 0, 1.0 / (1.0 + e), e / (1.0 + e))


def silu(z):
    return z * sigmoid(z)


def group_norm(x, w, groups, eps):
    """RMS norm of each of `groups` equal parts of the last axis by itself, then one weight per coordinate."""
    parts = x.reshape(x.shape[:-1] + (groups, x.shape[-1] // groups))
    return rms(parts, eps).reshape(x.shape) * w


def causal_conv(h, w):
    """h [T, C], w [C, taps]: the last tap multiplies the newest input, zeros before the start."""
    T, taps = h.shape[0], w.shape[1]
    out = np.zeros_like(h)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            out[back:] += w[:, j] * h[: T - back]
    return out


def rotate(x, pos, base):
    """x [T, ..., dims]: neighbours (2i, 2i + 1) turned by pos * base^(-2i / dims)."""
    dims = x.shape[-1]
    a = pos[:, None] * base ** (-np.arange(0, dims, 2) / dims)
    c, s = np.cos(a), np.sin(a)
    while c.ndim < x.ndim:
        c, s = c[:, None], s[:, None]
    u, v = x[..., 0::2], x[..., 1::2]
    out = np.empty_like(x)
    out[..., 0::2] = u * c - v * s
    out[..., 1::2] = v * c + u * s
    return out


def forget_gate(raw, lower):
    """raw, lower [..., channels] -> (f, 1 - f), the second without cancellation."""
    return lower + (1.0 - lower) * sigmoid(raw), (1.0 - lower) * sigmoid(-raw)


def hgrn_recurrence(q, f, k, v):
    """q, f, k [T, H, D], v [T, H, V] -> [T, H, V] from a zero state: S <- f S + k v^T, o = S^T q."""
    T, H, D = q.shape
    S, out = np.zeros((H, D, v.shape[2])), np.empty(v.shape)
    for t in range(T):
        S = f[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hdv,hd->hv", S, q[t])
    return out


def hgrn2(w, p, h, mx, eps):
    H, D, V, T = mx["heads"], mx["dim"], mx["vdim"], h.shape[0]
    q = silu(h @ w[p + "q"].T).reshape(T, H, D)
    v = (h @ w[p + "v"].T).reshape(T, H, V)
    f, k = forget_gate(h @ w[p + "f"].T + w[p + "f.b"], w[p + "lower"])
    o = hgrn_recurrence(q, f.reshape(T, H, D), k.reshape(T, H, D), v)
    return (rms(o, eps) * w[p + "norm"]).reshape(T, H * V) @ w[p + "o"].T


def latent_heads(w, p, h, mx, eps):
    """q [T, H, dim + rot] rotated, latent c [T, rank], shared rotated key part [T, rot]."""
    H, D, R, C, T = mx["heads"], mx["dim"], mx["rot_dim"], mx["kv_rank"], h.shape[0]
    pos = np.arange(T, dtype=np.float64)
    q = ((rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]) @ w[p + "uq"].T).reshape(T, H, D + R)
    q = np.concatenate([q[..., :D], rotate(q[..., D:], pos, mx["rot"]["base"])], axis=-1)
    kv = h @ w[p + "dkv"].T
    return q, rms(kv[:, :C], eps) * w[p + "dkv.norm"], rotate(kv[:, C:], pos, mx["rot"]["base"])


def sink_softmax(s, sink):
    """s [H, T, T] with -inf where nothing is seen; sink [H] counts once in every denominator."""
    m = np.maximum(s.max(axis=-1, keepdims=True), sink[:, None, None])
    e = np.exp(s - m)
    return e / (e.sum(axis=-1, keepdims=True) + np.exp(sink[:, None, None] - m))


def causal(s):
    T = s.shape[-1]
    return np.where(np.tril(np.ones((T, T), dtype=bool)), s, -np.inf)


def latent_attention(w, p, h, mx, eps):
    H, D, V, T = mx["heads"], mx["dim"], mx["vdim"], h.shape[0]
    q, c, kr = latent_heads(w, p, h, mx, eps)
    k = (c @ w[p + "uk"].T).reshape(T, H, D)
    v = (c @ w[p + "uv"].T).reshape(T, H, V)
    s = np.stack([(q[:, i, :D] @ k[:, i].T + q[:, i, D:] @ kr.T) * mx["scale"] for i in range(H)])
    a = sink_softmax(causal(s), w[p + "sink"])
    return np.stack([a[i] @ v[:, i] for i in range(H)], axis=1).reshape(T, H * V) @ w[p + "o"].T


def feed_forward(w, p, h):
    return np.maximum(h @ w[p + "up"].T + w[p + "up.b"], 0.0) ** 2 @ w[p + "down"].T + w[p + "down.b"]


def layer(w, cfg, i, x):
    spec, eps, g, m = cfg["layers"][i], cfg["norm"]["eps"], cfg["norm"]["groups"], cfg["residual_mult"]
    h = group_norm(x, w[f"l{i}.norm1"], g, eps)
    h = h + causal_conv(h, w[f"l{i}.canon1"])
    mix = {"hgrn2": hgrn2, "latent_attention": latent_attention}[spec["type"]]
    x = x + m * group_norm(mix(w, f"l{i}.mix.", h, spec["mixer"], eps), w[f"l{i}.norm1b"], g, eps)
    if spec["mlp"]:
        f = feed_forward(w, f"l{i}.mlp.", group_norm(x, w[f"l{i}.norm2"], g, eps))
        x = x + m * group_norm(f, w[f"l{i}.norm2b"], g, eps)
    return x


def layer_order(cfg):
    """(layer, pass or None when the layer does not open a pass) of every layer run."""
    lp, n = cfg["loop"], len(cfg["layers"])
    order = [(i, None) for i in range(lp["start"])]
    for t in range(lp["times"]):
        order += [(i, t if i == lp["start"] else None) for i in range(lp["start"], lp["stop"])]
    return order + [(i, None) for i in range(lp["stop"], n)]


def enter_pass(w, x, x0, t):
    return np.concatenate([x, x0], axis=-1) @ w["loop.in"].T + w["loop.step"][t]


def forward(w, cfg, tokens, want_layers=False):
    """Logits [T, vocab] of a whole sequence (and the residual stream after every layer run)."""
    x0 = w["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    x, per = x0, []
    for i, t in layer_order(cfg):
        if t is not None:
            x = enter_pass(w, x, x0, t)
        x = layer(w, cfg, i, x)
        per.append(x)
    logits = group_norm(x, w["final.norm"], cfg["norm"]["groups"], cfg["norm"]["eps"]) @ w["embed"].T
    return (logits, np.stack(per)) if want_layers else logits


def greedy(w, cfg, prompt, n_new):
    ids = list(prompt)
    for _ in range(n_new):
        ids.append(int(np.argmax(forward(w, cfg, ids)[-1])))
    return ids[len(prompt):]
