"""Plain, slow Tuzupel decoder in float64 numpy: one function per mechanism, whole sequences only, no cache, no code of
the package.  Weights are a dict name -> array, the configuration is the parsed config.json."""
import math

import numpy as np


def rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm_about_zero(x, w, eps):
    """Model norm: the stored weight is the difference from one."""
    return rms(x, eps) * (1.0 + w)


def sigmoid(z):
    e = np.exp(-np.abs(z))
    return np.where(z >= 0, 1.0 / (1.0 + e), e / (1.0 + e))


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# ---------------------------------------------------------------------------- streams
def stream_read(X, w_in):
    """X [T, S, N], w_in [S] -> [T, N]."""
    return np.einsum("tsn,s->tn", X, w_in)


def stream_write(X, y, mix, w_out):
    """New streams out of the old ones (mix is indexed [from, to]) and a sublayer's output y [T, N]."""
    return np.einsum("tsn,su->tun", X, mix) + w_out[None, :, None] * y[:, None, :]


# ---------------------------------------------------------------------------- attention
def frequencies(rot):
    """One frequency per pair, slow ones divided by the factor, a ramp in between."""
    if not rot:
        return np.zeros(0)
    d = rot["dims"]
    f = rot["base"] ** (-np.arange(0, d, 2) / d)
    sc = rot.get("scaling")
    if not sc:
        return f
    out = []
    for x in f:
        wave = 2.0 * math.pi / x
        if wave < sc["original"] / sc["high"]:
            out.append(x)
        elif wave > sc["original"] / sc["low"]:
            out.append(x / sc["factor"])
        else:
            s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
            out.append((1.0 - s) * x / sc["factor"] + s * x)
    return np.array(out)


def rotate(x, pos, f):
    """x [T, ..., dim]: neighbours (2i, 2i + 1) of the first 2 len(f) coordinates turned by pos * f[i]."""
    a = pos[:, None] * f
    c, s = np.cos(a), np.sin(a)
    while c.ndim < x.ndim:
        c, s = c[:, None], s[:, None]
    d = 2 * len(f)
    u, v = x[..., 0:d:2], x[..., 1:d:2]
    out = x.copy()
    out[..., 0:d:2] = u * c - v * s
    out[..., 1:d:2] = v * c + u * s
    return out


def sees(T, window=0, chunk=0):
    """[T, T] bool: may query i look at key j."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    m = j <= i
    if window:
        m &= i - j < window
    if chunk:
        m &= i // chunk == j // chunk
    return m


def edge(mx):
    return mx["mask"]["size"] if mx.get("mask") else 0


def softmax_over(s, seen, sink=None):
    """s [..., T, T]; sink [heads] (axis 0 of s) counts once in every denominator."""
    s = np.where(seen, s, -np.inf)
    m = s.max(axis=-1, keepdims=True)
    if sink is not None:
        m = np.maximum(m, sink[:, None, None])
    e = np.exp(s - m)
    den = e.sum(axis=-1, keepdims=True)
    if sink is not None:
        den = den + np.exp(sink[:, None, None] - m)
    return e / den


def attend(q, k, v, scale, seen, sink=None):
    """q [T, H, D], k [T, G, D], v [T, G, V] -> [T, H, V]; query head h reads key / value head h // (H / G)."""
    R = q.shape[1] // k.shape[1]
    k, v = np.repeat(k, R, axis=1), np.repeat(v, R, axis=1)
    a = softmax_over(np.einsum("ihd,jhd->hij", q, k) * scale, seen, sink)
    return np.einsum("hij,jhv->ihv", a, v)


def attention(w, p, h, mx, eps):
    H, G, D, V, T = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"], h.shape[0]
    pos, f = np.arange(T, dtype=np.float64), frequencies(mx.get("rot"))
    q = rotate(rms((h @ w[p + "q"].T).reshape(T, H, D), eps) * w[p + "q.norm"], pos, f)
    k = rotate(rms((h @ w[p + "k"].T).reshape(T, G, D), eps) * w[p + "k.norm"], pos, f)
    v = (h @ w[p + "v"].T).reshape(T, G, V)
    o = attend(q, k, v, mx["scale"], sees(T, chunk=edge(mx)), w[p + "sink"])
    return o.reshape(T, H * V) @ w[p + "o"].T


def latent_attention(w, p, h, mx, eps):
    H, D, V, T = mx["heads"], mx["dim"], mx["vdim"], h.shape[0]
    q = (h @ w[p + "q"].T).reshape(T, H, D)
    c = rms(h @ w[p + "dkv"].T, eps) * w[p + "dkv.norm"]
    k, v = (c @ w[p + "uk"].T).reshape(T, H, D), (c @ w[p + "uv"].T).reshape(T, H, V)
    return attend(q, k, v, mx["scale"], sees(T, window=edge(mx))).reshape(T, H * V) @ w[p + "o"].T


# ---------------------------------------------------------------------------- gated linear recurrence
def causal_conv(x, w, b):
    """x [T, C], w [C, taps]: the last tap multiplies the newest input, zeros before the start."""
    T, taps = x.shape[0], w.shape[1]
    out = np.tile(b, (T, 1))
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            out[back:] += w[:, j] * x[: T - back]
    return out


def block_gate(u, w, b):
    """u [T, C], w [blocks, n, n], b [blocks, n] -> sigmoid of every block's own linear map."""
    parts = u.reshape(u.shape[0], w.shape[0], w.shape[1])
    return sigmoid(np.einsum("tbi,boi->tbo", parts, w) + b).reshape(u.shape)


def linear_recurrence(u, r, i, lam, start=None):
    """S <- a S + sqrt(1 - a^2) i u with log a = -8 r softplus(lam); all [T, C], lam [C]."""
    log_a = -8.0 * r * softplus(lam)
    a, b = np.exp(log_a), np.sqrt(-np.expm1(2.0 * log_a)) * i * u
    S, out = np.zeros(u.shape[1]) if start is None else start, np.empty_like(u)
    for t in range(u.shape[0]):
        S = a[t] * S + b[t]
        out[t] = S
    return out


def rglru(w, p, h, mx, eps):
    y = gelu_tanh(h @ w[p + "y"].T + w[p + "y.b"])
    u = causal_conv(h @ w[p + "x"].T + w[p + "x.b"], w[p + "conv"], w[p + "conv.b"])
    r, i = block_gate(u, w[p + "ra"], w[p + "ra.b"]), block_gate(u, w[p + "ri"], w[p + "ri.b"])
    return (linear_recurrence(u, r, i, w[p + "lam"]) * y) @ w[p + "o"].T


# ---------------------------------------------------------------------------- experts
def glu_clamped(g, u, limit):
    g, u = np.minimum(g, limit), np.clip(u, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def expert(w, p, h, limit):
    return glu_clamped(h @ w[p + ".gate"].T, h @ w[p + ".up"].T, limit) @ w[p + ".down"].T


def router_scores(z):
    """Softmax over all router outputs [T, experts + identity]."""
    e = np.exp(z - z.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def route(z, correction, top, scale, forced=None):
    """Router logits -> (choices [T, top], weights [T, top]).  `forced`: choices that are made elsewhere."""
    s = router_scores(z)
    ids = np.argsort(-(s + correction), axis=-1, kind="stable")[:, :top] if forced is None else forced
    return ids, np.take_along_axis(s, ids, axis=-1) * scale


def shortfall(z, correction, ids):
    """Per token: by how much the best choice score left out exceeds the worst one taken (<= 0 for the right choice)."""
    c = router_scores(z) + correction
    taken = np.zeros(c.shape, dtype=bool)
    np.put_along_axis(taken, ids, True, axis=-1)
    assert (taken.sum(axis=-1) == ids.shape[1]).all()          # no expert twice
    left = np.where(taken, -np.inf, c).max(axis=-1)
    return left - np.where(taken, c, np.inf).min(axis=-1)


def experts(w, p, h, mlp, forced=None, short=None):
    r, E = mlp["router"], mlp["router"]["experts"]
    z = h @ w[p + "router"].T
    ids, wt = route(z, w[p + "correction"], r["top"], r["scale"], forced)
    if short is not None:
        short.append(shortfall(z, w[p + "correction"], ids))
    out = np.zeros_like(h)
    for e in range(E + r["identity"]):
        for j in range(r["top"]):
            t = np.nonzero(ids[:, j] == e)[0]
            if len(t):
                y = expert(w, f"{p}e{e}", h[t], mlp["expert"]["limit"]) if e < E else h[t]
                out[t] += wt[t, j][:, None] * y
    if mlp.get("shared"):
        out += sigmoid(h @ w[p + "shared.sg"].T) * expert(w, p + "shared", h, mlp["shared"]["limit"])
    return out


# ---------------------------------------------------------------------------- model
def layer(w, cfg, i, X, forced=None, short=None):
    spec, eps = cfg["layers"][i], cfg["norm"]["eps"]
    mix = {"attention": attention, "latent_attention": latent_attention, "rglru": rglru}[spec["type"]]
    subs = [(1, lambda h: mix(w, f"l{i}.mix.", h, spec["mixer"], eps))]
    if spec["mlp"]:
        subs.append((2, lambda h: experts(w, f"l{i}.mlp.", h, spec["mlp"], forced, short)))
    for q, f in subs:
        hc = f"l{i}.hc{q}."
        y = f(norm_about_zero(stream_read(X, w[hc + "in"]), w[f"l{i}.norm{q}"], eps))
        X = stream_write(X, y, w[hc + "mix"], w[hc + "out"])
    return X


def forward(w, cfg, tokens, want_layers=False, choices=None, short=None):
    """Logits [T, vocab] of a whole sequence (and the sum of the streams after every layer).  `choices`: layer -> experts
    [T, top] to use instead of the router's own; `short` collects the shortfall of every layer's choices."""
    x = w["embed"][np.asarray(tokens)]
    X, per = np.repeat(x[:, None, :], cfg["streams"], axis=1), []
    for i in range(len(cfg["layers"])):
        X = layer(w, cfg, i, X, None if choices is None else choices[i], short)
        per.append(X.sum(axis=1))
    z = norm_about_zero(X.sum(axis=1), w["final.norm"], cfg["norm"]["eps"]) @ w["head"].T
    cap = cfg.get("logit_softcap")
    logits = cap * np.tanh(z / cap) if cap else z
    return (logits, np.stack(per)) if want_layers else logits


def greedy(w, cfg, prompt, n_new):
    ids = list(prompt)
    for _ in range(n_new):
        ids.append(int(np.argmax(forward(w, cfg, ids)[-1])))
    return ids[len(prompt):]
