"""Plain, slow Ratilorn decoder in float64 numpy: one function per mechanism, whole sequences only, no cache, no code of
the package.  Weights are a dict name -> array, the configuration is the parsed config.json."""
import numpy as np


def rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm_about_zero(x, w, eps):
    """Model norm: the stored weight is the difference from one."""
    return rms(x, eps) * (1.0 + w)


def sigmoid(z):
    e = np.exp(-np.abs(z))
    return np.where(z >= 0, 1.0 / (1.0 + e), e / (1.0 + e))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def embedding(table, positions, tokens):
    return table[np.asarray(tokens)] + positions[: len(tokens)]


def heads_of(h, w, name, n):
    """Projection with its bias, one row of heads per token."""
    return (h @ w[name].T + w[name + ".b"]).reshape(h.shape[0], n, -1)


def scores(q, k, scale):
    """q [T, H, D], k [T, G, D] -> [H, T, T]; query head h reads key head h // (H / G)."""
    return np.einsum("ihd,jhd->hij", q, np.repeat(k, q.shape[1] // k.shape[1], axis=1)) * scale


def past(T):
    i = np.arange(T)
    return i[None, :] <= i[:, None]


def weighted_values(a, v):
    """a [H, T, T], v [T, G, V] -> [T, H, V]."""
    return np.einsum("hij,jhv->ihv", a, np.repeat(v, a.shape[0] // v.shape[1], axis=1))


# ---------------------------------------------------------------------------- sigmoid attention
def log_distance_bias(T, r1, r2):
    """[H, T, T]; distances ahead of the query do not count."""
    i = np.arange(T, dtype=np.float64)
    d = np.maximum(i[:, None] - i[None, :], 0.0)
    return r1[:, None, None] * np.log(1.0 + r2[:, None, None] * d)


def sigmoid_weights(s, offset):
    """One weight per visible key by itself, no sum over keys."""
    return np.where(past(s.shape[-1]), sigmoid(s + offset[:, None, None]), 0.0)


def mix_heads(a, talk):
    return np.einsum("hg,gij->hij", talk, a)


def mix_values(v, first, lam):
    return (1.0 - lam) * v + lam * first


def attention(w, p, h, mx, eps, first):
    """`first`: a list that holds the values of the first layer whose values are mixed, once it has run."""
    H, G, T = mx["heads"], mx["kv_heads"], h.shape[0]
    q, k = rms(heads_of(h, w, p + "q", H), eps), rms(heads_of(h, w, p + "k", G), eps)
    v = heads_of(h, w, p + "v", G)
    if mx.get("v_mix"):
        if first:
            v = mix_values(v, first[0], w[p + "vmix"])
        else:
            first.append(v)
    s = scores(q, k, mx["scale"]) - log_distance_bias(T, w[p + "r1"], w[p + "r2"])
    a = mix_heads(sigmoid_weights(s, w[p + "pb"]), w[p + "talk"])
    return weighted_values(a, v).reshape(T, -1) @ w[p + "o"].T


# ---------------------------------------------------------------------------- softmax attention beside a state space
def softmax_past(s):
    s = np.where(past(s.shape[-1]), s, -np.inf)
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def grouped_attention(w, p, h, mx, eps):
    H, G, T = mx["heads"], mx["kv_heads"], h.shape[0]
    q = rms(heads_of(h, w, p + "q", H), eps) * w[p + "q.norm"]
    k = rms(heads_of(h, w, p + "k", G), eps) * w[p + "k.norm"]
    a = softmax_past(scores(q, k, mx["scale"]))
    return weighted_values(a, heads_of(h, w, p + "v", G)).reshape(T, -1) @ w[p + "o"].T


def causal_conv(x, w, b):
    """x [T, C], w [C, taps]: the last tap multiplies the newest input, zeros before the start."""
    T, taps = x.shape[0], w.shape[1]
    out = np.tile(b, (T, 1))
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            out[back:] += w[:, j] * x[: T - back]
    return out


def state_space(x, B, C, dt, A_log, D, start=None):
    """x [T, H, V], B and C [T, G, N], dt [T, H] (positive) -> (y [T, H, V], state [H, N, V])."""
    T, H, V = x.shape
    R = H // B.shape[1]
    B, C = np.repeat(B, R, axis=1), np.repeat(C, R, axis=1)
    S, y = np.zeros((H, B.shape[2], V)) if start is None else start, np.empty_like(x)
    for t in range(T):
        decay = np.exp(-np.exp(A_log) * dt[t])
        S = decay[:, None, None] * S + dt[t][:, None, None] * B[t][:, :, None] * x[t][:, None, :]
        y[t] = np.einsum("hnv,hn->hv", S, C[t]) + D[:, None] * x[t]
    return y, S


def gated_group_norm(y, z, weight, groups, eps):
    """The gate first, then every one of the equal parts by its own root mean square."""
    g = y * silu(z)
    return rms(g.reshape(g.shape[0], groups, -1), eps).reshape(g.shape) * weight


def mamba2(w, p, h, mx, eps):
    H, V, N, G, T = mx["heads"], mx["vdim"], mx["state"], mx["groups"], h.shape[0]
    inner = H * V
    u = h @ w[p + "in"].T
    z, dt = u[:, :inner], softplus(u[:, -H:] + w[p + "dt_bias"])
    xbc = silu(causal_conv(u[:, inner:-H], w[p + "conv"], w[p + "conv.b"]))
    x, B, C = np.split(xbc, [inner, inner + G * N], axis=1)
    y, _ = state_space(x.reshape(T, H, V), B.reshape(T, G, N), C.reshape(T, G, N), dt, w[p + "A_log"], w[p + "D"])
    return gated_group_norm(y.reshape(T, inner), z, w[p + "norm"], mx["norm_groups"], eps) @ w[p + "o"].T


def parallel(w, p, h, mx, eps, first):
    left = grouped_attention(w, p + "left.", h, mx["left"], eps)
    right = mamba2(w, p + "right.", h, mx["right"], eps)
    return 0.5 * (rms(left, eps) * w[p + "left.out"] + rms(right, eps) * w[p + "right.out"])


# ---------------------------------------------------------------------------- feed-forward
def glu(w, p, h):
    return (silu(h @ w[p + ".gate"].T) * (h @ w[p + ".up"].T)) @ w[p + ".down"].T


def limited_choice(c, groups):
    """Choice scores with the experts outside the best groups at minus infinity."""
    if not groups:
        return c
    parts = c.reshape(c.shape[0], groups["count"], -1)
    score = np.sort(parts, axis=-1)[..., -2:].sum(axis=-1)
    best = np.argsort(-score, axis=-1, kind="stable")[:, : groups["keep"]]
    out = np.full(parts.shape, -np.inf)
    rows = np.arange(c.shape[0])[:, None]
    out[rows, best] = parts[rows, best]
    return out.reshape(c.shape)


def route(z, correction, r, forced=None):
    """Router logits -> (choices [T, top], weights [T, top]).  `forced`: choices that are made elsewhere."""
    s = sigmoid(z)
    c = limited_choice(s + correction, r.get("groups"))
    ids = np.argsort(-c, axis=-1, kind="stable")[:, : r["top"]] if forced is None else forced
    wt = np.take_along_axis(s, ids, axis=-1)
    return ids, wt / (wt.sum(axis=-1, keepdims=True) + 1e-20)


def shortfall(z, correction, r, ids):
    """Per token: by how much scores would have to differ for the choices to be right (<= 0: they are): the best choice score
    left out against the worst one taken, in every group that is used or kept by more than that, and the worst group used against
    the last one kept."""
    c, groups = sigmoid(z) + correction, r.get("groups")
    taken = np.zeros(c.shape, dtype=bool)
    np.put_along_axis(taken, ids, True, axis=-1)
    assert (taken.sum(axis=-1) == ids.shape[1]).all()          # no expert twice
    worst = np.where(taken, c, np.inf).min(axis=-1, keepdims=True)
    if not groups:
        return np.where(taken, -np.inf, c).max(axis=-1) - worst[:, 0]
    n, keep = groups["count"], groups["keep"]
    parts, hit = c.reshape(len(c), n, -1), taken.reshape(len(c), n, -1)
    score, used = np.sort(parts, axis=-1)[..., -2:].sum(axis=-1), hit.any(axis=-1)
    assert (used.sum(axis=-1) <= keep).all()
    order = -np.sort(-score, axis=-1)
    last, after = order[:, keep - 1: keep], order[:, keep: keep + 1] if keep < n else np.full((len(c), 1), -np.inf)
    left = np.where(hit, -np.inf, parts).max(axis=-1) - worst                  # of every group
    kept = np.where(score >= last, np.minimum(left, score - after), -np.inf)   # a group kept by little need not have been
    return np.maximum(np.maximum(np.where(used, left, kept).max(axis=-1), (last - np.where(used, score, np.inf)).max(axis=-1)), -1.0)


def experts(w, p, h, mlp, forced=None, short=None):
    r = mlp["router"]
    z = h @ w[p + "router"].T
    ids, wt = route(z, w[p + "correction"], r, forced)
    if short is not None:
        short.append(shortfall(z, w[p + "correction"], r, ids))
    out = np.zeros_like(h)
    for e in range(r["experts"]):
        for j in range(r["top"]):
            t = np.nonzero(ids[:, j] == e)[0]
            if len(t):
                out[t] += wt[t, j][:, None] * glu(w, f"{p}e{e}", h[t])
    return out + glu(w, p + "shared", h) if mlp.get("shared") else out


# ---------------------------------------------------------------------------- model
def layer(w, cfg, i, x, first, forced=None, short=None):
    spec, eps = cfg["layers"][i], cfg["norm"]["eps"]
    mix = {"attention": attention, "parallel": parallel}[spec["type"]]
    x = x + norm_about_zero(mix(w, f"l{i}.mix.", x, spec["mixer"], eps, first), w[f"l{i}.norm1"], eps)
    mlp = spec.get("mlp")
    if mlp:
        y = glu(w, f"l{i}.mlp", x) if mlp["kind"] == "dense" else experts(w, f"l{i}.mlp.", x, mlp, forced, short)
        x = x + norm_about_zero(y, w[f"l{i}.norm2"], eps)
    return x


def forward(w, cfg, tokens, want_layers=False, choices=None, short=None):
    """Logits [T, vocab] of a whole sequence (and the residual after every layer).  `choices`: layer -> experts [T, top] to use
    instead of the router's own; `short` collects the shortfall of every layer's choices."""
    x, per, first = embedding(w["embed"], w["pos"], tokens), [], []
    for i in range(len(cfg["layers"])):
        x = layer(w, cfg, i, x, first, None if choices is None else choices[i], short)
        per.append(x)
    logits = norm_about_zero(x, w["final.norm"], cfg["norm"]["eps"]) @ w["embed"].T * cfg["logit_scale"]
    return (logits, np.stack(per)) if want_layers else logits


def greedy(w, cfg, prompt, n_new):
    ids = list(prompt)
    for _ in range(n_new):
        ids.append(int(np.argmax(forward(w, cfg, ids)[-1])))
    return ids[len(prompt):]
