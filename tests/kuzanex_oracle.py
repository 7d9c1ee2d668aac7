"""Plain, slow Kuzanex decoder in float64 numpy: one function per mechanism, whole sequences only, no cache, no code of
the package.  Weights are a dict name -> array, the configuration is the parsed config.json."""
import numpy as np


def rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def sigmoid(z):
    return np.where(z >= 0, 1.0 / (1.0 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1.0 + np.exp(-np.abs(z))))


def softplus(z):
    return np.logaddexp(0.0, z)


def scalar_norm(x, g, eps):
    """RMS norm followed by one gain for every coordinate."""
    return rms(x, eps) * float(np.asarray(g).reshape(()))


def xielu(z, act):
    p, q = float(act[0]), float(act[1])
    pos = softplus(p) * z * z + 0.5 * z
    neg = (0.5 + softplus(q)) * (np.exp(np.minimum(z, 0.0)) - 1.0 - z) + 0.5 * z
    return np.where(z > 0, pos, neg)


def head_slopes(n_heads):
    return np.array([2.0 ** (-8.0 * (h + 1) / n_heads) for h in range(n_heads)])


def capped_scores(q, k, scale, softcap):
    """q [T, H, D], k [T, G, D] -> [H, T, T] scores of query i against key j, soft-capped."""
    T, H, _ = q.shape
    G = k.shape[1]
    s = np.empty((H, T, T))
    for h in range(H):
        s[h] = scale * (q[:, h] @ k[:, h // (H // G)].T)
    return softcap * np.tanh(s / softcap)


def distance_bias(s):
    H, T, _ = s.shape
    d = np.arange(T)[:, None] - np.arange(T)[None, :]
    return s - head_slopes(H)[:, None, None] * d


def mix_heads(s, talk):
    return np.einsum("hg,gij->hij", talk, s)


def window_mask(T, size):
    d = np.arange(T)[:, None] - np.arange(T)[None, :]
    return (d >= 0) & (d < size)


def sink_softmax(s, mask):
    """exp(s) / (1 + sum exp(s)) over the visible keys: the extra term is a key of score 0 without a value."""
    s = np.where(mask, s, -np.inf)
    m = np.maximum(s.max(axis=-1, keepdims=True), 0.0)
    e = np.exp(s - m)
    return e / (np.exp(-m) + e.sum(axis=-1, keepdims=True))


def attention(w, p, h, mx, eps):
    H, G, D, V = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    T = h.shape[0]
    q = (h @ w[p + "q"].T + w[p + "q.b"]).reshape(T, H, D)
    k = (h @ w[p + "k"].T + w[p + "k.b"]).reshape(T, G, D)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).reshape(T, G, V)
    q = rms(q, eps) * w[p + "q.norm"]
    k = rms(k, eps) * w[p + "k.norm"]
    s = mix_heads(distance_bias(capped_scores(q, k, mx["scale"], mx["softcap"])), w[p + "talk"])
    a = sink_softmax(s, window_mask(T, mx["mask"]["size"]))
    o = np.stack([a[i] @ v[:, i // (H // G)] for i in range(H)], axis=1)        # [T, H, V]
    o = o * sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(T, H * V) @ w[p + "o"].T


def mlstm_gates(i_raw, f_raw, cap):
    i = cap * np.tanh(i_raw / cap)
    f = -softplus(-(cap * np.tanh(f_raw / cap)))
    return i, f


def mlstm_recurrence(q, k, v, i, f):
    """q, k [T, H, D], v [T, H, V], log gates [T, H] -> [T, H, V], token by token from a zero state."""
    T, H, D = q.shape
    out = np.empty(v.shape)
    S, n, m = np.zeros((H, D, v.shape[2])), np.zeros((H, D)), np.zeros(H)
    for t in range(T):
        m_new = np.maximum(f[t] + m, i[t])
        a, b = np.exp(f[t] + m - m_new), np.exp(i[t] - m_new)
        S = a[:, None, None] * S + b[:, None, None] * (k[t][:, :, None] * v[t][:, None, :])
        n = a[:, None] * n + b[:, None] * k[t]
        m = m_new
        den = np.maximum(np.abs(np.einsum("hd,hd->h", n, q[t])), np.exp(-m)) + 1e-6
        out[t] = np.einsum("hdv,hd->hv", S, q[t]) / den[:, None]
    return out


def mlstm(w, p, h, mx, eps):
    H, D, V = mx["heads"], mx["dim"], mx["vdim"]
    T = h.shape[0]
    q = (h @ w[p + "q"].T).reshape(T, H, D) * D ** -0.5
    k = (h @ w[p + "k"].T).reshape(T, H, D)
    v = (h @ w[p + "v"].T).reshape(T, H, V)
    i, f = mlstm_gates(h @ w[p + "i"].T + w[p + "i.b"], h @ w[p + "f"].T + w[p + "f.b"], mx["gate_cap"])
    o = rms(mlstm_recurrence(q, k, v, i, f), eps).reshape(T, H * V)
    return (o * w[p + "norm"] * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def feed_forward(w, p, h):
    return xielu(h @ w[p + "up"].T + w[p + "up.b"], w[p + "act"]) @ w[p + "down"].T + w[p + "down.b"]


def layer(w, cfg, i, x):
    spec, eps, a = cfg["layers"][i], cfg["norm"]["eps"], cfg["postln_alpha"]
    mix = {"attention": attention, "mlstm": mlstm}[spec["type"]]
    x = scalar_norm(a * x + mix(w, f"l{i}.mix.", x, spec["mixer"], eps), w[f"l{i}.norm1"], eps)
    if spec.get("mlp"):
        x = scalar_norm(a * x + feed_forward(w, f"l{i}.mlp.", x), w[f"l{i}.norm2"], eps)
    return x


def forward(w, cfg, tokens, want_layers=False):
    """Logits [T, vocab] of a whole sequence (and the residual stream after every layer)."""
    x = w["embed"][np.asarray(tokens)]
    per = []
    for i in range(len(cfg["layers"])):
        x = layer(w, cfg, i, x)
        per.append(x)
    logits = scalar_norm(x, w["final.norm"], cfg["norm"]["eps"]) @ w["head"].T
    return (logits, np.stack(per)) if want_layers else logits


def greedy(w, cfg, prompt, n_new):
    ids = list(prompt)
    for _ in range(n_new):
        ids.append(int(np.argmax(forward(w, cfg, ids)[-1])))
    return ids[len(prompt):]
