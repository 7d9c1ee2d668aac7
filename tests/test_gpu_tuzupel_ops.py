"""Kernels of residual streams, plain attention with chunks and learned sinks, windowed latent attention, gated linear
recurrence and experts, each mechanism alone against the plain float64 functions of tuzupel_oracle."""
import numpy as np
import pytest
import torch

import tuzupel_oracle as K

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]


@pytest.fixture(scope="module")
def ops():
    from ninfer_fusion_b200 import load_native
    return load_native()


def rnd(seed, *shape, s=1.0, dtype=torch.float32):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(shape, generator=g) * s).to(dtype)


def f64(t):
    return t.detach().double().cpu().numpy()


def rel(got, want):
    got, want = np.asarray(got, dtype=np.float64), np.asarray(want, dtype=np.float64)
    assert np.isfinite(got).all()
    return float(np.abs(got - want).max() / max(1e-30, np.abs(want).max()))


def ints(x):
    return torch.tensor(x, dtype=torch.int32, device="cuda")


def pad_cols(t, n):
    out = torch.zeros(*t.shape[:-1], n, dtype=t.dtype)
    out[..., : t.shape[-1]] = t
    return out


# ---------------------------------------------------------------------------- streams
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("S,n", [(1, 90), (2, 64), (3, 208), (4, 2048), (4, 4096), (5, 136), (8, 5000), (16, 24), (4, 12288)])
def test_streams(ops, dt, S, n):
    """Read only, update by a GEMM's result, update by a mixture with identity choices and a gated shared part; the first
    update finds the embedding row in every stream."""
    T, N, eps, k, E, vocab = 5, (n + 7) // 8 * 8, 1e-3, 3, 4, 11
    X, mix, w_in, w_out, w = rnd(1, T, S, n), rnd(2, S, S), rnd(3, S), rnd(4, S), 1 + 0.3 * rnd(5, n)
    delta, gate = rnd(6, T, n) * 2, rnd(7, T, 3)
    ret, h, weight = rnd(8, T, k, n).to(dt), rnd(9, T, n).to(dt), rnd(10, T, k).abs()
    choice = torch.tensor([[0, 1, 2], [4, 0, 3], [5, 4, 1], [3, 2, 6], [4, 5, 6]])          # 4, 5, 6: identities
    table, ids = rnd(11, vocab, n).to(dt), torch.tensor([0, 10, 3, 3, 7])
    tol = 3e-6 if dt == torch.float32 else 6e-3
    dev = lambda t: pad_cols(t, N).contiguous().cuda()
    coef = (mix.cuda(), w_out.cuda(), w_in.cuda(), dev(w))
    sel = (choice < E)[..., None].numpy()
    mixed = K.sigmoid(f64(gate)[:, 1:2]) * f64(delta) + (f64(weight)[..., None] * np.where(sel, f64(ret), f64(h)[:, None])).sum(1)
    parts = {"none": (None,) * 6 + (0,), "sum": (dev(delta), None, None, None, None, None, 0),
             "mixture": (dev(delta), gate.cuda()[:, 1:2], ints(choice.tolist()), weight.cuda(), dev(ret).view(T * k, N), dev(h), E)}
    for what, part in parts.items():
        for first in (False, True):
            src = np.repeat(f64(table)[ids.numpy()][:, None], S, axis=1) if first else f64(X)
            new = {"none": src, "sum": K.stream_write(src, f64(delta), f64(mix), f64(w_out)),
                   "mixture": K.stream_write(src, mixed, f64(mix), f64(w_out))}[what]
            want = K.rms(K.stream_read(new, f64(w_in)), eps) * f64(w)
            xo = dev(X)
            out = parts["mixture"][5] if what == "mixture" else torch.empty((T, N), dtype=dt, device="cuda")     # in place of h
            keep = out.clone()
            upd = (None, None) if what == "none" else coef[:2]
            ops.stream_rows(None if first else xo, ints(ids.tolist()), dev(table), None if what == "none" else xo, *part, *upd, *coef[2:],
                            out, n, eps, False)
            assert rel(f64(out)[:, :n], want) < tol and not out[:, n:].any(), (what, first)
            if what != "none":
                assert rel(f64(xo)[..., :n], new) < (3e-6 if what == "sum" or dt == torch.float32 else 1e-5)
                assert not xo[..., n:].any()
            out.copy_(keep)
    y = torch.empty((T, N), device="cuda")
    ops.mixture_rows(*parts["mixture"], y, False)
    assert rel(f64(y)[:, :n], mixed) < 1e-5


# ---------------------------------------------------------------------------- attention
class Heads:
    """Sequences `lens` long of which the last `news` tokens are queries, rows scattered over shuffled pages; one key per
    sequence stands out."""

    def __init__(self, H, G, D, V, dt, lens, news, P, seed=0):
        self.lens, self.news, self.scale = lens, news, 2.0 * D ** -0.5
        per = [-(-n // P) for n in lens]
        perm = torch.randperm(sum(per) + 2, generator=torch.Generator().manual_seed(seed)).tolist()
        table = torch.full((len(lens), max(per)), -1, dtype=torch.int32)
        Dp, Vp = (D + 15) // 16 * 16, (V + 15) // 16 * 16
        kp, vp = torch.zeros(sum(per) + 2, G, P, Dp), torch.zeros(sum(per) + 2, G, P, Vp)
        self.q, self.k, self.v, q, row, kv = [], [], [], [], [], []
        at = 0
        for s, n in enumerate(lens):
            qs, ks, vs = (rnd(seed + 7 * s + i, n, h, d).to(dt).float() for i, (h, d) in enumerate(((H, D), (G, D), (G, V))))
            ks[n // 3] *= 3.0
            self.q.append(f64(qs)), self.k.append(f64(ks)), self.v.append(f64(vs))
            for b in range(per[s]):
                table[s, b] = perm[at]
                m = min(P, n - b * P)
                kp[perm[at], :, :m, :D] = ks[b * P: b * P + m].transpose(0, 1)
                vp[perm[at], :, :m, :V] = vs[b * P: b * P + m].transpose(0, 1)
                at += 1
            m = news[s]
            q.append(pad_cols(qs[n - m:], Dp).reshape(m, H * Dp))
            row += [s] * m
            kv += list(range(n - m + 1, n + 1))
        self.T, self.H, self.V, self.Vp = len(row), H, V, Vp
        self.args = (torch.cat(q).to(dt).cuda(), kp.to(dt).cuda(), vp.to(dt).cuda(), table.cuda(), ints(row), ints(kv))
        start = np.cumsum([0] + news)
        self.blocks = (ints([start[s] + o for s, m in enumerate(news) for o in range(0, m, 64)]),
                       ints([min(64, m - o) for m in news for o in range(0, m, 64)]))
        self.dt = dt

    def want(self, window, chunk, sink):
        out = []
        for q, k, v, n, m in zip(self.q, self.k, self.v, self.lens, self.news):
            out.append(K.attend(q, k, v, self.scale, K.sees(n, window, chunk), sink)[n - m:])
        return np.concatenate(out)

    def out(self):
        return torch.full((self.T, self.H * self.Vp), 9.0, dtype=self.dt, device="cuda")

    def get(self, out):
        o = out.view(self.T, self.H, self.Vp)
        assert not o[..., self.V:].any()
        return f64(o)[..., : self.V]


MASKS = [(0, 0), (37, 0), (0, 50), (0, 64), (64, 0), (1, 0), (40, 64), (0, 1)]


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,G,D,V,P", [(6, 2, 32, 48, 16), (5, 5, 20, 12, 8), (20, 1, 64, 64, 64), (8, 2, 128, 128, 64), (4, 2, 128, 64, 16),
                                       (3, 1, 160, 256, 64), (2, 2, 272, 48, 16)])
def test_attention_of_plain_scores(ops, dt, H, G, D, V, P):
    """Windows and chunks, learned sinks, portions and single tokens in one step, splits: every form against the oracle."""
    x = Heads(H, G, D, V, dt, [1, 130, 70, 300, 64, 129], [1, 130, 3, 75, 1, 64], P)
    sink = np.linspace(-1.0, 5.0, H)
    tol = 5e-6 if dt == torch.float32 else 1.2e-2
    forms = (D + 15) // 16 * 16, (V + 15) // 16 * 16
    for window, chunk in MASKS:
        for s in (None, sink):
            want = x.want(window, chunk, s)
            sinks = None if s is None else torch.tensor(s, dtype=torch.float32, device="cuda")
            shape = (window, x.scale, 0.0, 0.0, None, None, None)
            for split, n in ((320, 1), (64, 5)):
                po, ml = torch.empty(x.T * n * H * x.Vp, device="cuda"), torch.empty(x.T * n * H * 2, device="cuda")
                out = x.out()
                ops.head_mix_attention(*x.args, *shape, out, split, n, po, ml, False, chunk, sinks)
                assert rel(x.get(out), want) < tol, (window, chunk, split)
            if dt == torch.bfloat16 and ops.group_prefill_supported(*forms):
                out = x.out()
                ops.group_prefill(*x.args, window, chunk, x.scale, 0.0, sinks, out, *x.blocks, False)
                assert rel(x.get(out), want) < tol, (window, chunk)
    # a constant sink as well
    out = x.out()
    ops.head_mix_attention(*x.args, 0, x.scale, 0.0, 1.0, None, None, None, out, 320, 1, None, None, False)
    assert rel(x.get(out), x.want(0, 0, np.zeros(H))) < tol


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("D,R", [(20, 6), (64, 64), (128, 64), (48, 2), (272, 200)])
def test_norm_rotation_and_append(ops, dt, D, R):
    """Positions from the first to far beyond where a 32-bit product would be off; the rest of a head passes unturned."""
    H, G, V, P, eps = 3, 1, 24, 16, 1e-3
    Dp, Vp = (D + 15) // 16 * 16, 32
    pos = [0, 1, 15, 16, 511, 4000, 100000, 131071]
    T = len(pos)
    rot = {"base": 5e4, "dims": R, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 256}}
    f = K.frequencies(rot)
    q, k, v = rnd(1, T, H, D).to(dt), rnd(2, T, G, D).to(dt), rnd(3, T, G, V).to(dt)
    qn, kn = 1 + 0.2 * rnd(4, D), 1 + 0.2 * rnd(5, D)
    proj = torch.cat([pad_cols(q, Dp).reshape(T, -1), pad_cols(k, Dp).reshape(T, -1), pad_cols(v, Vp).reshape(T, -1)], 1).cuda()
    n_pages = max(pos) // P + 1
    table = torch.full((1, n_pages), -1, dtype=torch.int32)
    used = sorted({p // P for p in pos})
    for i, b in enumerate(used):
        table[0, b] = len(used) - 1 - i
    kp, vp = torch.zeros(len(used), G, P, Dp, dtype=dt, device="cuda"), torch.zeros(len(used), G, P, Vp, dtype=dt, device="cuda")
    out = torch.zeros(T, H * Dp, dtype=dt, device="cuda")
    ops.qkv_append(proj, 0, H * Dp, (H + G) * Dp, H, G, D, pad_cols(qn, Dp).cuda(), pad_cols(kn, Dp).cuda(), eps, ints([0] * T), ints(pos), table.cuda(),
                   out, kp, vp, P, False, torch.tensor(f, dtype=torch.float64, device="cuda"))
    p = np.array(pos, dtype=np.float64)
    tol = 3e-6 if dt == torch.float32 else 5e-3
    assert rel(f64(out).reshape(T, H, Dp)[..., :D], K.rotate(K.rms(f64(q), eps) * f64(qn), p, f)) < tol
    want = K.rotate(K.rms(f64(k), eps) * f64(kn), p, f)
    got = np.stack([f64(kp)[table[0, a // P], :, a % P, :D] for a in pos])
    assert rel(got, want) < tol
    assert rel(np.stack([f64(vp)[table[0, a // P], :, a % P, :V] for a in pos]), f64(v)) < 1e-6


# ---------------------------------------------------------------------------- latent attention in a window
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("window", [1, 20, 64, 65, 200, 0])
@pytest.mark.parametrize("H,D,V,C", [(3, 32, 16, 48), (20, 16, 32, 80), (2, 128, 128, 512)])
def test_latent_attention_in_a_window(ops, dt, H, D, V, C, window):
    """Unrotated queries; keys inside the window only, in the absorbed form (tokens, splits) and the expanded one (rows
    gathered from the window of the portion's first token on)."""
    P, scale = 16, 0.3
    lens, news = [1, 150, 90, 260, 64], [1, 150, 2, 70, 1]
    per = [-(-n // P) for n in lens]
    table = torch.full((len(lens), max(per)), -1, dtype=torch.int32)
    perm = torch.randperm(sum(per), generator=torch.Generator().manual_seed(1)).tolist()
    pages = torch.zeros(sum(per), 1, P, C)
    uk, uv = rnd(50, H, D, C, s=C ** -0.5).to(dt), rnd(51, H, V, C, s=C ** -0.5).to(dt)
    q, row, kv, want, at = [], [], [], [], 0
    for s, (n, m) in enumerate(zip(lens, news)):
        c, qs = rnd(s, n, C).to(dt), rnd(20 + s, n, H, D).to(dt)
        c[n // 3] *= 2
        for b in range(per[s]):
            table[s, b] = perm[at]
            pages[perm[at], 0, : min(P, n - b * P)] = c[b * P: (b + 1) * P].float()
            at += 1
        k, v = (np.einsum("hdc,jc->jhd", f64(u), f64(c)) for u in (uk, uv))
        want.append(K.attend(f64(qs), k, v, scale, K.sees(n, window))[n - m:])
        q.append(qs[n - m:].reshape(m, H * D))
        row += [s] * m
        kv += list(range(n - m + 1, n + 1))
    q, want, T = torch.cat(q).cuda(), np.concatenate(want), len(row)
    pages, table = pages.to(dt).cuda(), table.cuda()
    start = np.cumsum([0] + news)
    blocks = (ints([start[s] + o for s, m in enumerate(news) for o in range(0, m, 64)]), ints([min(64, m - o) for m in news for o in range(0, m, 64)]), 64)
    q_abs = torch.from_numpy(np.einsum("thd,hdc->thc", f64(q).reshape(T, H, D), f64(uk))).reshape(T, H * C).to(dt).cuda()
    freq = torch.zeros(0, dtype=torch.float64, device="cuda")
    row_d, kv_d, cu = ints(row), ints(kv), ints(start.tolist())
    args = (q_abs, q, pages, table, row_d, kv_d, H, 0, scale, freq, None)
    tol = 6e-6 if dt == torch.float32 else 2e-2

    def expand(o):
        return np.einsum("thc,hvc->thv", f64(o).reshape(T, H, C), f64(uv))
    out = torch.zeros((T, H * C), dtype=dt, device="cuda")
    ops.latent_token_attention(*args, out, False, window)
    assert rel(expand(out), want) < tol
    if dt == torch.float32:
        return
    keys = min(max(lens), window + 63) if window else max(lens)
    for split in (keys, 64, 32):
        n = -(-keys // split)
        po, ml = torch.empty(T * n * H * C, device="cuda"), torch.empty(T * n * H * 2, device="cuda")
        ops.latent_absorbed_attention(*args, out, *blocks, row_d, cu, 0, split, n, po, ml, False, window)
        assert rel(expand(out), want) < tol, split
    # expanded, for portions of 60 and more
    base, seqs, total = [], [], 0
    for s, (n, m) in enumerate(zip(lens, news)):
        first = max(0, n - m + 1 - window) if window else 0
        base.append([total, first] if m >= 60 else [-1, 0])
        if m >= 60:
            seqs.append([s, total, first, n - first])
            total += n - first
    rows = torch.zeros((total, C), dtype=dt, device="cuda")
    ops.latent_gather(pages, table, ints(seqs), max(s[3] for s in seqs), rows, False)
    c = rows.float().cpu()
    wide = torch.cat([torch.einsum("hdc,jc->jhd", u.float(), c).reshape(total, -1) for u in (uk, uv)], 1).to(dt).cuda()
    got = torch.full((T, H * V), 9.0, dtype=dt, device="cuda")
    ops.latent_expanded_attention(q, rows, wide, kv_d, H, C, 0, scale, freq, None, got, *blocks, row_d, ints(base), False, window)
    long = np.repeat(np.array(news) >= 60, news)
    assert rel(f64(got).reshape(T, H, V)[long], want[long]) < tol and (got[torch.from_numpy(~long).cuda()] == 9).all()


# ---------------------------------------------------------------------------- gated linear recurrence
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("blocks,width,taps", [(7, 16, 4), (1, 64, 7), (3, 28, 3), (2, 256, 4), (1, 192, 1), (2, 80, 2), (1, 544, 4)])
def test_gated_recurrence_over_cuts_and_batches(ops, dt, blocks, width, taps):
    """Three sequences in portions of all sizes on shuffled slots: in steps, and with the fused kernels (portions, single
    tokens).  Channels forget at once, almost never, and anything between; no other slot is touched."""
    np_ = (width + 15) // 16 * 16
    C, Cp = blocks * width, blocks * np_
    lens, slots, n_slots = [150, 70, 23], [4, 0, 2], 6

    def pad(t):                                       # [..., C] -> [..., Cp], block by block
        return pad_cols(t.reshape(*t.shape[:-1], blocks, width), np_).reshape(*t.shape[:-1], Cp)
    x, y = [rnd(s, n, C).to(dt) for s, n in enumerate(lens)], [rnd(9 + s, n, C).to(dt) for s, n in enumerate(lens)]
    conv, conv_b = rnd(20, C, taps), rnd(21, C, s=0.3)
    ga, gi = (rnd(22 + i, blocks, width, width, s=2 * width ** -0.5).to(torch.bfloat16) for i in range(2))
    ba, bi = rnd(24, blocks, width), rnd(25, blocks, width)
    lam = torch.linspace(-9.0, 2.0, C)[torch.randperm(C, generator=torch.Generator().manual_seed(0))]
    want, ends = [], []
    for xs, ys in zip(x, y):
        u = K.causal_conv(f64(xs), f64(conv), f64(conv_b))
        S = K.linear_recurrence(u, K.block_gate(u, f64(ga), f64(ba)), K.block_gate(u, f64(gi), f64(bi)), f64(lam))
        want.append(S * K.gelu_tanh(f64(ys)))
        ends.append(S)
    gates = torch.zeros(blocks, 2, np_, np_)
    gates[:, 0, :width, :width], gates[:, 1, :width, :width] = ga.float(), gi.float()
    gbias = torch.zeros(blocks, 2, np_)
    gbias[:, 0, :width], gbias[:, 1, :width] = ba, bi
    gates, gbias = gates.view(blocks, 2 * np_, np_).to(dt).cuda(), gbias.view(blocks, 2 * np_).cuda()
    rate = pad(8 * torch.nn.functional.softplus(lam.double())).float().cuda()
    cw, cb = torch.stack([pad(v) for v in conv.t()]).cuda(), pad(conv_b).cuda()
    fused = dt == torch.bfloat16 and bool(ops.rglru_fused_supported(np_))
    tol = 1e-5 if dt == torch.float32 else 2e-2
    for form in ("steps", "fused") if fused else ("steps",):
        ring, S = torch.full((n_slots, taps, Cp), 7.0, device="cuda"), torch.full((n_slots, Cp), 7.0, device="cuda")
        for s in slots:
            ring[s], S[s] = 0, 0
        at, step, got = [0, 0, 0], 0, [[], [], []]
        sizes = [[1, 1, 1], [64, 1, 2], [2, 33, 1], [65, 3, 7], [1, 1, 1], [1, 2, 4], [9, 40, 16]]
        while any(a < n for a, n in zip(at, lens)):
            todo = [(s, min(sizes[step % len(sizes)][s], lens[s] - at[s])) for s in range(3)]
            todo = [(s, n) for s, n in todo if n > 0]
            order = todo if step % 2 else todo[::-1]
            proj = torch.cat([torch.cat([pad(y[s][at[s]:at[s] + n]), pad(x[s][at[s]:at[s] + n])], 1) for s, n in order]).cuda()
            T, news = proj.shape[0], [n for _, n in order]
            cu = np.cumsum([0] + news)
            seq = ints(np.repeat(np.arange(len(order)), news).tolist())
            pos = ints([at[s] + i for s, n in order for i in range(n)])
            head = (proj, blocks, cw, cb, ints(cu.tolist()), seq, pos, ints([slots[s] for s, _ in order]), ring)
            out = torch.zeros(T, Cp, dtype=dt, device="cuda")
            for write in (False, True):              # a dry run first: it must leave the state as it is
                before = (ring.clone(), S.clone())
                if form == "steps":
                    u = torch.empty(T, Cp, dtype=dt, device="cuda")
                    ops.rglru_conv(*head, u, False)
                    raw = torch.einsum("tbi,boi->tbo", u.double().view(T, blocks, np_), gates.double()).float() + gbias
                    ops.rglru_scan(*head, u, raw.contiguous(), rate, S, out, write, False)
                else:
                    bs = ints([cu[i] + o for i, n in enumerate(news) for o in range(0, n, 64)])
                    bc = ints([min(64, n - o) for n in news for o in range(0, n, 64)])
                    ws = None
                    if max(news) > 1:
                        ws = torch.empty(int(ops.rglru_chunked_workspace_bytes(T, len(order), Cp)), dtype=torch.uint8, device="cuda")
                    ops.rglru(*head, gates, gbias, rate, S, out, bs, bc, ws, write, False)
                if not write:
                    assert torch.equal(ring, before[0]) and torch.equal(S, before[1])
            for i, (s, n) in enumerate(order):
                got[s].append(f64(out).reshape(T, blocks, np_)[cu[i]:cu[i + 1], :, :width].reshape(n, C))
                at[s] += n
                assert rel(f64(S[slots[s]]).reshape(blocks, np_)[:, :width].reshape(C), ends[s][at[s] - 1]) < tol, (form, s, at[s])
                for p in range(max(0, at[s] - taps), at[s]):
                    assert np.array_equal(f64(ring[slots[s], p % taps]).reshape(blocks, np_)[:, :width].reshape(C), f64(x[s][p]))
            step += 1
        for s in range(3):
            assert rel(np.concatenate(got[s]), want[s]) < tol, (form, s)
        others = [i for i in range(n_slots) if i not in slots]
        assert (ring[others] == 7).all() and (S[others] == 7).all()


def test_many_single_tokens_of_the_gated_recurrence(ops):
    """More sequences than one tile of tokens holds, each on its own slot, against the recurrence in steps."""
    blocks, n, taps, T = 2, 96, 4, 150
    C = blocks * n
    g = torch.Generator().manual_seed(3)
    slots = torch.randperm(T, generator=g)
    proj = rnd(1, T, 2 * C).to(torch.bfloat16).cuda()
    gates, gbias = rnd(2, blocks, 2 * n, n, s=n ** -0.5).to(torch.bfloat16).cuda(), rnd(3, blocks, 2 * n).cuda()
    rate, cw, cb = rnd(4, C).abs().cuda(), rnd(5, taps, C).cuda(), rnd(6, C).cuda()
    pos = torch.randint(0, 9, (T,), generator=g)
    seq = ints(list(range(T)))
    res = []
    for fused in (False, True):
        ring, S = rnd(7, T, taps, C).cuda(), rnd(8, T, C).cuda()
        out = torch.zeros(T, C, dtype=torch.bfloat16, device="cuda")
        head = (proj, blocks, cw, cb, ints(list(range(T + 1))), seq, ints(pos.tolist()), ints(slots.tolist()), ring)
        if fused:
            ops.rglru(*head, gates, gbias, rate, S, out, seq, seq, None, True, False)
        else:
            u = torch.empty(T, C, dtype=torch.bfloat16, device="cuda")
            ops.rglru_conv(*head, u, False)
            raw = torch.einsum("tbi,boi->tbo", u.double().view(T, blocks, n), gates.double()).float() + gbias
            ops.rglru_scan(*head, u, raw.contiguous(), rate, S, out, True, False)
        res.append((out, S, ring))
    assert rel(f64(res[1][0]), f64(res[0][0])) < 1e-2 and rel(f64(res[1][1]), f64(res[0][1])) < 1e-5 and torch.equal(res[1][2], res[0][2])


# ---------------------------------------------------------------------------- experts
@pytest.mark.parametrize("E,I,k", [(3, 0, 1), (8, 2, 2), (5, 3, 8), (64, 8, 6), (300, 20, 17), (512, 0, 4)])
def test_routing(ops, E, I, k):
    """Choice by corrected scores, weight by the scores alone, identities without rows, ties to the lower number."""
    T, n = 77, E + I
    z, corr = rnd(1, T, n, s=2.0), rnd(2, n, s=0.3)
    z[5] = 0.0
    corr[: n // 2] = corr[0].item()
    logits = torch.full((T, n + 3), 50.0)
    logits[:, :n] = z
    hist, ids = torch.zeros(E, dtype=torch.int32, device="cuda"), torch.zeros(T, k, dtype=torch.int32, device="cuda")
    weights, pos = torch.zeros(T, k, device="cuda"), torch.zeros(T, k, dtype=torch.int32, device="cuda")
    ops.moe_route_scored(logits.cuda(), E, I, k, corr.cuda(), 1.7, hist, ids, weights, pos, False)
    got = ids.cpu().numpy()
    assert K.shortfall(f64(z), f64(corr), got).max() < 1e-6
    assert np.array_equal(got[5], K.route(np.zeros((1, n)), f64(corr), k, 1.0)[0][0])
    assert rel(f64(weights), np.take_along_axis(K.router_scores(f64(z)), got.astype(np.int64), 1) * 1.7) < 2e-6
    flat, p = got.reshape(-1), pos.cpu().numpy().reshape(-1)
    for e in range(E):
        assert sorted(p[flat == e]) == list(range((flat == e).sum())) and int(hist[e]) == (flat == e).sum()
    assert (p[flat >= E] == -1).all()


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("case,layer", [("mixed", 0), ("mixed", 2), ("odd", 0), ("odd", 2), ("edges", 0), ("wide", 1)])
def test_experts(dt, case, layer):
    """The whole block on steps of 1 to 300 tokens, twice over with the same buffers: grouped GEMMs, bounded units, identities,
    the shared expert, padded widths."""
    import tuzupel_cases as C
    from ninfer_fusion_b200.models import tuzupel
    from ninfer_fusion_b200.models.experts import run_experts
    from ninfer_fusion_b200.models.layered import LayeredModel, LayeredWorkspace
    c, cfg, t, w = C.build(case)
    model = LayeredModel(cfg, tuzupel.pack(cfg, t.__getitem__, dt, "cuda:0"), "cuda:0")
    ws = LayeredWorkspace(cfg, 300, 8, "cuda:0", dt)
    spec, n, N = cfg.layers[layer].mlp, cfg.hidden, cfg.hidden_p
    for T in (1, 33, 300, 7):
        h = (rnd(T, T, n) * 1.5).to(dt)
        x, delta = pad_cols(h, N).cuda(), torch.full((T, N), 9.0, device="cuda")
        y = run_experts(model, ws.experts, T, f"text/layers/{layer}", spec, x, delta)
        out = torch.zeros((T, N), device="cuda")
        model.ops.mixture_rows(*y.values(), out, False)
        model.status.check()
        ids, short = y["choice"].cpu().numpy().astype(np.int64), []
        want = K.experts(w, f"l{layer}.mlp.", f64(h), c["layers"][layer]["mlp"], ids, short)
        assert short[0].max() < 1e-6
        assert rel(f64(out)[:, :n], want) < (5e-6 if dt == torch.float32 else 1.5e-2) and not out[:, n:].any()
        assert not ws.experts.hist.any()


@pytest.mark.parametrize("T", [1, 40, 300, 3000])
def test_bounded_units_and_soft_cap_in_gemm_epilogues(ops, T):
    """Every tile shape of the dense GEMM, the persistent kernel included."""
    Kd, F = 128, 5120
    x, wgu = rnd(1, T, Kd).to(torch.bfloat16), rnd(2, 2 * F, Kd, s=0.2).to(torch.bfloat16)
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    z = f64(x) @ f64(wgu).T
    for limit, slope, shift in ((1.5, 1.702, 1.0), (0.0, 1.0, 0.0)):
        out = torch.empty(T, F, dtype=torch.bfloat16, device="cuda")
        ops.gemm_bf16(x.cuda(), wgu.cuda(), out, 2, None, None, None, int(ops.gemm_pick_splits(T, 2 * F, Kd, 2)), status, False,
                      glu=[limit, slope, shift])
        g, u = z[:, :F], z[:, F:]
        want = K.glu_clamped(g, u, limit) if limit else g * K.sigmoid(g) * u
        assert rel(f64(out), want) < 6e-3
    cap = torch.tensor([5.0, 0.2], device="cuda")
    o32 = torch.empty(T, 2 * F, device="cuda")
    ops.gemm_bf16(x.cuda(), wgu.cuda(), None, 0, None, None, None, int(ops.gemm_pick_splits(T, 2 * F, Kd, 0)), status, False, 5, out32=o32, act_params=cap)
    assert rel(f64(o32), 5 * np.tanh(z / 5)) < 1e-5
    if T <= 300:
        ops.gemm_f32(x.float().cuda(), wgu.float().cuda(), None, None, 5, cap, o32, 0)
        assert rel(f64(o32), 5 * np.tanh(z / 5)) < 2e-6
    assert int(status) == 0
