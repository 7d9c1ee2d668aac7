"""Kernels of sigmoid attention, the state space, output norms with branches and grouped sigmoid routing, each mechanism alone
against the plain float64 functions of ratilorn_oracle."""
import numpy as np
import pytest
import torch

import ratilorn_oracle as K

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


# ---------------------------------------------------------------------------- embedding and row steps
@pytest.mark.parametrize("dt", DTYPES)
def test_embedding_with_positions(ops, dt):
    T, N, vocab, places = 6, 136, 11, 40
    table, pos = rnd(1, vocab, N).to(dt), rnd(2, places, N).to(dt)
    ids, at = [0, 10, 3, 3, 7, 1], [0, 39, 5, 6, 38, 0]
    x, xa = torch.empty(T, N, device="cuda"), torch.empty(T, N, dtype=dt, device="cuda")
    ops.embed_rows32(ints(ids), table.cuda(), x, xa, 1.0, False, ints(at), pos.cuda())
    want = f64(table)[ids] + f64(pos)[at]
    assert rel(f64(x), want) < 1e-7 and rel(f64(xa), want) < (1e-7 if dt == torch.float32 else 5e-3)


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("n", [24, 90, 208, 2048, 4096, 5000, 12288])
def test_output_norm_rows(ops, dt, n):
    """A GEMM's result, two branches, and a sum over experts with and without a gate; with the final norm and without."""
    T, N, eps, k, E = 5, (n + 7) // 8 * 8, 1e-3, 3, 4
    x, a, b = rnd(1, T, n), rnd(2, T, n) * 3, rnd(3, T, n) * 0.1
    w, wa, wb, wf = (1 + 0.3 * rnd(4 + i, n) for i in range(4))
    ret, weight, gate = rnd(9, T, k, n).to(dt), rnd(10, T, k).abs(), rnd(11, T, 2)
    choice = torch.tensor([[0, 1, 2], [3, 0, 1], [2, 1, 0], [3, 2, 1], [1, 3, 0]])
    dev = lambda t: pad_cols(t, N).contiguous().cuda()
    summed = (f64(weight)[..., None] * f64(ret)).sum(1)
    h = dev(rnd(12, T, n).to(dt))
    sel = (ints(choice.tolist()), weight.cuda(), dev(ret).view(T * k, N), h, E)
    none4, none7 = (None,) * 4, (None,) * 6 + (0,)
    forms = {"plain": (none4, (dev(a), None, None, None, None, None, 0), f64(a)),
             "pair": ((dev(a), dev(b), dev(wa), dev(wb)), none7, 0.5 * (K.rms(f64(a), eps) * f64(wa) + K.rms(f64(b), eps) * f64(wb))),
             "experts": (none4, (None, None, *sel), summed),
             "shared": (none4, (dev(a), None, *sel), summed + f64(a)),
             "gated": (none4, (dev(a), gate.cuda()[:, 1:2], *sel), summed + K.sigmoid(f64(gate)[:, 1:2]) * f64(a))}
    tol = 4e-6 if dt == torch.float32 else 5e-3
    for what, (branches, parts, y) in forms.items():
        new = f64(x) + K.rms(y, eps) * f64(w)
        for final in (False, True):
            xd, out = dev(x), torch.full((T, N), 9.0, dtype=dt, device="cuda")
            ops.branch_rows(xd, *branches, *parts, dev(w), dev(wf) if final else None, out, n, eps, False)
            assert rel(f64(xd)[:, :n], new) < 4e-6 and not xd[:, n:].any(), (what, final)
            assert rel(f64(out)[:, :n], K.rms(new, eps) * f64(wf) if final else new) < tol and not out[:, n:].any(), (what, final)


# ---------------------------------------------------------------------------- sigmoid attention
class Heads:
    """Sequences `lens` long of which the last `news` tokens are queries, rows scattered over shuffled pages; one key per
    sequence stands out."""

    def __init__(self, H, G, D, V, dt, lens, news, P, seed=0):
        self.lens, self.news, self.scale = lens, news, 1.5 * D ** -0.5
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

    def want(self, r1, r2, offset, talk, window=0):
        out = []
        for q, k, v, n, m in zip(self.q, self.k, self.v, self.lens, self.news):
            a = K.sigmoid_weights(K.scores(q, k, self.scale) - K.log_distance_bias(n, r1, r2), offset)
            if window:
                i = np.arange(n)
                a = a * (i[:, None] - i[None, :] < window)
            out.append(K.weighted_values(K.mix_heads(a, talk), v)[n - m:])
        return np.concatenate(out)

    def get(self, out):
        o = out.view(self.T, self.H, self.Vp)
        assert not o[..., self.V:].any()
        return f64(o)[..., : self.V]


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,G,D,V,P", [(6, 2, 32, 48, 16), (5, 5, 20, 12, 8), (16, 4, 64, 64, 64), (8, 2, 128, 128, 64), (32, 8, 96, 32, 64), (20, 1, 64, 64, 16),
                                       (40, 4, 16, 16, 16), (3, 1, 160, 256, 64), (2, 2, 272, 304, 16)])
def test_sigmoid_attention(ops, dt, H, G, D, V, P):
    """Portions and single tokens in one step, splits, with and without a window: every form against the oracle.  Weights of
    all sizes: offsets from -12 to 2, biases that vanish and that cut far keys off."""
    x = Heads(H, G, D, V, dt, [1, 130, 70, 300, 64, 129], [1, 130, 3, 75, 1, 64], P)
    r1, r2, offset = np.linspace(0.0, 2.0, H).astype(np.float32), np.linspace(5.0, 0.0, H).astype(np.float32), np.linspace(-12.0, 2.0, H).astype(np.float32)
    talk = np.random.default_rng(3).normal(size=(H, H)).astype(np.float32) * H ** -0.5
    dev = [torch.from_numpy(a).cuda() for a in (r1, r2, offset, talk)]
    tol = 5e-6 if dt == torch.float32 else 1.2e-2
    for window in (0, 37):
        want = x.want(r1, r2, offset, talk, window)
        shape, extra = (window, x.scale, 0.0, 0.0, dev[3], None, None), (True, *dev[:3])
        for split, n in ((320, 1), (64, 5)):
            po, ml = torch.empty(x.T * n * H * x.Vp, device="cuda"), torch.empty(x.T * n * H * 2, device="cuda")
            out = torch.full((x.T, H * x.Vp), 9.0, dtype=dt, device="cuda")
            ops.head_mix_attention(*x.args, *shape, out, split, n, po, ml, False, 0, None, *extra)
            assert rel(x.get(out), want) < tol, (window, split)
        if dt == torch.bfloat16:
            one = int(ops.head_mix_prefill_scratch(H, 300, window, 1, True))
            for blocks in (x.blocks[0].numel(), 2):           # all at a time, and as many as a small scratch holds
                scratch = torch.empty(one * blocks, dtype=torch.uint8, device="cuda")
                out = torch.full((x.T, H * x.Vp), 9.0, dtype=dt, device="cuda")
                ops.head_mix_prefill(*x.args, *shape, out, *x.blocks, 300, scratch, False, *extra)
                assert rel(x.get(out), want) < tol, (window, blocks)
    # without a bias, an offset or a mix
    out = torch.full((x.T, H * x.Vp), 9.0, dtype=dt, device="cuda")
    ops.head_mix_attention(*x.args, 0, x.scale, 0.0, 0.0, None, None, None, out, 320, 1, None, None, False, 0, None, True)
    assert rel(x.get(out), x.want(0 * r1, 0 * r2, 0 * offset, np.eye(H))) < tol


def test_far_keys_of_sigmoid_attention(ops):
    """One key that stands out at every distance up to 5000, decoded alone: small weights elsewhere keep their relative size."""
    H, G, D, V, P, n = 4, 2, 64, 64, 64, 5001
    q, k, v = torch.zeros(H, D), torch.zeros(n, G, D), torch.zeros(n, G, V)
    q[:, 0] = 8.0
    v[:, :, 0] = 1.0
    for far in (0, 1, 15, 16, 63, 64, 65, 1000, 4999, 5000):
        k.zero_()
        k[n - 1 - far, :, 0] = 8.0
        v[:, :, 1] = 0.0
        v[n - 1 - far, :, 1] = 1.0
        kp = torch.zeros((n + P - 1) // P * P, G, D)
        vp = torch.zeros_like(kp)
        kp[:n], vp[:n] = k, v
        pages = [t.view(-1, P, G, D).transpose(1, 2).contiguous().cuda() for t in (kp, vp)]
        r1, r2, off = np.array([0.5, 1.0, 0.0, 0.3]), np.array([1.0, 0.25, 0.0, 2.0]), np.array([-8.0, -9.0, -10.0, -11.0])
        d = n - 1 - np.arange(n)
        s = (f64(q) @ f64(k[:, 0]).T) * 0.2 - r1[:, None] * np.log(1 + r2[:, None] * d)
        a = K.sigmoid(s + off[:, None])
        want = np.stack([a.sum(1), a[:, n - 1 - far]], 1)
        for dt in DTYPES:
            dev = [torch.from_numpy(x).float().cuda() for x in (r1, r2, off)]
            out = torch.zeros(1, H * V, dtype=dt, device="cuda")
            po, ml = torch.empty(40 * H * V, device="cuda"), torch.empty(40 * H * 2, device="cuda")
            ops.head_mix_attention(q.reshape(1, -1).to(dt).cuda(), *(t.to(dt) for t in pages), torch.arange(pages[0].shape[0], dtype=torch.int32, device="cuda")[None],
                                   ints([0]), ints([n]), 0, 0.2, 0.0, 0.0, None, None, None, out, 128, 40, po, ml, False, 0, None, True, *dev)
            got = f64(out).reshape(H, V)[:, :2]
            assert (np.abs(got - want) < (1e-5 if dt == torch.float32 else 1.5e-2) * np.abs(want)).all(), (far, dt)


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("D,V", [(20, 24), (64, 48), (272, 144)])
def test_unit_norm_and_mixed_values(ops, dt, D, V):
    """q and k normed without weights, values kept for later layers, and mixed with those of an earlier one."""
    H, G, P, eps, lam = 3, 2, 16, 1e-3, 0.3125
    Dp, Vp = (D + 15) // 16 * 16, (V + 15) // 16 * 16
    pos = [0, 1, 15, 16, 40]
    T = len(pos)
    q, k, v, first = (rnd(i, T, h, d).to(dt) for i, (h, d) in enumerate(((H, D), (G, D), (G, V), (G, V))))
    proj = torch.cat([pad_cols(q, Dp).reshape(T, -1), pad_cols(k, Dp).reshape(T, -1), pad_cols(v, Vp).reshape(T, -1)], 1).cuda()
    table = ints([[2, 0, 1]])
    head = (proj, 0, H * Dp, (H + G) * Dp, H, G, D, None, None, eps, ints([0] * T), ints(pos), table)
    for mixed in (False, True):
        kp, vp = torch.zeros(3, G, P, Dp, dtype=dt, device="cuda"), torch.zeros(3, G, P, Vp, dtype=dt, device="cuda")
        out, buf = torch.zeros(T, H * Dp, dtype=dt, device="cuda"), pad_cols(first, Vp).reshape(T, -1).cuda()
        ops.qkv_append(*head, out, kp, vp, P, False, None, True, buf, torch.tensor([lam], device="cuda") if mixed else None)
        tol = 3e-6 if dt == torch.float32 else 5e-3
        assert rel(f64(out).reshape(T, H, Dp)[..., :D], K.rms(f64(q), eps)) < tol
        cells = [([2, 0, 1][a // P], a % P) for a in pos]
        assert rel(np.stack([f64(kp)[c, :, r, :D] for c, r in cells]), K.rms(f64(k), eps)) < tol
        want = K.mix_values(f64(v), f64(first), lam) if mixed else f64(v)
        assert rel(np.stack([f64(vp)[c, :, r, :V] for c, r in cells]), want) < tol
        assert np.array_equal(f64(buf).reshape(T, G, Vp)[..., :V], f64(first if mixed else v))


# ---------------------------------------------------------------------------- state space
def padded(t, parts):
    """Columns in runs of (count, true width, padded width)."""
    out, at = [], 0
    for n, w, wp in parts:
        out.append(pad_cols(t[..., at: at + n * w].reshape(*t.shape[:-1], n, w), wp).reshape(*t.shape[:-1], n * wp))
        at += n * w
    return torch.cat(out, -1)


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,V,N,G,taps", [(4, 32, 48, 2, 4), (3, 20, 24, 1, 1), (8, 16, 128, 4, 7), (6, 64, 64, 1, 4), (2, 144, 272, 1, 4), (5, 64, 128, 1, 2), (2, 80, 16, 2, 3),
                                         (1, 16, 500, 1, 4)])
def test_state_space_over_cuts_and_batches(ops, dt, H, V, N, G, taps):
    """Three sequences in portions of all sizes on shuffled slots: token by token and in chunks.  Heads forget at once, almost
    never, and anything between; no other slot is touched, and a dry run leaves the state as it is."""
    Vp, Np = (V + 15) // 16 * 16, (N + 15) // 16 * 16
    inner, K_, Kp = H * V, H * V + 2 * G * N, H * Vp + 2 * G * Np
    runs = [(H, V, Vp), (G, N, Np), (G, N, Np)]
    lens, slots, n_slots = [150, 70, 23], [4, 0, 2], 6
    x = [rnd(s, n, K_).to(dt) for s, n in enumerate(lens)]
    raw = [rnd(9 + s, n, H, s=2.0) + torch.linspace(-7.0, 2.0, H) for s, n in enumerate(lens)]
    conv, conv_b = rnd(20, K_, taps, s=taps ** -0.5), rnd(21, K_, s=0.3)
    A, D = torch.linspace(2.0, -2.0, H), rnd(22, H)
    want, ends = [], []
    for xs, rs in zip(x, raw):
        u = K.silu(K.causal_conv(f64(xs), f64(conv), f64(conv_b)))
        xx, B, C = np.split(u, [inner, inner + G * N], axis=1)
        args = (xx.reshape(-1, H, V), B.reshape(-1, G, N), C.reshape(-1, G, N), K.softplus(f64(rs)))
        want.append(K.state_space(*args, f64(A), f64(D))[0])
        ends.append(args)
    cw, cb = torch.stack([padded(v, runs) for v in conv.t()]).cuda(), padded(conv_b, runs).cuda()
    rate, skip = A.double().exp().float().cuda(), D.cuda()
    chunked = dt == torch.bfloat16 and bool(ops.ssd_chunked_supported(Np, Vp))
    tol = 1e-5 if dt == torch.float32 else 2e-2
    for form in ("tokens", "chunks") if chunked else ("tokens",):
        ring, S = torch.full((n_slots, taps, Kp), 7.0, device="cuda"), torch.full((n_slots, H, Vp, Np), 7.0, device="cuda")
        for s in slots:
            ring[s], S[s] = 0, 0
        at, step, got = [0, 0, 0], 0, [[], [], []]
        sizes = [[1, 1, 1], [64, 1, 2], [2, 33, 1], [65, 3, 7], [1, 1, 1], [1, 2, 4], [9, 40, 16]]
        while any(a < n for a, n in zip(at, lens)):
            todo = [(s, min(sizes[step % len(sizes)][s], lens[s] - at[s])) for s in range(3)]
            todo = [(s, n) for s, n in todo if n > 0]
            order = todo if step % 2 else todo[::-1]
            proj = torch.cat([padded(x[s][at[s]:at[s] + n], runs) for s, n in order])
            proj = torch.cat([torch.full((proj.shape[0], 16), 3.0, dtype=dt), proj], 1).cuda()       # columns that are somebody else's
            dts = torch.cat([raw[s][at[s]:at[s] + n] for s, n in order]).cuda()
            T, news = proj.shape[0], [n for _, n in order]
            cu = np.cumsum([0] + news)
            one = max(news) == 1
            ws = None
            if form == "chunks" and not one:
                ws = torch.empty(int(ops.ssd_chunked_workspace_bytes(T, len(order), H, Np, Vp)), dtype=torch.uint8, device="cuda")
            u = torch.empty(T * Kp, dtype=dt, device="cuda")
            out = torch.zeros(T, H * Vp, dtype=dt, device="cuda")
            for write in (False, True):
                before = (ring.clone(), S.clone())
                ops.ssd(proj, 16, dts, cw, cb, rate, skip, G, ints(cu.tolist()), ints(np.repeat(np.arange(len(order)), news).tolist()),
                        ints([at[s] + i for s, n in order for i in range(n)]), ints([slots[s] for s, _ in order]), ring, S, u, out, write, ws, False, one)
                if not write:
                    assert torch.equal(ring, before[0]) and torch.equal(S, before[1])
            for i, (s, n) in enumerate(order):
                got[s].append(f64(out).reshape(T, H, Vp)[cu[i]:cu[i + 1], :, :V])
                at[s] += n
                end = K.state_space(*(a[: at[s]] for a in ends[s]), f64(A), f64(D))[1]
                assert rel(f64(S[slots[s]])[:, :V, :N].transpose(0, 2, 1), end) < tol, (form, s, at[s])
                for p in range(max(0, at[s] - taps), at[s]):
                    assert np.array_equal(f64(ring[slots[s], p % taps]), f64(padded(x[s][p], runs)))
            step += 1
        for s in range(3):
            assert rel(np.concatenate(got[s]), want[s]) < tol, (form, s)
        others = [i for i in range(n_slots) if i not in slots]
        assert (ring[others] == 7).all() and (S[others] == 7).all()


@pytest.mark.parametrize("dt", DTYPES)
def test_a_state_that_hardly_decays(ops, dt):
    """One strong input at the first token, read back 700 tokens later through decays of 1e-4 per token, whatever the cuts."""
    H, V, N, T, taps = 2, 16, 16, 700, 1
    Kp = H * V + 2 * N
    x = torch.zeros(T, Kp)
    x[0, : H * V], x[0, H * V] = 20.0, 20.0                  # x and the first column of B at token 0
    x[-1, H * V + N] = 20.0                                  # the first column of C at the last token
    raw = torch.full((T, H), float(np.log(np.expm1(1e-2))))
    rate = torch.tensor([1e-2, 1e-1], device="cuda")
    dt_ = K.softplus(f64(raw))
    u = K.silu(f64(x))
    want, _ = K.state_space(u[:, : H * V].reshape(T, H, V), u[:, None, H * V: H * V + N], u[:, None, H * V + N:], dt_, np.log(f64(rate)), np.zeros(H))
    cw, cb = torch.ones(1, Kp, device="cuda"), torch.zeros(Kp, device="cuda")
    proj, raw = x.to(dt).cuda(), raw.cuda()
    for cuts in ([700], [1] * 700, [350, 1, 349], [2] * 350):
        for chunks in ((False, True) if dt == torch.bfloat16 and max(cuts) > 1 else (False,)):
            ring, S = torch.zeros(1, taps, Kp, device="cuda"), torch.zeros(1, H, V, N, device="cuda")
            at = 0
            for n in cuts:
                ws = torch.empty(int(ops.ssd_chunked_workspace_bytes(n, 1, H, N, V)), dtype=torch.uint8, device="cuda") if chunks else None
                out, buf = torch.zeros(n, H * V, dtype=dt, device="cuda"), torch.empty(n * Kp, dtype=dt, device="cuda")
                ops.ssd(proj[at:at + n], 0, raw[at:at + n], cw, cb, rate, torch.zeros(H, device="cuda"), 1, ints([0, n]), ints([0] * n), ints(list(range(at, at + n))),
                        ints([0]), ring, S, buf, out, True, ws if n > 1 else None, False, n == 1)
                at += n
            assert rel(f64(out)[-1].reshape(H, V), want[-1]) < (2e-5 if dt == torch.float32 else 1e-2), (cuts[0], chunks)


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,V,parts", [(4, 32, 2), (3, 20, 4), (5, 12, 1), (2, 48, 3), (64, 64, 8), (64, 64, 1), (2, 24, 6), (7, 16, 112)])
def test_gated_norm(ops, dt, H, V, parts):
    """Parts that are heads, several heads, or cut through heads; padded heads."""
    T, eps, Vp = 6, 1e-3, (V + 15) // 16 * 16
    y, z, w = rnd(1, T, H * V).to(dt), rnd(2, T, H * V).to(dt), 1 + 0.3 * rnd(3, H * V)
    pad = lambda t: padded(t, [(H, V, Vp)]).cuda()
    yd = torch.cat([pad(y), torch.full((T, 8), 5.0, dtype=dt, device="cuda")], 1)
    ops.ssd_gated_norm(yd[:, :-8], pad(z), pad(w), H, V, parts, eps, False)
    want = K.gated_group_norm(f64(y), f64(z), f64(w), parts, eps)
    got = f64(yd[:, :-8]).reshape(T, H, Vp)
    assert rel(got[..., :V].reshape(T, -1), want) < (3e-6 if dt == torch.float32 else 6e-3)
    assert not got[..., V:].any() and (yd[:, -8:] == 5).all()


# ---------------------------------------------------------------------------- routing
@pytest.mark.parametrize("E,k,groups", [(3, 1, None), (8, 2, (4, 1)), (12, 4, (3, 2)), (64, 6, (8, 3)), (300, 17, (20, 4)), (512, 4, (64, 40)), (512, 8, None), (6, 2, (6, 3)),
                                        (40, 33, (2, 2))])
def test_sigmoid_routing_in_groups(ops, E, k, groups):
    """Groups by their two best corrected scores, choices inside the best of them, weights divided by their sum."""
    T = 77
    z, corr = rnd(1, T, E, s=2.0), rnd(2, E, s=0.3) - 0.8
    logits = torch.full((T, E + 3), 50.0)
    logits[:, :E] = z
    hist, ids = torch.zeros(E, dtype=torch.int32, device="cuda"), torch.zeros(T, k, dtype=torch.int32, device="cuda")
    weights, pos = torch.zeros(T, k, device="cuda"), torch.zeros(T, k, dtype=torch.int32, device="cuda")
    ops.moe_route_scored(logits.cuda(), E, 0, k, corr.cuda(), 1.0, hist, ids, weights, pos, False, True, True, *(groups or (0, 0)))
    r = {"experts": E, "top": k}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    got = ids.cpu().numpy().astype(np.int64)
    assert K.shortfall(f64(z), f64(corr), r, got).max() < 1e-6
    assert rel(f64(weights), K.route(f64(z), f64(corr), r, got)[1]) < 2e-6
    flat, p = got.reshape(-1), pos.cpu().numpy().reshape(-1)
    for e in range(E):
        assert sorted(p[flat == e]) == list(range((flat == e).sum())) and int(hist[e]) == (flat == e).sum()


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("case,layer", [("mixed", 1), ("mixed", 2), ("odd", 0), ("many_heads", 2), ("mixed", 0), ("odd", 1)])
def test_feed_forwards(dt, case, layer):
    """Experts with a plain shared one or none, and dense gated units, on steps of 1 to 300 tokens with the same buffers."""
    import ratilorn_cases as C
    from ninfer_fusion_b200.models import ratilorn
    from ninfer_fusion_b200.models.experts import run_experts
    from ninfer_fusion_b200.models.layered import LayeredModel, LayeredWorkspace
    c, cfg, t, w = C.build(case)
    model = LayeredModel(cfg, ratilorn.pack(cfg, t.__getitem__, dt, "cuda:0"), "cuda:0")
    ws = LayeredWorkspace(cfg, 300, 8, "cuda:0", dt)
    spec, n, N, p = cfg.layers[layer].mlp, cfg.hidden, cfg.hidden_p, f"text/layers/{layer}"
    for T in (1, 33, 300, 7):
        h = (rnd(T, T, n) * 1.5).to(dt)
        x, tol = pad_cols(h, N).cuda(), 5e-6 if dt == torch.float32 else 1.5e-2
        if spec.kind == "glu":
            ws.xa[:T] = x
            model._feed_forward(ws, T, p, spec, None)
            out, want = ws.delta[:T], K.glu(w, f"l{layer}.mlp", f64(h))
        else:
            y = run_experts(model, ws.experts, T, p, spec, x, torch.full((T, N), 9.0, device="cuda"))
            out = torch.zeros((T, N), device="cuda")
            model.ops.mixture_rows(*y.values(), out, False)
            ids, short = y["choice"].cpu().numpy().astype(np.int64), []
            want = K.experts(w, f"l{layer}.mlp.", f64(h), c["layers"][layer]["mlp"], ids, short)
            assert short[0].max() < 1e-6 and not ws.experts.hist.any()
        model.status.check()
        assert rel(f64(out)[:, :n], want) < tol and not out[:, n:].any()
