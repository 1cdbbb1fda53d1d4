"""Each mechanism of the Lerosun kernels alone, against the oracle's equations in float64."""
import pytest
import torch

import lerosun_oracle as P

pytestmark = pytest.mark.gpu
DEV = "cuda"
BF, F32 = torch.bfloat16, torch.float32


def _rel(a, b):
    a, b = a.double().cpu(), b.double().cpu()
    return float((a - b).norm() / (b.norm() + 1e-30))


def _ok():
    from rumus_b200.ops import native
    return native.read_status() == 0


def p8(n):
    return (n + 7) // 8 * 8


def _pad(t, n):
    return torch.nn.functional.pad(t, (0, n - t.shape[-1]))


# ------------------------------------------------------------------------------------------ around the sub-layers
@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("D,T", [(64, 5), (50, 3), (1003, 40), (2052, 2), (9000, 3)])
def test_normed_embeddings(dt, D, T):
    from rumus_b200.ops import stream
    torch.manual_seed(D)
    table, g = torch.randn(30, D).to(dt) * 0.1, torch.tensor([1.7])
    ids = torch.randint(0, 30, (T,))
    ids[-1] = 99                                     # no such token
    for w in (torch.tensor([0.6]), torch.randn(D)):
        x, h = stream.embed_norm(ids.to(DEV), table.to(DEV), g.to(DEV), w.to(DEV), 1e-2, p8(D))
        want = P.embed(ids[:-1], table.double(), 1.7, 1e-2)
        assert _rel(x[:-1], want) < 1e-6 and bool((x[-1] == 0).all()) and bool((h[-1] == 0).all())
        assert _rel(h[:-1, :D], P.rms(want, 1e-2) * w.double()) < (4e-3 if dt == BF else 1e-6)
        assert bool((h[:, D:] == 0).all())


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("D,T", [(64, 5), (50, 3), (1003, 70), (2052, 300), (5000, 2), (13000, 2)])
def test_scaled_results_join_the_residual(dt, D, T):
    from rumus_b200.ops import stream
    torch.manual_seed(D)
    x, y, s = torch.randn(T, D), torch.randn(T, D), torch.randn(D)
    want = x.double() + s.double() * y.double()
    for w in (torch.tensor([0.6]), torch.randn(D)):
        for keep in (True, False):
            xd = x.to(DEV)
            h = stream.scaled_add_norm(xd, y.to(DEV), s.to(DEV), w.to(DEV), 1e-2, dt, p8(D), keep=keep)
            assert _rel(xd, want) < 1e-6 if keep else torch.equal(xd.cpu(), x)
            assert _rel(h[:, :D], P.rms(want, 1e-2) * w.double()) < (4e-3 if dt == BF else 1e-6)
            assert bool((h[:, D:] == 0).all())


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("F", [33, 64, 1000])
def test_gated_relu(dt, F):
    from rumus_b200.ops import stream
    gu = torch.randn(70, 2 * F).to(dt)
    out = torch.empty(70, F, device=DEV, dtype=dt)
    stream.glu(stream.GLU_RELU, gu.to(DEV), out)
    want = torch.relu(gu[:, :F].double()) * gu[:, F:].double()
    assert _rel(out, want) < (4e-3 if dt == BF else 1e-6) and bool(((out == 0).cpu() == (want == 0)).all())


# ------------------------------------------------------------------------------------------ attention
def _paged(ctxs, G, bs, dp, dt):
    """Pools with the pages of several sequences in a shuffled order, tables, and a reader of a sequence's rows."""
    need = [(c + bs - 1) // bs for c in ctxs]
    nb = sum(need) + 3
    kp, vp = torch.randn(nb, G, bs, dp, device=DEV).to(dt), torch.randn(nb, G, bs, dp, device=DEV).to(dt)
    perm = torch.randperm(nb)
    tab, k = torch.zeros(len(ctxs), max(need), dtype=torch.int32), 0
    for i, n in enumerate(need):
        tab[i, :n] = perm[k:k + n]
        k += n

    def rows(i):
        t = torch.arange(ctxs[i])
        b, o = tab[i, t // bs].long().to(DEV), (t % bs).to(DEV)
        return kp[b, :, o].double().cpu(), vp[b, :, o].double().cpu()

    return kp, vp, tab.to(DEV), rows


def _heads(q, rows, mix, scale, sink, size, offset):
    """q [T, H, d] and keys as they are (already rotated)."""
    k, v = rows
    H, G = q.shape[1], k.shape[1]
    s = P.talk(P.scores(q.double().cpu(), k, scale, torch.ones(H)), mix.double().cpu())
    none = torch.tensor(-1e30, dtype=torch.float64)
    return torch.stack([P.attend(s[h], v[:, h // (H // G)], none if sink is None else sink[h].double().cpu(), size, offset) for h in range(H)], 1)


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("H,G,dim,rot,rows", [(3, 1, 10, 6, 2), (4, 2, 24, 24, 0), (8, 1, 128, 64, 5), (6, 2, 200, 2, 9), (5, 5, 64, 0, 3),
                                             (12, 4, 20, 12, 4), (20, 1, 16, 8, 9)])
def test_after_the_projection(dt, H, G, dim, rot, rows):
    """Rotated and plain keys go to their cache rows; queries change in place or leave mixed."""
    from rumus_b200.ops import stream, talk
    torch.manual_seed(dim + H)
    T, bs, dp = 9, 4, p8(dim)
    proj = torch.cat([_pad(torch.randn(T, n, dim), dp).flatten(1) for n in (H, G)] + [torch.randn(T, 8)], 1).to(dt)
    pos, slots = torch.randint(0, 5000, (T,)), torch.randperm(5 * bs)[:T]
    slots[3] = -1
    mix = torch.randn(H, H)
    freq = 300.0 ** (-2.0 * torch.arange(max(rot, 2) // 2, dtype=torch.float64) / max(rot, 2))
    tab = stream.rotary_table(pos.to(DEV), freq.float().to(DEV), 1.0)
    kp, vp = (torch.full((5, G, bs, dp), 7.0, device=DEV, dtype=dt) for _ in range(2))
    got = proj.to(DEV)
    qmix = talk.talk_post(got, slots.to(DEV), kp, vp, mix.to(DEV), H, rows, **(dict(tab=tab, rot=rot) if rot else {}))
    x = proj[:, :(H + G) * dp].double().view(T, H + G, dp)
    want = P.rotate(x, pos.tolist(), {"dims": rot, "base": 300.0})
    tol = 4e-3 if dt == BF else 2e-4                # positions in the thousands, angles in 32 bits
    if rows:
        assert _rel(got[:rows, :H * dp].view(rows, H, dp), want[:rows, :H]) < tol
    assert torch.equal(got[rows:].cpu(), proj[rows:]) and torch.equal(got[:, H * dp:].cpu(), proj[:, H * dp:])
    if rows < T:
        q = want[rows:, :H].view(T - rows, G, H // G, dp)
        assert _rel(qmix, torch.einsum("hcr,tcrd->thcd", mix.double().view(H, G, H // G), q)) < tol
    else:
        assert qmix is None
    for t in range(T):
        s = int(slots[t])
        if s >= 0:
            assert _rel(kp[s // bs, :, s % bs], want[t, H:]) < tol and torch.equal(vp[s // bs, :, s % bs].cpu(), x[t, H:].to(dt))
    touched = torch.zeros(5 * bs, dtype=torch.bool)
    touched[slots[slots >= 0]] = True
    assert bool((kp.transpose(1, 2).reshape(5 * bs, -1)[~touched.to(DEV)] == 7).all())


def _mix(H):
    return (torch.eye(H) * (0.5 + torch.rand(H, 1)) + 0.4 * torch.randn(H, H) / H ** 0.5).to(DEV)


ROWS = [  # heads, kv heads, dim, window, page, contexts
    (4, 2, 48, 37, 16, [1, 4, 37, 38, 41, 42, 100]), (3, 3, 16, 64, 64, [63, 64, 65, 128, 129, 192, 300]),
    (8, 1, 128, 100, 64, [700, 130, 2, 99, 100, 101]), (10, 2, 72, 1, 8, [1, 2, 3, 64, 65]), (6, 2, 200, 50, 32, [49, 50, 51, 400]),
    (2, 1, 264, 20, 16, [5, 20, 21, 90]), (16, 4, 128, 130, 64, [130, 131, 194, 500]), (32, 8, 64, 300, 64, [64, 600]),
    (20, 1, 56, 1 << 30, 8, [8, 129, 500]), (12, 4, 64, 80, 48, [79, 80, 81, 143, 144, 200]), (32, 8, 128, 200, 64, [333]), (9, 9, 24, 70, 64, [69, 200]),
]


@pytest.mark.parametrize("dt,plain", [(BF, False), (BF, True), (F32, True)])
@pytest.mark.parametrize("case", ROWS)
@pytest.mark.parametrize("splits", [1, 0, 5])
def test_rows_of_talking_heads(dt, plain, case, splits):
    from rumus_b200.ops import talk
    H, G, dim, W, bs, ctxs = case
    torch.manual_seed(H + dim)
    kp, vp, tab, rows = _paged(ctxs, G, bs, dim, dt)
    n, mix = len(ctxs), _mix(H)
    q = (torch.randn(n, H, dim, device=DEV) * 2).to(dt)
    sink, gate = torch.randn(H, device=DEV), torch.randn(n, H, device=DEV).to(dt)
    for s, kind in ((sink, 2), (None, 0)):
        out = torch.full((n, H * dim + 8), 3.0, device=DEV, dtype=dt)
        talk.talk_rows_attention(q, kp, vp, tab, torch.tensor(ctxs, dtype=torch.int32, device=DEV), mix, s, gate if kind else None, kind,
                                 out[:, :H * dim], W, dim ** -0.5, max(ctxs), splits=splits, plain=plain)
        assert _ok() and bool((out[:, H * dim:] == 3).all())
        for i, c in enumerate(ctxs):
            want = _heads(q[i:i + 1], rows(i), mix, dim ** -0.5, s, W, c - 1)[0]
            if kind:
                want = want * P.sigmoid(gate[i].double().cpu())[:, None]
            assert _rel(out[i, :H * dim].view(H, dim), want) < (8e-3 if dt == BF else 5e-6), (i, c)


@pytest.mark.parametrize("H,G,dim,W,bs,segs", [
    (4, 2, 48, 37, 16, [(0, 23), (30, 60), (100, 29)]), (6, 2, 64, 80, 64, [(0, 300), (145, 140), (500, 2), (63, 129)]),
    (2, 1, 128, 30, 64, [(5, 130), (0, 128), (400, 9), (95, 40)]), (2, 2, 72, 1, 8, [(0, 65), (129, 127)]),
    (3, 1, 16, 200, 128, [(0, 200), (330, 130)]), (8, 4, 128, 64, 32, [(0, 70), (200, 130)]), (5, 5, 64, 65, 64, [(128, 128), (127, 3), (64, 64)]),
    (10, 5, 96, 90, 64, [(0, 140), (77, 60)]), (8, 8, 128, 1 << 30, 64, [(100, 130)]), (16, 16, 40, 50, 64, [(33, 70)]), (8, 1, 56, 129, 64, [(1, 300)]),
])
def test_prompts_of_talking_heads(H, G, dim, W, bs, segs):
    from rumus_b200.ops import talk
    from rumus_b200.ops.latent import prefill_items
    torch.manual_seed(dim + H)
    assert talk.prefill_covered(BF, H, G, dim, dim, bs, 1.0)
    kp, vp, tab, rows = _paged([s + n for s, n in segs], G, bs, dim, BF)
    T, row0, mix = sum(n for _, n in segs), 3, _mix(H)
    q, sink = (torch.randn(T, H, dim, device=DEV) * 1.5).to(BF), torch.randn(H, device=DEV)
    gate = torch.randn(T + row0, H, device=DEV).to(BF)
    qmix = torch.einsum("hcr,tcrd->thcd", mix.view(H, G, H // G), q.float().view(T, G, H // G, dim)).to(BF).contiguous()
    out = torch.full((T + row0, H * dim), 5.0, device=DEV, dtype=BF)
    at, r0 = [], row0
    for i, (s, n) in enumerate(segs):
        at.append((r0, n, i, s))
        r0 += n
    items = torch.tensor(prefill_items(at), dtype=torch.int32, device=DEV)
    talk.talk_prefill(qmix, row0, kp, vp, tab, items, sink, gate, 2, out, W, dim ** -0.5)
    assert _ok() and bool((out[:row0] == 5).all())
    for r0, n, i, s in at:
        want = _heads(q[r0 - row0:r0 - row0 + n], rows(i), mix, dim ** -0.5, sink, W, s) * P.sigmoid(gate[r0:r0 + n].double().cpu())[:, :, None]
        got, want = out[r0:r0 + n].double().cpu(), want.flatten(1)
        err = (got - want).norm(dim=1) / (want.norm(dim=1) + 1e-3 * want.norm() / n ** 0.5)
        assert float(err.max()) < 5e-2 and _rel(got, want) < 1.5e-2, (s, n)


@pytest.mark.parametrize("place", [0, 5, 63, 64, 70, 500])
@pytest.mark.parametrize("W", [1, 2, 63, 64, 65, 300])
def test_a_key_is_seen_exactly_inside_the_window(place, W):
    """One key that every query chooses, and whose values are all one, among quiet ones.  Only one head's own score is high;
    the others hear of it."""
    from rumus_b200.ops import talk
    from rumus_b200.ops.latent import prefill_items
    torch.manual_seed(place + W)
    H, G, dim, n, bs = 4, 2, 32, 900, 64
    kp, vp, tab, _ = _paged([n], G, bs, dim, BF)
    d = torch.randn(dim, device=DEV)
    d = d / d.norm()
    kp.mul_(0.05)
    vp.mul_(0.05)
    kp[int(tab[0, place // bs]), 1, place % bs] = (d * 20).to(BF)
    vp[int(tab[0, place // bs]), :, place % bs] = 1.0
    mix = torch.eye(H, device=DEV)
    mix[:, 3] = 1.0
    see = lambda p: 0 <= p - place < W
    at = sorted({p for p in (place - 1, place, place + 1, place + W - 1, place + W, place + W + 1, place + W + 70, 127, 128, n - 1) if 0 <= p < n})
    ctx = torch.tensor([p + 1 for p in at], dtype=torch.int32, device=DEV)

    def queries(rows):
        q = torch.zeros(rows, H, dim, device=DEV)
        q[:, 3] = d
        return q.to(BF)

    for plain in (False, True):
        out = torch.empty(len(at), H * dim, device=DEV, dtype=BF)
        talk.talk_rows_attention(queries(len(at)), kp, vp, tab.expand(len(at), -1).contiguous(), ctx, mix, None, None, 0, out, W, 1.0, n, plain=plain)
        heads = out.float().view(len(at), H, dim).mean(2).cpu()
        assert (heads.min(1).values > 0.9).tolist() == [see(p) for p in at] == (heads.max(1).values > 0.9).tolist(), plain
    for first, rows in ((0, 300), (max(0, place + W - 100), 190), (600, 128)):
        q = queries(rows)
        qmix = torch.einsum("hcr,tcrd->thcd", mix.view(H, G, H // G), q.float().view(rows, G, H // G, dim)).to(BF).contiguous()
        out = torch.empty(rows, H * dim, device=DEV, dtype=BF)
        items = torch.tensor(prefill_items([(0, rows, 0, first)]), dtype=torch.int32, device=DEV)
        talk.talk_prefill(qmix, 0, kp, vp, tab, items, None, None, 0, out, W, 1.0)
        heads = out.float().view(rows, H, dim).mean(2).cpu()
        want = [see(first + i) for i in range(rows)]
        assert (heads.min(1).values > 0.9).tolist() == want == (heads.max(1).values > 0.9).tolist(), first
    assert _ok()


# ------------------------------------------------------------------------------------------ gated delta rule
LENS, CUTS = [150, 3, 70, 260], [[1, 2, 70, 149], [1], [64], [5, 69, 197]]


def _rounds():
    """Portions of every sequence, round by round: (sequence, first token, tokens)."""
    ends = [c + [n] for c, n in zip(CUTS, LENS)]
    for k in range(max(len(e) for e in ends)):
        yield [(i, 0 if k == 0 else e[k - 1], e[k] - (0 if k == 0 else e[k - 1])) for i, e in enumerate(ends) if k < len(e)]


DELTA = [  # heads, kv heads, dim, vdim, taps, spread of the decays
    (5, 5, 24, 56, 3, 1.0), (2, 1, 128, 128, 4, 3.0), (3, 3, 10, 13, 2, 0.3), (6, 2, 64, 24, 1, 8.0), (2, 1, 104, 72, 5, 2.0),
    (6, 2, 40, 64, 4, 1.0),
    (2, 1, 200, 40, 3, 1.0), (1, 1, 24, 264, 4, 1.0),
]


@pytest.mark.parametrize("dt,way", [(BF, "chunks"), (BF, "rows"), (F32, "rows")])
@pytest.mark.parametrize("H,G,d,e,taps,spread", DELTA)
def test_delta_rule_with_a_decay_per_head(dt, way, H, G, d, e, taps, spread):
    """Convolutions, unit lengths, decays, the rule itself, output norm and gate over portions as short as one token (shorter
    than the convolution); decays from nearly none to nearly all in a step."""
    from rumus_b200.ops import recurrent
    dp, ep = p8(d), p8(e)
    if way == "chunks" and not recurrent.delta_chunks_covered(dt, dp, ep):
        pytest.skip("sizes that go token by token")
    torch.manual_seed(d + e + taps)
    places, eps, per, C = [2, 0, 4, 3], 1e-4, H // G, 2 * G * dp + H * ep
    raw = [torch.cat([_pad(torch.randn(n, G, d), dp).flatten(1), _pad(torch.randn(n, G, d), dp).flatten(1),
                      _pad(torch.randn(n, H, e), ep).flatten(1)], 1).to(dt) for n in LENS]
    few = [torch.randn(n, 2 * p8(H)) for n in LENS]                 # write strengths, then steps
    for f in few:
        f[:, p8(H):] *= spread
    gate = [_pad(torch.randn(n, H, e), ep).flatten(1).to(dt) for n in LENS]
    w = torch.zeros(taps, C)
    used = raw[0].abs().sum(0) > 0
    w[:, used] = torch.randn(taps, int(used.sum())) * taps ** -0.5
    dt_bias, A, norm = torch.randn(H), torch.randn(H), torch.randn(e)
    state = {"S": torch.randn(5, H, dp, ep, device=DEV), "conv": torch.randn(5, H, taps - 1, 2 * dp + ep, device=DEV).to(dt)}
    got = [[] for _ in LENS]
    for rnd in _rounds():
        rows, seqs = 0, []
        for i, s, n in rnd:
            seqs.append([rows, n, places[i], s])
            rows += n
        seqs = torch.tensor(seqs, dtype=torch.int32, device=DEV)
        take = lambda ts: torch.cat([ts[i][s:s + n] for i, s, n in rnd]).to(DEV)
        r, f = _pad(take(raw), C + 8), take(few)
        out = torch.full((rows, H * ep + 8), 5.0, device=DEV, dtype=dt)
        ins = (r, w.to(DEV), f[:, p8(H):], dt_bias.to(DEV), A.exp().to(DEV), f)
        rest = (seqs, state, take(gate), _pad(norm, ep).to(DEV), out[:, :H * ep], G, d, e, eps)
        if way == "rows":
            recurrent.delta_rows(*ins, *rest, per_head=True, silu=True)
        else:
            chunks = recurrent.cut([(int(s[0]), int(s[1])) for s in seqs.cpu()], recurrent.DELTA_CHUNK, DEV)
            recurrent.delta_chunks(*ins, chunks, *rest, per_head=True, silu=True)
        assert bool((out[:, H * ep:] == 5).all())
        at = 0
        for i, _, n in rnd:
            got[i].append(out[at:at + n, :H * ep].reshape(n, H, ep)[..., :e].double().cpu())
            at += n
    assert _ok()
    for i, n in enumerate(LENS):
        c = P.short_conv(raw[i].double(), w.double().T)
        if dt == BF:                     # the kernels keep convolved numbers in 16 bits
            c = c.to(BF).double()
        q, k, v = c[:, :G * dp].view(n, G, dp), c[:, G * dp:2 * G * dp].view(n, G, dp), c[:, 2 * G * dp:].view(n, H, ep)
        q, k = P.unit(q) * d ** -0.5, P.unit(k)
        g = torch.exp(-A.double().exp() * P.softplus(few[i][:, p8(H):p8(H) + H].double() + dt_bias.double()))
        beta, out = P.sigmoid(few[i][:, :H].double()), torch.cat(got[i])
        for h in range(H):
            o, S = P.delta_memory(q[:, h // per], k[:, h // per], v[:, h], g[:, h], beta[:, h])
            o = P.rms(o[:, :e], eps) * norm.double() * P.silu(gate[i].double().view(n, H, ep)[:, h, :e])
            assert _rel(out[:, h], o) < (2e-2 if dt == BF else 2e-5), (i, h)
            assert _rel(state["S"][places[i], h], S) < (1e-2 if dt == BF else 1e-5), (i, h)
        if taps > 1:
            last = torch.cat([torch.zeros(taps - 1, C).to(dt), raw[i]])[-(taps - 1):]
            for h in range(H):
                kh = h // per
                mine = torch.cat([last[:, kh * dp:(kh + 1) * dp], last[:, (G + kh) * dp:(G + kh + 1) * dp],
                                  last[:, 2 * G * dp + h * ep:2 * G * dp + (h + 1) * ep]], 1)
                assert torch.equal(state["conv"][places[i], h].cpu(), mine)
