"""Each mechanism of the Potodra kernels alone, against the oracle's equations in float64."""
import math

import pytest
import torch

import potodra_oracle as P

pytestmark = pytest.mark.gpu
DEV = "cuda"
BF, F32 = torch.bfloat16, torch.float32


def _rel(a, b):
    a, b = a.double().cpu(), b.double().cpu()
    return float((a - b).norm() / (b.norm() + 1e-30))


def _ok():
    from rumus_b200.ops import native
    return native.read_status() == 0


def _tol(dt):
    return 5e-3 if dt == BF else 3e-6


def p8(n):
    return (n + 7) // 8 * 8


def _pad(t, n):
    return torch.nn.functional.pad(t, (0, n - t.shape[-1]))


# ------------------------------------------------------------------------------------------ streams
@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("S,D,n_add,T", [(4, 64, 3, 5), (1, 50, 0, 3), (2, 1004, 2, 70), (3, 2050, 0, 2), (5, 40, 1, 300), (8, 4100, 4, 3)])
def test_streams_between_sublayers(dt, S, D, n_add, T):
    """Mixing, what every stream gains, the weighted sum and its norm; from equal streams, with and without a result."""
    from rumus_b200.ops import stream
    torch.manual_seed(S * D)
    ld = p8(D)
    w_in, w_out, mix, w = torch.randn(S), torch.randn(S), torch.randn(S, S), torch.randn(D)
    y, rows = torch.randn(T, D), torch.randn(T * n_add + 3, ld).to(dt)
    index = torch.randperm(T * n_add + 3)[:T * n_add].view(T, n_add).int()
    full = y.double() + (rows[index.long(), :D].double().sum(1) if n_add else 0)
    dev = lambda *ts: [t.to(DEV) for t in ts]
    gi, go, gm, gw, gy, gr, gx = dev(w_in, w_out, mix, w, y, rows, index)
    for equal in (True, False):
        x = torch.randn(T, 1 if equal else S, D).expand(-1, S, -1)
        xd = x.to(DEV) if not equal else x[:, 0].to(DEV).unsqueeze(1).expand(-1, S, -1)
        h, same = stream.stream_mix_norm(xd, gi, gw, 1e-2, dt, ld)
        assert same is xd
        assert _rel(h[:, :D], P.rms(P.streams_read(x.double(), w_in.double()), 1e-2) * w.double()) < _tol(dt)
        want = P.streams_write(x.double(), mix.double(), w_out.double(), full)
        add = (gr, gx) if n_add else None
        last, none = stream.stream_mix_norm(xd, gi, gw, 1e-2, dt, ld, y=gy, mix=gm, w_out=go, add=add, keep=False)
        h, new = stream.stream_mix_norm(xd, gi, gw, 1e-2, dt, ld, y=gy, mix=gm, w_out=go, add=add)
        assert none is None and torch.equal(last, h) and _rel(new, want) < 2e-6
        assert _rel(h[:, :D], P.rms(P.streams_read(want, w_in.double()), 1e-2) * w.double()) < _tol(dt)
        assert float(h[:, D:].abs().sum()) == 0


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("M,K,N", [(5, 64, 40), (300, 256, 512), (700, 72, 264)])
def test_squared_relu_in_the_product(dt, M, K, N):
    from rumus_b200.ops import native
    torch.manual_seed(M)
    a, w = torch.randn(M, K).to(dt), (torch.randn(N, K) * K ** -0.5).to(dt)
    got = native.gemm(a.to(DEV), w.to(DEV).t(), act="relu2", path=2 if dt == F32 else 0)
    assert _rel(got, torch.relu(a.double() @ w.double().T) ** 2) < _tol(dt)


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("F", [33, 64, 1000])
def test_gated_unit_with_a_gate_per_row(dt, F):
    from rumus_b200.ops import stream
    torch.manual_seed(F)
    wide = (torch.randn(9, 2 * F + 8) * 3).to(dt)
    out = torch.empty(9, F, device=DEV, dtype=dt)
    g = wide.to(DEV)
    stream.clamped_glu(g[:, :2 * F], out, 0.7, 1.702, 1.0, row_gate=g[:, 2 * F:])
    x = wide.double()
    gate, up = x[:, :F].clamp(max=0.7), x[:, F:2 * F].clamp(-0.7, 0.7)
    assert _rel(out, gate * P.sigmoid(1.702 * gate) * (up + 1) * P.sigmoid(x[:, 2 * F:2 * F + 1])) < _tol(dt)


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("T,K,N", [(1, 64, 3), (7, 1000, 16), (40, 256, 50)])
def test_few_outputs_in_32_bits(dt, T, K, N):
    from rumus_b200.ops import recurrent
    torch.manual_seed(K)
    h, w, b = torch.randn(T, K + 8).to(dt).to(DEV)[:, :K], torch.randn(N, K).to(dt), torch.randn(N)
    want = h.double().cpu() @ w.double().T
    assert _rel(recurrent.few_outputs(h, w.to(DEV)), want) < 1e-6
    assert _rel(recurrent.few_outputs(h, w.to(DEV), b.to(DEV)), want + b.double()) < 1e-6


# ------------------------------------------------------------------------------------------ attention
@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("H,G,dim,rot", [(3, 1, 10, 6), (4, 2, 24, 24), (2, 2, 128, 64), (2, 1, 200, 2), (3, 3, 64, 8), (2, 1, 20, 12)])
def test_rotation_of_neighbours_and_halves(dt, H, G, dim, rot):
    from rumus_b200.ops import stream, window
    from rumus_b200.ops.rotary import RotarySpec
    torch.manual_seed(dim)
    T, dp = 6, p8(dim)
    pos, spec = torch.tensor([0, 1, 5, 64, 1000, 3]), {"base": 1234.0, "dims": rot}
    q, k, v = torch.randn(T, H, dim).to(dt), torch.randn(T, G, dim).to(dt), torch.randn(T, G, 8).to(dt)
    f, m = RotarySpec.from_dict(spec).frequencies()
    tab = stream.rotary_table(pos.to(DEV), f.to(DEV), m)
    for neighbours in (True, False):
        proj = torch.cat([_pad(q, dp).flatten(1), _pad(k, dp).flatten(1), v.flatten(1)], 1).to(DEV)
        kp, vp = torch.zeros(2, G, 4, dp, dtype=dt, device=DEV), torch.zeros(2, G, 4, 8, dtype=dt, device=DEV)
        window.window_post(proj, torch.arange(T, device=DEV), kp, vp, H, dim, tab=tab, rot=rot, neighbours=neighbours)
        tol = 5e-3 if dt == BF else 3e-5
        assert _rel(proj[:, :H * dp].view(T, H, dp)[..., :dim], P.rotate(q.double(), pos, spec, neighbours)) < tol
        kr = kp.permute(0, 2, 1, 3).reshape(8, G, dp)[:T]
        assert _rel(kr[..., :dim], P.rotate(k.double(), pos, spec, neighbours)) < tol and float(kr[..., dim:].abs().sum()) == 0


def _paged(ctxs, G, bs, dp, vp, dt):
    """Pools with the pages of several sequences in a shuffled order, tables, and a reader of a sequence's rows."""
    need = [(c + bs - 1) // bs for c in ctxs]
    nb = sum(need) + 3
    kp, vp_ = torch.randn(nb, G, bs, dp, device=DEV).to(dt), torch.randn(nb, G, bs, vp, device=DEV).to(dt)
    perm = torch.randperm(nb)
    tab, k = torch.zeros(len(ctxs), max(need), dtype=torch.int32), 0
    for i, n in enumerate(need):
        tab[i, :n] = perm[k:k + n]
        k += n

    def rows(i):
        t = torch.arange(ctxs[i])
        b, o = tab[i, t // bs].long().to(DEV), (t % bs).to(DEV)
        return kp[b, :, o].double().cpu(), vp_[b, :, o].double().cpu()

    return kp, vp_, tab.to(DEV), rows


def _heads(q, rows, scale, cap, sink, mask, offset, out_scale):
    k, v = rows
    per = q.shape[1] // k.shape[1]
    return out_scale * torch.cat([P.attend(q[:, h].double().cpu(), k[:, h // per], v[:, h // per], scale, cap,
                                           None if sink is None else sink[h].double().cpu(), mask, offset) for h in range(q.shape[1])], -1)


ROWS = [  # heads, kv heads, dim, vdim, window, kept, cap, page, contexts
    (4, 2, 48, 40, 37, 5, 3.0, 16, [1, 4, 5, 6, 37, 38, 41, 42, 43, 100]),
    (3, 3, 16, 16, 64, 64, None, 64, [63, 64, 65, 128, 129, 192, 193, 300]),
    (8, 1, 128, 128, 100, 130, 20.0, 64, [700, 130, 2, 229, 230, 231, 232]),
    (10, 2, 72, 128, 1, 1, 0.7, 8, [1, 2, 3, 64, 65]),
    (6, 2, 200, 136, 50, 3, 5.0, 32, [49, 50, 51, 53, 54, 400]),
    (2, 1, 264, 400, 20, 17, None, 16, [5, 20, 21, 37, 38, 90]),
    (12, 4, 64, 56, 80, 7, 18.0, 64, [79, 80, 86, 87, 127, 128, 143, 144, 151, 200, 500]),
    (20, 1, 56, 104, 1 << 30, 0, 9.0, 8, [8, 129, 500]),
]


@pytest.mark.parametrize("dt,plain", [(BF, False), (BF, True), (F32, True)])
@pytest.mark.parametrize("case", ROWS)
@pytest.mark.parametrize("splits", [1, 0, 5])
def test_rows_with_kept_tokens_and_capped_scores(dt, plain, case, splits):
    from rumus_b200.ops import window
    H, G, dim, vdim, W, keep, cap, bs, ctxs = case
    torch.manual_seed(H + dim)
    kp, vp, tab, rows = _paged(ctxs, G, bs, dim, vdim, dt)
    q = (torch.randn(len(ctxs), H, dim, device=DEV) * 2).to(dt)
    sink, out = torch.randn(H, device=DEV), torch.empty(len(ctxs), H * vdim, device=DEV, dtype=dt)
    for s in (sink, None):
        window.window_rows_attention(q, kp, vp, tab, torch.tensor(ctxs, dtype=torch.int32, device=DEV), s, None, 0, out, W, dim ** -0.5,
                                     max(ctxs), splits=splits, plain=plain, keep=keep, cap=cap, out_scale=0.6)
        assert _ok()
        for i, c in enumerate(ctxs):
            want = _heads(q[i:i + 1], rows(i), dim ** -0.5, cap, s, {"size": W, "keep_first": keep}, c - 1, 0.6)
            assert _rel(out[i:i + 1], want) < (8e-3 if dt == BF else 5e-6), (i, c)


@pytest.mark.parametrize("H,G,dim,vdim,W,keep,cap,bs,segs", [
    (4, 2, 48, 40, 37, 5, 3.0, 16, [(0, 23), (30, 60), (100, 29)]), (6, 2, 64, 56, 80, 7, 18.0, 64, [(0, 300), (145, 140), (500, 2), (63, 129)]),
    (2, 1, 128, 128, 30, 70, None, 64, [(5, 130), (0, 128), (400, 9), (95, 40)]), (2, 2, 72, 64, 1, 1, 1.0, 8, [(0, 65), (129, 127)]),
    (3, 1, 16, 72, 200, 129, 6.0, 128, [(0, 200), (330, 130)]), (2, 1, 24, 16, 1 << 30, 0, 4.0, 32, [(0, 70), (200, 130)]),
    (1, 1, 8, 8, 64, 64, None, 64, [(128, 128), (127, 3), (64, 64)]),
])
def test_prompts_with_kept_tokens_and_capped_scores(H, G, dim, vdim, W, keep, cap, bs, segs):
    from rumus_b200.ops import window
    from rumus_b200.ops.latent import prefill_items
    torch.manual_seed(dim + vdim)
    kp, vp, tab, rows = _paged([s + n for s, n in segs], G, bs, dim, vdim, BF)
    T = sum(n for _, n in segs)
    q, sink = (torch.randn(T, H, dim, device=DEV) * 2).to(BF), torch.randn(H, device=DEV)
    out = torch.empty(T, H * vdim, device=DEV, dtype=BF)
    at, r0 = [], 0
    for i, (s, n) in enumerate(segs):
        at.append((r0, n, i, s))
        r0 += n
    items = torch.tensor(prefill_items(at), dtype=torch.int32, device=DEV)
    window.window_prefill(q, kp, vp, tab, items, sink, None, 0, out, W, dim ** -0.5, keep=keep, cap=cap, out_scale=1.7)
    assert _ok()
    for r0, n, i, s in at:
        want = _heads(q[r0:r0 + n], rows(i), dim ** -0.5, cap, sink, {"size": W, "keep_first": keep}, s, 1.7)
        got = out[r0:r0 + n].double().cpu()
        err = (got - want).norm(dim=1) / (want.norm(dim=1) + 1e-3 * want.norm() / n ** 0.5)
        assert float(err.max()) < 2e-2 and _rel(got, want) < 8e-3, (s, n)


@pytest.mark.parametrize("place", [0, 4, 5, 6, 63, 64, 69, 70, 500])
@pytest.mark.parametrize("W,keep", [(2, 5), (65, 5), (64, 70), (1, 64), (300, 1)])
def test_a_key_is_seen_exactly_while_kept_or_inside_the_window(place, W, keep):
    """One key that every query chooses, and whose values are all one, among quiet ones."""
    from rumus_b200.ops import window
    from rumus_b200.ops.latent import prefill_items
    torch.manual_seed(place + W)
    H, G, dim, vdim, n, bs = 4, 2, 32, 16, 900, 64
    kp, vp, tab, _ = _paged([n], G, bs, dim, vdim, BF)
    d = torch.randn(dim, device=DEV)
    d = d / d.norm()
    kp.mul_(0.05)
    vp.mul_(0.05)
    kp[int(tab[0, place // bs]), :, place % bs] = (d * 20).to(BF)
    vp[int(tab[0, place // bs]), :, place % bs] = 1.0
    see = lambda p: place <= p and (p - place < W or place < keep)
    at = sorted({p for p in (place - 1, place, place + 1, place + W - 1, place + W, place + W + 1, place + W + 70, 127, 128, n - 1) if 0 <= p < n})
    ctx = torch.tensor([p + 1 for p in at], dtype=torch.int32, device=DEV)
    q = d.to(BF).expand(len(at), H, dim).contiguous()
    for plain in (False, True):
        out = torch.empty(len(at), H * vdim, device=DEV, dtype=BF)
        window.window_rows_attention(q, kp, vp, tab.expand(len(at), -1).contiguous(), ctx, None, None, 0, out, W, 1.0, n, plain=plain, keep=keep,
                                     cap=30.0)
        assert (out.float().mean(1).cpu() > 0.9).tolist() == [see(p) for p in at], plain
    for first, rows in ((0, 300), (max(0, place + W - 100), 190), (600, 128)):
        q = d.to(BF).expand(rows, H, dim).contiguous()
        out = torch.empty(rows, H * vdim, device=DEV, dtype=BF)
        items = torch.tensor(prefill_items([(0, rows, 0, first)]), dtype=torch.int32, device=DEV)
        window.window_prefill(q, kp, vp, tab, items, None, None, 0, out, W, 1.0, keep=keep, cap=30.0)
        assert (out.float().mean(1).cpu() > 0.9).tolist() == [see(first + i) for i in range(rows)], first
    assert _ok()


# ------------------------------------------------------------------------------------------ recurrences
def _portions(lens, cuts):
    """Rounds of portions: sequence i is cut at cuts[i]; round r holds the r-th portion of every sequence that has one."""
    bounds = [[0] + list(c) + [n] for n, c in zip(lens, cuts)]
    for r in range(max(len(b) for b in bounds) - 1):
        yield [(i, b[r], b[r + 1] - b[r]) for i, b in enumerate(bounds) if r + 1 < len(b)]


def _batch(round_, places):
    seqs, row = [], 0
    for i, start, n in round_:
        seqs.append([row, n, places[i], start])
        row += n
    return torch.tensor(seqs, dtype=torch.int32, device=DEV), lambda ts: torch.cat([ts[i][s:s + n] for i, s, n in round_])


def _compare(got, want, dt, fp32_tol=2e-5):
    """Per token; 16-bit results may be off by their own rounding, and states by what the split products leave."""
    err = (got.double().cpu() - want).norm(dim=-1) / (want.norm(dim=-1) + 1e-30)
    assert float(err.max()) < (5e-3 if dt == BF else fp32_tol), float(err.max())


LENS, CUTS = [300, 1, 131, 64], [[128, 129, 257], [], [2, 3, 130], [9]]
MLSTM = [(3, 40, 56, 2.0, 11.0), (1, 128, 128, 8.0, 15.0), (3, 10, 13, 0.1, 3.0), (2, 64, 24, 30.0, 5.0), (2, 104, 72, 3.0, 8.0)]


@pytest.mark.parametrize("dt,way", [(BF, "chunks"), (BF, "rows"), (F32, "rows")])
@pytest.mark.parametrize("H,d,e,spread,cap", MLSTM + [(1, 200, 40, 2.0, 9.0), (1, 24, 264, 2.0, 9.0), (1, 300, 130, 2.0, 9.0)])
def test_matrix_memory(dt, way, H, d, e, spread, cap):
    """Several sequences in portions, in places of their own that hold another sequence's state before; gates from
    flat to saturated."""
    from rumus_b200.ops import recurrent
    dp, ep = p8(d), p8(e)
    if way == "chunks" and not recurrent.mlstm_chunks_covered(dt, dp, ep):
        pytest.skip("sizes that go token by token")
    torch.manual_seed(d + e)
    places, eps = [2, 0, 4, 3], 1e-4
    mk = lambda *s: [torch.randn(n, *s) for n in LENS]
    q, k, v, g = ([x.to(dt) for x in mk(H, w)] for w in (d, d, e, e))
    zi, zf = [x * spread for x in mk(H)], [x * spread + 2 for x in mk(H)]
    norm = torch.randn(H, e)
    state = {"S": torch.randn(5, H, dp, ep, device=DEV), "n": torch.randn(5, H, dp, device=DEV), "m": torch.randn(5, H, device=DEV)}
    rows = [torch.cat([_pad(q[i], dp).flatten(1), _pad(k[i], dp).flatten(1), _pad(v[i], ep).flatten(1), _pad(g[i], ep).flatten(1)], 1)
            for i in range(len(LENS))]
    gates = [torch.cat([zi[i], zf[i]], 1) for i in range(len(LENS))]
    got = [[] for _ in LENS]
    for rnd in _portions(LENS, CUTS):
        seqs, take = _batch(rnd, places)
        pr, gt = take(rows).to(DEV), take(gates).to(DEV)
        out = torch.full((pr.shape[0], H * ep + 8), 5.0, device=DEV, dtype=dt)
        rest = (state, pr[:, H * (2 * dp + ep):], _pad(norm, ep).flatten().to(DEV), out[:, :H * ep], d, e, cap, eps)
        if way == "rows":
            recurrent.mlstm_rows(pr, gt, seqs, *rest)
        else:
            chunks = recurrent.cut([(int(s[0]), int(s[1])) for s in seqs.cpu()], recurrent.MLSTM_CHUNK, DEV)
            recurrent.mlstm_chunks(pr, gt, chunks, seqs, *rest)
        assert bool((out[:, H * ep:] == 5).all())
        at = 0
        for i, _, n in rnd:
            got[i].append(out[at:at + n, :H * ep].reshape(n, H, ep)[..., :e].cpu())
            at += n
    assert _ok()
    for i in range(len(LENS)):
        out = torch.cat(got[i])
        for h in range(H):
            lo = lambda z: cap * torch.tanh(z.double() / cap)
            o, (S, n, m) = P.mlstm_memory(q[i][:, h].double() * d ** -0.5, k[i][:, h].double(), v[i][:, h].double(), lo(zi[i][:, h]),
                                          -P.softplus(-lo(zf[i][:, h])))
            _compare(out[:, h], P.rms(o, eps) * norm[h].double() * P.sigmoid(g[i][:, h].double()), dt, 5e-4)
            tol = 1e-4 if way == "chunks" else 1e-5
            assert _rel(state["S"][places[i], h, :d, :e], S) < tol and _rel(state["n"][places[i], h, :d], n) < tol
            assert abs(float(state["m"][places[i], h]) - float(m)) < 1e-4 * max(1.0, abs(float(m)))


def _delta_case(dt, H, G, d, e, taps, spread):
    C = 2 * G * p8(d) + H * p8(e)
    raw = [torch.cat([_pad(torch.randn(n, G, d), p8(d)).flatten(1), _pad(torch.randn(n, G, d), p8(d)).flatten(1),
                      _pad(torch.randn(n, H, e), p8(e)).flatten(1)], 1).to(dt) for n in LENS]
    a = [_pad(torch.randn(n, H, d) * spread, p8(d)).flatten(1) for n in LENS]
    b, gate = [torch.randn(n, H) for n in LENS], [_pad(torch.randn(n, H, e), p8(e)).flatten(1).to(dt) for n in LENS]
    w = torch.zeros(taps, C)
    w[:, raw[0].abs().sum(0) > 0] = torch.randn(taps, int((raw[0].abs().sum(0) > 0).sum())) * taps ** -0.5
    return raw, a, b, gate, w


DELTA = [(5, 5, 24, 56, 3, 1.0), (2, 1, 128, 128, 4, 3.0), (3, 3, 10, 13, 2, 0.3), (6, 2, 64, 24, 1, 8.0), (2, 1, 104, 72, 5, 2.0)]


@pytest.mark.parametrize("dt,way", [(BF, "chunks"), (BF, "rows"), (F32, "rows")])
@pytest.mark.parametrize("H,G,d,e,taps,spread", DELTA + [(2, 1, 200, 40, 3, 1.0), (1, 1, 24, 264, 4, 1.0), (1, 1, 300, 130, 2, 1.0)])
def test_delta_rule(dt, way, H, G, d, e, taps, spread):
    """Convolutions, unit lengths, decays and the rule itself over portions as short as one token (shorter than the
    convolution); decays from nearly none to nearly all in a step."""
    from rumus_b200.ops import recurrent
    dp, ep = p8(d), p8(e)
    if way == "chunks" and not recurrent.delta_chunks_covered(dt, dp, ep):
        pytest.skip("sizes that go token by token")
    torch.manual_seed(d + e + taps)
    places, eps, per = [2, 0, 4, 3], 1e-4, H // G
    raw, a, b, gate, w = _delta_case(dt, H, G, d, e, taps, spread)
    dt_bias, A, norm = torch.randn(H * dp), torch.randn(H), torch.randn(e)
    state = {"S": torch.randn(5, H, dp, ep, device=DEV), "conv": torch.randn(5, H, taps - 1, 2 * dp + ep, device=DEV).to(dt)}
    got = [[] for _ in LENS]
    for rnd in _portions(LENS, CUTS):
        seqs, take = _batch(rnd, places)
        r = _pad(take(raw), w.shape[1] + 8).to(DEV)
        steps = (take(a).to(DEV), dt_bias.to(DEV), A.exp().to(DEV), take(b).to(DEV))
        out = torch.full((r.shape[0], H * ep + 8), 5.0, device=DEV, dtype=dt)
        leave = (take(gate).to(DEV), _pad(norm, ep).to(DEV), out[:, :H * ep])
        if way == "rows":
            recurrent.delta_rows(r, w.to(DEV), *steps, seqs, state, *leave, G, d, e, eps)
        else:
            chunks = recurrent.cut([(int(s[0]), int(s[1])) for s in seqs.cpu()], recurrent.DELTA_CHUNK, DEV)
            recurrent.delta_chunks(r, w.to(DEV), *steps, chunks, seqs, state, *leave, G, d, e, eps)
        assert bool((out[:, H * ep:] == 5).all())
        at = 0
        for i, _, n in rnd:
            got[i].append(out[at:at + n, :H * ep].reshape(n, H, ep)[..., :e].cpu())
            at += n
    assert _ok()
    for i, n in enumerate(LENS):
        c = P.short_conv(raw[i].double(), w.double().T)
        q, k, v = c[:, :G * dp].view(n, G, dp), c[:, G * dp:2 * G * dp].view(n, G, dp), c[:, 2 * G * dp:].view(n, H, ep)
        q, k = P.unit(q) * d ** -0.5, P.unit(k)
        if dt == BF:                     # the kernels keep convolved values in 16 bits
            v = v.to(BF).double()
        g = torch.exp(-A.double().exp()[:, None] * P.softplus(a[i].double() + dt_bias.double()).view(n, H, dp))
        beta, out = P.sigmoid(b[i].double()), torch.cat(got[i])
        for h in range(H):
            o, S = P.delta_memory(q[:, h // per], k[:, h // per], v[:, h], g[:, h], beta[:, h])
            o = P.rms(o[:, :e], eps) * norm.double() * P.sigmoid(gate[i].double().view(n, H, ep)[:, h, :e])
            _compare(out[:, h], o, dt, 2e-4)
            assert _rel(state["S"][places[i], h], S) < (1e-3 if dt == BF else 1e-5)
        if taps > 1:
            last = torch.cat([torch.zeros(taps - 1, w.shape[1]).to(dt), raw[i]])[-(taps - 1):]
            for h in range(H):
                kh = h // per
                mine = torch.cat([last[:, kh * dp:(kh + 1) * dp], last[:, (G + kh) * dp:(G + kh + 1) * dp],
                                  last[:, 2 * G * dp + h * ep:2 * G * dp + (h + 1) * ep]], 1)
                assert torch.equal(state["conv"][places[i], h].cpu(), mine)


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("H,d,e", [(4, 24, 40), (7, 128, 128)])
def test_more_heads_than_ctas(dt, H, d, e):
    """Many sequences of zero to three tokens, new and old ones: the same results and states as each of them alone."""
    from rumus_b200.ops import recurrent
    torch.manual_seed(H)
    B, taps, cap = 600 // H + 20, 3, 9.0
    lens = [i % 4 for i in range(B)]
    start = [0 if i % 5 == 0 else 9 for i in range(B)]
    row = [sum(lens[:i]) for i in range(B)]
    T = sum(lens)
    seqs = torch.tensor([[row[i], lens[i], B - 1 - i, start[i]] for i in range(B)], dtype=torch.int32, device=DEV)
    old = {"S": torch.randn(B, H, d, e, device=DEV), "n": torch.randn(B, H, d, device=DEV), "m": torch.rand(B, H, device=DEV),
           "conv": torch.randn(B, H, taps - 1, 2 * d + e, device=DEV).to(dt)}
    proj, gates, norm = torch.randn(T, H * (2 * d + 2 * e), device=DEV).to(dt), torch.randn(T, 2 * H, device=DEV), torch.randn(H * e, device=DEV)
    gate = proj[:, H * (2 * d + e):]
    w, a, b = torch.randn(taps, H * (2 * d + e), device=DEV), torch.randn(T, H * d, device=DEV), torch.randn(T, H, device=DEV)
    bias, decay = torch.randn(H * d, device=DEV), torch.rand(H, device=DEV)

    def run(which, out_m, out_d, state):
        recurrent.mlstm_rows(proj, gates, which, state, gate, norm, out_m, d, e, cap, 1e-5)
        other = dict(state, S=state["S2"])
        recurrent.delta_rows(proj, w, a, bias, decay, b, which, other, gate, norm[:e].contiguous(), out_d, H, d, e, 1e-5)

    def fresh():
        return [torch.zeros(T, H * e, device=DEV, dtype=dt) for _ in range(2)] + [{**{k: t.clone() for k, t in old.items()}, "S2": old["S"].clone()}]

    many, alone = fresh(), fresh()
    run(seqs, *many)
    for i in range(0, B, 3):
        run(seqs[i:i + 1].contiguous(), *alone)
    assert _ok()
    for i in range(0, B, 3):
        rows, place = slice(row[i], row[i] + lens[i]), B - 1 - i
        for x, y in zip(many[:2], alone[:2]):
            assert torch.equal(x[rows], y[rows])
        for k in many[2]:
            assert torch.equal(many[2][k][place], alone[2][k][place]), k
    assert all(torch.equal(many[2][k][B - 1], old["S" if k == "S2" else k][B - 1]) for k in many[2])          # no tokens


def test_portions_without_tokens_change_nothing():
    """Padding of captured batches."""
    from rumus_b200.ops import recurrent
    state = {"S": torch.randn(2, 1, 8, 8, device=DEV), "n": torch.randn(2, 1, 8, device=DEV), "m": torch.randn(2, 1, device=DEV)}
    before = {k: t.clone() for k, t in state.items()}
    pr, out = torch.randn(3, 32, device=DEV), torch.full((3, 8), 7.0, device=DEV)
    seqs = torch.zeros(3, 4, dtype=torch.int32, device=DEV)
    recurrent.mlstm_rows(pr, torch.randn(3, 2, device=DEV), seqs, state, pr[:, 24:], torch.ones(8, device=DEV), out, 8, 8, 5.0, 1e-6)
    assert all(torch.equal(before[k], state[k]) for k in state) and bool((out == 7).all())


# ------------------------------------------------------------------------------------------ experts
@pytest.mark.parametrize("T,E,top,groups,keep,given", [
    (1, 10, 3, 5, 3, False), (5, 6, 2, 1, 1, False), (64, 64, 6, 8, 3, False), (100, 36, 5, 12, 2, True), (300, 16, 4, 4, 1, True),
    (9, 128, 5, 64, 9, False), (700, 8, 1, 8, 5, True), (33, 80, 7, 40, 11, False),
])
def test_routing_by_groups(T, E, top, groups, keep, given):
    from rumus_b200.ops import moe
    torch.manual_seed(T + E)
    h, w = torch.randn(T, 64).to(BF), (torch.randn(E, 64) * 2 * 64 ** -0.5).to(BF)
    # corrections often larger than the scores, and negative choice scores
    correction = torch.randn(E) - 0.5
    z = h.double() @ w.double().T
    counts = torch.zeros(E + 1, dtype=torch.int32, device=DEV)
    logits = z.float().to(DEV) if given else None
    r = moe.route(h.to(DEV), w.to(DEV), correction.to(DEV), counts, top, logits=logits, score=moe.SIGMOID, groups=groups, keep=keep)
    assert int(counts.abs().sum()) == 0
    s, clear = P.sigmoid(z), 0
    for t in range(T):
        want, margin = P.choose(s[t], correction.double(), top, {"count": groups, "keep": keep})
        if margin > 1e-5:
            clear += 1
            assert r.idx[t].tolist() == want, t
        torch.testing.assert_close(r.weight[t].double().cpu(), s[t][r.idx[t].long().cpu()], rtol=1e-5, atol=1e-6)
    assert clear > 0.9 * T
    slots = r.slot_of.cpu().flatten().long()
    assert len(set(slots.tolist())) == T * top and torch.equal(r.slot_weight.cpu()[slots], r.weight.cpu().flatten())


@pytest.mark.parametrize("dt,plain,tile", [(BF, False, 0), (BF, False, 32), (BF, False, 256), (BF, True, 0), (F32, True, 0)])
@pytest.mark.parametrize("T,E,top,dim,ff,limit", [(3, 8, 3, 264, 136, 0.5), (150, 4, 2, 64, 520, 7.0), (900, 4, 2, 136, 24, 1.0)])
def test_experts_with_clamped_units(dt, plain, tile, T, E, top, dim, ff, limit):
    from rumus_b200.ops import moe, stream
    torch.manual_seed(T + dim)
    w = {}
    for e in range(E):
        w[f"e{e}.gate"], w[f"e{e}.up"] = (torch.randn(ff, dim) * 2 * dim ** -0.5).to(dt), (torch.randn(ff, dim) * 2 * dim ** -0.5).to(dt)
        w[f"e{e}.down"] = (torch.randn(dim, ff) * ff ** -0.5).to(dt)
    w["router"], w["correction"] = (torch.randn(E, dim) * 2 * dim ** -0.5).to(dt), torch.randn(E) * 0.3
    for k in ("gate", "up"):
        w["shared." + k] = torch.zeros(8, dim).to(dt)
    w["shared.down"], w["shared.sg"] = torch.zeros(dim, 8).to(dt), torch.zeros(1, dim).to(dt)
    h = torch.randn(T, dim).to(dt)
    gu = moe.interleave(*(torch.stack([w[f"e{e}.{k}"] for e in range(E)]).to(DEV) for k in ("gate", "up")))
    wide = gu.shape[1] // 2
    dn = _pad(torch.stack([w[f"e{e}.down"] for e in range(E)]), wide).to(DEV)
    counts = torch.zeros(E + 1, dtype=torch.int32, device=DEV)
    hd = h.to(DEV)
    logits = (h.double() @ w["router"].double().T).float().to(DEV)
    r = moe.route(hd, w["router"].to(DEV), w["correction"].to(DEV), counts, top, logits=logits, plain=plain, tile=tile, score=moe.SIGMOID,
                  groups=2, keep=2)
    act, y = torch.empty(r.slots, wide, device=DEV, dtype=dt), torch.empty(r.slots, dim, device=DEV, dtype=dt)
    moe.grouped(hd, gu, r, act, gated=True, plain=plain, unit=(limit, 1.702, 1.0))
    moe.grouped(act, dn, r, y, gated=False, plain=plain)
    x = torch.zeros(T, dim, device=DEV)
    stream.rms_norm_stream(x, torch.ones(dim, device=DEV), None, 1e-6, dt, dim, add=(y, r.slot_of))
    margins = []
    want = P.mixture(h.double(), {k: t.double() for k, t in w.items()}, "", {
        "router": {"top": top, "groups": {"count": 2, "keep": 2}}, "expert": {"limit": limit}, "shared": {"limit": 1.0}}, margins)
    clear = margins[0] > 1e-5
    err = (x.double().cpu() - want).norm(dim=1)[clear] / want.norm(dim=1)[clear]
    assert _ok() and float(err.max()) < (3e-2 if dt == BF else 2e-5)
    assert math.isfinite(float(x.sum()))
