"""Each mechanism of the Nufupel kernels alone, against the oracle's equations in float64."""
import math

import pytest
import torch

import nufupel_oracle as N

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


# ------------------------------------------------------------------------------------------ around the mixers
@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("D,n_add", [(50, 3), (64, 1), (1004, 7), (2050, 2), (2052, 33)])
def test_norm_that_first_adds_rows(dt, D, n_add):
    from rumus_b200.ops import stream
    torch.manual_seed(D)
    T, ld = 5, p8(D)
    x = torch.randn(T, D, device=DEV)
    rows = torch.randn(T * n_add + 3, ld, device=DEV).to(dt)
    index = torch.randperm(T * n_add + 3, device=DEV)[:T * n_add].view(T, n_add).int()
    w = torch.randn(D, device=DEV)
    want = x.double() + rows[index.long(), :D].double().sum(1)
    y, _ = stream.rms_norm_stream(x, w, None, 1e-2, dt, ld, add=(rows, index))
    assert _rel(x, want) < 1e-6
    assert _rel(y[:, :D], N.rms_norm(want, w.double(), 1e-2)) < _tol(dt) and float(y[:, D:].abs().sum()) == 0


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("F", [33, 64, 1000])
def test_gated_units(dt, F):
    from rumus_b200.ops import stream
    torch.manual_seed(F)
    wide = (torch.randn(9, 2 * F + 16) * 3).to(dt)
    gu = wide[:, 8:8 + 2 * F]
    for kind, act in ((stream.GLU_GELU, N.gelu_tanh), (stream.GLU_SILU, N.silu)):
        buf = torch.full((9, F + 16), 7.0, device=DEV, dtype=dt)
        stream.glu(kind, wide.to(DEV)[:, 8:8 + 2 * F], buf[:, 8:8 + F])
        assert _rel(buf[:, 8:8 + F], act(gu[:, :F].double()) * gu[:, F:].double()) < _tol(dt)
        assert bool((buf[:, :8] == 7).all()) and bool((buf[:, 8 + F:] == 7).all())


def test_softcap():
    from rumus_b200.ops import stream
    z = torch.randn(5, 77, device=DEV) * 40
    want = N.softcap(z.double(), 12.5)
    assert _rel(stream.softcap_(z, 12.5), want) < 1e-6 and float(z.abs().max()) <= 12.5


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("H,G,dim,vdim,rot,bs", [
    (3, 1, 10, 13, None, 4), (4, 2, 24, 16, 24, 8), (6, 3, 42, 7, 10, 4), (8, 8, 128, 64, 64, 16), (2, 1, 200, 300, 2, 4),
])
def test_projection_to_queries_and_cache_rows(dt, H, G, dim, vdim, rot, bs):
    """Head norms, partial rotation with elements half a rotation apart, keys and values in the right cache rows."""
    from rumus_b200.ops import stream, window
    from rumus_b200.ops.rotary import RotarySpec
    torch.manual_seed(dim)
    T, dp, vp = 7, p8(dim), p8(vdim)
    spec = {"base": 1234.0, "dims": rot, "scaling": {"factor": 3.0, "low": 1.0, "high": 4.0, "original": 60}}
    pos = torch.tensor([0, 1, 5, 64, 1000, 3, 2])
    slots = torch.tensor([9, 0, 3, -1, 15, 14, 2])
    q, k, v = torch.randn(T, H, dim).to(dt), torch.randn(T, G, dim).to(dt), torch.randn(T, G, vdim).to(dt)
    pad = torch.nn.functional.pad
    proj = torch.cat([pad(q, (0, dp - dim)).flatten(1), pad(k, (0, dp - dim)).flatten(1), pad(v, (0, vp - vdim)).flatten(1),
                      torch.full((T, 8), 5.0).to(dt)], 1).to(DEV)
    kp = torch.full((16 // bs, G, bs, dp), 3.0, dtype=dt, device=DEV)
    vpool = torch.full((16 // bs, G, bs, vp), 3.0, dtype=dt, device=DEV)
    kw, wq, wk = {}, q.double(), k.double()
    if rot is not None:
        qn, kn = torch.rand(dim) + 0.5, torch.rand(dim) + 0.5
        f, m = RotarySpec.from_dict(spec).frequencies()
        kw = dict(tab=stream.rotary_table(pos.to(DEV), f.to(DEV), m), rot=rot, norms=(qn.to(DEV), kn.to(DEV)), eps=1e-3)
        wq = N.rotate(N.rms_norm(wq, qn.double(), 1e-3), pos.tolist(), spec)
        wk = N.rotate(N.rms_norm(wk, kn.double(), 1e-3), pos.tolist(), spec)
    window.window_post(proj, slots.to(DEV), kp, vpool, H, dim, **kw)
    got = proj.cpu()
    assert _rel(got[:, :H * dp].view(T, H, dp)[..., :dim], wq) < (5e-3 if dt == BF else 3e-5)
    assert bool((got[:, -8:] == 5).all())
    kr, vr = kp.permute(0, 2, 1, 3).reshape(16, G, dp).cpu(), vpool.permute(0, 2, 1, 3).reshape(16, G, vp).cpu()
    for t, s in enumerate(slots.tolist()):
        if s >= 0:
            assert _rel(kr[s, :, :dim], wk[t]) < (5e-3 if dt == BF else 3e-5)
            assert torch.equal(vr[s, :, :vdim], v[t])
            assert float(kr[s, :, dim:].abs().sum()) == 0 and float(vr[s, :, vdim:].abs().sum()) == 0
    idle = [s for s in range(16) if s not in slots.tolist()]
    assert bool((kr[idle] == 3).all()) and bool((vr[idle] == 3).all())


# ------------------------------------------------------------------------------------------ attention
def _paged(ctxs, G, bs, dp, vp, dt, extra=3):
    """Pools with the pages of several sequences in a shuffled order, tables, and a reader of a sequence's rows."""
    need = [(c + bs - 1) // bs for c in ctxs]
    nb = sum(need) + extra
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


def _want(q, rows, sink, gate, kind, mx, offset):
    """Oracle heads [n, H * vdim] of queries q [n, H, dim] at positions offset ..."""
    o = N.attention_heads(q.double().cpu(), *rows, sink.double().cpu(), mx, offset=offset)
    if kind == 1:
        o = o * torch.sigmoid(gate.double().cpu()).view(o.shape)
    elif kind == 2:
        o = o * torch.sigmoid(gate.double().cpu())[:, :o.shape[1], None]
    return o.flatten(1)


@pytest.mark.parametrize("dt,plain", [(BF, False), (BF, True), (F32, True)])
@pytest.mark.parametrize("H,G,dim,vdim,W,bs,ctxs,kind", [
    (4, 2, 48, 40, 37, 16, [1, 15, 16, 17, 36, 37, 38, 53, 100], 1),
    (3, 3, 16, 16, 64, 64, [63, 64, 65, 128, 129, 300], 2),
    (8, 1, 128, 128, 1000, 64, [4000, 130, 2, 999, 1000, 1001], 1),
    (10, 2, 72, 128, 1, 8, [1, 2, 64, 65], 2),
    (6, 2, 200, 136, 50, 32, [49, 50, 51, 400], 0),
    (2, 1, 264, 512, 20, 16, [5, 20, 21, 90], 1),
    (48, 2, 64, 64, 90, 48, [89, 91, 47, 48, 49], 2),
    (48, 2, 120, 40, 90, 64, [89, 91, 63, 64, 155, 300], 1),
    (20, 1, 56, 104, 130, 8, [8, 129, 130, 131, 500], 2),
    (32, 4, 128, 128, 300, 32, [1, 299, 300, 301, 640, 777, 4096], 1),
    (12, 4, 8, 24, 5000, 64, [700, 64], 1),
])
@pytest.mark.parametrize("splits", [1, 0, 5])
def test_row_attention(dt, plain, H, G, dim, vdim, W, bs, ctxs, kind, splits):
    """Contexts around page, tile and window borders; one to many query heads on a key/value head."""
    from rumus_b200.ops import window
    torch.manual_seed(H + dim)
    kp, vp, tab, rows = _paged(ctxs, G, bs, dim, vdim, dt)
    B, mx = len(ctxs), {"heads": H, "kv_heads": G, "scale": 2.0 * dim ** -0.5, "mask": {"size": W}}
    q = torch.randn(B, H * dim + 16, device=DEV).to(dt)[:, :H * dim].unflatten(1, (H, dim))
    gate = torch.randn(B, H * vdim if kind == 1 else p8(H), device=DEV).to(dt)
    sink = torch.randn(H, device=DEV) * 2
    out = torch.full((B, H * vdim + 8), 5.0, device=DEV, dtype=dt)
    window.window_rows_attention(q, kp, vp, tab, torch.tensor(ctxs, dtype=torch.int32, device=DEV), sink, gate if kind else None,
                                 kind, out[:, :H * vdim], W, mx["scale"], max(ctxs), splits=splits, plain=plain)
    assert _ok() and bool((out[:, H * vdim:] == 5).all())
    for i, c in enumerate(ctxs):
        want = _want(q[i:i + 1], rows(i), sink, gate[i:i + 1], kind, mx, c - 1)
        assert _rel(out[i:i + 1, :H * vdim], want) < (8e-3 if dt == BF else 5e-6), (i, c)


def _one_loud_key(place, n, G, dim, vdim, bs, dt):
    """A sequence of n quiet keys, one of which every query chooses and whose values are all one."""
    kp, vp, tab, _ = _paged([n], G, bs, dim, vdim, dt)
    d = torch.randn(dim, device=DEV)
    d = d / d.norm()
    kp.mul_(0.05)
    vp.mul_(0.05)
    b, o = int(tab[0, place // bs]), place % bs
    kp[b, :, o] = (d * 20).to(dt)
    vp[b, :, o] = 1.0
    return d.to(dt), kp, vp, tab


@pytest.mark.parametrize("dt,plain", [(BF, False), (BF, True), (F32, True)])
@pytest.mark.parametrize("place", [0, 1, 63, 64, 127, 128, 500, 1299])
@pytest.mark.parametrize("W", [1, 2, 64, 65, 777])
def test_rows_see_a_key_exactly_inside_the_window(dt, plain, place, W):
    from rumus_b200.ops import window
    torch.manual_seed(place + W)
    H, G, dim, vdim, n = 4, 2, 32, 16, 2200
    d, kp, vp, tab = _one_loud_key(place, n, G, dim, vdim, 64, dt)
    ctx = [c for c in (place, place + 1, place + 2, place + W - 1, place + W, place + W + 1, place + W + 40) if 0 < c <= n]
    q = d.expand(len(ctx), H, dim).contiguous()
    out = torch.empty(len(ctx), H * vdim, device=DEV, dtype=dt)
    window.window_rows_attention(q, kp, vp, tab.expand(len(ctx), -1).contiguous(), torch.tensor(ctx, dtype=torch.int32, device=DEV),
                                 None, None, 0, out, W, 1.0, n, plain=plain)
    seen = out.float().mean(1).cpu() > 0.9
    assert seen.tolist() == [c - W <= place < c for c in ctx]
    assert _ok()


def test_row_sink_takes_its_share():
    """A sink that weighs as much as all keys together halves the output."""
    from rumus_b200.ops import window
    H, n, W = 3, 40, 16
    kp = torch.zeros(1, 1, 64, 8, device=DEV)
    vp = torch.ones(1, 1, 64, 8, device=DEV)
    tab = torch.zeros(1, 1, dtype=torch.int32, device=DEV)
    sink = torch.tensor([math.log(W), -1e4, math.log(3 * W)], device=DEV)
    for splits in (1, 3):
        out = torch.empty(1, H * 8, device=DEV)
        window.window_rows_attention(torch.randn(1, H, 8, device=DEV), kp, vp, tab, torch.tensor([n], dtype=torch.int32, device=DEV),
                                     sink, None, 0, out, W, 1.0, n, splits=splits)
        torch.testing.assert_close(out.view(H, 8).mean(1).cpu(), torch.tensor([0.5, 1.0, 0.25]), rtol=1e-5, atol=1e-6)


@pytest.mark.parametrize("H,G,dim,vdim,W,bs,segs,kind", [
    (4, 2, 48, 40, 37, 16, [(0, 23)], 1), (4, 2, 48, 40, 37, 64, [(0, 300), (100, 29), (127, 2), (0, 1)], 2),
    (3, 1, 128, 128, 200, 64, [(5, 130), (0, 128), (1000, 9), (63, 129)], 1),
    (6, 3, 72, 64, 128, 128, [(0, 513), (129, 127), (128, 128)], 2), (2, 2, 64, 72, 129, 8, [(0, 129), (255, 257)], 0),
    (1, 1, 8, 8, 1, 32, [(0, 65), (31, 40)], 1), (5, 1, 104, 16, 4000, 256, [(0, 300), (700, 200)], 1),
    (2, 1, 16, 128, 64, 64, [(640, 64), (64, 65), (127, 200)], 0),
])
def test_prompt_attention(H, G, dim, vdim, W, bs, segs, kind):
    """Portions that start in the middle of a sequence, at and around page, tile and window borders, several in one
    launch."""
    from rumus_b200.ops import window
    from rumus_b200.ops.latent import prefill_items
    torch.manual_seed(dim + vdim + W)
    kp, vp, tab, rows = _paged([s + n for s, n in segs], G, bs, dim, vdim, BF)
    T, mx = sum(n for _, n in segs), {"heads": H, "kv_heads": G, "scale": 2.0 * dim ** -0.5, "mask": {"size": W}}
    q = torch.randn(T, H * dim + 24, device=DEV).to(BF)[:, :H * dim].unflatten(1, (H, dim))
    gate = torch.randn(T, H * vdim if kind == 1 else p8(H), device=DEV).to(BF)
    sink = torch.randn(H, device=DEV) * 2
    out = torch.full((T, H * vdim + 8), 5.0, device=DEV, dtype=BF)
    at, r0 = [], 0
    for i, (s, n) in enumerate(segs):
        at.append((r0, n, i, s))
        r0 += n
    items = torch.tensor(prefill_items(at), dtype=torch.int32, device=DEV)
    window.window_prefill(q, kp, vp, tab, items, sink, gate if kind else None, kind, out[:, :H * vdim], W, mx["scale"])
    assert _ok() and bool((out[:, H * vdim:] == 5).all())
    for r0, n, i, s in at:
        want = _want(q[r0:r0 + n], rows(i), sink, gate[r0:r0 + n], kind, mx, s)
        got = out[r0:r0 + n, :H * vdim].double().cpu()
        err = (got - want).norm(dim=1) / (want.norm(dim=1) + 1e-3 * want.norm() / n ** 0.5)
        assert float(err.max()) < 2e-2 and _rel(got, want) < 8e-3, (s, n)


@pytest.mark.parametrize("bs", [16, 64])
@pytest.mark.parametrize("place,first,W", [
    (0, 0, 50), (1, 200, 250), (127, 0, 64), (128, 100, 100), (129, 120, 129), (255, 250, 128), (256, 256, 127), (300, 290, 1),
    (64, 0, 2), (5, 130, 127), (190, 200, 300),
])
def test_prompt_rows_see_a_key_exactly_inside_the_window(place, first, W, bs):
    from rumus_b200.ops import window
    from rumus_b200.ops.latent import prefill_items
    torch.manual_seed(place)
    H, G, dim, vdim, n = 4, 2, 32, 16, 170
    d, kp, vp, tab = _one_loud_key(place, first + n, G, dim, vdim, bs, BF)
    q = d.expand(n, H, dim).contiguous()
    out = torch.empty(n, H * vdim, device=DEV, dtype=BF)
    items = torch.tensor(prefill_items([(0, n, 0, first)]), dtype=torch.int32, device=DEV)
    window.window_prefill(q, kp, vp, tab, items, None, None, 0, out, W, 1.0)
    seen = out.float().mean(1).cpu() > 0.9
    assert seen.tolist() == [place <= first + i < place + W for i in range(n)]
    assert _ok()


# ------------------------------------------------------------------------------------------ experts
@pytest.mark.parametrize("T,E,top,dim,given", [
    (1, 8, 3, 64, False), (5, 3, 1, 40, False), (64, 64, 6, 256, False), (100, 37, 37, 72, False), (300, 16, 2, 64, True),
    (2500, 33, 4, 48, True), (700, 3, 2, 40, True), (7, 1000, 40, 32, False), (9, 1, 1, 24, True),
])
def test_routing(T, E, top, dim, given):
    """Choices and weights as in the oracle; every pair has a slot of its own in its expert's run; the work items
    cover the slots; the counters are zero again."""
    from rumus_b200.ops import moe
    torch.manual_seed(T + E)
    h, w = torch.randn(T, dim).to(BF), (torch.randn(E, dim) * dim ** -0.5).to(BF)
    bias = torch.randn(E) * 0.3
    counts = torch.zeros(E + 1, dtype=torch.int32, device=DEV)
    z = h.double() @ w.double().T + bias.double()
    logits = torch.nn.functional.pad(z - bias.double(), (0, 8)).float().to(DEV) if given else None
    for _ in range(2):
        r = moe.route(h.to(DEV), w.to(DEV), bias.to(DEV), counts, top, logits=logits)
    assert int(counts.abs().sum()) == 0
    zt, it = z.topk(top, -1)
    # 32-bit sums may order two nearly equal logits the other way round: compare the chosen logits
    chosen = torch.gather(z, 1, r.idx.long().cpu())
    assert float((chosen - zt).abs().max()) < 1e-5
    assert all(len(set(row)) == top for row in r.idx.tolist())
    torch.testing.assert_close(r.weight.double().cpu(), torch.softmax(chosen, -1), rtol=1e-5, atol=1e-6)
    slots = r.slot_of.cpu().flatten().long()
    in_order = r.tile == moe.PAIR_TILE
    assert in_order == (T * top >= moe.PAIR_LOAD * E) and len(set(slots.tolist())) == T * top
    assert (r.rows is not None) == (in_order or T > moe.ROUTE_ROWS)
    assert torch.equal(r.slot_token.cpu()[slots], torch.arange(T).repeat_interleave(top).int())
    assert torch.equal(r.slot_weight.cpu()[slots], r.weight.cpu().flatten())
    if r.rows is not None:
        assert torch.equal(r.rows.cpu()[slots], h.repeat_interleave(top, 0))
    assert in_order or r.slots == T * top
    expert_of = torch.full((r.slots,), -1)
    expert_of[slots] = r.idx.cpu().flatten().long()
    used = expert_of[expert_of >= 0]
    assert bool((used[1:] >= used[:-1]).all())
    n = int(r.n_items)
    assert 0 < n <= r.max_items
    cover = []
    for i, (e, s0, k, _) in enumerate(r.items[:n].tolist()):
        assert 0 < k <= r.tile and bool((expert_of[s0:s0 + k] == e).all()) and (not in_order or s0 == i * r.tile)
        cover += range(s0, s0 + k)
    assert sorted(cover) == sorted(slots.tolist())


def _mixture_weights(E, dim, ff, dt):
    w = {}
    for e in range(E):
        w[f"e{e}.gate"], w[f"e{e}.up"] = (torch.randn(ff, dim) * dim ** -0.5).to(dt), (torch.randn(ff, dim) * dim ** -0.5).to(dt)
        w[f"e{e}.down"] = (torch.randn(dim, ff) * ff ** -0.5).to(dt)
    w["router"], w["router.b"] = (torch.randn(E, dim) * 2 * dim ** -0.5).to(dt), torch.randn(E).to(dt)
    w["shared.gate"] = w["shared.up"] = torch.zeros(8, dim).to(dt)
    w["shared.down"] = torch.zeros(dim, 8).to(dt)
    return w


@pytest.mark.parametrize("dt,plain,tile", [(BF, False, 0), (BF, False, 16), (BF, False, 64), (BF, False, 128), (BF, False, 256), (BF, True, 0),
                                           (F32, True, 0)])
@pytest.mark.parametrize("T,E,top,dim,ff", [
    (1, 4, 2, 64, 40), (3, 8, 3, 264, 136), (40, 5, 2, 72, 296), (70, 2, 1, 128, 128), (150, 3, 2, 64, 520), (600, 2, 2, 136, 24),
    (257, 1, 1, 64, 64), (90, 64, 6, 40, 8), (1500, 4, 2, 328, 200),
])
def test_experts(dt, plain, tile, T, E, top, dim, ff):
    """Routing, both grouped products and the weighted sum, for few and for hundreds of tokens per expert."""
    from rumus_b200.ops import moe, stream
    torch.manual_seed(T + dim)
    w = _mixture_weights(E, dim, ff, dt)
    h = torch.randn(T, dim + 8).to(dt).to(DEV)[:, :dim]
    gu = moe.interleave(*(torch.stack([w[f"e{e}.{k}"] for e in range(E)]).to(DEV) for k in ("gate", "up")))
    wide = gu.shape[1] // 2
    dn = torch.nn.functional.pad(torch.stack([w[f"e{e}.down"] for e in range(E)]), (0, wide - ff)).to(DEV)
    counts = torch.zeros(E + 1, dtype=torch.int32, device=DEV)
    logits = (h.float() @ w["router"].float().T.to(DEV)).contiguous() if dt == F32 or T > moe.ROUTE_ROWS else None
    hc = h.contiguous()
    r = moe.route(hc, w["router"].to(DEV), w["router.b"].float().to(DEV), counts, top, logits=logits, plain=plain,
                  tile=tile)
    act, y = torch.empty(r.slots, wide, device=DEV, dtype=dt), torch.full((r.slots, dim + 8), 3.0, device=DEV, dtype=dt)
    moe.grouped(h, gu, r, act, gated=True, plain=plain)
    moe.grouped(act, dn, r, y[:, :dim], gated=False, plain=plain)
    assert _ok() and bool((y[:, dim:] == 3).all())
    x = torch.zeros(T, dim, device=DEV)
    stream.rms_norm_stream(x, torch.ones(dim, device=DEV), None, 1e-6, dt, p8(dim), add=(y, r.slot_of))
    wd = {k: v.double() for k, v in w.items()}
    want = N.mixture(hc.double().cpu(), wd, "", {"router": {"top": top}})
    got = x.double().cpu()
    err = (got - want).norm(dim=1) / want.norm(dim=1)
    assert float(err.max()) < (3e-2 if dt == BF else 2e-5) and _rel(got, want) < (8e-3 if dt == BF else 3e-6)
