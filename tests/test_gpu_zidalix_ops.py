"""Each mechanism of the Zidalix kernels alone, against the oracle's equations in float64."""
import pytest
import torch

import zidalix_oracle as Z

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
    return 5e-3 if dt == BF else 2e-6


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("D", [50, 64, 1000, 2052])
def test_embedding_and_norms(dt, D):
    from rumus_b200.ops import latent
    torch.manual_seed(D)
    table = torch.randn(37, D).to(dt)
    ids = torch.tensor([0, 36, 5, 5, 17])
    x = latent.embed_scaled(ids.to(DEV), table.to(DEV), 1.7)
    assert x.dtype == F32 and _rel(x, Z.embed(ids, table.double(), 1.7)) < 1e-6
    w1, w2 = torch.randn(D), torch.randn(D)
    ldy = latent.pad8(D)
    y1, y2 = latent.rms_norm_stream(x, w1.to(DEV), w2.to(DEV), 1e-2, dt, ldy)
    for y, w in ((y1, w1), (y2, w2)):
        assert _rel(y[:, :D], Z.rms_norm(x.double().cpu(), w.double(), 1e-2)) < _tol(dt)
        assert float(y[:, D:].abs().sum()) == 0
    only, none = latent.rms_norm_stream(x, w1.to(DEV), None, 1e-2, dt, ldy)
    assert none is None and torch.equal(only, y1)


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("F", [33, 64, 1000])
def test_clamped_glu(dt, F):
    from rumus_b200.ops import latent
    torch.manual_seed(F)
    gu = (torch.randn(9, 2 * F) * 3).to(dt)
    buf = torch.full((9, F + 16), 7.0, device=DEV, dtype=dt)
    latent.clamped_glu(gu.to(DEV), buf[:, 8:8 + F], 1.25, 1.702, 1.0)
    g, u = gu[:, :F].double().clamp(max=1.25), gu[:, F:].double().clamp(-1.25, 1.25)
    assert _rel(buf[:, 8:8 + F], g * torch.sigmoid(1.702 * g) * (u + 1)) < _tol(dt)
    assert bool((buf[:, :8] == 7).all()) and bool((buf[:, 8 + F:] == 7).all())


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("rank,rot,dim,heads", [(21, 6, 10, 3), (72, 24, 40, 5), (200, 40, 96, 2), (9, 2, 7, 1)])
def test_latents_rotation_and_cache_rows(dt, rank, rot, dim, heads):
    """Queries rotated in place; latents normed, the shared key part rotated, both put into the right cache rows."""
    from rumus_b200.ops import latent
    from rumus_b200.ops.rotary import RotarySpec
    torch.manual_seed(rank)
    spec = {"base": 1234.0, "dims": rot, "scaling": {"factor": 3.0, "original": 40, "fast": 8.0, "slow": 1.0}}
    T, p8 = 7, latent.pad8
    pos = torch.tensor([0, 1, 5, 64, 1000, 3, 2])
    slots = torch.tensor([9, 0, 3, -1, 15, 14, 2])
    q, z = torch.randn(T, heads, dim + rot).to(dt), torch.randn(T, rank + rot).to(dt)
    wq = p8(dim) + p8(rot)
    proj = torch.zeros(T, heads * wq + p8(rank) + p8(rot) + 8, dtype=dt)
    for h in range(heads):
        proj[:, h * wq:h * wq + dim] = q[:, h, :dim]
        proj[:, h * wq + p8(dim):h * wq + p8(dim) + rot] = q[:, h, dim:]
    col = heads * wq
    proj[:, col:col + rank], proj[:, col + p8(rank):col + p8(rank) + rot] = z[:, :rank], z[:, rank:]
    proj = proj.to(DEV)
    freq, factor = RotarySpec.from_dict(spec).frequencies()
    tab = latent.rotary_table(pos.to(DEV), freq.to(DEV), factor)
    nw = torch.rand(rank) + 0.5
    pool = torch.full((4, 4, p8(rank) + p8(rot)), 3.0, dtype=dt, device=DEV)
    latent.latent_post(proj, tab, heads, p8(dim), rot, kv_col=col, norm_w=nw.to(DEV), slots=slots.to(DEV), pool=pool, rank=rank,
                       eps=1e-3)
    got = proj.cpu()
    want_q = Z.rotate(q[..., dim:].double(), pos.tolist(), spec)
    for h in range(heads):
        assert torch.equal(got[:, h * wq:h * wq + dim], q[:, h, :dim])
        assert _rel(got[:, h * wq + p8(dim):h * wq + p8(dim) + rot], want_q[:, h]) < (5e-3 if dt == BF else 2e-5)
    rows = pool.view(16, -1).cpu()
    c = Z.rms_norm(z[:, :rank].double(), nw.double(), 1e-3)
    kr = Z.rotate(z[:, rank:].double(), pos.tolist(), spec)
    for t, s in enumerate(slots.tolist()):
        if s >= 0:
            assert _rel(rows[s, :rank], c[t]) < _tol(dt)
            assert _rel(rows[s, p8(rank):p8(rank) + rot], kr[t]) < (5e-3 if dt == BF else 2e-5)
            assert float(rows[s, rank:p8(rank)].abs().sum()) == 0 and float(rows[s, p8(rank) + rot:].abs().sum()) == 0
    untouched = [s for s in range(16) if s not in slots.tolist()]
    assert bool((rows[untouched] == 3).all())


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("T,H,K,N", [(1, 5, 40, 64), (5, 3, 24, 96), (33, 16, 128, 512), (100, 2, 40, 136), (17, 5, 512, 8)])
@pytest.mark.parametrize("transposed", [False, True])
def test_head_matmul(dt, T, H, K, N, transposed):
    from rumus_b200.ops import latent
    torch.manual_seed(T + K)
    wide = torch.randn(T, H, K + 8, device=DEV).to(dt)
    a = wide[..., :K]
    w = (torch.randn(H, *((N, K) if transposed else (K, N)), device=DEV) * K ** -0.5).to(dt)
    g = torch.randn(T, H, N, device=DEV).to(dt)
    ref = torch.einsum("thk,hnk->thn" if transposed else "thk,hkn->thn", a.double(), w.double())
    for gate in (None, g):
        out = torch.empty(T, H, N, device=DEV, dtype=dt)
        latent.head_matmul(a, w, out, transposed, gate=gate)
        assert _rel(out, ref * torch.sigmoid(g.double()) if gate is not None else ref) < _tol(dt)
    assert _ok()


def _paged(ctxs, bs, width, dt, extra=3):
    need = [(c + bs - 1) // bs for c in ctxs]
    nb = sum(need) + extra
    pool = torch.randn(nb, bs, width, device=DEV).to(dt)
    perm = torch.randperm(nb)
    tab, k = torch.zeros(len(ctxs), max(need), dtype=torch.int32), 0
    for i, n in enumerate(need):
        tab[i, :n] = perm[k:k + n]
        k += n

    def rows(i):
        idx = torch.arange(ctxs[i])
        return pool[tab[i, idx // bs].long().to(DEV), (idx % bs).to(DEV)].double().cpu()

    return pool, tab.to(DEV), rows


@pytest.mark.parametrize("dt,plain", [(BF, False), (BF, True), (F32, True)])
@pytest.mark.parametrize("H,R,rot,bs,ctxs", [
    (5, 72, 24, 64, [1, 63, 64, 65, 128, 129]), (6, 96, 16, 16, [100, 777, 33, 16, 17]), (16, 512, 64, 64, [4000, 130, 2]),
    (20, 256, 64, 128, [300, 128, 127]), (33, 512, 64, 32, [500, 1]), (128, 512, 64, 64, [700, 64]), (3, 136, 24, 8, [90, 8, 9]),
    (5, 24, 8, 64, [70]),
])
def test_row_attention(dt, plain, H, R, rot, bs, ctxs):
    """Contexts that end just before, at and after page and tile borders; heads in one group and in several."""
    from rumus_b200.ops import latent
    torch.manual_seed(H + R)
    pool, tab, rows = _paged(ctxs, bs, R + rot, dt)
    B, scale = len(ctxs), 2.0 * (R + rot) ** -0.5
    qa, qr = torch.randn(B, H, R, device=DEV).to(dt), torch.randn(B, H, rot + 8, device=DEV).to(dt)[..., :rot]
    sink = torch.randn(H, device=DEV) * 2
    out = latent.latent_rows_attention(qa, qr, pool, tab, torch.tensor(ctxs, dtype=torch.int32, device=DEV), sink, scale,
                                       max(ctxs), plain=plain)
    for i in range(B):
        kv = rows(i)
        q = torch.cat([qa[i], qr[i]], -1).double().cpu()
        want = torch.stack([Z.sink_attention(q[h:h + 1], kv, kv[:, :R], scale, sink[h].double().cpu(), offset=ctxs[i] - 1)[0]
                            for h in range(H)])
        assert _rel(out[i], want) < (6e-3 if dt == BF else 1e-5), (i, ctxs[i])
    assert _ok()


@pytest.mark.parametrize("place", [0, 1, 62, 63, 64, 65, 511, 512, 1299])
def test_row_attention_finds_one_key(place):
    """One key among 1300 carries the whole answer; it lies at the first tokens, at page borders, at the end."""
    from rumus_b200.ops import latent
    torch.manual_seed(place)
    H, R, rot, n = 3, 80, 24, 1300
    pool, tab, _ = _paged([n], 64, R + rot, BF)
    pool[..., :R] = torch.randn_like(pool[..., :R]) * 0.1
    q = torch.randn(R + rot, device=DEV)
    key = (q / q.norm() * 12).to(BF)
    pool[int(tab[0, place // 64]), place % 64] = key
    qq = q.to(BF).expand(1, H, -1)
    for ctx in (n, place + 1):
        out = latent.latent_rows_attention(qq[..., :R].contiguous(), qq[..., R:].contiguous(), pool, tab,
                                           torch.tensor([ctx], dtype=torch.int32, device=DEV), None, 0.5, n)
        assert _rel(out[0, 0], key[:R]) < 2e-2
    if place:
        out = latent.latent_rows_attention(qq[..., :R].contiguous(), qq[..., R:].contiguous(), pool, tab,
                                           torch.tensor([place], dtype=torch.int32, device=DEV), None, 0.5, n)
        assert _rel(out[0, 0], key[:R]) > 0.5      # one context length earlier the key is out of sight


@pytest.mark.parametrize("H,D,rot,V,R,segs", [
    (3, 40, 24, 32, 72, [(0, 23)]), (5, 40, 24, 48, 72, [(0, 300), (100, 29), (127, 2), (0, 1)]),
    (3, 24, 16, 40, 96, [(5, 130), (0, 128), (1000, 9), (63, 129)]), (2, 128, 64, 128, 512, [(0, 513), (129, 127)]),
    (2, 96, 64, 64, 512, [(0, 200)]), (2, 64, 8, 72, 128, [(0, 129), (255, 257)]), (1, 8, 8, 8, 8, [(0, 65)]),
])
def test_prompt_attention(H, D, rot, V, R, segs):
    """Portions that start in the middle of a sequence, at and around tile borders, several in one launch."""
    from rumus_b200.ops import latent
    torch.manual_seed(D + R)
    T, keys = sum(n for _, n in segs), sum(s + n for s, n in segs)
    q = torch.randn(T, H, D + rot, device=DEV).to(BF)
    kv, rows = torch.randn(keys, H * (D + V), device=DEV).to(BF), torch.randn(keys, R + rot, device=DEV).to(BF)
    gate, sink = torch.randn(T, H * V, device=DEV).to(BF), torch.randn(H, device=DEV) * 2
    out = torch.full((T, H * V + 8), 5.0, device=DEV, dtype=BF)
    scale, at, r0, k0 = 2.0 * (D + rot) ** -0.5, [], 0, 0
    for s, n in segs:
        at.append((r0, n, k0, s))
        r0, k0 = r0 + n, k0 + s + n
    items = torch.tensor(latent.prefill_items(at), dtype=torch.int32, device=DEV)
    latent.latent_prefill(q, kv, rows, items, sink, gate, out[:, :H * V], D, V, R, scale)
    assert _ok() and bool((out[:, H * V:] == 5).all())
    kvc, rc, qc = kv.double().cpu(), rows.double().cpu(), q.double().cpu()
    for r0, n, k0, s in at:
        for h in range(H):
            k = torch.cat([kvc[k0:k0 + s + n, h * D:(h + 1) * D], rc[k0:k0 + s + n, R:]], -1)
            v = kvc[k0:k0 + s + n, H * D + h * V:H * D + (h + 1) * V]
            want = Z.sink_attention(qc[r0:r0 + n, h], k, v, scale, sink[h].double().cpu(), offset=s)
            want = want * torch.sigmoid(gate[r0:r0 + n, h * V:(h + 1) * V].double().cpu())
            assert _rel(out[r0:r0 + n, h * V:(h + 1) * V], want) < 8e-3, (s, n, h)


@pytest.mark.parametrize("place,first", [(0, 0), (1, 200), (127, 0), (128, 100), (129, 120), (255, 250), (256, 256)])
def test_prompt_attention_causal_edge(place, first):
    """A key that every query would choose: rows before it must not see it, it and later ones must."""
    from rumus_b200.ops import latent
    torch.manual_seed(place)
    H, D, rot, V, R, n = 2, 32, 16, 32, 16, 150
    keys = first + n
    d = torch.randn(D, device=DEV)
    q = (d.expand(n, H, D) + 0.05 * torch.randn(n, H, D, device=DEV)).to(BF)
    q = torch.cat([q, torch.zeros(n, H, rot, device=DEV, dtype=BF)], -1)
    kv = (torch.randn(keys, H * (D + V), device=DEV) * 0.05).to(BF)
    kv[place, :H * D] = (d / d.norm() * 20).to(BF).repeat(H)
    kv[place, H * D:] = 1.0
    rows = torch.zeros(keys, R + rot, device=DEV, dtype=BF)
    out = torch.empty(n, H * V, device=DEV, dtype=BF)
    items = torch.tensor(latent.prefill_items([(0, n, 0, first)]), dtype=torch.int32, device=DEV)
    latent.latent_prefill(q, kv, rows, items, None, None, out, D, V, R, 1.0)
    seen = out.float().mean(1).cpu() > 0.9
    assert seen.tolist() == [first + i >= place for i in range(n)]
    assert _ok()


def test_gather_of_several_prefixes():
    from rumus_b200.ops import latent
    torch.manual_seed(0)
    ctxs = [5, 64, 65, 1]
    pool, tab, rows = _paged(ctxs, 16, 40, BF)
    off = [0]
    for c in ctxs:
        off.append(off[-1] + c)
    out = latent.latent_gather(pool, tab, torch.tensor(off, dtype=torch.int32, device=DEV), off[-1]).double().cpu()
    for i in range(len(ctxs)):
        assert torch.equal(out[off[i]:off[i + 1]], rows(i))
