"""Nufupel through the serving engine: logits against the oracle for whole prompts, portions, decoding and mixed batches
with pages used again; window edges; greedy generation; the command-line trace replay.

32-bit runs have to match the float64 oracle to rounding, so a key, state or page that is wrong anywhere shows; 16-bit
runs are compared more loosely, and not at positions where rounding may choose another expert."""
import json
import os
import random
import subprocess

import pytest
import torch

import nufupel_oracle as N
from nufupel_models import CONFIGS, weights_for

pytestmark = pytest.mark.gpu
BF, F32 = torch.bfloat16, torch.float32
TOL = {F32: 3e-5, BF: 6e-2}
MARGIN = {F32: 1e-4, BF: 0.1}            # a choice of experts closer than this may go either way
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
_W, _REF = {}, {}


def _weights(name):
    if name not in _W:
        _W[name] = weights_for(CONFIGS[name], 5)
    return _W[name]


def _tokens(name, n, seed):
    return torch.randint(0, CONFIGS[name]["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def _reference(name, tokens):
    """(logits, smallest margin of every position over the mixtures)."""
    key = (name, tuple(tokens))
    if key not in _REF:
        margins = []
        out = N.forward(CONFIGS[name], _weights(name), tokens, margins=margins)
        _REF[key] = out, torch.stack(margins).min(0).values
    return _REF[key]


def _engine(name, dt, blocks=16, bs=64, live=4, **kw):
    from rumus_b200.models.nufupel import NufupelConfig
    from rumus_b200.serve import Engine, ServeConfig
    cfg = ServeConfig(model=NufupelConfig.from_dict(CONFIGS[name]), dtype=dt, num_blocks=blocks, block_size=bs, max_batch=live, **kw)
    return Engine(cfg, torch.device("cuda"), weights=_weights(name))


def _err(got, want):
    """Relative error per position: the largest, or three times the mean if that is more (peaked attention makes single
    positions sensitive to 16-bit rounding; most are far below)."""
    e = (got.double().cpu() - want).norm(dim=-1) / want.norm(dim=-1)
    return float(torch.maximum(e.max(), 3 * e.mean()))


def _off(got, ref, dt, rows=slice(None)):
    """Error of the logits of ``rows`` against ``_reference``'s, over positions whose choices of experts are clear.  In
    16 bits another choice at an unclear position also reaches later ones through their windows: the few largest
    errors count a fourth."""
    want, margin = ref[0][rows], ref[1][rows]
    clear = margin > MARGIN[dt]
    assert len(clear) < 10 or float(clear.float().mean()) > 0.4
    if not bool(clear.any()):
        return 0.0
    got, want = got[clear.to(got.device)], want[clear]
    if dt == F32:
        return _err(got, want)
    e = ((got.double().cpu() - want).norm(dim=-1) / want.norm(dim=-1)).sort().values
    few = len(e) // 20
    return max(float(e[len(e) - 1 - few]), 3 * float(e.mean()), float(e[-1]) / 4)


def _feed(eng, rid, tokens, cuts):
    """Logits of every token, fed in portions that end at ``cuts`` and the end."""
    out, at = [], 0
    for c in list(cuts) + [len(tokens)]:
        out.append(eng.feed([(rid, tokens[at:c], list(range(c - at)))]))
        at = c
    return torch.cat(out)


def _clean(eng):
    from rumus_b200.ops import native
    assert native.read_status() == 0 and eng.sched.free_blocks() == eng.cfg.num_blocks
    assert all(int(L.counts.abs().sum()) == 0 for L in eng.model.layers if L.mixture)


@pytest.mark.parametrize("dt", [F32, BF])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompts_and_portions(name, dt):
    """The same prompt whole, token by token, in portions of two, and cut around page, tile and window borders."""
    tokens = _tokens(name, 170, 1)
    ref = _reference(name, tokens)
    eng = _engine(name, dt)
    assert (eng.model.rows_per_portion is None) == (dt == F32 or name == "tall")
    assert _off(_feed(eng, 1, tokens, []), ref, dt) < TOL[dt]
    eng.release(1)
    schedules = {"single": list(range(1, 170)), "twos": list(range(2, 170, 2)), "borders": [63, 65, 127, 128, 130],
                 "ragged": [1, 4, 13, 64, 73, 82, 140, 149], "long then single": list(range(120, 170))}
    for label, cuts in schedules.items():
        assert _off(_feed(eng, 2, tokens, cuts), ref, dt) < TOL[dt], label
        eng.release(2)
    for n in (1, 2, 3, 8, 9):           # short sequences: only first tokens
        assert _off(_feed(eng, 3, tokens[:n], []), ref, dt, slice(n)) < TOL[dt], n
        eng.release(3)
    _clean(eng)


@pytest.mark.parametrize("dt", [F32, BF])
@pytest.mark.parametrize("name,bs", [("shared", 64), ("odd", 16), ("wide", 32), ("shared", 48)])
def test_mixed_batches_and_pages_used_again(name, dt, bs):
    """Up to four live sequences in one batch, portions beside single tokens, some left out of a step; the pool holds
    less than all sequences together, so blocks change hands."""
    rnd = random.Random(11)
    lens = [97, 5, 190, 33, 64, 130, 1, 71]
    seqs = {i: _tokens(name, n, 100 + i) for i, n in enumerate(lens)}
    eng = _engine(name, dt, blocks=448 // bs, bs=bs)
    handed = []
    waiting, live, at, got = list(seqs), [], {i: 0 for i in seqs}, {i: [] for i in seqs}
    guard = 0
    while waiting or live:
        guard += 1
        assert guard < 2000
        need = lambda i: (len(seqs[i]) + bs - 1) // bs
        while waiting and len(live) < 4 and sum(need(i) for i in live + waiting[:1]) <= eng.cfg.num_blocks:
            live.append(waiting.pop(0))
        batch = []
        for i in live:
            if rnd.random() < 0.25 and len(live) > 1:
                continue
            left = len(seqs[i]) - at[i]
            batch.append((i, min(left, rnd.choice([1, 1, 2, 3, 9, 17, 64, 128]))))
        if not batch:
            continue
        logits = eng.feed([(i, seqs[i][at[i]:at[i] + n], list(range(n))) for i, n in batch])
        for i, n in batch:
            got[i].append(logits[:n])
            logits = logits[n:]
            at[i] += n
            if at[i] == len(seqs[i]):
                handed.append(set(eng.sched.block_table(i, 64)))
                eng.release(i)
                live.remove(i)
    assert any(a & b for k, a in enumerate(handed) for b in handed[:k])          # blocks were used again
    for i in seqs:
        assert _off(torch.cat(got[i]), _reference(name, seqs[i]), dt) < TOL[dt], i
    _clean(eng)


@pytest.mark.parametrize("name", ["shared", "wide"])
def test_logits_do_not_depend_on_the_schedule(name):
    """16-bit logits of one position for different cuts and companions differ by rounding only: far less than they
    differ from another token's."""
    tokens, other = _tokens(name, 140, 21), _tokens(name, 90, 22)
    clear = _reference(name, tokens)[1] > MARGIN[BF]
    eng = _engine(name, BF)
    a = _feed(eng, 1, tokens, [])
    eng.release(1)
    eng.feed([(7, other[:60], [])])
    b = torch.cat([eng.feed([(7, other[60:61], []), (1, tokens[:70], list(range(70)))]),
                   eng.feed([(1, tokens[70:], list(range(70))), (7, other[61:], [])])])
    c = _feed(eng, 2, tokens, list(range(100, 140)))
    for x in (b, c):
        assert _err(x.cpu()[clear], a.double().cpu()[clear]) < 5e-2
    for r in (1, 2, 7):
        eng.release(r)
    _clean(eng)


@pytest.mark.parametrize("dt", [F32, BF])
def test_long_decoding(dt):
    """Two hundred single tokens after a prompt, past several pages and windows and a graph's context bucket."""
    tokens = _tokens("shared", 330, 31)
    eng = _engine("shared", dt)
    assert _off(_feed(eng, 1, tokens, list(range(130, 330))), _reference("shared", tokens), dt) < TOL[dt]
    assert eng.graph_replays >= 199
    eng.release(1)
    _clean(eng)


def _one_layer(kind, window):
    """One attention layer, nothing else: what it cannot see has no way into the logits."""
    m = {"heads": 4, "kv_heads": 2, "dim": 16, "vdim": 16, "scale": 0.4, "mask": {"size": window}}
    if kind == "attention_2":
        m["rot"] = {"base": 100.0, "dims": 8, "scaling": None}
    return {"architecture": "Nufupel", "width": 40, "vocab": 60, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.5},
            "logit_softcap": 30.0, "layers": [{"type": kind, "mixer": m, "mlp": None}]}


@pytest.mark.parametrize("dt", [F32, BF])
@pytest.mark.parametrize("kind", ["attention", "attention_2"])
@pytest.mark.parametrize("window", [1, 63, 64, 65, 130])
def test_a_token_counts_exactly_inside_the_window(kind, window, dt):
    """Another token at one place changes the logits up to window - 1 places further on and not one more, in prompts, in
    portions and in decoding."""
    name = f"{kind} {window}"
    CONFIGS[name] = _one_layer(kind, window)
    try:
        n, eng = 200, _engine(name, dt)
        tokens = _tokens(name, n, 41)
        for cuts in ([], [70, 72, 130, 139], list(range(150, n))):
            base = _feed(eng, 1, tokens, cuts)
            eng.release(1)
            for place in (0, 1, 63, 64, 65, 100):
                changed = list(tokens)
                changed[place] = (changed[place] + 7) % 60
                d = (_feed(eng, 1, changed, cuts) - base).float().norm(dim=1).cpu()
                eng.release(1)
                assert bool((d[:place] == 0).all()) and bool((d[place + window:] == 0).all())
                seen = d[place:min(n, place + window)]
                assert float((seen > 0).float().mean()) > 0.7 and float(seen[0]) > 0
        _clean(eng)
    finally:
        del CONFIGS[name]
        _W.pop(name, None)


@pytest.mark.parametrize("place", [0, 1, 63, 64, 127, 128, 200])
def test_a_far_token_reaches_later_logits(place):
    """Changing one early token changes the logits of later ones, within the windows' joint reach, exactly as in the
    oracle, in prompts and in decoding."""
    tokens = _tokens("shared", 220, 41)
    changed = list(tokens)
    changed[place] = (changed[place] + 7) % CONFIGS["shared"]["vocab"]
    a, b = _reference("shared", tokens)[0], _reference("shared", changed)
    d = (a - b[0]).norm(dim=-1) / a.norm(dim=-1)
    far = min(219, place + 150)
    assert float(d[far]) > 20 * TOL[F32]
    eng = _engine("shared", F32)
    for cuts in ([], [place + 1] if place else [1], list(range(212, 220))):
        assert _off(_feed(eng, 1, changed, cuts), b, F32) < TOL[F32]
        eng.release(1)


def test_greedy_generation_matches_the_oracle():
    """Through add_request / step, the scheduler's own portions: more requests than slots, prompts longer than the token
    budget, a pool small enough to preempt."""
    name = "shared"
    reqs = {i + 1: (_tokens(name, n, 60 + i), m) for i, (n, m) in enumerate([(70, 12), (3, 9), (40, 17), (1, 5), (100, 6), (9, 20)])}
    eng = _engine(name, F32, blocks=8, bs=16, live=3, token_budget=48)
    for rid, (p, m) in reqs.items():
        assert eng.add_request(rid, p, m)
    assert not eng.add_request(99, [1] * 200, 5)              # longer than the pool
    outs = {}
    while eng.has_work():
        for rid in eng.step():
            outs[rid] = eng.requests.pop(rid).output
    for rid, (p, m) in reqs.items():
        assert outs[rid] == N.greedy(CONFIGS[name], _weights(name), p, m), rid
    assert eng.sched.preemptions() > 0
    _clean(eng)


def test_greedy_generation_in_16_bits_follows_the_oracle_where_it_is_clear():
    """Every generated token is the oracle's choice, or one whose logit the oracle puts within rounding of it."""
    name = "wide"
    eng = _engine(name, BF, blocks=32, live=4, token_budget=64)
    reqs = {i + 1: (_tokens(name, n, 80 + i), 10) for i, n in enumerate([90, 12, 30])}
    for rid, (p, m) in reqs.items():
        assert eng.add_request(rid, p, m)
    while eng.has_work():
        for rid in eng.step():
            out, (p, _) = eng.requests.pop(rid).output, reqs[rid]
            ref, margin = _reference(name, p + out)
            for k, t in enumerate(out):
                row = ref[len(p) + k - 1]
                assert float(row.max() - row[t]) < 0.15 * float(row.std()) or float(margin[len(p) + k - 1]) < MARGIN[BF]
    _clean(eng)


def test_graphs_match_eager_decoding():
    tokens = _tokens("shared", 90, 51)
    outs = []
    for graphs in (True, False):
        eng = _engine("shared", BF, cuda_graphs=graphs)
        outs.append(_feed(eng, 1, tokens, list(range(60, 90))))
        assert (eng.graph_replays > 0) == graphs
    assert _err(outs[0], outs[1].double().cpu()) < 1e-2


def _save_model(name, folder):
    from rumus_b200.io.safetensors import save_tensors
    save_tensors(_weights(name), os.path.join(folder, "model.safetensors"))
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(CONFIGS[name], f)


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_replay(tmp_path, dtype):
    _save_model("odd", str(tmp_path))
    a, b = _tokens("odd", 90, 71), _tokens("odd", 40, 72)
    steps = [
        {"step": 0, "entries": [{"id": "p", "tokens": a[:70], "want": [0, 69]}], "end": []},
        {"step": 1, "entries": [{"id": "q", "tokens": b[:3], "want": []}], "end": []},
        {"step": 2, "entries": [{"id": "p", "tokens": a[70:71], "want": [0]}, {"id": "q", "tokens": b[3:], "want": [36, 1]}], "end": ["q"]},
        {"step": 5, "entries": [{"id": "p", "tokens": a[71:], "want": [18]}], "end": ["p"]},
        {"step": 6, "entries": [{"id": "p", "tokens": b, "want": [39]}], "end": ["p"]},      # a new sequence of that name
    ]
    out = tmp_path / "out"
    out.mkdir()
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", dtype, "--out", str(out),
                        "--max-tokens", "192"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True,
                       text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {k}" for k in (0, 1, 2, 5, 6)]
    assert not (out / "1.f32").exists()
    ra, rb = _reference("odd", a), _reference("odd", b)
    want = {0: [(ra, 0), (ra, 69)], 2: [(ra, 70), (rb, 39), (rb, 4)], 5: [(ra, 89)], 6: [(rb, 39)]}
    dt = getattr(torch, dtype)
    for k, rows in want.items():
        got = torch.frombuffer(bytearray((out / f"{k}.f32").read_bytes()), dtype=torch.float32).view(len(rows), -1)
        for g, (ref, i) in zip(got, rows):
            assert _off(g[None], ref, dt, slice(i, i + 1)) < TOL[dt], k


def test_engine_from_a_folder(tmp_path):
    from rumus_b200.serve.loading import load_engine
    _save_model("shared", str(tmp_path))
    eng = load_engine(str(tmp_path), torch.device("cuda"), F32, num_blocks=8, max_batch=2)
    tokens = _tokens("shared", 30, 91)
    assert _off(_feed(eng, 1, tokens, [20]), _reference("shared", tokens), F32) < TOL[F32]
