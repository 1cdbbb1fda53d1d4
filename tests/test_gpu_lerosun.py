"""Lerosun through the serving engine: logits against the oracle for whole prompts, portions, decoding and mixed batches
with pages and state places used again; window edges; passes of a loop; greedy generation; the command-line trace replay.

32-bit runs have to match the float64 oracle to rounding, so a key, state or page that is wrong anywhere shows; 16-bit
runs are compared more loosely."""
import json
import os
import random
import subprocess

import pytest
import torch

import lerosun_oracle as P
from lerosun_models import CONFIGS, weights_for

pytestmark = pytest.mark.gpu
BF, F32 = torch.bfloat16, torch.float32
TOL = {F32: 2e-4, BF: 0.12}
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
_W, _REF = {}, {}


def _weights(name):
    if name not in _W:
        _W[name] = weights_for(CONFIGS[name], 5)
    return _W[name]


def _tokens(name, n, seed):
    return torch.randint(0, CONFIGS[name]["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def _reference(name, tokens):
    key = (name, tuple(tokens))
    if key not in _REF:
        _REF[key] = P.forward(CONFIGS[name], _weights(name), tokens)
    return _REF[key]


def _engine(name, dt, blocks=16, bs=64, live=4, **kw):
    from rumus_b200.models.lerosun import LerosunConfig
    from rumus_b200.serve import Engine, ServeConfig
    cfg = ServeConfig(model=LerosunConfig.from_dict(CONFIGS[name]), dtype=dt, num_blocks=blocks, block_size=bs, max_batch=live, **kw)
    return Engine(cfg, torch.device("cuda"), weights=_weights(name))


def _off(got, ref, rows=slice(None)):
    """Largest error of the logits of ``rows`` against the oracle's."""
    want = ref[rows]
    return float(((got.double().cpu() - want).norm(dim=-1) / want.norm(dim=-1)).max())


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


@pytest.mark.parametrize("dt", [F32, BF])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompts_and_portions(name, dt):
    """The same prompt whole, token by token, in portions of two, and cut around page, tile, chunk and window borders."""
    tokens = _tokens(name, 200, 1)
    ref = _reference(name, tokens)
    eng = _engine(name, dt)
    assert (eng.model.rows_per_portion is None) == (dt == F32 or name == "tall")
    assert _off(_feed(eng, 1, tokens, []), ref) < TOL[dt]
    eng.release(1)
    schedules = {"single": list(range(1, 200)), "twos": list(range(2, 200, 2)), "borders": [63, 65, 127, 128, 130, 194],
                 "ragged": [1, 4, 13, 64, 73, 82, 140, 149], "long then single": list(range(150, 200))}
    for label, cuts in schedules.items():
        assert _off(_feed(eng, 2, tokens, cuts), ref) < TOL[dt], label
        eng.release(2)
    for n in (1, 2, 3, 8, 9):           # short sequences: only first tokens, where an earlier one's state lay
        assert _off(_feed(eng, 3, tokens[:n], []), ref, slice(n)) < TOL[dt], n
        eng.release(3)
    _clean(eng)


@pytest.mark.parametrize("dt", [F32, BF])
@pytest.mark.parametrize("name,bs", [("mixed", 64), ("odd", 16), ("wide", 32), ("mixed", 48), ("many", 128)])
def test_mixed_batches_with_pages_and_places_used_again(name, dt, bs):
    """Up to four live sequences in one batch, portions beside single tokens, some left out of a step; the pool holds
    less than all sequences together, so blocks and places change hands."""
    rnd = random.Random(11)
    lens = [97, 5, 190, 33, 64, 130, 1, 71]
    seqs = {i: _tokens(name, n, 100 + i) for i, n in enumerate(lens)}
    eng = _engine(name, dt, blocks=512 // bs if bs == 128 else 448 // bs, bs=bs)
    blocks, places = [], []
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
                blocks.append(set(eng.sched.block_table(i, 64)))
                places.append(int(eng.sched.places([i])))
                eng.release(i)
                live.remove(i)
    assert any(a & b for k, a in enumerate(blocks) for b in blocks[:k]) and len(set(places)) < len(places)
    for i in seqs:
        assert _off(torch.cat(got[i]), _reference(name, seqs[i])) < TOL[dt], i
    _clean(eng)


@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_logits_do_not_depend_on_the_schedule(name):
    """32-bit logits of one position for different cuts and companions differ by rounding only."""
    tokens, other = _tokens(name, 140, 21), _tokens(name, 90, 22)
    eng = _engine(name, F32)
    a = _feed(eng, 1, tokens, [])
    eng.release(1)
    eng.feed([(7, other[:60], [])])
    b = torch.cat([eng.feed([(7, other[60:61], []), (1, tokens[:70], list(range(70)))]),
                   eng.feed([(1, tokens[70:], list(range(70))), (7, other[61:], [])])])
    c = _feed(eng, 2, tokens, list(range(100, 140)))
    for x in (b, c):
        assert float(((x - a).norm(dim=1) / a.norm(dim=1)).max()) < 1e-4
    for r in (1, 2, 7):
        eng.release(r)
    _clean(eng)


@pytest.mark.parametrize("dt", [F32, BF])
def test_long_decoding(dt):
    """Two hundred single tokens after a prompt, past several pages, chunks and windows and a graph's context bucket."""
    tokens = _tokens("mixed", 330, 31)
    eng = _engine("mixed", dt)
    assert _off(_feed(eng, 1, tokens, list(range(130, 330))), _reference("mixed", tokens)) < TOL[dt]
    assert eng.graph_replays >= 199
    eng.release(1)
    _clean(eng)


@pytest.mark.parametrize("dt", [F32, BF])
@pytest.mark.parametrize("window,heads", [(1, (4, 2)), (63, (4, 4)), (64, (2, 1)), (65, (8, 2)), (20, (12, 1))])
def test_a_token_counts_exactly_inside_the_window(window, heads, dt):
    """One attention layer, nothing else: another token at one place changes the logits where that place is seen and
    nowhere else, in prompts, in portions and in decoding."""
    name = f"one {window}"
    m = {"heads": heads[0], "kv_heads": heads[1], "dim": 16, "vdim": 16, "scale": 0.05, "mask": {"size": window}, "rot": {"base": 100.0, "dims": 8}}
    CONFIGS[name] = {"architecture": "Lerosun", "width": 40, "vocab": 60, "norm": {"eps": 1e-6},
                     "layers": [{"type": "attention", "mixer": m, "mlp": None}]}
    try:
        n, eng = 200, _engine(name, dt)
        tokens = _tokens(name, n, 41)
        for cuts in ([], [70, 72, 130, 139], list(range(150, n))):
            base = _feed(eng, 1, tokens, cuts)
            eng.release(1)
            for place in (0, 1, 4, 63, 64, 69, 70, 100):
                changed = list(tokens)
                changed[place] = (changed[place] + 7) % 60
                d = (_feed(eng, 1, changed, cuts) - base).float().norm(dim=1).cpu()
                eng.release(1)
                end = min(n, place + window)
                assert bool((d[:place] == 0).all()) and bool((d[end:] == 0).all()), place
                assert float((d[place:end] > 0).float().mean()) > 0.7 and float(d[place]) > 0, place
        _clean(eng)
    finally:
        del CONFIGS[name]
        _W.pop(name, None)


def test_every_pass_of_a_loop_has_a_cache_and_state_of_its_own():
    eng = _engine("mixed", F32)
    runs = eng.model.model.runs
    assert len(eng.cache.k) == len(runs) == 8
    pools = [t.data_ptr() for t in eng.cache.k if t is not None] + [l["S"].data_ptr() for l in eng.cache.state.layers if l is not None]
    assert len(set(pools)) == len(pools) == 8
    tokens = _tokens("mixed", 60, 3)
    _feed(eng, 1, tokens, [40])
    a, b = eng.cache.k[1], eng.cache.k[4]                     # both passes of layer 1
    assert float(a.abs().sum()) > 0 and float((a - b).abs().sum()) > 0


@pytest.mark.parametrize("place", [0, 1, 63, 64, 127, 128, 190])
def test_a_far_token_reaches_later_logits(place):
    """Changing one early token changes the logits of later ones exactly as in the oracle, in prompts and in decoding."""
    tokens = _tokens("mixed", 220, 41)
    changed = list(tokens)
    changed[place] = (changed[place] + 7) % CONFIGS["mixed"]["vocab"]
    a, b = _reference("mixed", tokens), _reference("mixed", changed)
    assert float((a[219] - b[219]).norm() / a[219].norm()) > 4 * TOL[F32]
    eng = _engine("mixed", F32)
    for cuts in ([], [place + 1], list(range(212, 220))):
        assert _off(_feed(eng, 1, changed, cuts), b) < TOL[F32]
        eng.release(1)


def _greedy(name, prompt, n):
    out = list(prompt)
    for _ in range(n):
        out.append(int(P.forward(CONFIGS[name], _weights(name), out)[-1].argmax()))
    return out[len(prompt):]


def test_greedy_generation_matches_the_oracle():
    """Through add_request / step, the scheduler's own portions: more requests than places, prompts longer than the token
    budget, a pool small enough to preempt."""
    name = "mixed"
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
        assert outs[rid] == _greedy(name, p, m), rid
    assert eng.sched.preemptions() > 0
    _clean(eng)


def test_greedy_generation_in_16_bits_follows_the_oracle_where_it_is_clear():
    """Nearly every generated token is the oracle's choice, or one whose logit the oracle puts within rounding of it."""
    name = "wide"
    eng = _engine(name, BF, blocks=32, live=4, token_budget=64)
    reqs = {i + 1: (_tokens(name, n, 80 + i), 10) for i, n in enumerate([90, 12, 30])}
    for rid, (p, m) in reqs.items():
        assert eng.add_request(rid, p, m)
    good = []
    while eng.has_work():
        for rid in eng.step():
            out, (p, _) = eng.requests.pop(rid).output, reqs[rid]
            ref = _reference(name, p + out)
            for k, t in enumerate(out):
                row = ref[len(p) + k - 1]
                good.append(float(row.max() - row[t]) < 0.3 * float(row.std()))
    assert len(good) == 30 and sum(good) >= 27
    _clean(eng)


def test_graphs_match_eager_decoding():
    """Also portions of a few tokens, which go through the same graphs."""
    tokens = _tokens("mixed", 100, 51)
    outs = []
    for graphs in (True, False):
        eng = _engine("mixed", F32, cuda_graphs=graphs)
        outs.append(_feed(eng, 1, tokens, list(range(60, 90)) + [92, 97]))
        assert (eng.graph_replays > 0) == graphs
    assert float(((outs[0] - outs[1]).norm(dim=1) / outs[1].norm(dim=1)).max()) < 1e-5


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
            assert _off(g[None], ref, slice(i, i + 1)) < 2 * TOL[dt], (k, i)


def test_engine_from_a_folder(tmp_path):
    from rumus_b200.serve.loading import load_engine
    _save_model("mixed", str(tmp_path))
    eng = load_engine(str(tmp_path), torch.device("cuda"), F32, num_blocks=8, max_batch=2)
    tokens = _tokens("mixed", 30, 91)
    assert _off(_feed(eng, 1, tokens, [20]), _reference("mixed", tokens)) < TOL[F32]
    assert eng.cache.state.bytes_per_sequence() > 0 and eng.cache.bytes_per_token() > 0
