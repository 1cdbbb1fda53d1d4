"""What the serving-model benchmarks share: measured peaks, event timing, kernel reports, engine throughput."""
from __future__ import annotations

import json
import os
import sys

import torch

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, ROOT)


def peaks():
    try:
        with open(os.path.join(ROOT, "MEASURED_PEAKS.json")) as f:
            d = json.load(f)
        return d["hbm_gbs"] * 1e9, d["bf16_tflops"] * 1e12, "of measured"
    except OSError:
        return 6.65e12, 1.59e15, "of fallback"


def event_ms(fn, n=5, warm=3):
    for _ in range(warm):
        fn()
    ts = []
    for _ in range(n):
        torch.cuda.synchronize()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        fn()
        b.record()
        torch.cuda.synchronize()
        ts.append(a.elapsed_time(b))
    return sorted(ts)[len(ts) // 2]


def graph_us(calls, reps=3):
    """Device time per call: the calls of one list (different operands each) captured into a graph."""
    for c in calls:
        c()
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g):
        for _ in range(reps):
            for c in calls:
                c()
    return event_ms(g.replay) * 1e3 / (reps * len(calls))


class Reports:
    """Prints one JSON line per kernel: time, roofline time, their ratio, and the same of a like kernel."""

    def __init__(self, size: str, out: list):
        self.size, self.out = size, out
        self.hbm, self.tc, self.note = peaks()

    def __call__(self, kernel, us, bytes_=0, flops=0, like=None):
        bound = max(bytes_ / self.hbm, flops / self.tc) * 1e6
        r = {"kernel": kernel, "size": self.size, "us": round(us, 2), "roofline_us": round(bound, 2), "fraction": round(bound / us, 3),
             "bound": "bytes" if bytes_ / self.hbm >= flops / self.tc else "flops", "peak": self.note}
        if like:
            r["like"] = like["kernel"]
            r["like_fraction"] = like["fraction"]
            r["distance_ratio"] = round(like["fraction"] / (bound / us), 2)
        self.out.append(r)
        print(json.dumps(r), flush=True)
        return r


def copies(bytes_each: int, least: int = 1) -> int:
    """How many operand copies together exceed L2 well."""
    return max(least, -(-300_000_000 // max(1, bytes_each)))


def engine_row(name, size, mc, layers, out, P=2048, ctx=2048, vocab=32000):
    """Prompts of ``P`` tokens as one ragged batch, then decoding at a context of ``ctx``, through ``Engine.feed``."""
    from rumus_b200.ops import native
    from rumus_b200.serve import Engine, ServeConfig
    eng = Engine(ServeConfig(model=mc, num_blocks=64 * 36 + 64, max_batch=64, max_seq_len=2304), torch.device("cuda"))
    g = torch.Generator().manual_seed(0)
    prompts = [torch.randint(0, vocab, (P,), generator=g).tolist() for _ in range(64)]
    row = {"model": name, "size": size, "layers": layers}
    for nseq in (1, 4):
        def prefill():
            eng.feed([(i, prompts[i], [P - 1]) for i in range(nseq)])
            for i in range(nseq):
                eng.release(i)
        ms = event_ms(prefill, n=3, warm=2)
        row[f"prefill_{nseq}x{P}_ms"] = round(ms, 3)
        row[f"prefill_{nseq}x{P}_tok_s"] = round(nseq * P / ms * 1e3)
    for i in range(64):
        eng.feed([(i, prompts[i][:ctx - 1], [])])
    # every sequence goes on with a token of its own, as real ones would
    for B in (1, 16, 64):
        ms = event_ms(lambda: eng.feed([(i, [prompts[i][7]], [0]) for i in range(B)]), n=7, warm=3)
        st = next(v for (b, _), v in eng._graphs.items() if b == B)
        dev_ms = event_ms(st.graph.replay)
        row[f"decode_b{B}_step_ms"], row[f"decode_b{B}_stack_ms"] = round(ms, 3), round(dev_ms, 3)
        row[f"decode_b{B}_tok_s"] = round(B / ms * 1e3)
    row["device_status"] = native.read_status()
    out.append(row)
    print(json.dumps(row), flush=True)
    del eng
    torch.cuda.empty_cache()
