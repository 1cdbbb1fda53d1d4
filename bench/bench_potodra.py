"""Potodra against the framework's closest model (Nufupel: windows, sinks, mixtures of experts with a shared one, fp32
residual) at equal size, and every kernel of its decoder stack against its roofline beside the like kernel.

    python bench.py --potodra            (or: python bench/bench_potodra.py [--kernels] [--models] [--size NAME])

Models: random weights, ``--layers`` layers of a real model's size, attention, two matrix memories and a parallel layer
in turn; the first layer's feed-forward dense, the others mixtures; four streams.  Prompts of 2048 tokens as one ragged
batch, then decoding at a context of 2048 with 1, 16 and 64 sequences through ``Engine.feed`` (CUDA graphs), CUDA-event
times.  The layers' weights and caches of a step exceed L2.  Kernels: captured into a graph over rotating operand copies
that together exceed L2, CUDA-event time of a replay divided by the launches in it.

The recurrent kernels have no like kernel in another model; they stand beside what does the same job there, prompt
attention and single-row attention.  Their rooflines count the vectors that enter and leave a head and one pass over its
state, in the state's recurrent form.
"""
from __future__ import annotations

import argparse
import os
import sys

import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))

from bench_nufupel import SIZES, nufupel_config  # noqa: E402
from serving_common import Reports, copies, engine_row, graph_us  # noqa: E402

from rumus_b200.models.potodra import PotodraConfig  # noqa: E402
from rumus_b200.ops import latent, moe, native, recurrent, stream, window  # noqa: E402

WINDOW, KEEP, CAP, STREAMS, TAPS, GROUPS, OPEN = 1024, 16, 30.0, 4, 4, 8, 4


def potodra_config(size, layers, vocab=32000):
    width, heads, kv, ff, E, top, eff, sff = SIZES[size]
    att = {"heads": heads, "kv_heads": kv, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "rot": {"base": 1e6, "dims": 128}}
    mem = {"heads": heads, "dim": 128, "vdim": 128}
    mixers = [("attention", {**att, "mask": {"size": WINDOW, "keep_first": KEEP}, "softcap": CAP}), ("mlstm", {**mem, "gate_cap": 15.0}),
              ("mlstm", {**mem, "gate_cap": 15.0}),
              ("parallel", {"left": att, "right": {**mem, "kv_heads": heads, "conv": TAPS}, "left_scale": 0.5, "right_scale": 0.5})]
    entries = []
    for i in range(layers):
        mlp = {"kind": "dense", "ff": ff} if i == 0 else \
            {"kind": "moe", "router": {"experts": E, "top": top, "groups": {"count": GROUPS, "keep": OPEN}},
             "expert": {"ff": eff, "limit": 7.0}, "shared": {"ff": sff, "limit": 7.0}}
        entries.append({"type": mixers[i % 4][0], "mixer": mixers[i % 4][1], "mlp": mlp})
    return PotodraConfig.from_dict({"vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0}, "streams": STREAMS,
                                    "layers": entries})


def bench_models(size, layers, out):
    engine_row("potodra", size, potodra_config(size, layers), layers, out)
    engine_row("nufupel", size, nufupel_config(size, layers), layers, out)


def bench_kernels(size, out):
    width, H, G, ff, E, top, eff, sff = SIZES[size]
    report = Reports(size, out)
    dev, bf = "cuda", torch.bfloat16
    D = V = 128

    def rnd(*s, scale=1.0):
        return (torch.randn(*s, device=dev) * scale).to(bf)

    # ---- prompt mixers
    S, n = 4096, 2
    nb = S // 64
    kp, vp = rnd(nb, G, 64, D), rnd(nb, G, 64, V)
    tab = torch.randperm(nb, device=dev).int().view(1, -1)
    items = torch.tensor(latent.prefill_items([(0, S, 0, 0)]), dtype=torch.int32, device=dev)
    q, o, gate, sink = rnd(S, H, D), rnd(S, H * V), rnd(S, H * V), torch.zeros(H, device=dev)
    prompt = {}
    for W in (WINDOW, S):
        pairs = sum(min(W, i + 1) for i in range(S))
        cost = dict(flops=H * pairs * (D + V) * 2, bytes_=S * (3 * H + 2 * G) * D * 2)
        us = graph_us([lambda: window.window_prefill(q, kp, vp, tab, items, sink, gate, 1, o, W, D ** -0.5)] * n)
        prompt[W] = report(f"window_prefill W{W} (Nufupel)", us, **cost)
        cost["bytes_"] -= S * H * V * 2
        us = graph_us([lambda: window.window_prefill(q, kp, vp, tab, items, sink, None, 0, o, W, D ** -0.5, keep=KEEP, cap=CAP)] * n)
        report(f"window_prefill W{W} kept {KEEP} capped", us, **cost, like=prompt[W])
        us = graph_us([lambda: window.window_prefill(q, kp, vp, tab, items, None, None, 0, o, W, D ** -0.5)] * n)
        report(f"window_prefill W{W} plain", us, **cost, like=prompt[W])
    del kp, vp
    taps, norm, dt, decay = torch.randn(TAPS, 3 * H * D, device=dev), torch.ones(H * V, device=dev), torch.full((H * D,), -4.0, device=dev), \
        torch.ones(H, device=dev)

    def memory(places):
        return {"S": torch.zeros(places, H, D, V, device=dev), "n": torch.zeros(places, H, D, device=dev), "m": torch.zeros(places, H, device=dev),
                "conv": torch.zeros(places, H, TAPS - 1, 3 * D, device=dev, dtype=bf)}

    for nseq, L in ((1, S), (4, 2048)):
        T, state = nseq * L, memory(nseq)
        seqs = torch.tensor([[i * L, L, i, 0] for i in range(nseq)], dtype=torch.int32, device=dev)
        cuts = {c: recurrent.cut([(i * L, L) for i in range(nseq)], c, dev) for c in (recurrent.MLSTM_CHUNK, recurrent.DELTA_CHUNK)}
        pj, gates, mix = rnd(T, 4 * H * D), torch.randn(T, 2 * H, device=dev), rnd(T, H * V)
        us = graph_us([lambda: recurrent.mlstm_chunks(pj, gates, cuts[recurrent.MLSTM_CHUNK], seqs, state, pj[:, 3 * H * D:], norm, mix, D, V, 15.0,
                                                      1e-6)] * n)
        report(f"mlstm_chunks {nseq} x {L}", us, flops=T * H * 4 * D * V, bytes_=T * H * (5 * 2 * D + 8) + nseq * H * D * V * 4, like=prompt[S])
        step, beta = torch.randn(T, H * D, device=dev), torch.randn(T, H, device=dev)
        us = graph_us([lambda: recurrent.delta_chunks(pj, taps, step, dt, decay, beta, cuts[recurrent.DELTA_CHUNK], seqs, state, pj[:, 3 * H * D:],
                                                      norm, mix, H, D, V, 1e-6)] * n)
        report(f"delta_chunks {nseq} x {L}", us, flops=T * H * 6 * D * V, bytes_=T * H * (5 * 2 * D + 4 * D + 4) + nseq * H * D * V * 4,
               like=prompt[S])
        del pj, mix, step

    # ---- single rows
    for B, ctx in ((1, 8192), (16, 4096), (64, 2048), (64, 1024)):
        bs, nb = 64, B * ctx // 64
        tab = torch.randperm(nb, device=dev).int().view(B, -1)
        cl = torch.full((B,), ctx, dtype=torch.int32, device=dev)
        m = copies(nb * bs * G * D * 4)
        kc, vc = [rnd(nb, G, bs, D) for _ in range(m)], [rnd(nb, G, bs, D) for _ in range(m)]
        ql, gt, ow = rnd(B, H, D), rnd(B, H * V), rnd(B, H * V)
        cost = dict(bytes_=B * ctx * G * D * 4 + 2 * B * H * D * 2, flops=B * ctx * H * D * 4)
        us = graph_us([lambda i=i: window.window_rows_attention(ql, kc[i], vc[i], tab, cl, sink, gt, 1, ow, ctx, D ** -0.5, ctx) for i in range(m)])
        like = report(f"window_rows b{B} W{ctx} (Nufupel)", us, **cost)
        us = graph_us([lambda i=i: window.window_rows_attention(ql, kc[i], vc[i], tab, cl, sink, None, 0, ow, ctx - KEEP, D ** -0.5, ctx, keep=KEEP,
                                                                cap=CAP) for i in range(m)])
        report(f"window_rows b{B} W{ctx - KEEP} kept {KEEP} capped", us, **cost, like=like)
        del kc, vc
        if ctx == 1024:
            continue
        bytes_ = B * H * (D * V * 8 + 5 * D * 2)
        m = copies(B * H * D * V * 8)
        states = [memory(B) for _ in range(m)]
        seqs = torch.tensor([[i, 1, i, 5] for i in range(B)], dtype=torch.int32, device=dev)
        pj, gates, step, beta = rnd(B, 4 * H * D), torch.randn(B, 2 * H, device=dev), torch.randn(B, H * D, device=dev), torch.randn(B, H, device=dev)
        us = graph_us([lambda i=i: recurrent.mlstm_rows(pj, gates, seqs, states[i], pj[:, 3 * H * D:], norm, ow, D, V, 15.0, 1e-6)
                       for i in range(m)])
        report(f"mlstm_rows b{B}", us, bytes_=bytes_, flops=B * H * 4 * D * V, like=like)
        us = graph_us([lambda i=i: recurrent.delta_rows(pj, taps, step, dt, decay, beta, seqs, states[i], pj[:, 3 * H * D:], norm, ow, H, D, V, 1e-6)
                       for i in range(m)])
        report(f"delta_rows b{B}", us, bytes_=bytes_ + B * H * D * (4 + 12 * (TAPS - 1)), flops=B * H * 6 * D * V, like=like)
        del states

    # ---- products with weights
    for T in (1, 16, 64, 512, 2048, 8192):
        x = rnd(T, width)
        m = copies(2 * ff * width * 2, 2)
        ws = [rnd(2 * ff, width) for _ in range(m)]
        us = graph_us([lambda i=i: native.gemm(x, ws[i].t()) for i in range(m)], reps=1)
        gu_like = report(f"gemm gate|up (Nufupel) {width}->{2 * ff} t{T}", us, bytes_=2 * ff * width * 2 + T * (2 * ff + width) * 2,
                         flops=4 * T * ff * width)
        del ws
        m = copies(ff * width * 2, 2)
        ws, xk, res = [rnd(width, ff) for _ in range(m)], rnd(T, ff), torch.randn(T, width, device=dev)
        us = graph_us([lambda i=i: native.gemm(xk, ws[i].t(), residual=res, out_dtype=torch.float32) for i in range(m)], reps=1)
        dn_like = report(f"gemm down + residual (Nufupel) {ff}->{width} t{T}", us, bytes_=ff * width * 2 + T * (ff * 2 + width * 8),
                         flops=2 * T * ff * width)
        us = graph_us([lambda i=i: native.gemm(xk, ws[i].t(), out_dtype=torch.float32) for i in range(m)], reps=1)
        report(f"gemm down {ff}->{width} t{T}", us, bytes_=ff * width * 2 + T * (ff * 2 + width * 4), flops=2 * T * ff * width, like=dn_like)
        ws = [w.view(ff, width) for w in ws]
        us = graph_us([lambda i=i: native.gemm(x, ws[i].t(), act="relu2") for i in range(m)], reps=1)
        report(f"gemm up, squared relu {width}->{ff} t{T}", us, bytes_=ff * width * 2 + T * (ff + width) * 2, flops=2 * T * ff * width, like=gu_like)
        del ws
        for what, N, biased in (("attention", (H + 2 * G) * D, True), ("memory", 4 * H * D, False), ("parallel", (H + 2 * G) * D + 3 * H * D + 2 * D, True)):
            m = copies(N * width * 2, 2)
            ws, bias = [rnd(N, width) for _ in range(m)], rnd(N) if biased else None
            us = graph_us([lambda i=i: native.gemm(x, ws[i].t(), bias=bias) for i in range(m)], reps=1)
            report(f"gemm input of {what} {width}->{N} t{T}", us, bytes_=N * width * 2 + T * (N + width) * 2, flops=2 * T * N * width, like=gu_like)
            del ws
        for what, K in (("heads", H * V), ("both halves", 2 * H * V)):
            m = copies(K * width * 2, 2)
            ws, xk = [rnd(width, K) for _ in range(m)], rnd(T, K)
            us = graph_us([lambda i=i: native.gemm(xk, ws[i].t(), out_dtype=torch.float32) for i in range(m)], reps=1)
            report(f"gemm output of {what} {K}->{width} t{T}", us, bytes_=K * width * 2 + T * (K * 2 + width * 4), flops=2 * T * K * width,
                   like=dn_like)
            del ws
        low = rnd(T, D)
        ws = [rnd(H * D, D) for _ in range(copies(H * D * D * 2 + T * H * D * 4, 2))]
        us = graph_us([lambda i=i: native.gemm(low, ws[i].t(), out_dtype=torch.float32) for i in range(len(ws))], reps=1)
        report(f"gemm low rank {D}->{H * D} t{T}", us, bytes_=H * D * D * 2 + T * (D * 2 + H * D * 4), flops=2 * T * D * H * D, like=gu_like)
        few = [rnd(2 * H, width) for _ in range(8)]
        fn = (lambda i: recurrent.few_outputs(x, few[i])) if T <= recurrent.FEW_ROWS else (lambda i: native.gemm(x, few[i].t(), out_dtype=torch.float32))
        us = graph_us([lambda i=i: fn(i) for i in range(8)], reps=1)
        report(f"few outputs {width}->{2 * H} t{T}", us, bytes_=2 * H * width * 2 + T * width * 2 + T * H * 8, flops=4 * T * H * width, like=gu_like)
        # experts
        m = max(2, min(3, copies(E * 3 * eff * width * 2)))
        gu = [rnd(E, 2 * eff, width) for _ in range(m)]
        rt, rb, counts = rnd(E, width, scale=width ** -0.5), torch.zeros(E, device=dev), torch.zeros(E + 1, device=dev, dtype=torch.int32)

        def routing(**kw):
            lg = native.gemm(x, rt.t(), out_dtype=torch.float32) if T > moe.ROUTE_ROWS else None
            return moe.route(x, rt, rb, counts, top, logits=lg, **kw)

        cost = dict(bytes_=T * width * 2 + E * width * 2 + (T * (top + 1) * width * 2 if T > moe.ROUTE_ROWS else 0), flops=2 * T * E * width)
        like = report(f"route (Nufupel) t{T}", graph_us([routing]), **cost)
        kw = dict(score=moe.SIGMOID, groups=GROUPS, keep=OPEN)
        report(f"route by groups t{T}", graph_us([lambda: routing(**kw)]), **cost, like=like)
        r = routing(**kw)
        used = len(r.idx.unique())
        act = torch.empty(r.slots, eff, device=dev, dtype=bf)
        cost = dict(bytes_=used * 2 * eff * width * 2 + T * width * 2 + T * top * eff * 2, flops=4 * T * top * eff * width)
        like = report(f"moe gate|up (Nufupel) t{T}", graph_us([lambda i=i: moe.grouped(x, gu[i], r, act, True) for i in range(m)]), **cost)
        us = graph_us([lambda i=i: moe.grouped(x, gu[i], r, act, True, unit=(7.0, 1.702, 1.0)) for i in range(m)])
        report(f"moe gate|up, clamped t{T}", us, **cost, like=like)
        del gu

    # ---- around the sub-layers
    for T in (1, 64, 8192):
        m = copies(T * width * 4 * STREAMS) if T > 1 else 8
        xs = [torch.randn(T, STREAMS, width, device=dev) for _ in range(m)]
        flat = [t.view(T * STREAMS, width)[:T] for t in xs]
        w, ws = torch.ones(width, device=dev), torch.ones(STREAMS, device=dev)
        us = graph_us([lambda i=i: stream.rms_norm_stream(flat[i], w, None, 1e-6, bf, width) for i in range(m)])
        like = report(f"rms_norm_stream (Nufupel) t{T}", us, bytes_=T * width * 6)
        mix, y = torch.eye(STREAMS, device=dev), torch.randn(T, width, device=dev)
        us = graph_us([lambda i=i: stream.stream_mix_norm(xs[i], ws, w, 1e-6, bf, width, y=y, mix=mix, w_out=ws) for i in range(m)])
        report(f"stream_mix_norm t{T}", us, bytes_=T * width * (8 * STREAMS + 6), like=like)
        rows, idx = rnd(T * top, width), torch.randperm(T * top, device=dev).int().view(T, top)
        us = graph_us([lambda i=i: stream.rms_norm_stream(flat[i], w, None, 1e-6, bf, width, add=(rows, idx)) for i in range(m)])
        like = report(f"rms_norm_stream + {top} expert rows (Nufupel) t{T}", us, bytes_=T * width * (10 + 2 * top))
        us = graph_us([lambda i=i: stream.stream_mix_norm(xs[i], ws, w, 1e-6, bf, width, y=y, mix=mix, w_out=ws, add=(rows, idx)) for i in range(m)])
        report(f"stream_mix_norm + {top} expert rows t{T}", us, bytes_=T * width * (8 * STREAMS + 6 + 2 * top), like=like)
        del xs, flat, rows
    T, m = 8192, 4
    gus = [rnd(T, 2 * sff + 8) for _ in range(m)]
    og = torch.empty(T, sff, device=dev, dtype=bf)
    us = graph_us([lambda i=i: stream.glu(stream.GLU_SILU, gus[i][:, :2 * sff], og) for i in range(m)])
    like = report("glu silu (Nufupel)", us, bytes_=T * sff * 6)
    us = graph_us([lambda i=i: stream.clamped_glu(gus[i][:, :2 * sff], og, 7.0, 1.702, 1.0, row_gate=gus[i][:, 2 * sff:]) for i in range(m)])
    report("clamped_glu with a row gate", us, bytes_=T * sff * 6, like=like)
    del gus
    pj = [rnd(T, (H + 2 * G) * D) for _ in range(m)]
    kp, vp, slots = rnd(T // 64, G, 64, D), rnd(T // 64, G, 64, V), torch.arange(T, device=dev)
    tabr = torch.rand(T, D // 2, 2, device=dev)
    hn = torch.ones(D, device=dev)
    us = graph_us([lambda i=i: window.window_post(pj[i], slots, kp, vp, H, D, tab=tabr, rot=D, norms=(hn, hn), eps=1e-6) for i in range(m)])
    like = report("window_post, norms and rotation (Nufupel)", us, bytes_=T * (H * D * 4 + 2 * G * D * 4 + D * 4))
    for nb_ in (False, True):
        us = graph_us([lambda i=i: window.window_post(pj[i], slots, kp, vp, H, D, tab=tabr, rot=D, neighbours=nb_) for i in range(m)])
        report(f"window_post, rotation of {'neighbours' if nb_ else 'halves'}", us, bytes_=T * (H * D * 4 + 2 * G * D * 4 + D * 4), like=like)
    assert native.read_status() == 0


def main(argv=None):
    ap = argparse.ArgumentParser()
    ap.add_argument("--size", default=None, choices=list(SIZES))
    ap.add_argument("--layers", type=int, default=8)
    ap.add_argument("--models", action="store_true")
    ap.add_argument("--kernels", action="store_true")
    a = ap.parse_args(argv)
    both = not (a.models or a.kernels)
    rows = []
    for size in [a.size] if a.size else list(SIZES):
        if a.kernels or both:
            bench_kernels(size, rows)
        if a.models or both:
            bench_models(size, a.layers, rows)
    return 0


if __name__ == "__main__":
    sys.exit(main())
