"""Lerosun against the framework's closest model (Potodra: a gated delta rule, windows, sinks, fp32 residual) at equal size,
and every kernel of its decoder stack against its roofline beside the like kernel.

    python bench.py --lerosun            (or: python bench/bench_lerosun.py [--kernels] [--models] [--size NAME])

Models: random weights, ``--layers`` layers of a real model's size: three delta rules and an attention layer in turn, each with
a gated feed-forward.  Potodra with its own mixers in turn and dense feed-forwards of as many weights.  Prompts of 2048 tokens as
one ragged batch, then decoding at a context of 2048 with 1, 16 and 64 sequences through ``Engine.feed`` (CUDA graphs), CUDA-event
times.  The layers' weights and caches of a step exceed L2.  Kernels: captured into a graph over rotating operand copies
that together exceed L2, CUDA-event time of a replay divided by the launches in it.

Rooflines count what the mechanism needs: a talking head's scores cost one product with its own key/value head and a mixture of
the heads' scores, whatever way the kernel goes about it; a recurrence the vectors that enter and leave a head and one pass
over its state, in its recurrent form.
"""
from __future__ import annotations

import argparse
import os
import sys

import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))

from bench_nufupel import SIZES  # noqa: E402
from bench_potodra import CAP, KEEP, TAPS, WINDOW, potodra_config  # noqa: E402
from serving_common import Reports, copies, engine_row, graph_us  # noqa: E402

from rumus_b200.models.lerosun import LerosunConfig  # noqa: E402
from rumus_b200.models.potodra import DenseConfig, PotodraConfig, PotodraLayer  # noqa: E402
from rumus_b200.ops import latent, native, recurrent, stream, talk, window  # noqa: E402


def lerosun_config(size, layers, vocab=32000):
    width, heads, kv, ff = SIZES[size][:4]
    att = {"heads": heads, "kv_heads": kv, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "rot": {"base": 1e6, "dims": 128},
           "mask": {"size": WINDOW}}
    mem = {"heads": heads, "kv_heads": heads, "dim": 128, "vdim": 128, "conv": TAPS}
    entries = [{"type": "attention" if i % 4 == 3 else "delta", "mixer": att if i % 4 == 3 else mem, "mlp": {"kind": "dense", "ff": ff}}
               for i in range(layers)]
    return LerosunConfig.from_dict({"vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "layers": entries, "loop": None})


def dense_potodra_config(size, layers, vocab=32000):
    """Its feed-forward has two matrices where Lerosun's has three."""
    c = potodra_config(size, layers, vocab)
    dense = tuple(PotodraLayer(L.mixer, DenseConfig(SIZES[size][3] * 3 // 2)) for L in c.layers)
    return PotodraConfig(c.vocab_size, c.d_model, c.norm_eps, c.embedding_scale, c.streams, dense)


def bench_models(size, layers, out):
    engine_row("lerosun", size, lerosun_config(size, layers), layers, out)
    engine_row("potodra (dense)", size, dense_potodra_config(size, layers), layers, out)


def bench_kernels(size, out):
    width, H, G, ff = SIZES[size][:4]
    report = Reports(size, out)
    dev, bf = "cuda", torch.bfloat16
    D = 128

    def rnd(*s, scale=1.0):
        return (torch.randn(*s, device=dev) * scale).to(bf)

    mix = torch.eye(H, device=dev) + 0.1 * torch.randn(H, H, device=dev)
    # ---- prompt mixers
    S, n = 4096, 2
    nb = S // 64
    kp, vp = rnd(nb, G, 64, D), rnd(nb, G, 64, D)
    tab = torch.randperm(nb, device=dev).int().view(1, -1)
    items = torch.tensor(latent.prefill_items([(0, S, 0, 0)]), dtype=torch.int32, device=dev)
    q, qm, o, gate, sink = rnd(S, H, D), rnd(S, H, G, D), rnd(S, H * D), rnd(S, H), torch.zeros(H, device=dev)
    for W in (WINDOW, S):
        pairs = sum(min(W, i + 1) for i in range(S))
        us = graph_us([lambda: window.window_prefill(q, kp, vp, tab, items, sink, None, 0, o, W, D ** -0.5, keep=KEEP, cap=CAP)] * n)
        like = report(f"window_prefill W{W} kept {KEEP} capped (Potodra)", us, flops=H * pairs * D * 4, bytes_=S * (2 * H + 2 * G) * D * 2)
        us = graph_us([lambda: talk.talk_prefill(qm, 0, kp, vp, tab, items, sink, gate, 2, o, W, D ** -0.5)] * n)
        report(f"talk_prefill W{W}", us, flops=H * pairs * (D * 4 + H * 2), bytes_=S * (2 * H + 2 * G) * D * 2, like=like)
    del kp, vp, q, qm, o
    taps, norm, decay = torch.randn(TAPS, 3 * H * D, device=dev), torch.ones(D, device=dev), torch.ones(H, device=dev)

    def memory(places):
        return {"S": torch.zeros(places, H, D, D, device=dev), "conv": torch.zeros(places, H, TAPS - 1, 3 * D, device=dev, dtype=bf)}

    def delta(fn, per_head, T, mid):
        """A call with steps per head or per channel; operands of ``T`` tokens."""
        pj, few, steps = rnd(T, 4 * H * D), torch.randn(T, 2 * H, device=dev), torch.randn(T, H * D, device=dev)
        mixed, wide = rnd(T, H * D), torch.full((H if per_head else H * D,), -4.0, device=dev)
        a = few[:, H:] if per_head else steps
        kw = dict(per_head=True, silu=True) if per_head else {}
        return lambda state: fn(pj, taps, a, wide, decay, few, *mid, state, pj[:, 3 * H * D:], norm, mixed, H, D, D, 1e-6, **kw)

    for nseq, L in ((1, S), (4, 2048)):
        T, state = nseq * L, memory(nseq)
        seqs = torch.tensor([[i * L, L, i, 0] for i in range(nseq)], dtype=torch.int32, device=dev)
        cuts = recurrent.cut([(i * L, L) for i in range(nseq)], recurrent.DELTA_CHUNK, dev)
        vectors = T * H * 5 * 2 * D + nseq * H * D * D * 4
        fn = delta(recurrent.delta_chunks, False, T, (cuts, seqs))
        like = report(f"delta_chunks {nseq} x {L}, decay per channel (Potodra)", graph_us([lambda: fn(state)] * n), flops=T * H * 6 * D * D,
                      bytes_=vectors + T * H * (4 * D + 4))
        fn = delta(recurrent.delta_chunks, True, T, (cuts, seqs))
        report(f"delta_chunks {nseq} x {L}, decay per head", graph_us([lambda: fn(state)] * n), flops=T * H * 6 * D * D,
               bytes_=vectors + T * H * 8, like=like)
        del fn

    # ---- single rows
    for B, ctx in ((1, 8192), (16, 4096), (64, 2048), (64, 1024)):
        bs, nb = 64, B * ctx // 64
        tab = torch.randperm(nb, device=dev).int().view(B, -1)
        cl = torch.full((B,), ctx, dtype=torch.int32, device=dev)
        m = copies(nb * bs * G * D * 4)
        kc, vc = [rnd(nb, G, bs, D) for _ in range(m)], [rnd(nb, G, bs, D) for _ in range(m)]
        ql, gt, ow = rnd(B, H, D), rnd(B, H), rnd(B, H * D)
        cost = dict(bytes_=B * ctx * G * D * 4 + 2 * B * H * D * 2, flops=B * ctx * H * D * 4)
        us = graph_us([lambda i=i: window.window_rows_attention(ql, kc[i], vc[i], tab, cl, sink, None, 0, ow, ctx - KEEP, D ** -0.5, ctx, keep=KEEP,
                                                                cap=CAP) for i in range(m)])
        like = report(f"window_rows b{B} W{ctx - KEEP} kept {KEEP} capped (Potodra)", us, **cost)
        us = graph_us([lambda i=i: talk.talk_rows_attention(ql, kc[i], vc[i], tab, cl, mix, sink, gt, 2, ow, ctx, D ** -0.5, ctx) for i in range(m)])
        report(f"talk_rows b{B} W{ctx}", us, **cost, like=like)
        del kc, vc
        if ctx == 1024:
            continue
        m = copies(B * H * D * D * 8)
        states = [memory(B) for _ in range(m)]
        seqs = torch.tensor([[i, 1, i, 5] for i in range(B)], dtype=torch.int32, device=dev)
        bytes_ = B * H * (D * D * 8 + 5 * D * 2 + 12 * D * (TAPS - 1))
        fn = delta(recurrent.delta_rows, False, B, (seqs,))
        like = report(f"delta_rows b{B}, decay per channel (Potodra)", graph_us([lambda i=i: fn(states[i]) for i in range(m)]),
                      bytes_=bytes_ + B * H * D * 4, flops=B * H * 6 * D * D)
        fn = delta(recurrent.delta_rows, True, B, (seqs,))
        report(f"delta_rows b{B}, decay per head", graph_us([lambda i=i: fn(states[i]) for i in range(m)]), bytes_=bytes_ + B * H * 8,
               flops=B * H * 6 * D * D, like=like)
        del states, fn

    # ---- products with weights
    for T in (1, 16, 64, 512, 2048, 8192):
        x = rnd(T, width)

        def product(what, K, N, like=None, bias=False, **kw):
            ws, xs = [rnd(N, K) for _ in range(copies(N * K * 2, 2))], x if K == width else rnd(T, K)
            b, out4 = rnd(N) if bias else None, kw.get("out_dtype") == torch.float32
            us = graph_us([lambda i=i: native.gemm(xs, ws[i].t(), bias=b, **kw) for i in range(len(ws))], reps=1)
            return report(f"gemm {what} {K}->{N} t{T}", us, bytes_=N * K * 2 + T * (N * (4 if out4 else 2) + K * 2), flops=2 * T * K * N, like=like)

        pad = stream.pad8(H)
        up = product("up, squared relu (Potodra)", width, ff * 3 // 2, act="relu2")
        dn = product("down (Potodra)", ff * 3 // 2, width, out_dtype=torch.float32)
        att = product("input of attention (Potodra)", width, (H + 2 * G) * D, bias=True)
        par = product("input of delta and attention (Potodra)", width, (H + 2 * G) * D + 3 * H * D + 2 * D, bias=True)
        hd = product("output of heads (Potodra)", H * D, width, out_dtype=torch.float32)
        product("gate|up", width, 2 * ff, up)
        product("down", ff, width, dn, out_dtype=torch.float32)
        product("input of attention", width, (H + G) * D + pad, att, bias=True)
        product("input of delta", width, 4 * H * D, par)
        product("output of heads", H * D, width, hd, out_dtype=torch.float32)
        one = None
        for what, rows in (("one number (Potodra)", pad), ("two numbers", 2 * pad)):
            few = [rnd(rows, width) for _ in range(8)]
            if T <= recurrent.FEW_ROWS:
                us = graph_us([lambda w=w: recurrent.few_outputs(x, w) for w in few], reps=1)
            else:
                us = graph_us([lambda w=w: native.gemm(x, w.t(), out_dtype=torch.float32) for w in few], reps=1)
            one = report(f"few outputs, {what} a head {width}->{rows} t{T}", us, bytes_=rows * width * 2 + T * width * 2 + T * rows * 4,
                         flops=2 * T * rows * width, like=one)

    # ---- around the sub-layers
    for T in (1, 64, 8192):
        m = copies(T * width * 4) if T > 1 else 8
        xs, ys = [torch.randn(T, 4, width, device=dev) for _ in range(m)], [torch.randn(T, width, device=dev) for _ in range(m)]
        w, ws, sc, one = torch.ones(width, device=dev), torch.ones(4, device=dev), torch.ones(width, device=dev), torch.ones(1, device=dev)
        eye = torch.eye(4, device=dev)
        us = graph_us([lambda i=i: stream.stream_mix_norm(xs[i], ws, w, 1e-6, bf, width, y=ys[i], mix=eye, w_out=ws) for i in range(m)])
        like = report(f"stream_mix_norm, 4 streams t{T} (Potodra)", us, bytes_=T * width * 38)
        flat = [t.view(-1)[:T * width].view(T, width) for t in xs]
        us = graph_us([lambda i=i: stream.scaled_add_norm(flat[i], ys[i], sc, one, 1e-6, bf, width) for i in range(m)])
        report(f"scaled_add_norm t{T}", us, bytes_=T * width * 14, like=like)
        del xs, ys, flat
        tables, ids = [rnd(32000, width) for _ in range(3)], torch.randint(0, 32000, (T,), device=dev)
        us = graph_us([lambda i=i: stream.embed_scaled(ids, tables[i], 1.0) for i in range(3)])
        like = report(f"embed_scaled t{T} (Potodra)", us, bytes_=T * width * 6)
        us = graph_us([lambda i=i: stream.embed_norm(ids, tables[i], one, one, 1e-6, width) for i in range(3)])
        report(f"embed_norm t{T}", us, bytes_=T * width * 8, like=like)
        del tables
    T, m = 8192, 4
    gus, og = [rnd(T, 2 * ff) for _ in range(m)], torch.empty(T, ff, device=dev, dtype=bf)
    us = graph_us([lambda i=i: stream.clamped_glu(gus[i], og, 7.0, 1.702, 1.0) for i in range(m)])
    like = report("clamped_glu (Potodra)", us, bytes_=T * ff * 6)
    us = graph_us([lambda i=i: stream.glu(stream.GLU_RELU, gus[i], og) for i in range(m)])
    report("glu relu", us, bytes_=T * ff * 6, like=like)
    del gus
    kp, vp, tabr = rnd(T // 64, G, 64, D), rnd(T // 64, G, 64, D), torch.rand(T, D // 2, 2, device=dev)
    for t in (64, T):
        slots, cols = torch.arange(t, device=dev), t * D * 4
        pj = [rnd(t, (H + 2 * G) * D) for _ in range(m)]
        us = graph_us([lambda i=i: window.window_post(pj[i], slots, kp, vp, H, D, tab=tabr[:t], rot=D) for i in range(m)])
        like = report(f"window_post t{t} (Potodra)", us, bytes_=t * (H * D * 4 + 2 * G * D * 4) + cols)
        us = graph_us([lambda i=i: talk.talk_post(pj[i], slots, kp, vp, mix, H, t, tab=tabr[:t], rot=D) for i in range(m)])
        report(f"talk_post t{t}, rows", us, bytes_=t * (H * D * 4 + 3 * G * D * 2) + cols, like=like)
        us = graph_us([lambda i=i: talk.talk_post(pj[i], slots, kp, vp, mix, H, 0, tab=tabr[:t], rot=D) for i in range(m)])
        report(f"talk_post t{t}, mixed queries", us, bytes_=t * (H * D * 2 + H * G * D * 2 + 3 * G * D * 2) + cols, flops=t * H * H * D * 2, like=like)
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
