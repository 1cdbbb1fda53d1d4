"""Nufupel against the framework's closest models (Zidalix: the same residual stream, gates and sinks, bf16 weights; INT4
Llama: keys and values in the cache) at equal size, and every kernel of its decoder stack against its roofline beside
the like kernel of those models.

    python bench.py --nufupel            (or: python bench/bench_nufupel.py [--kernels] [--models] [--size NAME])

Models: random weights, ``--layers`` layers of a real model's size; both kinds of attention in turn, the first layer's
feed-forward dense, the others mixtures whose active experts and shared expert together have the dense width.  Prompts
of 2048 tokens as one ragged batch, then decoding at a context of 2048 with 1, 16 and 64 sequences through
``Engine.feed`` (CUDA graphs), CUDA-event times.  The layers' weights and caches of a step exceed L2.  Kernels: captured
into a graph over rotating operand copies that together exceed L2, CUDA-event time of a replay divided by the launches
in it.
"""
from __future__ import annotations

import argparse
import os
import sys

import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))

from bench_zidalix import llama_config, zidalix_config  # noqa: E402
from serving_common import Reports, copies, engine_row, graph_us  # noqa: E402

from rumus_b200.models.nufupel import NufupelConfig  # noqa: E402
from rumus_b200.ops import functional as F, latent, moe, native, stream, window  # noqa: E402

SIZES = {  # width, heads, kv_heads, dense ff, experts, top, expert ff, shared ff
    "2b": (2048, 16, 4, 5632, 32, 4, 1024, 1536),
    "7b": (4096, 32, 8, 11008, 32, 4, 2048, 2816),
}
WINDOWS = (1024, 2048)      # of "attention" and "attention_2"


def nufupel_config(size, layers, vocab=32000):
    width, heads, kv, ff, E, top, eff, sff = SIZES[size]
    entries = []
    for i in range(layers):
        m = {"heads": heads, "kv_heads": kv, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "mask": {"size": WINDOWS[i % 2]}}
        if i % 2:
            m["rot"] = {"base": 1e6, "dims": 64, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}
        mlp = {"kind": "dense", "ff": ff} if i == 0 else \
            {"kind": "moe", "router": {"experts": E, "top": top}, "expert": {"ff": eff}, "shared": {"ff": sff}}
        entries.append({"type": "attention_2" if i % 2 else "attention", "mixer": m, "mlp": mlp})
    return NufupelConfig.from_dict({"vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0},
                                    "logit_softcap": 30.0, "layers": entries})


def bench_models(size, layers, out):
    width, heads, kv, ff = SIZES[size][:4]
    engine_row("nufupel", size, nufupel_config(size, layers), layers, out)
    engine_row("zidalix", size, zidalix_config(width, heads, ff, 512, layers), layers, out)
    engine_row("llama-int4", size, llama_config(width, heads, heads, ff, layers), layers, out)


def bench_kernels(size, out):
    width, H, G, ff, E, top, eff, sff = SIZES[size]
    report = Reports(size, out)
    dev, bf = "cuda", torch.bfloat16
    D = V = 128

    def rnd(*s, scale=1.0):
        return (torch.randn(*s, device=dev) * scale).to(bf)

    # ---- prompt attention
    S, n = 4096, 2
    R, rot = 512, 64
    qz, kv, rows, gate, o = rnd(S, H, D + rot), rnd(S, H * (D + V)), rnd(S, R + rot), rnd(S, H * V), rnd(S, H * V)
    sink = torch.zeros(H, device=dev)
    items = torch.tensor(latent.prefill_items([(0, S, 0, 0)]), dtype=torch.int32, device=dev)
    us = graph_us([lambda: latent.latent_prefill(qz, kv, rows, items, sink, gate, o, D, V, R, 192 ** -0.5)] * n)
    like = report("latent_prefill (Zidalix)", us, flops=H * S * S / 2 * (D + rot + V) * 2, bytes_=S * H * (D + rot + D + 3 * V) * 2)
    q, k, v = rnd(1, S, H, D), rnd(1, S, H, D), rnd(1, S, H, D)
    us = graph_us([lambda: F.flash_attention(q, k, v, True, D ** -0.5)] * n)
    report("flash_attn_fwd (Llama)", us, flops=H * S * S / 2 * (D + V) * 2, bytes_=4 * S * H * D * 2)
    del qz, kv, rows, q, k, v
    nb = S // 64
    kp, vp = rnd(nb, G, 64, D), rnd(nb, G, 64, V)
    tab = torch.randperm(nb, device=dev).int().view(1, -1)
    qw, hg = rnd(S, H, D), rnd(S, H)
    for W, kind in ((512, 1), (1024, 1), (2048, 2), (S, 1)):
        us = graph_us([lambda: window.window_prefill(qw, kp, vp, tab, items, sink, gate if kind == 1 else hg, kind, o, W, D ** -0.5)] * n)
        pairs = sum(min(W, i + 1) for i in range(S))
        report(f"window_prefill W{W}", us, flops=H * pairs * (D + V) * 2, bytes_=S * (2 * H + 2 * G + (H if kind == 1 else 0)) * D * 2,
               like=like)
    del kp, vp

    # ---- single rows
    from rumus_b200.serve.llama import paged_decode_attention
    for B, ctx in ((1, 8192), (16, 4096), (64, 2048), (64, 1024)):
        bs, nb = 64, B * ctx // 64
        tab = torch.randperm(nb, device=dev).int().view(B, -1)
        cl = torch.full((B,), ctx, dtype=torch.int32, device=dev)
        m = copies(nb * bs * H * D * 4)
        kc, vc = [rnd(nb, bs, H, D) for _ in range(m)], [rnd(nb, bs, H, D) for _ in range(m)]
        ql = rnd(B, H, D)
        us = graph_us([lambda i=i: paged_decode_attention(ql, kc[i], vc[i], tab, cl, D ** -0.5, ctx) for i in range(m)])
        paged = report(f"paged_decode_attn (Llama) b{B} ctx{ctx}", us, bytes_=B * ctx * H * D * 4, flops=B * ctx * H * D * 4)
        del kc, vc
        m = copies(nb * bs * (R + rot) * 2)
        pools = [rnd(nb, bs, R + rot) for _ in range(m)]
        qa, qr = rnd(B, H, R), rnd(B, H, rot)
        us = graph_us([lambda i=i: latent.latent_rows_attention(qa, qr, pools[i], tab, cl, sink, 192 ** -0.5, ctx) for i in range(m)])
        lat = report(f"latent_decode + merge (Zidalix) b{B} ctx{ctx}", us, bytes_=B * ctx * (R + rot) * 2 + 2 * B * H * R * 2,
                     flops=B * ctx * H * (2 * R + rot) * 2)
        del pools
        m = copies(nb * bs * G * D * 4)
        kc, vc = [rnd(nb, G, bs, D) for _ in range(m)], [rnd(nb, G, bs, D) for _ in range(m)]
        gt, ow = rnd(B, H * V), rnd(B, H * V)
        us = graph_us([lambda i=i: window.window_rows_attention(ql, kc[i], vc[i], tab, cl, sink, gt, 1, ow, ctx, D ** -0.5, ctx)
                       for i in range(m)])
        report(f"window_rows b{B} W{ctx}", us, bytes_=B * ctx * G * D * 4 + 3 * B * H * D * 2, flops=B * ctx * H * D * 4,
               like=max(paged, lat, key=lambda r: r["fraction"]))
        del kc, vc

    # ---- products with weights: the dense feed-forward of the same active width is the like kernel of the experts
    gu_like, dn_like = {}, {}
    for T in (1, 16, 64, 512, 2048, 8192):
        x = rnd(T, width)
        N = 2 * ff
        m = copies(N * width * 2, 2)
        ws = [rnd(N, width) for _ in range(m)]
        us = graph_us([lambda i=i: native.gemm(x, ws[i].t()) for i in range(m)], reps=1)
        gu_like[T] = report(f"gemm gate|up (Zidalix) {width}->{N} t{T}", us, bytes_=N * width * 2 + T * (N + width) * 2, flops=2 * T * N * width)
        del ws
        m = copies(ff * width * 2, 2)
        ws, xk, res = [rnd(width, ff) for _ in range(m)], rnd(T, ff), torch.randn(T, width, device=dev)
        us = graph_us([lambda i=i: native.gemm(xk, ws[i].t(), residual=res, out_dtype=torch.float32) for i in range(m)], reps=1)
        dn_like[T] = report(f"gemm down + residual (Zidalix) {ff}->{width} t{T}", us, bytes_=ff * width * 2 + T * (ff * 2 + width * 8),
                            flops=2 * T * ff * width)
        del ws
        Np = (H + 2 * G) * D + H * V + 2 * sff
        m = copies(Np * width * 2, 2)
        ws = [rnd(Np, width) for _ in range(m)]
        us = graph_us([lambda i=i: native.gemm(x, ws[i].t()) for i in range(m)], reps=1)
        report(f"gemm input {width}->{Np} t{T}", us, bytes_=Np * width * 2 + T * (Np + width) * 2, flops=2 * T * Np * width, like=gu_like[T])
        Ko = H * V + sff
        m = copies(Ko * width * 2, 2)
        ws, xk = [rnd(width, Ko) for _ in range(m)], rnd(T, Ko)
        us = graph_us([lambda i=i: native.gemm(xk, ws[i].t(), residual=res, out_dtype=torch.float32) for i in range(m)], reps=1)
        report(f"gemm output + residual {Ko}->{width} t{T}", us, bytes_=Ko * width * 2 + T * (Ko * 2 + width * 8), flops=2 * T * Ko * width,
               like=dn_like[T])
        del ws, xk
        # experts
        m = max(2, min(3, copies(E * 3 * eff * width * 2)))
        gu, dn = [rnd(E, 2 * eff, width) for _ in range(m)], [rnd(E, width, eff) for _ in range(m)]
        rt, rb, counts = rnd(E, width, scale=width ** -0.5), torch.zeros(E, device=dev), torch.zeros(E + 1, device=dev, dtype=torch.int32)

        def routing():
            lg = native.gemm(x, rt.t(), out_dtype=torch.float32) if T > moe.ROUTE_ROWS else None
            return moe.route(x, rt, rb, counts, top, logits=lg)

        us = graph_us([routing])
        r = routing()
        report(f"route t{T}" + (" with sorted rows" if r.rows is not None else ""), us,
               bytes_=T * width * 2 + E * width * 2 + (T * (top + 1) * width * 2 if r.rows is not None else 0), flops=2 * T * E * width)
        used = len(r.idx.unique())
        act, y = torch.empty(r.slots, eff, device=dev, dtype=bf), torch.empty(r.slots, width, device=dev, dtype=bf)
        us = graph_us([lambda i=i: moe.grouped(x, gu[i], r, act, True) for i in range(m)])
        report(f"moe gate|up t{T} ({used} experts, tile {r.tile})", us, bytes_=used * 2 * eff * width * 2 + T * width * 2 + T * top * eff * 2,
               flops=2 * T * top * 2 * eff * width, like=gu_like[T])
        us = graph_us([lambda i=i: moe.grouped(act, dn[i], r, y, False) for i in range(m)])
        report(f"moe down t{T}", us, bytes_=used * eff * width * 2 + T * top * (eff + width) * 2, flops=2 * T * top * eff * width, like=dn_like[T])
        del gu, dn

    # ---- elementwise over a prompt batch
    T, m = 8192, 4
    xs = [torch.randn(T, width, device=dev) for _ in range(m)]
    w = torch.ones(width, device=dev)
    us = graph_us([lambda i=i: latent.rms_norm_stream(xs[i], w, w, 1e-6, bf, width) for i in range(m)])
    like = report("rms_norm_stream, two weights (Zidalix)", us, bytes_=T * width * 8)
    us = graph_us([lambda i=i: stream.rms_norm_stream(xs[i], w, None, 1e-6, bf, width) for i in range(m)])
    report("rms_norm_stream, one weight", us, bytes_=T * width * 6, like=like)
    y, idx = rnd(T * top, width), torch.randperm(T * top, device=dev).int().view(T, top)
    us = graph_us([lambda i=i: stream.rms_norm_stream(xs[i], w, None, 1e-6, bf, width, add=(y, idx)) for i in range(m)])
    report(f"rms_norm_stream + {top} expert rows", us, bytes_=T * width * (10 + 2 * top), like=like)
    del y, xs
    gus = [rnd(T, 2 * ff) for _ in range(m)]
    og = torch.empty(T, H * V + ff, device=dev, dtype=bf)[:, H * V:]
    us = graph_us([lambda i=i: latent.clamped_glu(gus[i], og, 7.0, 1.702, 1.0) for i in range(m)])
    like = report("clamped_glu (Zidalix)", us, bytes_=T * ff * 6)
    for kind, nm in ((stream.GLU_GELU, "gelu"), (stream.GLU_SILU, "silu")):
        us = graph_us([lambda i=i: stream.glu(kind, gus[i], og) for i in range(m)])
        report(f"glu {nm}", us, bytes_=T * ff * 6, like=like)
    del gus, og
    tabr, slots = torch.rand(T, rot // 2, 2, device=dev), torch.arange(T, device=dev)
    N = H * (D + rot) + R + rot + H * V
    pj, pool, nw = [rnd(T, N) for _ in range(m)], rnd(T // 64, 64, R + rot), torch.ones(R, device=dev)
    us = graph_us([lambda i=i: latent.latent_post(pj[i], tabr, H, D, rot, kv_col=H * (D + rot), norm_w=nw, slots=slots, pool=pool, rank=R,
                                                  eps=1e-6) for i in range(m)])
    like = report("latent_post (Zidalix)", us, bytes_=T * (H * rot * 4 + (R + rot) * 4 + rot * 4))
    Np = (H + 2 * G) * D + H * V + 2 * sff
    pj = [rnd(T, Np) for _ in range(m)]
    kp, vp, hn = rnd(T // 64, G, 64, D), rnd(T // 64, G, 64, V), torch.ones(D, device=dev)
    us = graph_us([lambda i=i: window.window_post(pj[i], slots, kp, vp, H, D, tab=tabr, rot=rot, norms=(hn, hn), eps=1e-6) for i in range(m)])
    report("window_post, norms and rotation", us, bytes_=T * (H * D * 4 + 2 * G * D * 4 + rot * 4), like=like)
    us = graph_us([lambda i=i: window.window_post(pj[i], slots, kp, vp, H, D) for i in range(m)])
    report("window_post, plain", us, bytes_=T * 2 * G * D * 4, like=like)
    del pj
    lg = [torch.randn(64, 32000, device=dev) for _ in range(40)]
    us = graph_us([lambda i=i: stream.softcap_(lg[i], 30.0) for i in range(40)], reps=1)
    report("softcap 64 x 32000", us, bytes_=64 * 32000 * 8, like=like)
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
