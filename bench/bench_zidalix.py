"""Zidalix against the framework's closest model (INT4 Llama) at equal size, and every kernel of its decoder
stack against its roofline beside the like kernel of that model.

    python bench.py --zidalix            (or: python bench/bench_zidalix.py [--kernels] [--models] [--size NAME])

Models: random weights, ``--layers`` layers of a real model's size; prompts of 2048 tokens as one ragged batch,
then decoding at a context of 2048 with 1, 16 and 64 sequences through ``Engine.feed`` (CUDA graphs), CUDA-event
times.  The layers' weights and caches of a step exceed L2.  Kernels: captured into a graph over rotating operand
copies that together exceed L2, CUDA-event time of a replay divided by the launches in it.
"""
from __future__ import annotations

import argparse
import os
import sys

import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))

from serving_common import Reports, engine_row, graph_us  # noqa: E402

from rumus_b200.models.llama import LlamaConfig  # noqa: E402
from rumus_b200.models.zidalix import ZidalixConfig  # noqa: E402
from rumus_b200.ops import functional as F, latent, native  # noqa: E402

SIZES = {  # width, heads, ff, kv_rank
    "2b": (2048, 16, 5632, 512),
    "7b": (4096, 32, 11008, 512),
    "7b-128h": (4096, 128, 11008, 512),   # on request: as many heads as make decoding compute bound
}


def zidalix_config(width, heads, ff, rank, layers, vocab=32000):
    rot = {"base": 1e6, "dims": 64, "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}
    mixer = {"heads": heads, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": rank, "scale": 192 ** -0.5, "rot": rot}
    entries = []
    for i in range(layers):
        m = dict(mixer)
        if i % 4 == 3:
            m["kv_from"] = i - 1              # every fourth layer reads its predecessor's latents
        entries.append({"type": "latent_attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff, "limit": 7.0}})
    return ZidalixConfig.from_dict({"vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0},
                                    "logit_scale": 1.0, "layers": entries})


def llama_config(width, heads, kv_heads, ff, layers, vocab=32000):
    return LlamaConfig(vocab_size=vocab, seq_len=4096, d_model=width, num_heads=heads, num_kv_heads=kv_heads, num_layers=layers,
                       ffn_dim=ff)


def bench_models(size, layers, out):
    width, heads, ff, rank = SIZES[size]
    engine_row("zidalix", size, zidalix_config(width, heads, ff, rank, layers), layers, out)
    if heads == width // 128:
        engine_row("llama-int4", size, llama_config(width, heads, heads, ff, layers), layers, out)


def bench_kernels(size, out):
    width, H, ff, R = SIZES[size]
    report = Reports(size, out)
    dev, bf = "cuda", torch.bfloat16
    D, rot, V = 128, 64, 128
    like_h = width // 128

    def rnd(*s, scale=1.0):
        return (torch.randn(*s, device=dev) * scale).to(bf)

    # ---- prompt attention
    S, n = 4096, 2
    q, k, v = rnd(1, S, like_h, D), rnd(1, S, like_h, D), rnd(1, S, like_h, D)
    us = graph_us([lambda: F.flash_attention(q, k, v, True, D ** -0.5)] * n)
    like = report("flash_attn_fwd (Llama)", us, flops=like_h * S * S / 2 * (D + D) * 2, bytes_=4 * S * like_h * D * 2)
    T = S
    qz, kv, rows, gate, o = rnd(T, H, D + rot), rnd(T, H * (D + V)), rnd(T, R + rot), rnd(T, H * V), rnd(T, H * V)
    sink = torch.zeros(H, device=dev)
    items = torch.tensor(latent.prefill_items([(0, S, 0, 0)]), dtype=torch.int32, device=dev)
    us = graph_us([lambda: latent.latent_prefill(qz, kv, rows, items, sink, gate, o, D, V, R, 192 ** -0.5)] * n)
    report("latent_prefill", us, flops=H * S * S / 2 * (D + rot + V) * 2, bytes_=S * H * (D + rot + D + 3 * V) * 2, like=like)

    # ---- decode attention
    for B, ctx in ((1, 8192), (16, 4096), (64, 2048)):
        bs, nb = 64, B * ctx // 64
        tab = torch.randperm(nb, device=dev).int().view(B, -1)
        cl = torch.full((B,), ctx, dtype=torch.int32, device=dev)
        from rumus_b200.serve.llama import paged_decode_attention
        m = max(1, -(-300_000_000 // (nb * bs * like_h * D * 4)))
        kc = [rnd(nb, bs, like_h, D) for _ in range(m)]
        vc = [rnd(nb, bs, like_h, D) for _ in range(m)]
        ql = rnd(B, like_h, D)
        us = graph_us([lambda i=i: paged_decode_attention(ql, kc[i], vc[i], tab, cl, D ** -0.5, ctx) for i in range(m)])
        like = report(f"paged_decode_attn (Llama) b{B} ctx{ctx}", us, bytes_=B * ctx * like_h * D * 2 * 2,
                      flops=B * ctx * like_h * D * 4)
        del kc, vc
        m = max(1, -(-300_000_000 // (nb * bs * (R + rot) * 2)))
        pools = [rnd(nb, bs, R + rot) for _ in range(m)]
        qa, qr = rnd(B, H, R), rnd(B, H, rot)
        us = graph_us([lambda i=i: latent.latent_rows_attention(qa, qr, pools[i], tab, cl, sink, 192 ** -0.5, ctx) for i in range(m)])
        report(f"latent_decode + merge b{B} ctx{ctx}", us, bytes_=B * ctx * (R + rot) * 2 + 2 * B * H * R * 2,
               flops=B * ctx * H * (R + rot + R) * 2, like=like)
        del pools

    # ---- projections per head around it: like kernel = the INT4 product of the same bytes class
    from rumus_b200.nn.quant import QuantizedTensor, qmatmul_int4
    for B in (1, 16, 64):
        m = max(2, -(-300_000_000 // (width * width // 2)))
        wq = [QuantizedTensor.from_f32(torch.randn(width, width, device=dev) * 0.02, 128, torch.float16).to(dev) for _ in range(m)]
        x = rnd(B, width)
        us = graph_us([lambda i=i: qmatmul_int4(x, wq[i]) for i in range(m)], reps=1)
        like = report(f"qmatmul_int4 {width}x{width} (Llama) b{B}", us, bytes_=width * width // 2, flops=2 * B * width * width)
        del wq
        m = max(2, min(64, -(-300_000_000 // (H * D * R * 2))))
        uk = [rnd(H, D, R) for _ in range(m)]
        uv = [rnd(H, V, R) for _ in range(m)]
        a, c, g1 = rnd(B, H, D), rnd(B, H, R), rnd(B, H, V)
        oa, oc = torch.empty(B, H, R, device=dev, dtype=bf), torch.empty(B, H, V, device=dev, dtype=bf)
        us = graph_us([lambda i=i: latent.head_matmul(a, uk[i], oa, False) for i in range(m)])
        report(f"head_gemm into latent space b{B}", us, bytes_=H * D * R * 2 + B * H * (D + R) * 2, flops=2 * B * H * D * R, like=like)
        us = graph_us([lambda i=i: latent.head_matmul(c, uv[i], oc, True, gate=g1) for i in range(m)])
        report(f"head_gemm out of latent space + gate b{B}", us, bytes_=H * V * R * 2 + B * H * (2 * V + R) * 2,
               flops=2 * B * H * V * R, like=like)
        del uk, uv
        N = H * (D + rot) + R + rot + H * V
        m = max(2, -(-300_000_000 // (N * width * 2)))
        ws = [rnd(N, width) for _ in range(m)]
        us = graph_us([lambda i=i: native.gemm(x, ws[i].t()) for i in range(m)])
        report(f"gemm {width}->{N} b{B}", us, bytes_=N * width * 2, flops=2 * B * N * width, like=like)
        del ws
        K = H * V + ff
        m = max(2, -(-300_000_000 // (K * width * 2)))
        ws, xk, res = [rnd(width, K) for _ in range(m)], rnd(B, K), torch.randn(B, width, device=dev)
        us = graph_us([lambda i=i: native.gemm(xk, ws[i].t(), residual=res, out_dtype=torch.float32) for i in range(m)])
        report(f"gemm {K}->{width} + residual b{B}", us, bytes_=K * width * 2, flops=2 * B * K * width, like=like)
        del ws

    # ---- elementwise over a prompt batch
    T, m = 8192, 4
    xs16 = [rnd(T, width) for _ in range(m)]
    w16 = torch.ones(width, device=dev, dtype=bf)
    us = graph_us([lambda i=i: native.norm_fwd(xs16[i], w16, None, 1e-6, True) for i in range(m)])
    like = report("rms norm (Llama)", us, bytes_=T * width * 4)
    xs = [torch.randn(T, width, device=dev) for _ in range(m)]
    w = torch.ones(width, device=dev)
    us = graph_us([lambda i=i: latent.rms_norm_stream(xs[i], w, w, 1e-6, bf, width) for i in range(m)])
    report("rms_norm_stream, two weights", us, bytes_=T * width * 8, like=like)
    gus = [rnd(T, 2 * ff) for _ in range(m)]
    us = graph_us([lambda i=i: native.swiglu_fwd(gus[i]) for i in range(m)])
    like = report("swiglu (Llama)", us, bytes_=T * ff * 6)
    og = torch.empty(T, H * V + ff, device=dev, dtype=bf)[:, H * V:]
    us = graph_us([lambda i=i: latent.clamped_glu(gus[i], og, 7.0, 1.702, 1.0) for i in range(m)])
    report("clamped_glu", us, bytes_=T * ff * 6, like=like)
    del gus
    kq, vq = rnd(T, like_h * 128), rnd(T, like_h * 128)
    slots = torch.arange(T, device=dev)
    xq = [rnd(T, 3 * width) for _ in range(m)]
    us = graph_us([lambda i=i: native.rope_(xq[i], T, 1, 2 * like_h, 128, 0, 10000.0, False, pos_ids=slots) for i in range(m)])
    like = report("rope q, k (Llama)", us, bytes_=T * 2 * width * 4)
    N = H * (D + rot) + R + rot + H * V
    pj = [rnd(T, N) for _ in range(m)]
    tab = torch.rand(T, rot // 2, 2, device=dev)
    pool = rnd(T // 64, 64, R + rot)
    nw = torch.ones(R, device=dev)
    us = graph_us([lambda i=i: latent.latent_post(pj[i], tab, H, D, rot, kv_col=H * (D + rot), norm_w=nw, slots=slots, pool=pool,
                                                  rank=R, eps=1e-6) for i in range(m)])
    report("latent_post", us, bytes_=T * (H * rot * 4 + (R + rot) * 4 + rot * 4), like=like)
    tabs = torch.arange(T // 64, device=dev, dtype=torch.int32).view(1, -1)
    off = torch.tensor([0, T], dtype=torch.int32, device=dev)
    pools = [rnd(T // 64, 64, R + rot) for _ in range(16)]
    us = graph_us([lambda i=i: latent.latent_gather(pools[i], tabs, off, T) for i in range(16)])
    report("latent_gather", us, bytes_=T * (R + rot) * 4, like=like)
    ids = torch.randint(0, 32000, (T,), device=dev)
    emb = rnd(32000, width)
    us = graph_us([lambda: native.embedding_fwd(ids, emb)] * m)
    like = report("embedding (Llama)", us, bytes_=T * width * 4)
    us = graph_us([lambda: latent.embed_scaled(ids, emb, 2.0)] * m)
    report("embed_scaled", us, bytes_=T * width * 6, like=like)
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
    for size in [a.size] if a.size else ["2b", "7b"]:
        if a.kernels or both:
            bench_kernels(size, rows)
        if a.models or both:
            bench_models(size, a.layers, rows)
    return 0


if __name__ == "__main__":
    sys.exit(main())
