"""Small Potodra configurations and weights for the tests: sizes that are not multiples of eight, windows and kept tokens
shorter and longer than pages and tiles, layers without a feed-forward, one to five streams, groups of one and several
experts."""
import torch


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, top, count, keep, ff, limit, shared, shared_limit):
    return {"kind": "moe", "router": {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}},
            "expert": {"ff": ff, "limit": limit}, "shared": {"ff": shared, "limit": shared_limit}}


def _att(heads, kv_heads, dim, vdim, scale, rot, base):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"base": base, "dims": rot}}


def _window(heads, kv_heads, dim, vdim, size, keep, cap, scale, rot, mlp=None, base=3000.0):
    return {"type": "attention", "mlp": mlp,
            "mixer": {**_att(heads, kv_heads, dim, vdim, scale, rot, base), "mask": {"size": size, "keep_first": keep}, "softcap": cap}}


def _memory(heads, dim, vdim, cap, mlp=None):
    return {"type": "mlstm", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}


def _parallel(left, right, left_scale, right_scale, mlp=None):
    heads, kv_heads, dim, vdim, conv = right
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": _att(*left), "right": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv},
                      "left_scale": left_scale, "right_scale": right_scale}}


def _model(width, vocab, streams, layers, emb=1.3, eps=1e-5):
    return {"architecture": "Potodra", "width": width, "vocab": vocab, "streams": streams, "norm": {"eps": eps}, "embedding": {"scale": emb},
            "layers": layers}


CONFIGS = {
    # nothing is a multiple of eight, sizes change from layer to layer
    "odd": _model(50, 67, 3, [
        _parallel((3, 1, 10, 13, 0.5, 6, 500.0), (3, 3, 9, 11, 2), 0.7, 1.3, _dense(33)),
        _memory(2, 7, 13, 6.0, _moe(6, 2, 3, 2, 19, 1.5, 27, 0.8)),
        _window(6, 2, 12, 20, 21, 5, 4.0, 0.4, 10, None),
        _memory(3, 20, 5, 11.0, _dense(17)),
    ]),
    # every kind twice, shared queries and keys, many taps, one stream more than usual
    "mixed": _model(64, 96, 5, [
        _window(4, 2, 16, 24, 64, 64, 9.0, 0.3, 16, _moe(8, 3, 4, 2, 40, 2.0, 56, 1.1)),
        _parallel((4, 4, 24, 16, 0.25, 8, 900.0), (4, 2, 16, 32, 5), 1.1, 0.6, _moe(12, 4, 3, 2, 24, 0.7, 16, 3.0)),
        _memory(4, 16, 16, 8.0),
        _window(2, 1, 32, 16, 65, 3, 15.0, 0.25, 32, _dense(48)),
        _parallel((2, 1, 16, 40, 0.4, 16, 77.0), (6, 3, 24, 8, 4), 0.5, 0.9),
    ], emb=0.8, eps=1e-3),
    # beyond one 64-wide tile in every direction, two streams
    "wide": _model(136, 200, 2, [
        _memory(2, 104, 72, 14.0, _dense(200)),
        _window(4, 2, 104, 72, 100, 70, 30.0, 0.12, 40, _moe(40, 4, 10, 4, 72, 5.0, 136, 4.0)),
        _parallel((3, 1, 72, 128, 0.13, 72, 2e4), (2, 1, 128, 104, 3), 0.8, 0.8, _moe(5, 5, 1, 1, 33, 1.0, 24, 1.0)),
    ]),
    # sizes the tiled kernels leave to the plain ones; one stream
    "tall": _model(48, 80, 1, [
        _window(2, 1, 160, 40, 30, 9, 12.0, 0.09, 20, _moe(4, 1, 2, 1, 24, 1.0, 24, 2.0)),
        _memory(1, 136, 264, 9.0),
        _parallel((3, 3, 40, 264, 0.2, 4, 60.0), (1, 1, 200, 136, 3), 1.0, 1.0, _dense(24)),
    ]),
}


def weights_for(cfg, seed, sharp=2.0, dtype=torch.bfloat16):
    """Random weights in which every mechanism shows: peaked attention, gates and decays of all strengths, streams that
    mix.  Routers are scaled up, so that few choices of experts are close."""
    from rumus_b200.models.potodra import PotodraConfig
    g = torch.Generator().manual_seed(seed)
    c = PotodraConfig.from_dict(cfg)
    n, out = c.streams, {}
    ranks = {i: (5 + i, 9 + i) for i, e in enumerate(cfg["layers"]) if e["type"] == "parallel"}
    for k, shape in c.weight_shapes(ranks).items():
        last = k.rsplit(".", 1)[-1]
        r = torch.randn(shape, generator=g)
        if last in ("norm", "norm1", "norm2"):
            t = 1.0 + 0.3 * r
        elif last == "in":
            t = (1.0 + 0.5 * r) / n
        elif last == "out":
            t = 0.7 + 0.4 * r
        elif last == "mix":
            t = 0.8 * torch.eye(n) + 0.2 * r / n ** 0.5
        elif last == "dt_bias":
            t = r - 3.0
        elif last == "conv":
            t = r * shape[1] ** -0.5
        elif k.endswith(".f.b"):
            t = 2.0 + 2.0 * r
        elif last == "correction":
            t = 0.3 * r
        elif len(shape) == 1:
            t = r
        elif k == "embed":
            t = r
        else:
            t = r * shape[1] ** -0.5
            t = t * (sharp if last == "q" and "right" not in k else 3.0 if last == "router" else 1.0)
        out[k] = t.to(dtype)
    return out
