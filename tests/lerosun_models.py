"""Small Lerosun configurations and weights for the tests: sizes that are not multiples of eight, windows shorter and longer
than pages and tiles, rotations of a part of a head and of all of it, layers without a feed-forward, loops at the start, in the
middle and absent, convolutions of one and many taps."""
import torch


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _att(heads, kv_heads, dim, window, rot, scale, mlp=None, base=3000.0):
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale,
                                                       "mask": {"size": window}, "rot": {"base": base, "dims": rot}}}


def _delta(heads, kv_heads, dim, vdim, conv, mlp=None):
    return {"type": "delta", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def _model(width, vocab, layers, loop=None, eps=1e-5):
    return {"architecture": "Lerosun", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers,
            "loop": loop and dict(zip(("start", "stop", "times"), loop))}


CONFIGS = {
    # nothing is a multiple of eight, three passes from the first layer on
    "odd": _model(50, 67, [
        _delta(3, 3, 9, 11, 2, _dense(33)),
        _att(3, 1, 10, 21, 6, 0.5, None, 500.0),
        _att(6, 3, 12, 5, 12, 0.4, _dense(17)),
    ], (0, 2, 3)),
    # shared queries and keys, one tap and five, a loop in the middle, windows of a page and one more
    "mixed": _model(64, 96, [
        _delta(4, 2, 16, 32, 5),
        _att(4, 2, 24, 64, 16, 0.3, _dense(48), 900.0),
        _delta(6, 3, 24, 8, 1, _dense(40)),
        _att(2, 1, 32, 65, 32, 0.25, None, 77.0),
        _delta(2, 2, 40, 24, 4),
    ], (1, 4, 2), eps=1e-3),
    # beyond one 64-wide tile in every direction; heads in pairs and one by one; the loop ends with the last layer
    "wide": _model(136, 200, [
        _att(8, 4, 104, 100, 40, 0.12, _dense(200), 2e4),
        _delta(2, 1, 104, 72, 4, _dense(136)),
        _att(9, 3, 128, 70, 128, 0.1, None),
        _delta(3, 3, 128, 104, 3),
    ], (2, 4, 2)),
    # queries that fill tensor memory and shared memory; no loop
    "many": _model(72, 80, [
        _att(16, 8, 128, 130, 64, 0.1, _dense(24)),
        _att(9, 9, 40, 33, 8, 0.2),
        _delta(4, 4, 64, 128, 2),
    ]),
    # sizes the tiled kernels leave to the plain ones
    "tall": _model(48, 80, [
        _att(2, 1, 160, 30, 20, 0.09, _dense(24), 60.0),
        _delta(1, 1, 200, 136, 3),
        _att(10, 1, 16, 40, 4, 0.4),
        _delta(2, 1, 24, 264, 4, _dense(33)),
    ], (3, 4, 1)),
}


def weights_for(cfg, seed, sharp=2.0, dtype=torch.bfloat16):
    """Random weights in which every mechanism shows: peaked attention, heads that listen to each other, decays of all
    strengths, layer scales and temperatures away from one."""
    from rumus_b200.models.lerosun import LerosunConfig
    g = torch.Generator().manual_seed(seed)
    out = {}
    for k, shape in LerosunConfig.from_dict(cfg).weight_shapes().items():
        last = k.rsplit(".", 1)[-1]
        r = torch.randn(shape, generator=g)
        if last in ("norm", "norm1", "norm2", "temp"):
            t = 1.0 + 0.3 * r
        elif last in ("ls1", "ls2"):
            t = 0.6 + 0.3 * r
        elif last == "talk":
            t = 0.8 * torch.eye(shape[0]) + 0.5 * r / shape[0] ** 0.5
        elif last == "dt_bias":
            t = r - 3.0
        elif last == "conv":
            t = r * shape[1] ** -0.5
        elif k == "embed" or len(shape) == 1:
            t = r
        else:
            t = r * shape[1] ** -0.5 * (sharp if last in ("q", "k") else 1.0)
        out[k] = t.to(dtype)
    return out
