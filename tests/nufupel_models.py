"""Small Nufupel configurations and weights for the tests: sizes that are not multiples of eight, windows shorter and
longer than pages and tiles, layers without a feed-forward, layers that use another's weights."""
import torch

BANDS = {"factor": 3.0, "low": 1.0, "high": 4.0, "original": 60}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, top, ff, shared):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}, "shared": {"ff": shared}}


def _plain(heads, kv_heads, dim, vdim, window, scale, mlp=None, **kw):
    """Attention without positions."""
    return {"type": "attention", "mlp": mlp, **kw,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": window}}}


def _turned(heads, kv_heads, dim, vdim, window, scale, rot, mlp=None, *, base=10000.0, scaling=BANDS, **kw):
    """Attention with head norms and rotation."""
    e = _plain(heads, kv_heads, dim, vdim, window, scale, mlp, **kw)
    e["type"] = "attention_2"
    e["mixer"]["rot"] = {"base": base, "dims": rot, "scaling": scaling}
    return e


def _again(layers, j):
    """A layer with the weights of layer j."""
    return {**layers[j], "weights_of": j}


def _model(width, vocab, layers, emb=1.7, cap=9.0, eps=1e-5):
    return {"architecture": "Nufupel", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": emb},
            "logit_softcap": cap, "layers": layers}


def _configs():
    # nothing is a multiple of eight, sizes change from layer to layer
    odd = [
        _turned(3, 1, 10, 13, 21, 0.31, 6, _dense(33)),
        _plain(5, 5, 7, 5, 70, 0.4, None),
        _plain(6, 2, 12, 20, 3, 0.3, _moe(5, 2, 19, 27)),
        _turned(4, 2, 14, 9, 45, 0.3, 14, _moe(3, 1, 50, 11), base=777.0, scaling=None),
    ]
    odd.append(_again(odd, 2))
    # weights used several times, of both kinds, before and after one another
    shared = [
        _plain(4, 2, 16, 24, 64, 0.25, _moe(8, 3, 40, 56)),
        _turned(2, 1, 32, 16, 65, 0.2, 16, _dense(48)),
    ]
    shared += [_again(shared, 0), _turned(6, 2, 24, 16, 17, 0.3, 24, _moe(6, 6, 16, 8), base=500.0), _again(shared, 1), _again(shared, 0)]
    # beyond one 64-wide tile in every direction
    wide = [
        _turned(4, 2, 104, 72, 100, 0.12, 40, _moe(40, 4, 72, 136)),
        _plain(9, 3, 72, 128, 150, 0.14, _dense(200)),
    ]
    wide.append(_again(wide, 0))
    # outside what the prompt kernel covers: the row kernel takes over
    tall = [
        _plain(2, 1, 160, 40, 30, 0.08, _moe(2, 1, 24, 24)),
        _turned(3, 3, 40, 264, 80, 0.2, 8, None),
        _plain(16, 1, 8, 16, 200, 0.3, _dense(24)),
    ]
    return {"odd": _model(50, 67, odd), "shared": _model(64, 96, shared, emb=0.8, cap=20.0, eps=1e-3),
            "wide": _model(136, 200, wide, cap=5.0), "tall": _model(48, 80, tall)}


CONFIGS = _configs()


def weights_for(cfg, seed, sharp=2.5, dtype=torch.bfloat16):
    """Random weights whose attention is peaked (queries scaled by ``sharp``): with flat scores a key that is missing
    among hundreds would hardly show.  Routers are scaled up too, so that few choices of experts are close."""
    from rumus_b200.models.nufupel import NufupelConfig
    g = torch.Generator().manual_seed(seed)
    out = {}
    for k, shape in NufupelConfig.from_dict(cfg).weight_shapes().items():
        if k.endswith("norm1") or k == "final.norm":
            t = 0.3 * torch.randn(shape, generator=g)
        elif k.endswith(".norm"):
            t = (1.0 + 0.3 * torch.randn(shape, generator=g)) * (sharp if k.endswith("q.norm") else 1.0)
        elif k.endswith("sink") or k.endswith("router.b"):
            t = torch.randn(shape, generator=g)
        elif k == "embed":
            t = torch.randn(shape, generator=g)
        else:
            t = torch.randn(shape, generator=g) * shape[1] ** -0.5
            t = t * (sharp if k.endswith("mix.q") else 3.0 if k.endswith("router") else 1.0)
        out[k] = t.to(dtype)
    return out
