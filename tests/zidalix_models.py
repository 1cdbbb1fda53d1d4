"""Small Zidalix configurations and weights for the tests: sizes that are not multiples of eight, heads that
differ from layer to layer, layers without a feed-forward, layers that read another's latents."""
import torch

YARN = {"factor": 3.0, "original": 48, "fast": 16.0, "slow": 1.0}


def _layer(heads, dim, rot_dim, vdim, rank, scale, *, base=10000.0, scaling=YARN, kv_from=None, ff=40, limit=0.9):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "scale": scale,
         "rot": {"base": base, "dims": rot_dim, "scaling": scaling}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}


def _model(width, vocab, layers, emb=1.7, logit=0.6, eps=1e-5):
    return {"architecture": "Zidalix", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": emb},
            "logit_scale": logit, "layers": layers}


CONFIGS = {
    # nothing is a multiple of eight, sizes change from layer to layer
    "odd": _model(50, 67, [
        _layer(3, 10, 6, 13, 21, 0.31, ff=33),
        _layer(1, 7, 14, 5, 9, 0.22, base=777.0, ff=None),
        _layer(5, 12, 2, 20, 30, 0.4, scaling=None, ff=71, limit=2.5),
    ]),
    # two layers with latents of their own feed three others
    "shared": _model(64, 96, [
        _layer(2, 16, 8, 16, 24, 0.25),
        _layer(4, 8, 8, 24, 24, 0.3, kv_from=0, ff=56, limit=0.4),
        _layer(3, 16, 8, 16, 24, 0.2),
        _layer(2, 24, 8, 8, 24, 0.35, kv_from=2, ff=None),
        _layer(6, 8, 8, 16, 24, 0.25, kv_from=0),
    ], emb=0.8, logit=1.3, eps=1e-3),
    # beyond one 64-wide tile in every direction
    "wide": _model(136, 200, [
        _layer(2, 96, 40, 104, 200, 0.09, ff=72),
        _layer(9, 72, 40, 80, 200, 0.1, kv_from=0, ff=160, limit=3.0),
    ]),
    # outside what the tensor-core attention kernels cover: the plain kernel takes over
    "tall": _model(48, 80, [
        _layer(2, 160, 72, 40, 24, 0.08),
        _layer(2, 16, 8, 136, 600, 0.25),
    ]),
}


def weights_for(cfg, seed, sharp=2.5, dtype=torch.bfloat16):
    """Random weights whose attention is peaked (queries scaled by ``sharp``): with flat scores a key that is
    missing among hundreds would hardly show."""
    from rumus_b200.models.zidalix import ZidalixConfig
    g = torch.Generator().manual_seed(seed)
    out = {}
    for k, shape in ZidalixConfig.from_dict(cfg).weight_shapes().items():
        if "norm" in k:
            t = 1.0 + 0.3 * torch.randn(shape, generator=g)
        elif k.endswith("sink"):
            t = 1.0 + torch.randn(shape, generator=g)
        elif k == "embed":
            t = torch.randn(shape, generator=g)
        else:
            t = torch.randn(shape, generator=g) * shape[1] ** -0.5 * (sharp if k.endswith("mix.q") else 1.0)
        out[k] = t.to(dtype)
    return out
