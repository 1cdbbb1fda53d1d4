"""Nufupel without a GPU: configuration, registry, rotary frequencies, work items, tile sizes, and the oracle itself."""
import json

import pytest
import torch

import nufupel_oracle as N
from nufupel_models import CONFIGS, weights_for

from rumus_b200.models import registry
from rumus_b200.models.nufupel import DenseConfig, MixtureConfig, NufupelConfig
from rumus_b200.ops.rotary import BandScaling, RotarySpec


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_configuration_lists_the_weights(name):
    cfg = NufupelConfig.from_dict(CONFIGS[name])
    w = weights_for(CONFIGS[name], 0)
    cfg.check_weights(w)
    assert cfg.num_params() == sum(t.numel() for t in w.values())
    for i, e in enumerate(CONFIGS[name]["layers"]):
        own = "weights_of" not in e
        assert (f"l{i}.norm1" in w) == own and cfg.layers[i].owner == e.get("weights_of", i)
        assert (f"l{i}.mix.q.norm" in w) == (own and e["type"] == "attention_2")
        kind = (e["mlp"] or {}).get("kind")
        assert (f"l{i}.mlp.e0.gate" in w) == (own and kind == "moe") and (f"l{i}.mlp.gate" in w) == (own and kind == "dense")
        assert isinstance(cfg.layers[i].mlp, {"moe": MixtureConfig, "dense": DenseConfig, None: type(None)}[kind])
    missing = dict(w)
    del missing["l0.mix.sink"]
    with pytest.raises(ValueError, match="sink"):
        cfg.check_weights(missing)
    with pytest.raises(ValueError, match="unexpected"):
        cfg.check_weights({**w, "l0.mix.b": torch.ones(1)})
    with pytest.raises(ValueError, match="shape"):
        cfg.check_weights({**w, "head": w["head"][:, :-1]})


def _edit(name, fn):
    d = json.loads(json.dumps(CONFIGS[name]))
    fn(d)
    return d


def test_configurations_outside_the_design_are_refused():
    bad = [
        lambda d: d["layers"][2].update(weights_of=2),                   # itself
        lambda d: d["layers"][2].update(weights_of=5),                   # a layer without weights
        lambda d: d["layers"][2].update(weights_of=9),                   # no layer
        lambda d: d["layers"][2].update(weights_of=1),                   # a layer of another kind
        lambda d: d["layers"][2]["mixer"]["mask"].update(size=9),        # differs from its owner
        lambda d: d["layers"][1]["mixer"]["rot"].update(dims=34),        # more than a head has
        lambda d: d["layers"][1]["mixer"]["rot"].update(dims=7),
        lambda d: d["layers"][1]["mixer"]["rot"].update(scaling={"factor": 2.0}),
        lambda d: d["layers"][3]["mixer"].update(kv_heads=4),
        lambda d: d["layers"][3]["mixer"]["mask"].update(size=0),
        lambda d: d["layers"][3]["mlp"]["router"].update(top=7),
        lambda d: d["layers"][3]["mlp"].update(kind="sparse"),
        lambda d: d["layers"][3].update(type="something"),
    ]
    NufupelConfig.from_dict(_edit("shared", lambda d: None))
    for fn in bad:
        with pytest.raises(ValueError):
            NufupelConfig.from_dict(_edit("shared", fn))


def test_registry_finds_the_architecture(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps(CONFIGS["odd"]))
    cfg = registry.load_config(str(tmp_path))
    assert isinstance(cfg, NufupelConfig) and registry.architecture_of(cfg).name == "Nufupel"
    assert registry.architecture("Nufupel").serving_class().__name__ == "NufupelServing"


@pytest.mark.parametrize("rot", [
    {"base": 10000.0, "dims": 64, "scaling": {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 2048}},
    {"base": 500000.0, "dims": 16, "scaling": {"factor": 8.0, "low": 2.0, "high": 32.0, "original": 512}},
    {"base": 100.0, "dims": 8, "scaling": {"factor": 1.5, "low": 3.0, "high": 3.0, "original": 64}},      # no band between
    {"base": 10000.0, "dims": 32, "scaling": None},
    {"base": 10000.0, "dims": 2},
])
def test_rotary_frequencies(rot):
    f, m = RotarySpec.from_dict(rot).frequencies()
    want = torch.tensor(N.frequencies(rot["base"], rot["dims"], rot.get("scaling")), dtype=torch.float64)
    torch.testing.assert_close(f.double(), want, rtol=1e-6, atol=0)
    assert m == 1.0


def test_band_scaling_has_three_regimes():
    base, dims, sc = 10000.0, 64, {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 256}
    plain = RotarySpec(base, dims).frequencies()[0]
    ratio = RotarySpec(base, dims, BandScaling(**sc)).frequencies()[0] / plain
    kept, slowed = (ratio == 1).sum(), (ratio - 1 / 8).abs().lt(1e-6).sum()
    assert kept > 0 and slowed > 0 and kept + slowed < dims // 2 and bool((ratio[1:] <= ratio[:-1] + 1e-6).all())


def test_oracle_notices_a_missing_mechanism():
    """With the tests' weights every mechanism shows in the logits, so agreeing with the oracle means having it."""
    cfg = CONFIGS["shared"]
    w = weights_for(cfg, 3)
    tok = torch.randint(0, cfg["vocab"], (90,), generator=torch.Generator().manual_seed(0)).tolist()
    ref = N.forward(cfg, w, tok)

    def differs(cfg2=cfg, w2=w, tok2=tok):
        d = N.forward(cfg2, w2, tok2)[-1] - ref[-1]
        return float(d.norm() / ref[-1].norm())

    def window(i, size):
        return dict(cfg2=_edit("shared", lambda d: d["layers"][i]["mixer"]["mask"].update(size=size)))

    edits = {
        "sink": dict(w2={**w, "l0.mix.sink": torch.full_like(w["l0.mix.sink"], -1e4)}),
        "window": window(0, 63), "longer window": window(1, 66), "short window": window(3, 16),
        "gate per number": dict(w2={**w, "l0.mix.g": torch.zeros_like(w["l0.mix.g"])}),
        "gate per head": dict(w2={**w, "l1.mix.g": torch.zeros_like(w["l1.mix.g"])}),
        "head norm": dict(w2={**w, "l1.mix.k.norm": torch.ones_like(w["l1.mix.k.norm"])}),
        "scaling": dict(cfg2=_edit("shared", lambda d: [e["mixer"]["rot"].update(scaling=None) for e in d["layers"] if "rot" in e["mixer"]])),
        "part of a head": dict(cfg2=_edit("shared", lambda d: d["layers"][1]["mixer"]["rot"].update(dims=32))),
        "top": dict(cfg2=_edit("shared", lambda d: d["layers"][0]["mlp"]["router"].update(top=2))),
        "router bias": dict(w2={**w, "l0.mlp.router.b": torch.zeros_like(w["l0.mlp.router.b"])}),
        "shared expert": dict(w2={**w, "l0.mlp.shared.down": torch.zeros_like(w["l0.mlp.shared.down"])}),
        "norm around zero": dict(w2={**w, "l0.norm1": w["l0.norm1"] * 0}),
        "softcap": dict(cfg2=_edit("shared", lambda d: d.update(logit_softcap=1e4))),
        "token a window back": dict(tok2=tok[:89 - 63] + [(tok[89 - 63] + 1) % cfg["vocab"]] + tok[89 - 62:]),
    }
    for name, kw in edits.items():
        assert differs(**kw) > 1e-3, name


def test_slots_per_work_item_follow_the_load():
    from rumus_b200.ops.moe import PAIR_LOAD, PAIR_TILE, slot_tile
    assert slot_tile(3, 8, False) == 16 and slot_tile(16 * 8, 8, False) == 16 and slot_tile(16 * 8 + 1, 8, False) == 32
    assert slot_tile(PAIR_LOAD * 8 - 1, 8, False) <= 128
    assert slot_tile(PAIR_LOAD * 8, 8, False) == PAIR_TILE and slot_tile(10 ** 6, 8, True) == 16


def test_gates_and_ups_in_turns():
    from rumus_b200.ops.moe import interleave
    g, u = torch.randn(3, 40, 5), torch.randn(3, 40, 5)
    w = interleave(g, u)
    assert w.shape == (3, 128, 5)
    assert torch.equal(w[:, :32], g[:, :32]) and torch.equal(w[:, 32:64], u[:, :32])
    assert torch.equal(w[:, 64:72], g[:, 32:]) and torch.equal(w[:, 96:104], u[:, 32:])
    assert float(w[:, 72:96].abs().sum()) == 0 and float(w[:, 104:].abs().sum()) == 0


def test_parts_of_the_native_build_exist():
    from rumus_b200 import build
    cu, cpp = build.PARTS[registry.architecture("Nufupel").parts]
    _, _, cu_files, cpp_files = build._sources("window")
    assert len(cu_files) == len(cu) and len(cpp_files) == len(cpp)
    assert len(cu_files) < len(build._sources()[2])


def test_nufupel_has_no_cpu_path():
    from rumus_b200.serve import Engine, ServeConfig
    with pytest.raises(RuntimeError, match="CUDA"):
        Engine(ServeConfig(model=NufupelConfig.from_dict(CONFIGS["odd"]), num_blocks=4), torch.device("cpu"))


def test_oracle_runs_one_token_at_a_time_alike():
    """The oracle's attention of the last query alone equals its row of the whole."""
    g = torch.Generator().manual_seed(1)
    q, k, v = (torch.randn(12, 3, n, generator=g, dtype=torch.float64) for n in (8, 8, 5))
    mx = {"heads": 3, "kv_heads": 3, "scale": 0.4, "mask": {"size": 5}}
    sink = torch.randn(3, generator=g, dtype=torch.float64)
    whole = N.attention_heads(q, k, v, sink, mx)
    for t in range(12):
        torch.testing.assert_close(N.attention_heads(q[t:t + 1], k[:t + 1], v[:t + 1], sink, mx, offset=t), whole[t:t + 1])
        lo = max(0, t - 4)
        for h in range(3):
            e = torch.exp(k[lo:t + 1, h] @ q[t, h] * 0.4)
            torch.testing.assert_close(whole[t, h], (e @ v[lo:t + 1, h]) / (e.sum() + sink[h].exp()))
