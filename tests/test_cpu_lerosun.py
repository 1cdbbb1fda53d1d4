"""Lerosun without a GPU: configuration, weight list, registry, order of the layers, and the oracle itself."""
import copy
import json

import pytest
import torch

import lerosun_oracle as P
from lerosun_models import CONFIGS, weights_for

from rumus_b200.models import registry
from rumus_b200.models.lerosun import LerosunConfig, TalkingAttentionConfig
from rumus_b200.models.potodra import DeltaConfig


def _edit(name, fn):
    d = copy.deepcopy(CONFIGS[name])
    fn(d)
    return d


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_configuration_lists_the_weights(name):
    cfg, w = LerosunConfig.from_dict(CONFIGS[name]), weights_for(CONFIGS[name], 0)
    cfg.check_weights(w)
    kinds = {"attention": TalkingAttentionConfig, "delta": DeltaConfig}
    for i, e in enumerate(CONFIGS[name]["layers"]):
        assert type(cfg.layers[i].mixer) is kinds[e["type"]]
        assert (f"l{i}.mix.talk" in w) == (e["type"] == "attention") == (f"l{i}.mix.v" not in w)
        assert (f"l{i}.norm2" in w) == (f"l{i}.ls2" in w) == (e["mlp"] is not None)
    assert w["embed.norm"].shape == w["l0.norm1"].shape == w["final.norm"].shape == ()
    assert sum(t.numel() for t in w.values()) == cfg.num_params()
    gone = dict(w)
    del gone["l0.ls1"]
    with pytest.raises(ValueError, match="ls1"):
        cfg.check_weights(gone)
    with pytest.raises(ValueError, match="unexpected"):
        cfg.check_weights({**w, "l0.mix.z": torch.ones(1)})
    with pytest.raises(ValueError, match="shape"):
        cfg.check_weights({**w, "embed": w["embed"][:, :-1]})
    assert set(cfg.random_weights()) == set(w)


def test_a_layer_without_feed_forward_may_carry_its_norm():
    cfg, w = LerosunConfig.from_dict(CONFIGS["odd"]), weights_for(CONFIGS["odd"], 0)
    cfg.check_weights({**w, "l1.norm2": torch.ones(()), "l1.ls2": torch.ones(50)})
    with pytest.raises(ValueError, match="unexpected"):
        cfg.check_weights({**w, "l3.norm2": torch.ones(())})


def test_bad_configurations_are_refused():
    bad = [
        lambda d: d["layers"][0].update(type="recurrent"),
        lambda d: d["layers"][1]["mixer"].update(kv_heads=3),
        lambda d: d["layers"][1]["mixer"].update(vdim=16),
        lambda d: d["layers"][1]["mixer"]["rot"].update(dims=15),
        lambda d: d["layers"][1]["mixer"]["rot"].update(dims=26),
        lambda d: d["layers"][1]["mixer"]["mask"].update(size=0),
        lambda d: d["layers"][1]["mlp"].update(kind="moe"),
        lambda d: d["layers"][1]["mlp"].update(ff=0),
        lambda d: d["layers"][0]["mixer"].update(kv_heads=3),
        lambda d: d["layers"][0]["mixer"].update(conv=0),
        lambda d: d["loop"].update(stop=6),
        lambda d: d["loop"].update(start=5),
        lambda d: d["loop"].update(times=0),
    ]
    LerosunConfig.from_dict(_edit("mixed", lambda d: None))
    for fn in bad:
        with pytest.raises(ValueError):
            LerosunConfig.from_dict(_edit("mixed", fn))


def test_layers_run_in_the_order_of_the_loop():
    runs = {"odd": [0, 1, 0, 1, 0, 1, 2], "mixed": [0, 1, 2, 3, 1, 2, 3, 4], "wide": [0, 1, 2, 3, 2, 3], "many": [0, 1, 2], "tall": [0, 1, 2, 3]}
    for name, want in runs.items():
        assert LerosunConfig.from_dict(CONFIGS[name]).runs == want == P.order(CONFIGS[name])
    assert LerosunConfig.from_dict(_edit("odd", lambda d: d.pop("loop"))).runs == [0, 1, 2]


def test_registry_finds_the_architecture(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps(CONFIGS["odd"]))
    cfg = registry.load_config(str(tmp_path))
    assert isinstance(cfg, LerosunConfig) and registry.architecture_of(cfg).name == "Lerosun"
    assert registry.architecture("Lerosun").serving_class().__name__ == "LerosunServing"


def test_parts_of_the_native_build_exist():
    from rumus_b200 import build
    part = registry.architecture("Lerosun").parts
    cu, cpp = build.PARTS[part]
    _, _, cu_files, cpp_files = build._sources(part)
    assert len(cu_files) == len(cu) and len(cpp_files) == len(cpp)


def test_lerosun_has_no_cpu_path():
    from rumus_b200.serve import Engine, ServeConfig
    with pytest.raises(RuntimeError, match="CUDA"):
        Engine(ServeConfig(model=LerosunConfig.from_dict(CONFIGS["odd"]), num_blocks=4), torch.device("cpu"))


def test_oracle_notices_a_missing_mechanism():
    """With the tests' weights every mechanism shows in the logits, so agreeing with the oracle means having it."""
    name = "mixed"
    cfg, w = CONFIGS[name], weights_for(CONFIGS[name], 3)
    tok = torch.randint(0, cfg["vocab"], (150,), generator=torch.Generator().manual_seed(0)).tolist()
    ref = P.forward(cfg, w, tok)

    def differs(cfg2=cfg, w2=w):
        return float((P.forward(cfg2, w2, tok)[-1] - ref[-1]).norm() / ref[-1].norm())

    def changed(**kw):
        return dict(w2={**w, **{k.replace("__", "."): f(w[k.replace("__", ".")]) for k, f in kw.items()}})

    def mixer(i, **kw):
        return dict(cfg2=_edit(name, lambda d: d["layers"][i]["mixer"].update(**kw)))

    zero, one = lambda t: t * 0, lambda t: t * 0 + 1
    edits = {
        "sink": changed(l1__mix__sink=lambda t: t * 0 - 1e4), "window": mixer(1, mask={"size": 63}), "longer window": mixer(3, mask={"size": 66}),
        "query bias": changed(l1__mix__q__b=zero), "key bias": changed(l3__mix__k__b=zero), "temperature": changed(l1__mix__temp=one),
        "talk": changed(l1__mix__talk=lambda t: torch.eye(4)), "who listens to whom": changed(l1__mix__talk=lambda t: t.T.contiguous()),
        "part of a head": mixer(1, rot={"base": 900.0, "dims": 14}), "base": mixer(3, rot={"base": 78.0, "dims": 32}),
        "scale": mixer(1, scale=0.32), "gate per head": changed(l3__mix__g=zero),
        "oldest tap": changed(l0__mix__k__conv=lambda t: t * (torch.arange(5) > 0)), "decay": changed(l0__mix__A_log=lambda t: t + 0.5),
        "decay bias": changed(l2__mix__dt_bias=lambda t: t + 0.5), "decay projection": changed(l2__mix__a=zero),
        "write strength": changed(l0__mix__b=zero), "output gate": changed(l4__mix__g=lambda t: t * 0.5), "head norm": changed(l4__mix__norm=one),
        "layer scale": changed(l1__ls1=one), "scale of the feed-forward": changed(l2__ls2=one), "norm": changed(l3__norm1=lambda t: t * 1.2),
        "embedding norm": changed(embed__norm=lambda t: t * 1.2), "up": changed(l1__mlp__up=zero), "act": changed(l1__mlp__gate=lambda t: -t),
        "passes": dict(cfg2=_edit(name, lambda d: d["loop"].update(times=3))), "start": dict(cfg2=_edit(name, lambda d: d["loop"].update(start=2))),
        "stop": dict(cfg2=_edit(name, lambda d: d["loop"].update(stop=3))),
    }
    for what, kw in edits.items():
        assert differs(**kw) > 1e-3, what


def test_oracle_against_closed_forms():
    g = torch.Generator().manual_seed(2)
    T, d, e, H = 6, 4, 3, 4
    rnd = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    # without decay and with full strength the delta rule stores the last value of a key exactly
    k, v = P.unit(rnd(T, d)), rnd(T, e)
    k = k / k.norm(dim=1, keepdim=True)
    ones = torch.ones(T, dtype=torch.float64)
    o, S = P.delta_memory(k, k, v, ones, ones)
    torch.testing.assert_close(o, v)
    # orthogonal keys never meet: what is read back has only decayed
    k = torch.eye(d, dtype=torch.float64)
    gs, beta = torch.rand(d, generator=g, dtype=torch.float64), torch.rand(d, generator=g, dtype=torch.float64)
    o, S = P.delta_memory(k, k, v[:d], gs, beta)
    torch.testing.assert_close(S, torch.stack([gs[t + 1:].prod() * beta[t] * v[t] for t in range(d)]))
    # mixing scores or queries is the same
    q, ks, mix, temp = rnd(T, H, d), rnd(T, 2, d), rnd(H, H), rnd(H)
    s = P.talk(P.scores(q, ks, 0.7, temp), mix)
    wide = torch.stack([torch.stack([sum(mix[h, 2 * c + r] * temp[2 * c + r] * q[:, 2 * c + r] for r in range(2)) for c in range(2)], 1) for h in range(H)])
    torch.testing.assert_close(s, 0.7 * torch.einsum("htcd,scd->hts", wide, ks))
    # a sink takes part of the weight and gives nothing
    x = torch.zeros(1, T, dtype=torch.float64)
    torch.testing.assert_close(P.attend(x, torch.ones(T, 1, dtype=torch.float64), torch.tensor(0.0, dtype=torch.float64), T, T - 1), torch.full((1, 1), T / (T + 1), dtype=torch.float64))
    assert [P.visible(9, j, 3) for j in (6, 7, 9, 10)] == [False, True, True, False]
