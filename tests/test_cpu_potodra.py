"""Potodra without a GPU: configuration, registry, places of the scheduler, chunks, and the oracle itself."""
import json

import pytest
import torch

import potodra_oracle as P
from potodra_models import CONFIGS, weights_for

from rumus_b200.models import registry
from rumus_b200.models.potodra import AttentionConfig, MlstmConfig, ParallelConfig, PotodraConfig


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_configuration_lists_the_weights(name):
    cfg, w = PotodraConfig.from_dict(CONFIGS[name]), weights_for(CONFIGS[name], 0)
    cfg.check_weights(w)
    kinds = {"attention": AttentionConfig, "mlstm": MlstmConfig, "parallel": ParallelConfig}
    for i, e in enumerate(CONFIGS[name]["layers"]):
        assert type(cfg.layers[i].mixer) is kinds[e["type"]]
        assert (f"l{i}.mix.sink" in w) == (e["type"] == "attention") and f"l{i}.mix.left.sink" not in w
        assert (f"l{i}.mix.right.q.conv" in w) == (e["type"] == "parallel")
        assert (f"l{i}.norm2" in w) == (f"l{i}.hc2.mix" in w) == (e["mlp"] is not None)
    gone = dict(w)
    del gone["l0.hc1.out"]
    with pytest.raises(ValueError, match="hc1.out"):
        cfg.check_weights(gone)
    with pytest.raises(ValueError, match="unexpected"):
        cfg.check_weights({**w, "l0.mix.z": torch.ones(1)})
    with pytest.raises(ValueError, match="shape"):
        cfg.check_weights({**w, "embed": w["embed"][:, :-1]})


def test_inner_widths_come_from_the_tensors():
    cfg, w = PotodraConfig.from_dict(CONFIGS["odd"]), weights_for(CONFIGS["odd"], 0)
    assert w["l0.mix.right.a1"].shape[0] != w["l0.mix.right.g1"].shape[0]
    with pytest.raises(ValueError, match="a2"):
        cfg.check_weights({**w, "l0.mix.right.a1": w["l0.mix.right.a1"][:-1]})


def test_a_layer_without_feed_forward_may_carry_its_norm():
    cfg, w = PotodraConfig.from_dict(CONFIGS["odd"]), weights_for(CONFIGS["odd"], 0)
    cfg.check_weights({**w, "l2.norm2": torch.ones(50), "l2.hc2.in": torch.ones(3), "l2.hc2.out": torch.ones(3), "l2.hc2.mix": torch.eye(3)})


def _edit(name, fn):
    d = json.loads(json.dumps(CONFIGS[name]))
    fn(d)
    return d


def test_configurations_outside_the_design_are_refused():
    bad = [
        lambda d: d.update(streams=0),
        lambda d: d["layers"][0].update(type="something"),
        lambda d: d["layers"][0]["mixer"].update(kv_heads=3),
        lambda d: d["layers"][0]["mixer"]["rot"].update(dims=17),
        lambda d: d["layers"][0]["mixer"]["rot"].update(dims=18),
        lambda d: d["layers"][0]["mixer"]["mask"].update(size=0),
        lambda d: d["layers"][0]["mixer"]["mask"].update(keep_first=-1),
        lambda d: d["layers"][0]["mixer"].update(softcap=0.0),
        lambda d: d["layers"][0]["mlp"].update(kind="sparse"),
        lambda d: d["layers"][0]["mlp"]["router"]["groups"].update(count=3),      # 8 experts
        lambda d: d["layers"][0]["mlp"]["router"]["groups"].update(keep=5),
        lambda d: d["layers"][0]["mlp"]["router"].update(top=5),                  # two groups of two are open
        lambda d: d["layers"][1]["mixer"]["right"].update(kv_heads=3),
        lambda d: d["layers"][1]["mixer"]["right"].update(conv=0),
    ]
    PotodraConfig.from_dict(_edit("mixed", lambda d: None))
    for fn in bad:
        with pytest.raises(ValueError):
            PotodraConfig.from_dict(_edit("mixed", fn))


def test_registry_finds_the_architecture(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps(CONFIGS["odd"]))
    cfg = registry.load_config(str(tmp_path))
    assert isinstance(cfg, PotodraConfig) and registry.architecture_of(cfg).name == "Potodra"
    assert registry.architecture("Potodra").serving_class().__name__ == "PotodraServing"


def test_parts_of_the_native_build_exist():
    from rumus_b200 import build
    part = registry.architecture("Potodra").parts
    cu, cpp = build.PARTS[part]
    _, _, cu_files, cpp_files = build._sources(part)
    assert len(cu_files) == len(cu) and len(cpp_files) == len(cpp)


def test_potodra_has_no_cpu_path():
    from rumus_b200.serve import Engine, ServeConfig
    with pytest.raises(RuntimeError, match="CUDA"):
        Engine(ServeConfig(model=PotodraConfig.from_dict(CONFIGS["odd"]), num_blocks=4), torch.device("cpu"))


def test_places_belong_to_running_sequences():
    """A sequence keeps its place while it runs; places of ended and preempted ones are given again; never two alike."""
    from rumus_b200.serve import Scheduler
    s = Scheduler(8, 16, 3, 64)
    for rid in (5, 6, 7):
        s.extend(rid, 3)
    first = s.places([5, 6, 7]).tolist()
    assert sorted(first) == [0, 1, 2]
    with pytest.raises(RuntimeError):
        s.extend(8, 1)
    s.extend(6, 20)
    assert s.places([6, 5]).tolist() == [first[1], first[0]]
    s.abort(6)
    with pytest.raises(KeyError):
        s.places([6])
    s.extend(8, 1)
    assert s.places([8, 7]).tolist() == [first[1], first[2]]
    for rid in (5, 7, 8):
        s.abort(rid)
    # the scheduler's own: 40 tokens each in 3 blocks, 8 blocks: growing past a block's end preempts the youngest
    for rid in (1, 2, 3):
        assert s.add(rid, 40, 30) == 0
    seen, preempted = {}, False
    for _ in range(400):
        dec, pre = s.schedule()
        if not dec and not pre:
            break
        now = dec + [p[0] for p in pre]
        places = s.places(now).tolist()
        assert len(set(places)) == len(places)
        for rid, place, start in [(d, p, 1) for d, p in zip(dec, places)] + [(p[0], q, p[1]) for p, q in zip(pre, places[len(dec):])]:
            assert start == 0 or seen[rid] == place          # another place only from the beginning
            seen[rid] = place
        s.commit(dec, pre)
        preempted = preempted or s.preemptions() > 0
    assert preempted and s.free_blocks() == 8


def test_cutting_portions_into_chunks():
    from rumus_b200.ops.recurrent import cut
    c = cut([(3, 130), (200, 64), (264, 1)], 64, "cpu")
    assert c.items[:, :3].tolist() == [[3, 64, 0], [67, 64, 0], [131, 2, 0], [200, 64, 1], [264, 1, 2]]
    assert c.first.tolist() == [0, 3, 4, 5] and c.size == 64


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

    edits = {
        "sink": changed(l0__mix__sink=lambda t: t * 0 - 1e4), "cap": mixer(0, softcap=1e6), "window": mixer(0, mask={"size": 63, "keep_first": 64}),
        "kept tokens": mixer(0, mask={"size": 64, "keep_first": 63}), "few kept tokens": mixer(3, mask={"size": 65, "keep_first": 2}),
        "key bias": changed(l0__mix__q__b=lambda t: t * 0), "value bias": changed(l0__mix__v__b=lambda t: t * 0),
        "part of a head": mixer(1, left={**cfg["layers"][1]["mixer"]["left"], "rot": {"base": 900.0, "dims": 6}}),
        "input gate": changed(l2__mix__i=lambda t: t * 0), "forget bias": changed(l2__mix__f__b=lambda t: t * 0 + 9),
        "gate cap": mixer(2, gate_cap=2.0), "memory norm": changed(l2__mix__norm=lambda t: t * 0 + 1),
        "oldest tap": changed(l1__mix__right__k__conv=lambda t: t * (torch.arange(5) > 0)), "decay": changed(l1__mix__right__A_log=lambda t: t + 0.5),
        "decay bias": changed(l1__mix__right__dt_bias=lambda t: t + 0.5), "decay projection": changed(l1__mix__right__a2=lambda t: t * 0),
        "write strength": changed(l1__mix__right__b=lambda t: t * 0), "output gate": changed(l1__mix__right__g2=lambda t: t * 0),
        "scales": mixer(1, left_scale=0.6, right_scale=1.1), "connections": changed(l2__hc1__mix=lambda t: t.T.contiguous()),
        "connections out": changed(l2__hc1__out=lambda t: t * 0 + 1), "connections in": changed(l3__hc2__in=lambda t: t.flip(0)),
        "correction": changed(l0__mlp__correction=lambda t: t * 0), "shared gate": changed(l0__mlp__shared__sg=lambda t: t * 0),
        "groups": dict(cfg2=_edit(name, lambda d: [d["layers"][i]["mlp"]["router"]["groups"].update(keep=3) for i in (0, 1)])),
        "expert limit": dict(cfg2=_edit(name, lambda d: d["layers"][0]["mlp"]["expert"].update(limit=2.2))),
        "shared limit": dict(cfg2=_edit(name, lambda d: d["layers"][0]["mlp"]["shared"].update(limit=1.2))),
    }
    for what, kw in edits.items():
        assert differs(**kw) > 1e-3, what


def test_oracle_recurrences_go_on_from_where_they_were():
    """The oracle's memories against their closed forms on short sequences."""
    g = torch.Generator().manual_seed(2)
    T, d, e = 6, 4, 3
    q, k, v = (torch.randn(T, n, generator=g, dtype=torch.float64) for n in (d, d, e))
    i, f = torch.randn(T, generator=g, dtype=torch.float64), -P.softplus(torch.randn(T, generator=g, dtype=torch.float64))
    o, (S, n, m) = P.mlstm_memory(q, k, v, i, f)
    w = torch.tensor([[float(torch.exp(f[j + 1:t + 1].sum() + i[j])) if j <= t else 0.0 for j in range(T)] for t in range(T)], dtype=torch.float64)
    num, den = (w * (q @ k.T)) @ v, (w * (q @ k.T)).sum(1)
    run, ms = 0.0, []
    for t in range(T):
        run = max(float(f[t]) + run, float(i[t]))
        ms.append(run)
    ms = torch.tensor(ms, dtype=torch.float64)
    torch.testing.assert_close(o, num * torch.exp(-ms)[:, None] / (torch.maximum((den * torch.exp(-ms)).abs(), torch.exp(-ms)) + 1e-6)[:, None])
    torch.testing.assert_close(S, torch.einsum("j,jd,je->de", w[-1] * torch.exp(-ms[-1]), k, v))
    # the delta rule without decay and with full strength stores the last value of a key exactly
    k1 = k / k.norm(dim=1, keepdim=True)
    o, S = P.delta_memory(k1, k1, v, torch.ones(T, d, dtype=torch.float64), torch.ones(T, dtype=torch.float64))
    torch.testing.assert_close(o, v)
    torch.testing.assert_close(k1[-1] @ S, v[-1])
