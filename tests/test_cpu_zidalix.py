"""Zidalix without a GPU: configuration, registry, rotary frequencies, checkpoint files, caller-driven
sequences of the scheduler, work items of the prompt kernel, and the oracle itself."""
import json

import pytest
import torch

import zidalix_oracle as Z
from zidalix_models import CONFIGS, weights_for

from rumus_b200.models import registry
from rumus_b200.models.zidalix import ZidalixConfig
from rumus_b200.ops.rotary import RotarySpec


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_configuration_lists_the_weights(name):
    cfg = ZidalixConfig.from_dict(CONFIGS[name])
    w = weights_for(CONFIGS[name], 0)
    cfg.check_weights(w)
    assert cfg.num_params() == sum(t.numel() for t in w.values())
    for i, e in enumerate(CONFIGS[name]["layers"]):
        assert (f"l{i}.mix.dkv" in w) == (e["mixer"].get("kv_from") is None)
        assert (f"l{i}.norm2" in w) == (e["mlp"] is not None)
    missing = dict(w)
    del missing["l0.mix.sink"]
    with pytest.raises(ValueError, match="sink"):
        cfg.check_weights(missing)
    idle = {f"l{i}.norm2": torch.ones(cfg.d_model) for i, e in enumerate(CONFIGS[name]["layers"]) if e["mlp"] is None}
    cfg.check_weights({**w, **idle})
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
        lambda d: d["layers"][1]["mixer"].update(kv_from=1),             # itself
        lambda d: d["layers"][1]["mixer"].update(kv_from=2),             # a later layer
        lambda d: d["layers"][2]["mixer"].update(kv_from=1),             # a layer without latents
        lambda d: d["layers"][1]["mixer"].update(kv_rank=8),             # another latent size
        lambda d: d["layers"][1]["mixer"]["rot"].update(base=77.0),      # another rotation
        lambda d: d["layers"][0]["mixer"]["rot"].update(dims=6),
        lambda d: d["layers"][0].update(type="something"),
        lambda d: d["layers"][0]["mlp"].update(kind="sparse"),
    ]
    base = _edit("shared", lambda d: None)
    assert base["layers"][1]["mixer"]["kv_from"] == 0
    for fn in bad:
        with pytest.raises(ValueError):
            ZidalixConfig.from_dict(_edit("shared", fn))


def test_registry_finds_the_architecture(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps(CONFIGS["odd"]))
    cfg = registry.load_config(str(tmp_path))
    assert isinstance(cfg, ZidalixConfig) and registry.architecture_of(cfg).name == "Zidalix"
    assert registry.architecture("Zidalix").serving_class().__name__ == "ZidalixServing"
    with pytest.raises(ValueError, match="unknown architecture"):
        registry.architecture("nothing")
    llama = registry.architecture("Llama").config_class().from_dict({"architecture": "Llama", "num_layers": 3})
    assert llama.num_layers == 3 and registry.architecture_of(llama).name == "Llama"


@pytest.mark.parametrize("rot", [
    {"base": 10000.0, "dims": 64, "scaling": {"factor": 4.0, "original": 2048, "fast": 32.0, "slow": 1.0}},
    {"base": 500000.0, "dims": 16, "scaling": {"factor": 8.0, "original": 128, "fast": 8.0, "slow": 2.0}},
    {"base": 100.0, "dims": 8, "scaling": {"factor": 1.5, "original": 64, "fast": 4.0, "slow": 4.0}},   # empty ramp
    {"base": 10000.0, "dims": 32, "scaling": None},
    {"base": 10000.0, "dims": 2},
])
def test_rotary_frequencies(rot):
    f, m = RotarySpec.from_dict(rot).frequencies()
    want, wm = Z.yarn(rot["base"], rot["dims"], rot.get("scaling"))
    torch.testing.assert_close(f.double(), torch.tensor(want, dtype=torch.float64), rtol=1e-6, atol=0)
    assert abs(m - wm) < 1e-12
    assert (m > 1) == (rot.get("scaling") is not None)


def test_oracle_notices_a_missing_mechanism():
    """With the tests' weights every mechanism shows in the logits, so agreeing with the oracle means having it."""
    cfg = CONFIGS["shared"]
    w = weights_for(cfg, 3)
    tok = torch.randint(0, cfg["vocab"], (60,), generator=torch.Generator().manual_seed(0)).tolist()
    ref = Z.forward(cfg, w, tok)

    def differs(cfg2=cfg, w2=w, tok2=tok):
        d = Z.forward(cfg2, w2, tok2)[-1] - ref[-1]
        return float(d.norm() / ref[-1].norm())

    edits = {
        "sink": dict(w2={**w, "l0.mix.sink": torch.full_like(w["l0.mix.sink"], -1e4)}),
        "first token": dict(tok2=[(tok[0] + 1) % cfg["vocab"]] + tok[1:]),
        "kv_from": dict(cfg2=_edit("shared", lambda d: d["layers"][3]["mixer"].update(kv_from=0))),
        "limit": dict(cfg2=_edit("shared", lambda d: d["layers"][0]["mlp"].update(limit=1e4))),
        "scaling": dict(cfg2=_edit("shared", lambda d: [e["mixer"]["rot"].update(scaling=None) for e in d["layers"]])),
        "gate": dict(w2={**w, "l1.mix.g": torch.zeros_like(w["l1.mix.g"])}),
    }
    for name, kw in edits.items():
        assert differs(**kw) > 1e-3, name


def test_tensor_files_keep_dtypes(tmp_path):
    from rumus_b200.io.safetensors import load_safetensors, load_tensors, save_safetensors, save_tensors
    t = {"a": torch.randn(3, 5).bfloat16(), "b": torch.arange(7, dtype=torch.int32), "c": torch.randn(2, 2),
         "d": torch.randn(4).half(), "e": torch.zeros(0, 3).bfloat16()}
    p = str(tmp_path / "m.safetensors")
    save_tensors(t, p)
    back = load_tensors(p)
    assert set(back) == set(t) and all(back[k].dtype == t[k].dtype and torch.equal(back[k], t[k]) for k in t)
    import safetensors.torch as st
    theirs = st.load_file(p)
    assert all(torch.equal(theirs[k], t[k]) for k in t)
    with pytest.raises(ValueError, match="F32"):
        load_safetensors(p)
    save_safetensors({"x": t["c"]}, p)
    assert torch.equal(load_tensors(p)["x"], t["c"]) and torch.equal(load_safetensors(p)["x"], t["c"])
    with open(p, "r+b") as f:
        f.truncate(40)
    with pytest.raises(ValueError):
        load_tensors(p)


def test_caller_driven_sequences_share_the_pool():
    from rumus_b200.serve import Scheduler
    s = Scheduler(num_blocks=6, block_size=4, max_batch=2, token_budget=64)
    assert s.extend(10, 5) == 0 and s.free_blocks() == 4
    assert s.extend(10, 3) == 5 and s.free_blocks() == 4          # 8 tokens fill two blocks
    assert s.extend(10, 1) == 8 and s.free_blocks() == 3
    first = s.block_table(10, 8)
    assert len(set(first)) == 3
    assert s.extend(11, 2) == 0
    with pytest.raises(RuntimeError, match="slot"):
        s.extend(12, 1)
    with pytest.raises(RuntimeError, match="free blocks"):
        s.extend(11, 60)
    assert s.extend(11, 1) == 2 and s.free_blocks() == 2           # the failed call changed nothing
    s.abort(10)
    assert s.free_blocks() == 5 and s.num_running() == 1
    assert s.extend(12, 9) == 0 and set(s.block_table(12, 8)) & set(first)
    # scheduled requests run beside them and never preempt them
    s.abort(12)
    assert s.add(1, 4, 12) == 0
    for _ in range(30):
        dec, pre = s.schedule()
        assert all(i == 1 for i in dec) and all(q[0] == 1 for q in pre)
        if s.commit(dec, pre):
            break
    with pytest.raises(RuntimeError):
        s.add(5, 1, 1)
        s.extend(5, 1)
    assert s.block_table(11, 8)


def test_prompt_work_items_cover_every_row_once():
    from rumus_b200.ops.latent import QUERY_TILE, prefill_items
    segs = [(0, 300, 0, 0), (300, 2, 300, 77), (302, 128, 379, 1000), (430, 129, 1507, 5)]
    items = prefill_items(segs)
    rows = sorted(r for q, n, _, _ in items for r in range(q, q + n))
    assert rows == list(range(559)) and all(0 < n <= QUERY_TILE for _, n, _, _ in items)
    ends = [p + n for _, n, _, p in items]
    assert ends == sorted(ends, reverse=True)
    for q, n, k0, p in items:
        s = max((x for x in segs if x[0] <= q), key=lambda x: x[0])
        assert k0 == s[2] and p == s[3] + q - s[0]


def test_parts_of_the_native_build_exist():
    from rumus_b200 import build
    cu, cpp = build.PARTS[registry.architecture("Zidalix").parts]
    _, _, cu_files, cpp_files = build._sources("latent")
    assert len(cu_files) == len(cu) and len(cpp_files) == len(cpp)
    assert len(cu_files) < len(build._sources()[2])


def test_zidalix_has_no_cpu_path():
    from rumus_b200.serve import Engine, ServeConfig
    with pytest.raises(RuntimeError, match="CUDA"):
        Engine(ServeConfig(model=ZidalixConfig.from_dict(CONFIGS["odd"]), num_blocks=4), torch.device("cpu"))
