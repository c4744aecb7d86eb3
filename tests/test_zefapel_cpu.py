"""Zefapel without a GPU: its configuration, its plan, the cache's storage for it, and the engine's step logic over it
with the kernels replaced by their plain torch restatement (tests/torch_ops.py), against the plain implementation
(tests/plain_zefapel.py); and the plain implementation's own parts where a slip would hide."""

import copy
import math

import pytest
import torch

import plain_zefapel as plain
from torch_ops import TorchOps
from zefapel_helpers import CONFIGS, assert_logits, config, plain_logits, prompts, write_folder


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("zefapel")
    return {name: write_folder(root / name, name) for name in CONFIGS}


def cpu_engine(folder, **kw):
    from kernel_rush_kawk_b200 import Engine

    args = dict(dtype="float32", device="cpu", ops=TorchOps(torch.float32), max_tokens=1024, max_slots=5,
                max_context=512, use_cuda_graphs=False)
    args.update(kw)
    return Engine(folder, **args)


def test_config_reads_back_and_is_found_by_its_name(folders):
    from kernel_rush_kawk_b200 import ZefapelConfig, read_config

    for name in CONFIGS:
        arch, cfg = read_config(folders[name])
        assert arch.name == "Zefapel" and isinstance(cfg, ZefapelConfig)
        assert ZefapelConfig.from_dict(cfg.to_dict()) == cfg
        assert cfg.embedding_scale == CONFIGS[name]["embedding"]["scale"]


@pytest.mark.parametrize("damage, word", [
    (lambda c: c["layers"][1].__setitem__("type", "attention"), "type"),
    (lambda c: c["layers"][2]["mixer"].pop("gate_cap"), "gate_cap"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("tau", 0), "tau"),
    (lambda c: c["layers"][1]["mixer"].pop("q_rank"), "q_rank"),
    (lambda c: c["layers"][1]["mixer"]["rot"].__setitem__("dims", 6), "rot_dim"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("fast"), "fast"),
    (lambda c: c["layers"][3]["mixer"].__setitem__("kv_from", 3), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].__setitem__("kv_from", 0), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].__setitem__("kv_rank", 16), "kv_rank"),
    (lambda c: c["layers"][0]["mlp"]["router"].__setitem__("top", 5), "top"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].__setitem__("count", 3), "groups"),
    (lambda c: c["layers"][0]["mlp"]["router"].__setitem__("identity", -1), "identity"),
    (lambda c: c["layers"][1].__setitem__("mlp", {"kind": "wide", "ff": 8}), "dense"),
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c.__setitem__("layers", []), "layers"),
])
def test_config_faults_are_named(damage, word):
    from kernel_rush_kawk_b200 import ConfigError, ZefapelConfig

    raw = copy.deepcopy(CONFIGS["za"])
    damage(raw)
    with pytest.raises(ConfigError, match=word):
        ZefapelConfig.from_dict(raw)


def test_plan_names_every_tensor_and_each_layer_asks_the_cache_for_what_it_keeps():
    from kernel_rush_kawk_b200.config.registry import get_architecture
    from kernel_rush_kawk_b200.engine.model import PartTree
    from kernel_rush_kawk_b200.parts import KVNeed, StateNeed

    cfg = config("za")
    tree = PartTree(get_architecture("Zefapel").plan(cfg))
    names = tree.expected_tensors()
    shape = lambda n: tuple(names[n].shape)
    assert shape("l0.norm1.alpha") == () and shape("l0.norm1.b") == (64,) and shape("l0.ls1") == (64,)
    assert shape("l0.mix.a1") == (5, 64) and shape("l0.mix.a2") == (60, 5) and shape("l0.mix.norm") == (12,)
    assert shape("l2.mix.norm") == (80,) and shape("l2.mix.i") == (2, 64)
    assert shape("l0.mlp.router") == (8, 64) and shape("l0.mlp.correction") == (8,)
    assert "l0.mlp.e5.up" not in names and "l0.mlp.e0.gate" not in names and shape("l0.mlp.shared.sg") == (1, 64)
    assert shape("l1.mix.dkv") == (40, 64) and "l3.mix.dkv" not in names and "l3.mix.dkv.norm" not in names
    assert "l2.norm2" not in names and "l2.ls2" not in names and "final.norm.alpha" in names and "head" in names
    needs = tree.cache_needs()
    assert needs[0] == StateNeed((3, 20, 12), "float32")
    assert needs[1] == KVNeed(1, 40, None, values=False)  # a latent row and its rotated key part
    assert needs[2] == (StateNeed((2, 24, 40), "float32"), StateNeed((2, 25), "float32"))
    assert needs[3] == ("from", 1)


def test_frequencies_of_the_scaled_rotation():
    """Pairs below the ramp keep their frequency, pairs beyond it are divided by the factor, one in between is mixed;
    without scaling nothing changes; a ramp of no width is a step. By hand for 16 dimensions and base 100."""
    from kernel_rush_kawk_b200.parts.latent_attention import scaled_frequencies

    s = {"factor": 4.0, "original": 64, "fast": 4.0, "slow": 0.5}
    at = lambda turns: 16 * math.log(64 / (2 * math.pi * turns)) / (2 * math.log(100.0))
    assert (math.floor(at(4.0)), math.ceil(at(0.5))) == (1, 6)
    f, factor = scaled_frequencies(16, 100.0, s)
    base = [100.0 ** (-2.0 * i / 16) for i in range(8)]
    ramp = [0.0, 0.0, 0.2, 0.4, 0.6, 0.8, 1.0, 1.0]
    assert torch.allclose(f, torch.tensor([b / 4 * r + b * (1 - r) for b, r in zip(base, ramp)], dtype=torch.float64), rtol=1e-12)
    assert abs(factor - (0.1 * math.log(4.0) + 1.0)) < 1e-12
    assert torch.allclose(scaled_frequencies(16, 100.0, None)[0], torch.tensor(base, dtype=torch.float64))
    assert scaled_frequencies(16, 100.0, None)[1] == 1.0
    for c in CONFIGS.values():
        for layer in c["layers"]:
            rot = layer["mixer"].get("rot")
            if rot is not None:
                mine, by = scaled_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
                theirs, factor = plain.rotation(rot)
                assert torch.allclose(mine, torch.tensor(theirs, dtype=torch.float64), rtol=1e-12) and abs(by - factor) < 1e-12


def test_choice_is_within_the_kept_groups_and_weights_are_not_renormalised():
    """Struck-out scores count as minus infinity: with corrections that make every score negative the choice still comes
    from the kept groups."""
    z = torch.tensor([2.0, 0.0, 1.0, 1.5, -1.0, 0.5], dtype=torch.float64)
    corr = torch.tensor([-2.0, -1.0, -1.2, -1.3, -1.1, -1.4], dtype=torch.float64)
    s = torch.softmax(z, 0)
    idx, w = plain.choose(z, corr, 2, {"count": 3, "keep": 1})
    c = s + corr
    best = max(range(3), key=lambda g: c[2 * g:2 * g + 2].max())
    assert sorted(idx) == [2 * best, 2 * best + 1] and torch.equal(w, s[idx])
    assert abs(w.sum() - 1.0) > 0.1
    ops = TorchOps(torch.float32)
    experts, weights, _, passed = ops.moe_route_softmax_groups(torch.eye(1), z.float()[:, None], corr.float(), 2, 3, 1, 3)
    got = {int(e): float(a) for e, a in zip(experts[0], weights[0]) if e >= 0}
    assert set(got) == {i for i in idx if i < 3}
    assert abs(float(passed[0]) - float(sum(s[i] for i in idx if i >= 3))) < 1e-6


@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompts_portions_and_single_tokens_agree_with_the_plain_implementation(folders, name):
    from kernel_rush_kawk_b200 import StepEntry

    eng = cpu_engine(folders[name])
    ids = prompts(name, [90])[0]
    ref = plain_logits(folders[name], ids)
    for pieces in ([90], [50, 2, 3, 35], [70] + [1] * 20):
        slot = eng.cache.alloc()
        got, start = [], 0
        for n in pieces:
            got.append(eng.step([StepEntry(slot, ids[start:start + n], list(range(n)))]))
            start += n
        eng.cache.free(slot)
        assert_logits(torch.cat(got), ref, "float32", f"{name}, pieces {pieces[:4]}")
    eng.cache.check()


def test_unequal_batch_against_each_alone_and_reused_slots(folders):
    from kernel_rush_kawk_b200 import StepEntry

    eng = cpu_engine(folders["za"])
    for seed in (3, 4):  # the second time over, slots and pages hold the first batch's leavings
        seqs = prompts("za", [40, 1, 70, 13], seed=seed)
        slots = [eng.cache.alloc() for _ in seqs]
        heads = [len(ids) - 2 if len(ids) > 2 else len(ids) for ids in seqs]
        first = eng.step([StepEntry(s, ids[:n], [n - 1]) for s, ids, n in zip(slots, seqs, heads)])
        for i, (ids, n) in enumerate(zip(seqs, heads)):
            assert_logits(first[i:i + 1], plain_logits(folders["za"], ids)[n - 1:n], "float32", f"batched prompt {i}")
        live = [(s, ids) for s, ids in zip(slots, seqs) if len(ids) > 2]
        for back in (2, 1):
            got = eng.step([StepEntry(s, [ids[-back]], [0]) for s, ids in live])
            for i, (s, ids) in enumerate(live):
                ref = plain_logits(folders["za"], ids)
                assert_logits(got[i:i + 1], ref[len(ids) - back:len(ids) - back + 1], "float32", f"batched token of sequence {i}")
        for s in slots:
            eng.cache.free(s)
        eng.cache.check()


def test_presets_build_their_plans_and_are_served_by_name():
    from kernel_rush_kawk_b200 import ZefapelConfig
    from kernel_rush_kawk_b200.config.registry import get_architecture, preset_config
    from kernel_rush_kawk_b200.engine.model import PartTree

    for name in ZefapelConfig.preset_names():
        cfg = preset_config(name)
        assert PartTree(get_architecture("Zefapel").plan(cfg), 64).expected_tensors()
    assert "zefapel_tiny" in ZefapelConfig.preset_names()


def test_command_line_writes_a_preset_as_a_model_folder(tmp_path):
    from kernel_rush_kawk_b200 import cli, read_config

    assert cli.main(["write-random", "--preset", "zefapel_tiny", "--seed", "1", "--out", str(tmp_path / "m")]) == 0
    arch, cfg = read_config(tmp_path / "m")
    assert arch.name == "Zefapel" and len(cfg.layers) == 4
    steps = list(cpu_engine(tmp_path / "m", max_tokens=256, max_context=256).generate([[5, 6, 7], [9]], 3))
    assert len(steps) == 3 and all(len(s) == 2 for s in steps)
