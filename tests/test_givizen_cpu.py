"""Givizen without a GPU: its configuration, its plan, the cache's storage for it, and the engine's step logic over it
with the kernels replaced by their plain torch restatement (tests/torch_ops.py), against the plain implementation
(tests/plain_givizen.py); and the plain implementation's own parts where a slip would hide."""

import copy
import math

import pytest
import torch

import plain_givizen as plain
from givizen_helpers import CONFIGS, assert_logits, config, plain_logits, prompts, write_folder
from torch_ops import TorchOps


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("givizen")
    return {name: write_folder(root / name, name) for name in CONFIGS}


def cpu_engine(folder, **kw):
    from kernel_rush_kawk_b200 import Engine

    args = dict(dtype="float32", device="cpu", ops=TorchOps(torch.float32), max_tokens=1024, max_slots=5,
                max_context=512, use_cuda_graphs=False)
    args.update(kw)
    return Engine(folder, **args)


def test_config_reads_back_and_is_found_by_its_name(folders):
    from kernel_rush_kawk_b200 import GivizenConfig, read_config

    for name in CONFIGS:
        arch, cfg = read_config(folders[name])
        assert arch.name == "Givizen" and isinstance(cfg, GivizenConfig)
        assert GivizenConfig.from_dict(cfg.to_dict()) == cfg
        assert cfg.logit_softcap == CONFIGS[name].get("logit_softcap")


@pytest.mark.parametrize("damage, word", [
    (lambda c: c["layers"][1].__setitem__("type", "attention_3"), "type"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("kv_heads", 3), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["mask"].__setitem__("size", 0), "size"),
    (lambda c: c["layers"][0]["mixer"]["q_temp"].pop("coef"), "coef"),
    (lambda c: c["layers"][0]["mixer"]["q_temp"].__setitem__("every", 2.5), "every"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][1]["mixer"].__setitem__("softcap", 0), "softcap"),
    (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "dense"), "moe"),
    (lambda c: c["layers"][0]["mlp"]["expert"].pop("limit"), "limit"),
    (lambda c: c["layers"][0]["mlp"]["shared"].pop("ff"), "ff"),
    (lambda c: c["layers"][0]["mlp"]["router"].__setitem__("top", 7), "top"),
    (lambda c: c.__setitem__("logit_softcap", -1.0), "logit_softcap"),
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c.__setitem__("layers", []), "layers"),
])
def test_config_faults_are_named(damage, word):
    from kernel_rush_kawk_b200 import ConfigError, GivizenConfig

    raw = copy.deepcopy(CONFIGS["ga"])
    damage(raw)
    with pytest.raises(ConfigError, match=word):
        GivizenConfig.from_dict(raw)


def test_plan_names_every_tensor_and_each_layer_asks_the_cache_for_what_it_keeps():
    from kernel_rush_kawk_b200.config.registry import get_architecture
    from kernel_rush_kawk_b200.engine.model import PartTree
    from kernel_rush_kawk_b200.parts import KVNeed

    tree = PartTree(get_architecture("Givizen").plan(config("ga")))
    names = tree.expected_tensors()
    shape = lambda n: tuple(names[n].shape)
    assert shape("l0.mix.q") == (64, 64) and shape("l0.mix.k") == (32, 64) and shape("l0.mix.v") == (48, 64)
    assert shape("l0.mix.o") == (64, 96) and shape("l0.mix.q.norm") == (16,) and shape("l0.mix.sink") == (4,)
    assert "l0.mix.g" not in names and shape("l1.mix.g") == (3, 64)
    assert not {"l1.mix.q.norm", "l1.mix.k.norm", "l1.mix.sink"} & set(names)
    assert shape("l0.mlp.router") == (6, 64) and shape("l0.mlp.e5.gate") == (40, 64) and shape("l0.mlp.shared.down") == (64, 72)
    assert "l0.mlp.correction" not in names and "l0.mlp.router.b" not in names
    assert "l2.norm1" in names and "l2.norm2" not in names and "final.norm" in names and "head" in names
    needs = tree.cache_needs()
    assert needs[0] == KVNeed(2, 16, 20, 24) and needs[1] == KVNeed(1, 24, 33, 16)
    assert needs[2] == KVNeed(2, 40, 1, 12) and needs[3] == KVNeed(3, 8, 64)
    assert PartTree(get_architecture("Givizen").plan(config("gb"))).cache_needs()[3] == KVNeed(1, 64, None)


def test_options_that_do_not_go_together_are_refused():
    from kernel_rush_kawk_b200.parts import RoutedExperts, ScaledEmbedding, SinkWindowAttention

    base = {"hidden": 32, "heads": 2, "kv_heads": 1, "dim": 8, "scale": 0.3, "window": 9, "eps": 1e-5}
    SinkWindowAttention({**base, "qk_norm": "head_rms", "softcap": 3.0, "distance_bias": True, "q_temp": (0.5, 4)})
    for bad in ({"talk": True}, {"chunk": 8}, {"qk_norm": "head", "value_norm": True}, {"q_temp": (0.5, 4), "value_mix": "first"},
                {"softcap": 0.0}, {"q_temp": (0.5, 0)}, {"qk_norm": "heads"}):
        with pytest.raises(ValueError):
            SinkWindowAttention({**base, **bad})
    with pytest.raises(ValueError):
        ScaledEmbedding({"vocab": 5, "hidden": 4, "rounded": True, "copies": 2})
    with pytest.raises(ValueError):
        RoutedExperts({"hidden": 8, "experts": 4, "top": 5, "intermediate": 8, "scoring": "sigmoid"})


def test_temperature_and_slopes_by_hand():
    assert plain.temperature(0, 0.5, 64) == 1.0 and plain.temperature(62, 0.5, 64) == 1.0
    assert abs(plain.temperature(63, 0.5, 64) - (1 + 0.5 * math.log(2))) < 1e-12  # position 63 is the 64th
    assert abs(plain.temperature(127, 0.5, 64) - (1 + 0.5 * math.log(3))) < 1e-12
    assert abs(plain.temperature(0, 2.0, 1) - (1 + 2 * math.log(2))) < 1e-12
    assert plain.slopes(8) == [2.0 ** -(h + 1) for h in range(8)] and plain.slopes(1) == [2.0 ** -8]
    assert abs(plain.slopes(3)[0] - 2.0 ** (-8 / 3)) < 1e-15


def test_the_softmax_by_hand():
    """One head, three keys, window 2: the first key is out of sight; the cap comes before the bias; the sink gets neither."""
    q = torch.tensor([[[1.0]], [[1.0]], [[2.0]]], dtype=torch.float64)
    k = torch.tensor([[[9.0]], [[3.0]], [[-1.0]]], dtype=torch.float64)
    v = torch.tensor([[[100.0]], [[1.0]], [[-2.0]]], dtype=torch.float64)
    out = plain.biased_window_softmax(q, k, v, 0.5, 2, softcap=2.0, sink=torch.tensor([0.7], dtype=torch.float64))
    near, far = 2 * math.tanh(-0.5), 2 * math.tanh(1.5) - 2.0 ** -8
    e = [math.exp(far), math.exp(near), math.exp(0.7)]
    assert abs(out[2, 0, 0].item() - (e[0] * 1.0 + e[1] * -2.0) / sum(e)) < 1e-12


def test_the_weight_multiplies_the_experts_input():
    """With clamped inputs expert(w h) and w expert(h) differ; the sum is over the former."""
    g = torch.Generator().manual_seed(1)
    r = lambda *s: torch.randn(s, generator=g, dtype=torch.float64)
    w = {"router": r(3, 8), **{f"e{e}.{k}": r(*s) for e in range(3) for k, s in (("gate", (5, 8)), ("up", (5, 8)), ("down", (8, 5)))}}
    h = r(4, 8)
    mlp = {"router": {"experts": 3, "top": 2}, "expert": {"ff": 5, "limit": 0.8}}
    got = plain.routed_ff(h, w, "", mlp)
    for t in range(4):
        s = torch.sigmoid(w["router"] @ h[t])
        best = s.argsort(descending=True)[:2].tolist()
        inside = sum(plain.expert(s[e] * h[t], w, f"e{e}.", 0.8) for e in best)
        outside = sum(s[e] * plain.expert(h[t], w, f"e{e}.", 0.8) for e in best)
        assert torch.allclose(got[t], inside) and (inside - outside).abs().max() > 1e-2


@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompts_portions_and_single_tokens_agree_with_the_plain_implementation(folders, name):
    from kernel_rush_kawk_b200 import StepEntry

    eng = cpu_engine(folders[name])
    ids = prompts(name, [150])[0]
    ref = plain_logits(folders[name], ids)
    for pieces in ([150], [80, 2, 3, 65], [110] + [1] * 40):
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

    eng = cpu_engine(folders["ga"])
    for seed in (3, 4):  # the second time over, slots and pages hold the first batch's leavings
        seqs = prompts("ga", [40, 1, 70, 13], seed=seed)
        slots = [eng.cache.alloc() for _ in seqs]
        heads = [len(ids) - 2 if len(ids) > 2 else len(ids) for ids in seqs]
        first = eng.step([StepEntry(s, ids[:n], [n - 1]) for s, ids, n in zip(slots, seqs, heads)])
        for i, (ids, n) in enumerate(zip(seqs, heads)):
            assert_logits(first[i:i + 1], plain_logits(folders["ga"], ids)[n - 1:n], "float32", f"batched prompt {i}")
        live = [(s, ids) for s, ids in zip(slots, seqs) if len(ids) > 2]
        for back in (2, 1):
            got = eng.step([StepEntry(s, [ids[-back]], [0]) for s, ids in live])
            for i, (s, ids) in enumerate(live):
                ref = plain_logits(folders["ga"], ids)
                assert_logits(got[i:i + 1], ref[len(ids) - back:len(ids) - back + 1], "float32", f"batched token of sequence {i}")
        for s in slots:
            eng.cache.free(s)
        eng.cache.check()


def test_presets_build_their_plans_and_are_served_by_name():
    from kernel_rush_kawk_b200 import GivizenConfig
    from kernel_rush_kawk_b200.config.registry import get_architecture, preset_config
    from kernel_rush_kawk_b200.engine.model import PartTree

    for name in GivizenConfig.preset_names():
        cfg = preset_config(name)
        assert PartTree(get_architecture("Givizen").plan(cfg), 64).expected_tensors()
    assert "givizen_tiny" in GivizenConfig.preset_names()


def test_command_line_writes_a_preset_as_a_model_folder(tmp_path):
    from kernel_rush_kawk_b200 import cli, read_config

    assert cli.main(["write-random", "--preset", "givizen_tiny", "--seed", "1", "--out", str(tmp_path / "m")]) == 0
    arch, cfg = read_config(tmp_path / "m")
    assert arch.name == "Givizen" and len(cfg.layers) == 3
    steps = list(cpu_engine(tmp_path / "m", max_tokens=256, max_context=256).generate([[5, 6, 7], [9]], 3))
    assert len(steps) == 3 and all(len(s) == 2 for s in steps)
