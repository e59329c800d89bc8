"""The Zuvepel configuration and description without a GPU: the round trip of config.json, the errors, which parts a layer
gets, the schedule of a loop, what the cache is asked to hold, ranks that are the checkpoint's, and the plain
implementation's own small pieces."""
from __future__ import annotations

import copy

import pytest
import torch

from zuvepel_models import CONFIGS, low_ranks


def described(raw):
    from thintensor_b200.config.registry import load_config

    arch, config = load_config(copy.deepcopy(raw))
    return config, arch.describe(config)


def test_round_trip_and_description():
    from thintensor_b200.engine.model import DecoderModel

    for name, raw in CONFIGS.items():
        config, spec = described(raw)
        assert config.architecture == "Zuvepel" and config.to_dict() == raw, name
        assert all(layer.arrangement == "parallel" and layer.params == {"scale": raw["residual_mult"]} for layer in spec.layers)
        declared = DecoderModel(spec, torch.float32, None).weight_declarations()
        assert declared["head"].shape == (raw["vocab"], raw["width"]) and declared["final.norm.b"].shape == (raw["width"],)
        for index, layer in enumerate(raw["layers"]):
            m, p = layer["mixer"], f"l{index}."
            assert (p + "norm2.b" in declared) == (layer["mlp"] is not None) and p + "norm1.b" in declared
            if layer["type"] == "attention":
                assert declared[p + "mix.g"].shape == (m["heads"], raw["width"])
                assert declared[p + "mix.v.b"].shape == (m["kv_heads"] * m["vdim"],) and p + "mix.o.b" not in declared
            elif layer["type"] == "channel_delta":
                assert declared[p + "mix.dt_bias"].shape == (m["heads"] * m["dim"],) and declared[p + "mix.A_log"].shape == (m["heads"],)
                assert declared[p + "mix.a2"].shape[0] == m["heads"] * m["dim"] and declared[p + "mix.g2"].shape[0] == m["heads"] * m["vdim"]
            else:
                assert declared[p + "mix.a2.b"].shape == (m["heads"] * m["dim"],) and declared[p + "mix.norm"].shape == (m["vdim"],)


@pytest.mark.parametrize("loop,runs", [
    (None, [(0, False), (1, False), (2, False)]),
    ({"start": 0, "stop": 2, "times": 2}, [(0, False), (1, False), (0, True), (1, False), (2, False)]),
    ({"start": 0, "stop": 1, "times": 4}, [(0, False), (0, True), (0, True), (0, True), (1, False), (2, False)]),
    ({"start": 1, "stop": 3, "times": 2}, [(0, False), (1, False), (2, False), (1, True), (2, False)]),
    ({"start": 2, "stop": 3, "times": 2}, [(0, False), (1, False), (2, False), (2, True)]),
    ({"start": 0, "stop": 3, "times": 1}, [(0, False), (1, False), (2, False)]),
])
def test_schedule_of_a_loop(loop, runs):
    import plain_zuvepel

    from thintensor_b200.engine.model import DecoderModel

    raw = copy.deepcopy(CONFIGS["a"])
    raw.pop("loop")
    if loop:
        raw["loop"] = loop
    _, spec = described(raw)
    assert [(run.layer, run.add_embedding) for run in spec.schedule] == runs == plain_zuvepel.schedule(raw)
    assert all(run.cache_from is None for run in spec.schedule)
    kv, state, _ = DecoderModel(spec, torch.float32, None).cache_needs()       # every pass has an entry of its own
    assert len(kv) == len(runs) and [need is not None for need in kv] == [layer == 0 for layer, _ in runs]
    assert [len(s) for s in state] == [{0: 0, 1: 2, 2: 1}[layer] for layer, _ in runs]


def test_what_the_cache_is_asked_for():
    from thintensor_b200.engine.model import DecoderModel
    from thintensor_b200.parts.base import KVNeed

    _, spec = described(CONFIGS["b"])
    kv, state, _ = DecoderModel(spec, torch.float32, None).cache_needs()
    assert kv == [None, KVNeed(3, 20, 150, 36), None]
    assert [[tuple(s.shape) for s in needs] for needs in state] == [[(2, 30, 72)], [], [(3, 8, 136), (0, 2 * 136 + 24)]]


def test_which_keys_a_chunked_layer_sees():
    from thintensor_b200.parts import MIXERS

    part = MIXERS.build("attention", {"hidden": 8, "heads": 2, "kv_heads": 1, "head_dim": 4, "chunk": 5})
    assert part.reach == -5 and [part.visible_keys(p) for p in range(7)] == [1, 2, 3, 4, 5, 1, 2]
    for tokens in (1, 4, 5, 6, 10, 13):
        assert part.visible_pairs(tokens) == sum(part.visible_keys(p) for p in range(tokens))
    window = MIXERS.build("attention", {"hidden": 8, "heads": 2, "kv_heads": 1, "head_dim": 4, "window": 5})
    assert window.reach == 5 and window.visible_pairs(9) == sum(window.visible_keys(p) for p in range(9))
    with pytest.raises(ValueError, match="not both"):
        MIXERS.build("attention", {"hidden": 8, "heads": 2, "kv_heads": 1, "head_dim": 4, "chunk": 5, "window": 3})


def test_ranks_are_the_checkpoints():
    """A tensor may differ from its declaration along a free axis only."""
    from thintensor_b200.engine.model import DecoderModel
    from thintensor_b200.parts.recurrent import LowRankProduct
    from thintensor_b200.weights.loader import compare

    _, spec = described(CONFIGS["a"])
    declared = DecoderModel(spec, torch.float32, None).weight_declarations()
    stored = {name: decl.shape for name, decl in low_ranks(declared).items()}
    assert stored["l1.mix.a1"] != declared["l1.mix.a1"].shape and compare(declared, stored) == ([], [], [])
    wrong = dict(stored)
    wrong["l1.mix.a1"] = (7, 95)
    assert len(compare(declared, wrong)[2]) == 1
    wrong["l1.mix.a1"] = (7, 96, 1)
    assert len(compare(declared, wrong)[2]) == 1
    with pytest.raises(ValueError, match="takes 4"):
        LowRankProduct({"down": torch.zeros(3, 8), "up": torch.zeros(6, 4)}, "down", "up", 0, "x")


@pytest.mark.parametrize("change,needle", [
    (lambda c: c["layers"][0].update(type="mamba2"), "known"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "rotated part"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "multiple"),
    (lambda c: c["layers"][1]["mixer"].pop("conv"), "conv"),
    (lambda c: c["layers"][2]["mixer"].update(tau=0.0), "tau"),
    (lambda c: c["layers"][1].update(mlp={"kind": "moe"}), "dense"),
    (lambda c: c["loop"].update(stop=4), "loop"),
    (lambda c: c["loop"].update(start=2), "loop"),
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c.update(layers=[]), "layers"),
])
def test_errors(change, needle):
    from thintensor_b200.config.base import ConfigError
    from thintensor_b200.config.registry import load_config

    raw = copy.deepcopy(CONFIGS["a"])
    change(raw)
    with pytest.raises(ConfigError, match=needle):
        load_config(raw)


def test_what_may_be_left_out():
    """A mask, a rotation, key/value heads, a factor, an embedding scale and a loop that are not given do not exist."""
    raw = copy.deepcopy(CONFIGS["a"])
    for key in ("loop", "residual_mult", "embedding"):
        raw.pop(key)
    for key in ("mask", "rot", "kv_heads"):
        raw["layers"][0]["mixer"].pop(key)
    config, spec = described(raw)
    assert (config.residual_mult, config.embedding_scale, config.loop) == (1.0, 1.0, None)
    params = spec.layers[0].parts["mixer"].params
    assert params["kv_heads"] == 6 and params["chunk"] is None and params["position"] is None


def test_plain_pieces():
    """The oracle's own mechanisms against their definitions in another form."""
    import plain_zuvepel as plain

    g = torch.Generator().manual_seed(5)
    x = torch.randn(6, 3, 8, generator=g, dtype=torch.float64)
    turned = plain.rotate_halves(x, torch.arange(6), {"dims": 4, "base": 50.0})
    assert torch.equal(turned[..., 4:], x[..., 4:]) and torch.equal(turned[0], x[0])
    assert torch.allclose(turned[..., 0] ** 2 + turned[..., 2] ** 2, x[..., 0] ** 2 + x[..., 2] ** 2)      # 0 is paired with 2
    q, k, v = (torch.randn(5, 2, n, generator=g, dtype=torch.float64) for n in (4, 4, 3))
    # decay one: linear attention is the causal sum of (q_t . k_j) v_j
    out = plain.linear_attention(q, k, v, torch.ones(5, 2, 4, dtype=torch.float64))
    want = torch.einsum("hts,shv->thv", torch.einsum("thd,shd->hts", q, k).tril(), v)
    assert torch.allclose(out, want)
    # beta one, decay one and orthonormal keys: the delta rule stores v_j under k_j
    eye = torch.eye(4, dtype=torch.float64)[:, None, :].repeat(1, 2, 1)
    one = torch.ones(4, 2, dtype=torch.float64)
    out = plain.delta_rule(eye, eye, v[:4], one, torch.ones(4, 2, 4, dtype=torch.float64))
    assert torch.allclose(out, v[:4])
