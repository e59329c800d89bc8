"""The Zezilix configuration, description, cache needs and random weights (no GPU)."""
from __future__ import annotations

import json

import pytest
import torch

from thintensor_b200.config.base import ConfigError
from thintensor_b200.config.registry import load_config
from thintensor_b200.config.zezilix import DenseSizes, LatentAttentionSizes, MoeSizes, WkvSizes, ZezilixConfig
from thintensor_b200.engine.model import DecoderModel
from zezilix_models import CONFIGS, write_model


def described(name):
    arch, config = load_config(json.loads(json.dumps(CONFIGS[name])))
    return config, arch.describe(config)


@pytest.mark.parametrize("name", list(CONFIGS))
def test_round_trip(name):
    config, _ = described(name)
    assert isinstance(config, ZezilixConfig) and config.to_dict() == CONFIGS[name]
    assert ZezilixConfig.from_dict(config.to_dict()) == config


def test_typed_sizes():
    config, _ = described("a")
    assert config.streams == 3 and config.residual_mult == 0.7 and (config.loop.start, config.loop.stop, config.loop.times) == (0, 2, 2)
    first, second, third = config.layers
    assert isinstance(first.mixer, LatentAttentionSizes) and first.mixer.q_rank == 56 and isinstance(first.mlp, DenseSizes) and first.mlp.limit == 1.1
    assert second.mixer == WkvSizes(4, 24) and second.mlp == MoeSizes(5, 2, 40, 1.7)
    assert third.mixer.q_rank is None and third.mlp is None
    raw = json.loads(json.dumps(CONFIGS["b"]))
    del raw["streams"], raw["residual_mult"]
    assert load_config(raw)[1].streams == 1 and load_config(raw)[1].residual_mult == 1.0


def edited(change):
    raw = json.loads(json.dumps(CONFIGS["a"]))
    change(raw)
    return raw


@pytest.mark.parametrize("change,needle", [
    (lambda r: r.pop("norm"), "norm"),
    (lambda r: r.pop("layers"), "layers"),
    (lambda r: r.pop("vocab"), "vocab"),
    (lambda r: r.update(streams=0), "streams"),
    (lambda r: r["layers"][0].update(type="attention"), "attention"),
    (lambda r: r["layers"][0]["mixer"].pop("q_rank"), "q_rank"),
    (lambda r: r["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda r: r["layers"][0]["mixer"]["rot"].update(dims=10), "rotated part"),
    (lambda r: r["layers"][0]["mlp"].pop("limit"), "limit"),
    (lambda r: r["layers"][0]["mlp"].update(limit=-1.0), "limit"),
    (lambda r: r["layers"][1]["mlp"]["router"].update(top=6), "top"),
    (lambda r: r["layers"][1]["mlp"].update(kind="wide"), "kind"),
    (lambda r: r["layers"][1]["mixer"].pop("heads"), "heads"),
    (lambda r: r["loop"].update(stop=4), "loop"),
])
def test_errors_name_the_place(change, needle):
    with pytest.raises(ConfigError) as err:
        load_config(edited(change))
    assert needle in str(err.value)


def test_schedule_and_parts():
    config, spec = described("c")
    assert [run.layer for run in spec.schedule] == [0, 1, 2, 3, 2, 3, 2, 3] and spec.streams == 2
    assert not any(run.add_embedding or run.cache_from is not None for run in spec.schedule)
    first = spec.layers[0]
    assert first.arrangement == "pre_norm" and first.params == {"scale": 1.0}
    assert first.parts["mixer"].params["gate"] == "elementwise" and first.parts["mixer"].params["q_rank"] is None
    assert first.parts["mixer"].params["position"].params["interleaved"] is True
    assert spec.layers[2].parts["mixer"].params["gate"] is None and spec.layers[2].parts["mixer"].params["q_rank"] == 72
    assert spec.layers[1].parts["ffn"].params["weight_scale"] == 1.3 and spec.layers[1].parts["ffn"].params["gated"] is False
    assert spec.embedding.params["norm_eps"] == 1e-6
    _, without_loop = described("b")
    assert [run.layer for run in without_loop.schedule] == [0, 1, 2]


def test_tensor_names_and_shapes():
    _, spec = described("a")
    declared = DecoderModel(spec, torch.float32, None).weight_declarations()
    shapes = {name: decl.shape for name, decl in declared.items()}
    assert shapes["embed"] == (211, 96) and shapes["embed.norm"] == (96,) and shapes["head"] == (211, 96) and shapes["final.norm"] == (96,)
    assert shapes["l0.hc1.mix"] == (3, 3) and shapes["l0.hc2.in"] == (3,) and shapes["l0.hc2.out"] == (3,) and shapes["l0.ls1"] == (96,)
    assert shapes["l0.mix.uq"] == (3 * 28, 56) and shapes["l0.mix.dkv"] == (48, 96) and shapes["l0.mix.uv"] == (72, 40) and "l0.mix.g" not in shapes
    assert shapes["l2.mix.g"] == (72, 96) and shapes["l2.mix.q"] == (64, 96) and "l2.mix.dq" not in shapes and "l2.norm2" not in shapes
    assert shapes["l1.mix.mu.w"] == (96,) and shapes["l1.mix.u"] == (4, 24) and shapes["l1.mix.w0"] == (96,)
    assert declared["l1.mix.w1"].fits((7, 96)) and declared["l1.mix.w2"].fits((96, 7)) and not declared["l1.mix.w1"].fits((7, 95))
    assert shapes["l1.mlp.e4.up"] == (40, 96) and shapes["l1.mlp.e4.down"] == (96, 40) and "l1.mlp.e0.gate" not in shapes
    assert shapes["l1.mlp.router"] == (5, 96)


def test_cache_needs_of_every_pass():
    """Two runs of a looped layer keep a cache and states each; a latent layer keeps one row a token."""
    _, spec = described("a")
    kv, states, source = DecoderModel(spec, torch.float32, None).cache_needs()
    assert [None if n is None else (n.kv_heads, n.head_dim, n.v_dim, n.window) for n in kv] == [
        (1, 48, 0, None), None, (1, 48, 0, None), None, (1, 44, 0, None)]
    assert [[tuple(s.shape) for s in entry] for entry in states] == [[], [(4, 24, 24), (96,)], [], [(4, 24, 24), (96,)], []]
    assert all(s.dtype == torch.float32 for entry in states for s in entry) and source == [None] * 5


def test_streams_go_with_weights_for_them():
    from dataclasses import replace

    from thintensor_b200.parts.spec import LayerSpec

    _, spec = described("a")
    with pytest.raises(ValueError, match="streams"):
        DecoderModel(replace(spec, streams=None), torch.float32, None)
    bare = LayerSpec("pre_norm", {k: v for k, v in spec.layers[0].parts.items() if not k.endswith("streams")}, spec.layers[0].params)
    with pytest.raises(ValueError, match="streams"):
        DecoderModel(replace(spec, layers=(bare,) + spec.layers[1:]), torch.float32, None)


def test_random_weights_and_the_plain_reader(tmp_path):
    """A written folder holds exactly the declared tensors, and the plain implementation runs it."""
    import plain_zezilix

    folder = write_model(tmp_path / "a", "a", "bfloat16")
    config, weights = plain_zezilix.read_model(folder)
    _, spec = described("a")
    assert set(weights) == set(DecoderModel(spec, torch.float32, None).weight_declarations())
    logits = plain_zezilix.forward(config, weights, [5, 17, 3, 100])
    assert logits.shape == (4, 211) and bool(torch.isfinite(logits).all())


def test_plain_pieces():
    """The oracle's own pieces on cases worked out by hand."""
    import plain_zezilix as plain

    streams = torch.tensor([[[1.0, 2.0]], [[10.0, 20.0]]], dtype=torch.float64)
    mixed = plain.hyper_write(streams, torch.tensor([[1.0, 0.5], [0.0, 2.0]], dtype=torch.float64), torch.tensor([3.0, -1.0], dtype=torch.float64),
                              torch.tensor([[1.0, 1.0]], dtype=torch.float64))
    assert mixed.tolist() == [[[4.0, 5.0]], [[19.5, 40.0]]]               # from (row) to (column)
    one = torch.ones(1, 1, 1, dtype=torch.float64)
    out = plain.bonus_recurrence(one.repeat(3, 1, 1), one.repeat(3, 1, 1), torch.tensor([[[2.0]], [[3.0]], [[5.0]]], dtype=torch.float64),
                                 0.5 * one.repeat(3, 1, 1), 10.0 * torch.ones(1, 1, dtype=torch.float64))
    assert out.flatten().tolist() == [20.0, 2.0 + 30.0, 0.5 * 2.0 + 3.0 + 50.0]      # the token's own decay comes after it is read
    turned = plain.rotate_pairs(torch.tensor([[[1.0, 0.0, 7.0]]], dtype=torch.float64), torch.tensor([1]), {"dims": 2, "base": 10.0})
    assert torch.allclose(turned.flatten(), torch.tensor([torch.cos(torch.tensor(1.0)), torch.sin(torch.tensor(1.0)), 7.0]).double(), atol=1e-6)
