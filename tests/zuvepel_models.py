"""Tiny Zuvepel configurations with random weights for the tests, the plain implementation's outputs for them, and the
judge that compares an engine's logits with those.  The configurations differ from one another in every size; between
them they cover: one key/value head for all query heads, one for each and one for several, key and value sizes that differ and
that are equal, chunks that end inside the first cache block, span more than two blocks and are absent, a rotation of the
whole head, of a part of it and none, recurrences with key sizes in every register class, query/key heads shared and not,
convolutions of 1, 3 and 5 taps, products of low rank with odd ranks that differ from layer to layer, loops over the first
layers, over later ones and none, layers without a feed-forward, factors and embedding scales on both sides of one, and
one model whose attention heads have tensor-core sizes."""
from __future__ import annotations

import json
from pathlib import Path

import torch


def _dense(ff):
    return {"kind": "dense", "ff": ff}


CONFIGS = {
    # a chunk inside the first block; two passes over the first two layers
    "a": {
        "architecture": "Zuvepel", "vocab": 211, "width": 96, "norm": {"eps": 1e-5}, "residual_mult": 0.7, "embedding": {"scale": 1.5},
        "loop": {"start": 0, "stop": 2, "times": 2},
        "layers": [
            {"type": "attention", "mlp": _dense(136), "mixer": {
                "heads": 6, "kv_heads": 2, "dim": 16, "vdim": 24, "mask": {"size": 21}, "rot": {"dims": 8, "base": 500.0}, "scale": 0.3}},
            {"type": "channel_delta", "mlp": _dense(72), "mixer": {"heads": 4, "kv_heads": 2, "dim": 24, "vdim": 40, "conv": 3}},
            {"type": "gla", "mlp": None, "mixer": {"heads": 3, "dim": 20, "vdim": 12, "tau": 8.0}},
        ],
    },
    # no loop; large key sizes; a chunk over more than two blocks; no rotation; one tap
    "b": {
        "architecture": "Zuvepel", "vocab": 130, "width": 72, "norm": {"eps": 1e-6}, "residual_mult": 1.3, "embedding": {"scale": 0.5},
        "loop": {"start": 1, "stop": 3, "times": 1},
        "layers": [
            {"type": "gla", "mlp": _dense(102), "mixer": {"heads": 2, "dim": 72, "vdim": 30, "tau": 24.0}},
            {"type": "attention", "mlp": None, "mixer": {"heads": 3, "kv_heads": 3, "dim": 20, "vdim": 36, "mask": {"size": 150}, "scale": 0.25}},
            {"type": "channel_delta", "mlp": _dense(64), "mixer": {"heads": 3, "kv_heads": 1, "dim": 136, "vdim": 8, "conv": 1}},
        ],
    },
    # attention heads of tensor-core sizes, one layer without chunks; three passes over the layers in the middle; the factor 1
    "c": {
        "architecture": "Zuvepel", "vocab": 160, "width": 128, "norm": {"eps": 1e-6}, "residual_mult": 1.0, "embedding": {"scale": 2.0},
        "loop": {"start": 1, "stop": 3, "times": 3},
        "layers": [
            {"type": "channel_delta", "mlp": _dense(160), "mixer": {"heads": 2, "kv_heads": 2, "dim": 64, "vdim": 48, "conv": 5}},
            {"type": "attention", "mlp": _dense(192), "mixer": {
                "heads": 4, "kv_heads": 2, "dim": 64, "vdim": 64, "mask": {"size": 100}, "rot": {"dims": 64, "base": 10000.0}, "scale": 0.125}},
            {"type": "gla", "mlp": _dense(96), "mixer": {"heads": 1, "dim": 32, "vdim": 64, "tau": 4.0}},
            {"type": "attention", "mlp": _dense(96), "mixer": {
                "heads": 4, "kv_heads": 1, "dim": 128, "vdim": 128, "rot": {"dims": 64, "base": 100000.0}, "scale": 0.09}},
        ],
    },
}
SEEDS = {"a": 3, "b": 4, "c": 6}


def _rank(name: str, drawn: int) -> int:
    """A rank for the products of low rank of layer ``l<i>.``, which is the tensors' alone: another one in every layer and for the
    gate than for the decay; multiples of eight (tensor-core products in bfloat16) in the first layer, odd in the others."""
    layer = int(name[1:name.index(".")])
    if layer == 0:
        return 8 if name[-2] == "a" else 32
    return 5 + 2 * layer if name[-2] == "a" else 9 + 2 * layer


def low_ranks(declared):
    """The declarations with the tests' own ranks in place of those that random weights are drawn with by default."""
    out = {}
    for name, decl in declared.items():
        if decl.free:
            (axis,) = decl.free
            shape = list(decl.shape)
            shape[axis] = _rank(name, shape[axis])
            decl = type(decl)(tuple(shape), init=decl.init, free=decl.free)
        out[name] = decl
    return out


def shape_weights(tensors: dict[str, torch.Tensor], seed: int) -> dict[str, torch.Tensor]:
    """Rescale the drawn weights so that every mechanism moves the logits: hidden states and logits of order one, peaked
    attention, biases and gates away from zero, decays spread between fast ones and ones that carry hundreds of tokens."""
    g = torch.Generator().manual_seed(seed + 1000)
    out = {}
    for name, t in tensors.items():
        leaf = name.split(".", 1)[1] if name.startswith("l") and "." in name else name
        if name in ("embed", "head"):
            t = t * 30.0
        elif leaf.startswith("norm") and leaf.endswith(".b") or name == "final.norm.b":
            t = torch.randn(t.shape, generator=g) * 0.3
        elif leaf.endswith("A_log"):
            t = torch.rand(t.shape, generator=g) * 3.0 - 5.0
        elif leaf.endswith("dt_bias"):
            t = torch.rand(t.shape, generator=g) * 3.0 - 2.0
        elif leaf == "mix.a2.b":
            t = torch.rand(t.shape, generator=g) * 4.0 - 1.0
        elif leaf.endswith(".b") and leaf.startswith("mix."):
            t = torch.randn(t.shape, generator=g) * 0.5
        elif leaf.endswith(".conv"):
            t = torch.randn(t.shape, generator=g) * 0.6
        elif leaf in ("mix.q", "mix.k"):
            t = t * 20.0
        elif "norm" in leaf:
            pass
        elif leaf.startswith("mix.") or leaf.startswith("mlp."):
            t = t * 10.0
        out[name] = t
    return out


def write_model(folder: Path, name: str, stored: str = "float32", config: dict | None = None, seed: int | None = None) -> Path:
    from thintensor_b200.config.registry import load_config
    from thintensor_b200.engine.model import DecoderModel
    from thintensor_b200.weights.random_init import STORED_DTYPES, random_tensors
    from thintensor_b200.weights.safetensors_io import write_safetensors

    config = CONFIGS[name] if config is None else config
    seed = SEEDS[name] if seed is None else seed
    arch, typed = load_config(config)
    declared = low_ranks(DecoderModel(arch.describe(typed), torch.float32, None).weight_declarations())
    tensors = shape_weights(random_tensors(declared, seed, torch.float32), seed)
    tensors = {k: v.to(STORED_DTYPES[stored]) for k, v in tensors.items()}
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(config, indent=1))
    write_safetensors(folder / "model.safetensors", tensors)
    return folder


_oracle: dict = {}


def oracle_logits(folder: Path, tokens: list[int]) -> torch.Tensor:
    """float64 logits [T, vocab] of the plain implementation for one whole sequence."""
    import plain_zuvepel

    model_key = ("model", str(folder))
    if model_key not in _oracle:
        _oracle[model_key] = plain_zuvepel.read_model(folder)
    key = (str(folder), tuple(tokens))
    if key not in _oracle:
        cfg, weights = _oracle[model_key]
        with torch.no_grad():
            _oracle[key] = plain_zuvepel.forward(cfg, weights, tokens)
    return _oracle[key]


def oracle_sensitivity(folder: Path, tokens: list[int]) -> torch.Tensor:
    """Per position, one minus the cosine between the plain implementation's logits and its logits with every operand of
    a matrix product narrowed to bfloat16 on the way: how far the rounding of activations alone carries that position."""
    import plain_zuvepel

    key = ("sensitivity", str(folder), tuple(tokens))
    if key not in _oracle:
        want = oracle_logits(folder, tokens)
        cfg, weights = _oracle[("model", str(folder))]
        with torch.no_grad():
            other = plain_zuvepel.forward(cfg, weights, tokens, narrow=lambda x: x.to(torch.bfloat16).to(x.dtype))
        _oracle[key] = 1.0 - torch.nn.functional.cosine_similarity(want, other, dim=-1)
    return _oracle[key]


class Judge:
    """Compares rows of logits with the plain implementation's.  float32: every logit within 5e-5 of the request's largest
    one.  bfloat16: the cosine with the plain logits, position by position, against ``1 - cos <= 1e-3 + 4 s``, s being how
    far the plain implementation itself moves at that position when it narrows its activations to bfloat16.  Another
    rounding of the same quantities can carry a sensitive position a little further; so over a test up to one position in
    twenty-five (and one) may exceed its bound, while the mean of ``1 - cos`` stays within 0.002 of the mean bound."""

    def __init__(self, dtype, folder):
        self.dtype, self.folder, self.away, self.over, self.notes, self.bounds = dtype, folder, [], 0, [], []

    def add(self, got, tokens, rows, what):
        rows = list(rows)
        want = oracle_logits(self.folder, tokens)[rows]
        got = got.double().cpu().reshape(-1, got.shape[-1])
        assert got.shape == want.shape and torch.isfinite(got).all(), what
        if self.dtype == "float32":
            scale = max(1.0, float(want.abs().max()))
            err = (got - want).abs().max(dim=-1).values
            worst = int(err.argmax())
            assert float(err[worst]) <= 5e-5 * scale, f"{what}: position {rows[worst]}: max |diff| {float(err[worst]):.3e} with logits up to {scale:.3f}"
            return
        away = 1.0 - torch.nn.functional.cosine_similarity(got, want, dim=-1)
        bound = 1e-3 + 4.0 * oracle_sensitivity(self.folder, tokens)[rows]
        bad = away > bound
        if bool(bad.any()):
            worst = int((away / bound).argmax())
            self.notes.append(f"{what}: position {rows[worst]} has cosine {1 - float(away[worst]):.5f}, rounding alone allows {1 - float(bound[worst]):.5f}")
        self.over += int(bad.sum())
        self.away.append(away)
        self.bounds.append(bound)

    def done(self):
        if self.dtype == "bfloat16":
            away = torch.cat(self.away)
            assert self.over <= 1 + away.numel() // 25, f"{self.over} of {away.numel()} positions beyond their bound; " + "; ".join(self.notes[:4])
            allowed = 0.002 + float(torch.cat(self.bounds).mean())
            assert float(away.mean()) <= allowed, f"mean cosine {float(1.0 - away.mean()):.5f}, rounding alone allows {1.0 - allowed:.5f}"
