"""Tiny Zezilix configurations with random weights for the tests, the plain implementation's outputs for them, and the
judge that compares an engine's logits with those.  The configurations differ from one another in every size; between
them they cover: one, two and three residual streams, loops over the first layers, over later ones and none, both kinds of
latent attention with heads whose key and value sizes are equal, differ, and are padded to either tensor-core size or too large for
it, rotated parts of two numbers up to most of a head, recurrences with head sizes in every register class, ranks that tensor-core
products take and odd ones, mixtures of which a token takes one expert, several and all, routing and residual factors on
both sides of one, dense units with a clamp that bites, layers without a feed-forward, and one model whose sizes reach the grouped
product, the ungated product's own epilogue and the expanded prompt form."""
from __future__ import annotations

import json
from pathlib import Path

import torch


def _dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def _moe(experts, top, ff, scale):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}}


CONFIGS = {
    # three streams; two passes over the first two layers
    "a": {
        "architecture": "Zezilix", "vocab": 211, "width": 96, "norm": {"eps": 1e-5}, "residual_mult": 0.7, "streams": 3,
        "loop": {"start": 0, "stop": 2, "times": 2},
        "layers": [
            {"type": "latent_attention", "mlp": _dense(136, 1.1), "mixer": {
                "heads": 3, "dim": 20, "rot_dim": 8, "vdim": 24, "kv_rank": 40, "q_rank": 56, "scale": 0.3, "rot": {"dims": 8, "base": 500.0}}},
            {"type": "wkv", "mlp": _moe(5, 2, 40, 1.7), "mixer": {"heads": 4, "dim": 24}},
            {"type": "latent_attention_2", "mlp": None, "mixer": {
                "heads": 2, "dim": 12, "rot_dim": 20, "vdim": 36, "kv_rank": 24, "scale": 0.25, "rot": {"dims": 20, "base": 3000.0}}},
        ],
    },
    # one stream; no loop; large heads; one expert a token (in the last layer: a close call that rounding decides stays at its position)
    "b": {
        "architecture": "Zezilix", "vocab": 130, "width": 72, "norm": {"eps": 1e-6}, "residual_mult": 1.2, "streams": 1,
        "layers": [
            {"type": "wkv", "mlp": _dense(64, 0.8), "mixer": {"heads": 2, "dim": 136}},
            {"type": "latent_attention_2", "mlp": _moe(3, 3, 50, 2.0), "mixer": {
                "heads": 5, "dim": 110, "rot_dim": 34, "vdim": 16, "kv_rank": 36, "scale": 0.1, "rot": {"dims": 34, "base": 10000.0}}},
            {"type": "wkv", "mlp": _moe(4, 1, 24, 0.6), "mixer": {"heads": 3, "dim": 70}},
        ],
    },
    # tensor-core sizes: heads padded to 64 and to 128, grouped products, the experts' epilogue; three passes over the last two layers
    "c": {
        "architecture": "Zezilix", "vocab": 160, "width": 128, "norm": {"eps": 1e-6}, "residual_mult": 1.0, "streams": 2,
        "loop": {"start": 2, "stop": 4, "times": 3},
        "layers": [
            {"type": "latent_attention_2", "mlp": _dense(160, 1.5), "mixer": {
                "heads": 3, "dim": 72, "rot_dim": 32, "vdim": 100, "kv_rank": 64, "scale": 0.11, "rot": {"dims": 32, "base": 100000.0}}},
            {"type": "wkv", "mlp": _moe(8, 4, 128, 1.3), "mixer": {"heads": 2, "dim": 128}},
            {"type": "latent_attention", "mlp": _moe(6, 2, 64, 0.9), "mixer": {
                "heads": 4, "dim": 32, "rot_dim": 16, "vdim": 56, "kv_rank": 48, "q_rank": 72, "scale": 0.16, "rot": {"dims": 16, "base": 10000.0}}},
            {"type": "wkv", "mlp": _dense(96, 1.0), "mixer": {"heads": 4, "dim": 32}},
        ],
    },
}
SEEDS = {"a": 3, "b": 4, "c": 6}


def low_ranks(declared):
    """The declarations with a rank of the tests' own for the decays of every layer, which is the tensors' alone: multiples of eight
    (tensor-core products in bfloat16) in odd layers, odd in even ones."""
    out = {}
    for name, decl in declared.items():
        if decl.free:
            layer = int(name[1:name.index(".")])
            (axis,) = decl.free
            shape = list(decl.shape)
            shape[axis] = 8 * (layer + 1) if layer % 2 else 7 + 2 * layer
            decl = type(decl)(tuple(shape), init=decl.init, free=decl.free)
        out[name] = decl
    return out


def shape_weights(tensors: dict[str, torch.Tensor], seed: int) -> dict[str, torch.Tensor]:
    """Rescale the drawn weights so that every mechanism moves the logits: logits of order one, peaked attention, blends of the
    previous row from none to all of it, decays spread between fast ones and ones that carry hundreds of tokens, a bonus and gates
    of order one, routing scores that differ, streams that are read and written differently."""
    g = torch.Generator().manual_seed(seed + 1000)
    out = {}
    for name, t in tensors.items():
        leaf = name.split(".", 1)[1] if name.startswith("l") and "." in name else name
        if name == "head":
            t = t * 30.0
        elif leaf.startswith("mix.mu."):
            t = torch.rand(t.shape, generator=g)
        elif leaf == "mix.w0":
            t = torch.rand(t.shape, generator=g) * 6.0 - 6.0
        elif leaf == "mix.u":
            t = torch.randn(t.shape, generator=g)
        elif leaf.startswith("ls"):
            t = 1.0 + 0.4 * torch.randn(t.shape, generator=g)
        elif leaf.endswith(".in") or leaf.endswith(".out"):
            t = 0.8 + 0.4 * torch.randn(t.shape, generator=g)
        elif leaf.startswith("hc"):
            t = t + 0.15 * torch.randn(t.shape, generator=g)
        elif "norm" in leaf:
            pass
        elif leaf in ("mix.q", "mix.uq", "mix.dkv"):
            t = t * 12.0
        elif leaf == "mlp.router":
            t = t * 12.0
        elif leaf.startswith("mlp.e"):                  # experts that are alike in part: a close call of the router that rounding decides
            t = t * 6.0                                 # the other way then carries a position no further than other roundings may
            expert, matrix = leaf[len("mlp.e"):].split(".")
            if int(expert) > 0:
                t = 0.8 * out[name.replace(f".e{expert}.{matrix}", f".e0.{matrix}")] + 0.6 * t
        elif leaf.startswith("mlp."):
            t = t * 6.0
        elif leaf.startswith("mix."):
            t = t * 8.0
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
    import plain_zezilix

    model_key = ("model", str(folder))
    if model_key not in _oracle:
        _oracle[model_key] = plain_zezilix.read_model(folder)
    key = (str(folder), tuple(tokens))
    if key not in _oracle:
        cfg, weights = _oracle[model_key]
        with torch.no_grad():
            _oracle[key] = plain_zezilix.forward(cfg, weights, tokens)
    return _oracle[key]


def oracle_sensitivity(folder: Path, tokens: list[int]) -> torch.Tensor:
    """Per position, one minus the cosine between the plain implementation's logits and its logits with every operand of
    a matrix product narrowed to bfloat16 on the way: how far the rounding of activations alone carries that position.  The
    larger of two roundings of the same precision, on grids a little apart: a router's close call may fall with one and stand with the other."""
    import plain_zezilix

    key = ("sensitivity", str(folder), tuple(tokens))
    if key not in _oracle:
        want = oracle_logits(folder, tokens)
        cfg, weights = _oracle[("model", str(folder))]
        with torch.no_grad():
            others = [plain_zezilix.forward(cfg, weights, tokens, narrow=lambda x, f=factor: (x * f).to(torch.bfloat16).to(x.dtype) / f) for factor in (1.0, 1.37)]
        _oracle[key] = torch.stack([1.0 - torch.nn.functional.cosine_similarity(want, other, dim=-1) for other in others]).max(dim=0).values
    return _oracle[key]


def oracle_float32_error(folder: Path, tokens: list[int]) -> torch.Tensor:
    """Per position, the largest difference between the plain implementation's logits in float32 and in float64."""
    import plain_zezilix

    key = ("float32", str(folder), tuple(tokens))
    if key not in _oracle:
        want = oracle_logits(folder, tokens)
        cfg, weights = _oracle[("model", str(folder))]
        with torch.no_grad():
            other = plain_zezilix.forward(cfg, weights, tokens, dtype=torch.float32)
        _oracle[key] = (other.double() - want).abs().max(dim=-1).values
    return _oracle[key]


class Judge:
    """Compares rows of logits with the plain implementation's.  float32: every logit within 5e-5 of the request's largest
    one, or within eight times what the plain implementation itself differs by at that position when it computes in float32 (a
    first token's read-out, say, is ill-conditioned where the sum of its bonus products nearly vanishes).  bfloat16: the cosine with the plain logits, position by position, against ``1 - cos <= 1e-3 + 4 s``, s being how
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
            if float(err.max()) > 5e-5 * scale:
                err = err - 8.0 * oracle_float32_error(self.folder, tokens)[rows]
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
