"""Typed configuration of the Zuvepel decoder, read from its config.json.

config.json gives ``vocab``, ``width``, ``norm.eps``, ``residual_mult`` (what both sublayers' outputs are multiplied by; absent:
1), ``embedding.scale`` (the token rows' factor; absent: 1), ``loop`` (``start``, ``stop``, ``times``: layers ``start .. stop - 1`` run
``times`` times in a row; absent: every layer runs once) and ``layers``: a list whose entries name the layer's mixer (``type``:
``attention``, ``channel_delta`` or ``gla``), the mixer's sizes (``mixer``) and the feed-forward (``mlp``: ``{"kind": "dense", "ff": n}``,
or null for a layer without one).  An attention mixer's ``mask.size`` is the size of the chunks a position's keys come from
(absent: all keys), its ``rot`` the rotation (absent: none).  Ranks of products of low rank are not in config.json but in the
tensors' shapes.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any

from .base import ConfigError
from .famalorn import _float, _int
from .kerepel import DenseSizes
from .neruzen import Rotation

ARCHITECTURE = "Zuvepel"


def _kv_heads(raw: dict, heads: int, where: str) -> int:
    kv_heads = _int(raw, "kv_heads", where) if raw.get("kv_heads") is not None else heads
    if heads % kv_heads:
        raise ConfigError(f"config.json: {where}: {heads} heads are not a multiple of {kv_heads} key/value heads")
    return kv_heads


@dataclass(frozen=True)
class AttentionSizes:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int | None           # mask.size; None: every earlier position is seen
    rot: Rotation | None

    @staticmethod
    def from_dict(raw: dict, where: str) -> "AttentionSizes":
        heads, dim, mask = _int(raw, "heads", where), _int(raw, "dim", where), raw.get("mask")
        return AttentionSizes(heads, _kv_heads(raw, heads, where), dim, _int(raw, "vdim", where), _float(raw, "scale", where),
                              _int(mask, "size", where + ".mask") if mask else None, Rotation.from_dict(raw.get("rot"), where + ".rot", dim))

    def to_dict(self) -> dict:
        out: dict[str, Any] = {"dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads}
        if self.chunk is not None:
            out["mask"] = {"size": self.chunk}
        if self.rot is not None:
            out["rot"] = self.rot.to_dict()
        out.update({"scale": self.scale, "vdim": self.vdim})
        return out


@dataclass(frozen=True)
class ChannelDeltaSizes:
    heads: int
    kv_heads: int               # query/key heads
    dim: int
    vdim: int
    conv: int                   # taps of the short convolutions

    @staticmethod
    def from_dict(raw: dict, where: str) -> "ChannelDeltaSizes":
        heads = _int(raw, "heads", where)
        return ChannelDeltaSizes(heads, _kv_heads(raw, heads, where), _int(raw, "dim", where), _int(raw, "vdim", where), _int(raw, "conv", where))

    def to_dict(self) -> dict:
        return {"conv": self.conv, "dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "vdim": self.vdim}


@dataclass(frozen=True)
class GlaSizes:
    heads: int
    dim: int
    vdim: int
    tau: float

    @staticmethod
    def from_dict(raw: dict, where: str) -> "GlaSizes":
        sizes = GlaSizes(_int(raw, "heads", where), _int(raw, "dim", where), _int(raw, "vdim", where), _float(raw, "tau", where))
        if sizes.tau <= 0.0:
            raise ConfigError(f"config.json: {where}: tau is positive, got {sizes.tau}")
        return sizes

    def to_dict(self) -> dict:
        return {"dim": self.dim, "heads": self.heads, "tau": self.tau, "vdim": self.vdim}


MIXERS = {"attention": AttentionSizes, "channel_delta": ChannelDeltaSizes, "gla": GlaSizes}


@dataclass(frozen=True)
class ZuvepelLayer:
    type: str
    mixer: Any                  # AttentionSizes, ChannelDeltaSizes or GlaSizes
    mlp: DenseSizes | None      # None: the layer has no feed-forward

    def to_dict(self) -> dict:
        return {"mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict(), "type": self.type}


@dataclass(frozen=True)
class Loop:
    start: int
    stop: int
    times: int

    def to_dict(self) -> dict:
        return {"start": self.start, "stop": self.stop, "times": self.times}


@dataclass(frozen=True)
class ZuvepelConfig:
    vocab: int
    width: int
    eps: float
    layers: tuple[ZuvepelLayer, ...]
    residual_mult: float = 1.0
    embedding_scale: float = 1.0
    loop: Loop | None = None
    eos_token_ids: tuple[int, ...] = ()
    architecture: str = ARCHITECTURE

    @staticmethod
    def from_dict(raw: dict[str, Any]) -> "ZuvepelConfig":
        norm = raw.get("norm")
        if not isinstance(norm, dict):
            raise ConfigError("config.json is missing the 'norm' entry with its eps")
        entries = raw.get("layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError("config.json needs a non-empty list 'layers'")
        layers: list[ZuvepelLayer] = []
        for index, entry in enumerate(entries):
            where = f"layers[{index}]"
            kind = entry.get("type") if isinstance(entry, dict) else None
            if kind not in MIXERS:
                raise ConfigError(f"config.json: {where} has type {kind!r}; known: {', '.join(MIXERS)}")
            if not isinstance(entry.get("mixer"), dict):
                raise ConfigError(f"config.json: {where} needs the sizes of its mixer")
            mlp = entry.get("mlp")
            if mlp is not None and not (isinstance(mlp, dict) and mlp.get("kind") == "dense"):
                raise ConfigError(f"config.json: {where}.mlp must be null or of kind 'dense'")
            layers.append(ZuvepelLayer(kind, MIXERS[kind].from_dict(entry["mixer"], where + ".mixer"),
                                       None if mlp is None else DenseSizes(_int(mlp, "ff", where + ".mlp"))))
        loop = None
        if raw.get("loop"):
            loop = Loop(*(_int(raw["loop"], key, "loop", least) for key, least in (("start", 0), ("stop", 1), ("times", 1))))
            if not loop.start < loop.stop <= len(layers):
                raise ConfigError(f"config.json: loop runs layers {loop.start} .. {loop.stop - 1} of {len(layers)}")
        embedding = raw.get("embedding") or {}
        eos = raw.get("eos_token_id")
        eos_ids = () if eos is None else tuple(int(e) for e in (eos if isinstance(eos, (list, tuple)) else [eos]))
        return ZuvepelConfig(_int(raw, "vocab", "the model"), _int(raw, "width", "the model"), _float(norm, "eps", "norm"), tuple(layers),
                             _float(raw, "residual_mult", "the model") if raw.get("residual_mult") is not None else 1.0,
                             _float(embedding, "scale", "embedding") if embedding.get("scale") is not None else 1.0, loop, eos_ids)

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = {"architecture": self.architecture, "embedding": {"scale": self.embedding_scale},
                               "layers": [layer.to_dict() for layer in self.layers]}
        if self.loop is not None:
            out["loop"] = self.loop.to_dict()
        out.update({"norm": {"eps": self.eps}, "residual_mult": self.residual_mult, "vocab": self.vocab, "width": self.width})
        if self.eos_token_ids:
            out["eos_token_id"] = list(self.eos_token_ids)
        return out
