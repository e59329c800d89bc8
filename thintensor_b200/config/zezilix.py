"""Typed configuration of the Zezilix decoder, read from its config.json.

config.json gives ``vocab``, ``width``, ``norm.eps``, ``streams`` (copies of the residual stream; absent: 1), ``residual_mult`` (what
every sublayer's output is multiplied by; absent: 1), ``loop`` (``start``, ``stop``, ``times``: layers ``start .. stop - 1`` run ``times``
times in a row; absent: every layer runs once) and ``layers``: a list whose entries name the layer's mixer (``type``:
``latent_attention``, ``latent_attention_2`` or ``wkv``), the mixer's sizes (``mixer``) and the feed-forward (``mlp``: ``{"kind":
"dense", "ff": n, "limit": c}``, ``{"kind": "moe", "expert": {"ff": n}, "router": {"experts": E, "top": k, "scale": s}}``, or null for
a layer without one).  The two kinds of latent attention differ in their queries and their output gate.  The rank of the
decays' product of low rank is not in config.json but in the tensors' shapes.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any

from .base import ConfigError
from .famalorn import _float, _int
from .neruzen import Rotation
from .zuvepel import Loop

ARCHITECTURE = "Zezilix"


@dataclass(frozen=True)
class LatentAttentionSizes:
    heads: int
    dim: int                # unrotated query/key numbers per head
    rot_dim: int            # rotated query/key numbers per head; the key's are shared by all heads
    vdim: int
    kv_rank: int
    scale: float
    rot: Rotation | None
    q_rank: int | None      # None: direct queries

    @staticmethod
    def from_dict(raw: dict, where: str, low_rank_queries: bool) -> "LatentAttentionSizes":
        rot_dim = _int(raw, "rot_dim", where)
        return LatentAttentionSizes(_int(raw, "heads", where), _int(raw, "dim", where), rot_dim, _int(raw, "vdim", where),
                                    _int(raw, "kv_rank", where), _float(raw, "scale", where),
                                    Rotation.from_dict(raw.get("rot"), where + ".rot", rot_dim),
                                    _int(raw, "q_rank", where) if low_rank_queries else None)

    def to_dict(self) -> dict:
        out: dict[str, Any] = {"dim": self.dim, "heads": self.heads, "kv_rank": self.kv_rank}
        if self.q_rank is not None:
            out["q_rank"] = self.q_rank
        if self.rot is not None:
            out["rot"] = self.rot.to_dict()
        out.update({"rot_dim": self.rot_dim, "scale": self.scale, "vdim": self.vdim})
        return out


@dataclass(frozen=True)
class WkvSizes:
    heads: int
    dim: int                # of a head's receptances, keys and values alike

    @staticmethod
    def from_dict(raw: dict, where: str) -> "WkvSizes":
        return WkvSizes(_int(raw, "heads", where), _int(raw, "dim", where))

    def to_dict(self) -> dict:
        return {"dim": self.dim, "heads": self.heads}


@dataclass(frozen=True)
class DenseSizes:
    ff: int
    limit: float            # the clamp of the gated unit

    @staticmethod
    def from_dict(raw: dict, where: str) -> "DenseSizes":
        sizes = DenseSizes(_int(raw, "ff", where), _float(raw, "limit", where))
        if sizes.limit <= 0.0:
            raise ConfigError(f"config.json: {where}: the limit is positive, got {sizes.limit}")
        return sizes

    def to_dict(self) -> dict:
        return {"ff": self.ff, "kind": "dense", "limit": self.limit}


@dataclass(frozen=True)
class MoeSizes:
    experts: int
    top: int
    ff: int
    scale: float            # of the chosen experts' scores

    @staticmethod
    def from_dict(raw: dict, where: str) -> "MoeSizes":
        router, expert = raw.get("router"), raw.get("expert")
        if not isinstance(router, dict) or not isinstance(expert, dict):
            raise ConfigError(f"config.json: {where} needs 'router' and 'expert'")
        sizes = MoeSizes(_int(router, "experts", where + ".router"), _int(router, "top", where + ".router"), _int(expert, "ff", where + ".expert"),
                         _float(router, "scale", where + ".router") if router.get("scale") is not None else 1.0)
        if sizes.top > sizes.experts:
            raise ConfigError(f"config.json: {where}: top {sizes.top} of {sizes.experts} experts")
        return sizes

    def to_dict(self) -> dict:
        return {"expert": {"ff": self.ff}, "kind": "moe", "router": {"experts": self.experts, "scale": self.scale, "top": self.top}}


MIXER_TYPES = ("latent_attention", "latent_attention_2", "wkv")


@dataclass(frozen=True)
class ZezilixLayer:
    type: str
    mixer: Any              # LatentAttentionSizes or WkvSizes
    mlp: Any                # DenseSizes, MoeSizes, or None: the layer has no feed-forward

    def to_dict(self) -> dict:
        return {"mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict(), "type": self.type}


@dataclass(frozen=True)
class ZezilixConfig:
    vocab: int
    width: int
    eps: float
    layers: tuple[ZezilixLayer, ...]
    streams: int = 1
    residual_mult: float = 1.0
    loop: Loop | None = None
    eos_token_ids: tuple[int, ...] = ()
    architecture: str = ARCHITECTURE

    @staticmethod
    def from_dict(raw: dict[str, Any]) -> "ZezilixConfig":
        norm = raw.get("norm")
        if not isinstance(norm, dict):
            raise ConfigError("config.json is missing the 'norm' entry with its eps")
        entries = raw.get("layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError("config.json needs a non-empty list 'layers'")
        layers: list[ZezilixLayer] = []
        for index, entry in enumerate(entries):
            where = f"layers[{index}]"
            kind = entry.get("type") if isinstance(entry, dict) else None
            if kind not in MIXER_TYPES:
                raise ConfigError(f"config.json: {where} has type {kind!r}; known: {', '.join(MIXER_TYPES)}")
            if not isinstance(entry.get("mixer"), dict):
                raise ConfigError(f"config.json: {where} needs the sizes of its mixer")
            mixer = (WkvSizes.from_dict(entry["mixer"], where + ".mixer") if kind == "wkv"
                     else LatentAttentionSizes.from_dict(entry["mixer"], where + ".mixer", kind == "latent_attention"))
            mlp = entry.get("mlp")
            if mlp is None:
                feed = None
            elif isinstance(mlp, dict) and mlp.get("kind") == "dense":
                feed = DenseSizes.from_dict(mlp, where + ".mlp")
            elif isinstance(mlp, dict) and mlp.get("kind") == "moe":
                feed = MoeSizes.from_dict(mlp, where + ".mlp")
            else:
                raise ConfigError(f"config.json: {where}.mlp must be null or of kind 'dense' or 'moe'")
            layers.append(ZezilixLayer(kind, mixer, feed))
        loop = None
        if raw.get("loop"):
            loop = Loop(*(_int(raw["loop"], key, "loop", least) for key, least in (("start", 0), ("stop", 1), ("times", 1))))
            if not loop.start < loop.stop <= len(layers):
                raise ConfigError(f"config.json: loop runs layers {loop.start} .. {loop.stop - 1} of {len(layers)}")
        eos = raw.get("eos_token_id")
        eos_ids = () if eos is None else tuple(int(e) for e in (eos if isinstance(eos, (list, tuple)) else [eos]))
        return ZezilixConfig(_int(raw, "vocab", "the model"), _int(raw, "width", "the model"), _float(norm, "eps", "norm"), tuple(layers),
                             _int(raw, "streams", "the model") if raw.get("streams") is not None else 1,
                             _float(raw, "residual_mult", "the model") if raw.get("residual_mult") is not None else 1.0, loop, eos_ids)

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = {"architecture": self.architecture, "layers": [layer.to_dict() for layer in self.layers]}
        if self.loop is not None:
            out["loop"] = self.loop.to_dict()
        out.update({"norm": {"eps": self.eps}, "residual_mult": self.residual_mult, "streams": self.streams, "vocab": self.vocab,
                    "width": self.width})
        if self.eos_token_ids:
            out["eos_token_id"] = list(self.eos_token_ids)
        return out
