"""Residual streams in several copies, and factors on a sublayer's output.

``hyper`` (Zhu et al., "Hyper-Connections", in its static form): the stream comes in S copies.  A sublayer reads a weighted sum of
them, and afterwards every copy becomes a weighted sum of the old copies plus its own multiple of the sublayer's output.
``channel``: a factor per channel on a sublayer's output before the stream takes it.  Both parts only hold their numbers; the
arrangement hands them, as a :class:`~thintensor_b200.parts.base.Delta`, to the norm kernel that follows the sublayer, which
updates the copies, forms the next sublayer's input and norms it in one pass over the rows, in float32.
"""
from __future__ import annotations

import torch

from ..kernels import api
from .base import SCALES, STREAM_MIXES, Part, WeightDecl


@STREAM_MIXES.register("hyper")
class HyperConnection(Part):
    NAMES = {"read": "read", "write": "write", "mix": "mix"}

    def __init__(self, streams: int, names: dict | None = None):
        self.streams = int(streams)
        if not 1 <= self.streams <= api.MAX_STREAMS:
            raise ValueError(f"the kernels take 1 to {api.MAX_STREAMS} residual streams, not {streams}")
        self.names = {**self.NAMES, **(names or {})}
        self.read: torch.Tensor | None = None
        self.write: torch.Tensor | None = None
        self.mix: torch.Tensor | None = None

    def weights(self) -> dict[str, WeightDecl]:
        n = self.names
        return {n["read"]: WeightDecl((self.streams,), init="norm"), n["write"]: WeightDecl((self.streams,), init="norm"),
                n["mix"]: WeightDecl((self.streams, self.streams), init="identity")}

    def bind(self, tensors, dtype, device) -> None:
        self.read, self.write, self.mix = (tensors[self.names[key]].to(torch.float32).contiguous() for key in ("read", "write", "mix"))

    def vectors(self) -> list[torch.Tensor]:
        return [self.read, self.write, self.mix]

    def device_driven(self) -> bool:
        return True


@SCALES.register("channel")
class ChannelScale(Part):
    def __init__(self, dim: int, name: str = "scale"):
        self.dim, self.name = int(dim), name
        self.weight: torch.Tensor | None = None

    def weights(self) -> dict[str, WeightDecl]:
        return {self.name: WeightDecl((self.dim,), init="norm")}

    def bind(self, tensors, dtype, device) -> None:
        self.weight = tensors[self.name].to(torch.float32).contiguous()

    def vectors(self) -> list[torch.Tensor]:
        return [self.weight]

    def device_driven(self) -> bool:
        return True
