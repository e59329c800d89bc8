"""Interfaces of the parts a layer is made of, and one registry for each role.

A part is built from the parameters of its :class:`~thintensor_b200.parts.spec.PartSpec`
alone.  It declares the tensors it needs under names of its own, is handed those
tensors once, and is then run with a :class:`~thintensor_b200.engine.context.StepContext`.
No part knows which model it is in, which layer it is, or what the checkpoint calls
its tensors.

Roles and what each must provide:

* ``Norm``: ``forward(ctx, residual, delta, out, rows=None)`` adds ``delta`` (the not
  yet added output of the part before it, possibly several partial sums) into the
  float32 residual stream and writes the normalised rows to ``out``.
* ``PositionEncoding``: an object a mixer is given at construction.  Its ``kind`` says how
  positions enter the mixer (``"rotary"``: queries and keys are rotated, the mixer's kernels
  take the table that ``rotary()`` returns; ``"none"``); a mixer refuses kinds it cannot apply.
* ``Mixer``: ``forward(ctx, x, cache, states) -> Delta``; declares with ``cache_need()`` /
  ``state_needs()`` what the cache must hold for it: keys and values, and any number of
  per-sequence state tensors of fixed size, each with a shape and dtype of its own.
* ``FeedForward``: ``forward(ctx, x) -> Delta``.
* ``Embedding``: ``forward(ctx, tokens, residual, states)``; it may declare per-sequence states like a mixer
  (the previous token, say).  ``Head``: ``forward(ctx, x) -> logits``.
* ``InputShift``: ``forward(ctx, x, states) -> tensor``: what a mixer reads instead of the normed rows themselves
  (a blend with the previous token's rows, kept as a per-sequence state).
* ``SideInput``: ``forward(ctx, residual, pending) -> Delta``: what a layer adds at its end from the stream itself and the
  step's tokens (a gated slice of a second token embedding, say).
* ``DepthMix``: the weights with which a layer's end mixes the results of the layers so far (``weights()`` only; the
  arrangement hands them to the norm that follows).
* ``StreamMix``: the weights with which a sublayer reads and writes a residual stream that comes in several copies, and
  ``Scale``: a factor per channel on a sublayer's output (both ``weights()`` only, for the norm kernels as well).
* ``Arrangement``: wires norms, mixer and feed-forward around the residual stream.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Callable

import torch


@dataclass(frozen=True)
class WeightDecl:
    """A tensor a part needs.  ``init`` tells the random-weights mode how to draw it:
    ``normal`` is N(0, 0.02), ``norm`` is 1 + N(0, 0.1), ``small`` is N(0, 0.1), ``depth`` is N(0, 0.3) with one added to the last number,
    ``identity`` is N(0, 0.1) with one added on the diagonal of a square matrix, ``zeros`` is zero.  ``free`` lists axes whose extent the checkpoint decides (the rank of a product of low rank, say); ``shape``
    then holds what random weights are drawn with, and the part reads the real extent off the tensor it is bound to.
    ``alias_of`` names a checkpoint tensor (full name) to use instead when this one is
    absent from the checkpoint; with ``prefer_alias`` it is used even when this one is
    stored (a tied output head, whose stored copy is ignored)."""

    shape: tuple[int, ...]
    init: str = "normal"
    optional: bool = False
    alias_of: str | None = None
    prefer_alias: bool = False
    integer: bool = False
    free: tuple[int, ...] = ()

    def fits(self, shape) -> bool:
        return len(shape) == len(self.shape) and all(have == want or (axis in self.free and have > 0)
                                                     for axis, (have, want) in enumerate(zip(shape, self.shape)))


@dataclass(frozen=True)
class KVNeed:
    """Keys and values a mixer wants kept for each sequence: ``kv_heads`` heads of
    ``head_dim`` numbers per token (values: ``value_dim``, if given; 0: no value pool at all, for a mixer whose
    values are read out of the key rows, like a shared latent); ``window`` = only the last so many tokens."""

    kv_heads: int
    head_dim: int
    window: int | None = None
    value_dim: int | None = None        # numbers per value head where they differ from the keys' (None: head_dim)
    every: int = 1                      # one entry for each ``every`` tokens: entry n belongs to tokens n * every .. n * every + every - 1

    @property
    def v_dim(self) -> int:
        return self.head_dim if self.value_dim is None else self.value_dim


@dataclass(frozen=True)
class StateNeed:
    """Per-sequence state of fixed size: one tensor of ``shape`` and ``dtype`` for each
    sequence, zero when the sequence starts."""

    shape: tuple[int, ...]
    dtype: torch.dtype = torch.float32


@dataclass(frozen=True)
class PostNorm:
    """An RMS norm applied to a sublayer's output before the stream takes it: ``v / sqrt(mean(v^2) + eps) * (weight + offset)``."""

    weight: torch.Tensor        # float32 [hidden]
    eps: float
    offset: float = 0.0


@dataclass(frozen=True)
class DepthStep:
    """The stream after the addition is result ``index`` of ``results`` (float32 ``[count, tokens, hidden]``; result 0 is the
    embedding's output); what goes on is ``sum(weights[j] * results[j] for j <= index)``.  Without ``weights`` the
    stream is only kept (the embedding's output, before the first layer)."""

    results: torch.Tensor
    index: int
    weights: torch.Tensor | None    # float32 [index + 1]


@dataclass(frozen=True)
class StreamStep:
    """A residual stream in several copies ``x_s`` (float32 ``[streams, tokens, hidden]``).  With y the sublayer's output (after its
    scales), copy t becomes ``sum(mix[s, t] * x_s) + write[t] * y`` and what the norm takes is ``sum(read[t] * x_t)`` of the new
    copies.  ``mix`` None: the copies stay; ``write`` / ``read`` None: ones.  ``spread``: only the first copy is there so far (the
    embedding's output), and the others start equal to it."""

    mix: torch.Tensor | None = None     # float32 [streams, streams], from (row) and to (column)
    write: torch.Tensor | None = None   # float32 [streams]
    read: torch.Tensor | None = None    # float32 [streams]
    spread: bool = False


@dataclass
class Delta:
    """What a mixer or feed-forward adds to the residual stream: float32
    ``[splits, tokens, hidden]``; the sum over ``splits`` is the value.  The norm that
    follows does the sum and the addition.  ``tensor`` is None when the part has already
    added its result into the stream itself (``ctx.residual``, where the arrangement offers it).

    ``post``: the sum is normalised (RMS norm with this weight) before it is added.  ``depth``: after the
    addition the stream is kept as a layer's result and replaced by a weighted sum of the results so far.
    Both are carried out by the norm that follows, in its one pass over the row.

    ``gain`` (float32 ``[hidden]``) multiplies the sum channel by channel.  ``streams``: the stream comes in several copies, into
    which the sum goes and from which the norm that follows reads as the step says.

    ``second``: another sublayer's partial sums, added to the first's.  ``scale`` multiplies both.  ``addend`` (float32
    ``[tokens, hidden]``) is added as it is.  The norm that follows does these too."""

    tensor: torch.Tensor | None
    post: "PostNorm | None" = None
    depth: "DepthStep | None" = None
    second: torch.Tensor | None = None
    scale: float = 1.0
    addend: torch.Tensor | None = None
    gain: torch.Tensor | None = None
    streams: "StreamStep | None" = None

    @property
    def plain(self) -> bool:
        """Whether the delta is nothing but the sum of ``tensor``."""
        return self.post is None and self.depth is None and not self.branched and not self.streamed

    @property
    def streamed(self) -> bool:
        """Whether the delta goes through the kernel for scaled outputs and several streams."""
        return self.gain is not None or self.streams is not None

    @property
    def branched(self) -> bool:
        return self.second is not None or self.scale != 1.0 or self.addend is not None

    @property
    def splits(self) -> int:
        return 0 if self.tensor is None else self.tensor.shape[0]


class Part:
    """Common behaviour: declared weights and binding."""

    def weights(self) -> dict[str, WeightDecl]:
        return {}

    def bind(self, tensors: dict[str, torch.Tensor], dtype: torch.dtype, device: torch.device) -> None:
        """Receive the declared tensors (already on ``device``, in their stored dtype
        unless the engine runs in float32, ``dtype`` being the activation dtype) and
        prepare what kernels need."""

    def projections(self) -> list:
        """The part's weight matrices as :class:`~thintensor_b200.parts.linear.Linear` objects, each
        listed once and each multiplied with every token once per step: what the byte and FLOP
        models of the benchmarks count.  A view of another projection's rows is not listed."""
        return []

    def vectors(self) -> list[torch.Tensor]:
        """Other tensors a step reads once whatever its tokens (a norm's weight)."""
        return []

    def device_driven(self) -> bool:
        """Whether ``forward`` takes everything that changes from step to step from device memory
        (``ctx.tokens``, ``ctx.cu``, ``ctx.len_before``, ``ctx.slots``, the block tables) and, for steps
        of one shape (tokens, sequences, table width, wanted rows), launches the same kernels with
        the same host-side arguments.  Such a step can be captured in a CUDA graph once and
        replayed; a part that looks at ``ctx.host_slots`` / ``host_new`` / ``host_before`` or
        computes on the host must say no.  The engine replays only if every part says yes."""
        return False


class Norm(Part):
    def forward(self, ctx, residual: torch.Tensor, delta: Delta | None, out: torch.Tensor, rows: torch.Tensor | None = None) -> None:
        raise NotImplementedError

    def forward_pair(self, ctx, residual: torch.Tensor, delta: Delta | None, out: torch.Tensor, other: "Norm", other_out: torch.Tensor) -> None:
        """Add ``delta`` into the stream and take two norms of it, this one and ``other``.  Norms that can share one pass
        over a row override this."""
        self.forward(ctx, residual, delta, out)
        other.forward(ctx, residual, None, other_out)


@dataclass(frozen=True)
class RotaryTable:
    """What a kernel needs to rotate queries and keys: ``inv_freq`` float32 ``[rotary_dim / 2]`` on
    the device (the angle of pair i at position p is ``p * inv_freq[i]``), ``rotary_dim`` numbers at
    the front of each head are rotated (0: none), cosine and sine are multiplied by
    ``attention_scaling``.  ``signature`` identifies the table's contents."""

    inv_freq: torch.Tensor
    rotary_dim: int
    attention_scaling: float = 1.0
    signature: int = 0      # equal for tables with equal numbers (0: unknown): layers with equal tables can share what a step derives from them
    interleaved: bool = False   # pairs are (2i, 2i + 1) instead of (i, i + rotary_dim / 2)


class PositionEncoding(Part):
    """``kind`` is one of ``"rotary"`` and ``"none"``.  A rotary encoding implements ``rotary()``
    (valid after ``bind``); other kinds of encoding (learned tables, additive biases) would add a
    kind and the method that goes with it, and the mixers that can apply it would accept the kind."""

    kind: str = "none"

    def rotary(self) -> RotaryTable:
        raise NotImplementedError(f"a position encoding of kind {self.kind!r} has no rotary table")


class Mixer(Part):
    def cache_need(self) -> KVNeed | None:
        return None

    def summary_need(self) -> KVNeed | None:
        """A second, coarser cache beside the mixer's keys and values: one key and one value for each ``every`` tokens
        (the means of whole blocks of tokens, say).  ``forward`` finds it as ``cache.summary``."""
        return None

    def state_needs(self) -> list[StateNeed]:
        """Per-sequence state tensors of fixed size, zero when a sequence starts; ``forward`` gets
        one tensor ``[slots, *shape]`` for each, in this order."""
        return []

    def forward(self, ctx, x: torch.Tensor, cache, states: list[torch.Tensor]) -> Delta:
        raise NotImplementedError


class FeedForward(Part):
    def forward(self, ctx, x: torch.Tensor) -> Delta:
        raise NotImplementedError


class Embedding(Part):
    def state_needs(self) -> list[StateNeed]:
        """Per-sequence state tensors of fixed size, zero when a sequence starts (see :meth:`Mixer.state_needs`)."""
        return []

    def forward(self, ctx, tokens: torch.Tensor, residual: torch.Tensor, states: list[torch.Tensor] | None = None) -> None:
        raise NotImplementedError


class InputShift(Part):
    """Replaces a mixer's input rows by a function of them and of the rows of the tokens before."""

    def state_needs(self) -> list[StateNeed]:
        return []

    def forward(self, ctx, x: torch.Tensor, states: list[torch.Tensor]) -> torch.Tensor:
        raise NotImplementedError


class SideInput(Part):
    """Something a layer adds to the stream at its end that is no function of a norm of the stream: it reads the stream
    itself (with the layer's last delta added) and the step's tokens.  ``forward(ctx, residual, pending) -> Delta`` adds
    ``pending`` into the stream and returns what the next norm is to add."""

    def forward(self, ctx, residual: torch.Tensor, pending: "Delta | None") -> "Delta":
        raise NotImplementedError


class Head(Part):
    def forward(self, ctx, x: torch.Tensor) -> torch.Tensor:
        raise NotImplementedError


class Arrangement:
    """How one layer's parts are wired.  ``roles`` lists the part roles it needs and
    the registry each comes from; ``run`` returns the delta still to be added."""

    roles: dict[str, str] = {}
    optional: tuple[str, ...] = ()      # roles a layer may leave out

    def __init__(self, parts: dict[str, Part]):
        self.parts = parts

    def mixers(self) -> list[Mixer]:
        """The layer's mixers (a layer with an attention and a recurrent branch side by side has
        two); each gets a cache and states of its own."""
        return []

    def state_needs(self) -> list[StateNeed]:
        """Per-sequence states of the arrangement itself (of a part of its that is no mixer); ``run`` finds them
        behind the mixers': ``states[len(mixers())]``."""
        return []

    def run(self, ctx, residual: torch.Tensor, pending: Delta | None, caches: list, states: list[list[torch.Tensor]]) -> Delta | None:
        """``caches[i]`` and ``states[i]`` belong to ``mixers()[i]``; an arrangement with states of its own gets one
        more entry of each behind them."""
        raise NotImplementedError

    def device_driven(self) -> bool:
        """See :meth:`Part.device_driven`: an arrangement answers for itself and its parts."""
        return False


class Registry:
    """kind -> class, for one role."""

    def __init__(self, role: str):
        self.role = role
        self._classes: dict[str, Callable[..., Any]] = {}

    def register(self, kind: str):
        def decorate(cls):
            if kind in self._classes:
                raise ValueError(f"{self.role} {kind!r} is already registered")
            self._classes[kind] = cls
            return cls

        return decorate

    def unregister(self, kind: str) -> None:
        self._classes.pop(kind, None)

    def build(self, kind: str, params: dict[str, Any]):
        if kind not in self._classes:
            raise KeyError(f"no {self.role} of kind {kind!r}; registered: {', '.join(sorted(self._classes))}")
        return self._classes[kind](**params)

    def kinds(self) -> list[str]:
        return sorted(self._classes)


NORMS = Registry("norm")
POSITION_ENCODINGS = Registry("position encoding")
MIXERS = Registry("mixer")
FEED_FORWARDS = Registry("feed-forward")
DEPTH_MIXES = Registry("depth mix")
STREAM_MIXES = Registry("stream mix")
SCALES = Registry("scale")
EMBEDDINGS = Registry("embedding")
SHIFTS = Registry("input shift")
SIDES = Registry("side input")
HEADS = Registry("head")
ARRANGEMENTS = Registry("arrangement")

REGISTRIES = {
    "norm": NORMS,
    "position": POSITION_ENCODINGS,
    "mixer": MIXERS,
    "ffn": FEED_FORWARDS,
    "depth": DEPTH_MIXES,
    "streams": STREAM_MIXES,
    "scale": SCALES,
    "embedding": EMBEDDINGS,
    "shift": SHIFTS,
    "side": SIDES,
    "head": HEADS,
    "arrangement": ARRANGEMENTS,
}
