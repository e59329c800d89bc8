"""How a layer's parts are wired around the residual stream.

``pre_norm``: ``h += mixer(norm(h)); h += ffn(norm(h))``, the order of
thinruntime/gpu_runtime.py:10114-10390.  The residual stream is float32; a part's
output is handed on as a :class:`Delta` and added by the next norm's kernel, so the
layer's second addition is done by the following layer's first norm (or by the final
norm).  For long prompts the output projections add their product into the stream themselves
(their tensor-core kernel's epilogue reads and writes the tile once, which spares the
norm kernel a read of the product and a write of the stream); the delta is then empty.

``sandwich``: every sublayer stands between two norms, ``h += norm_after(mixer(norm_before(h)))`` and the same for the
feed-forward, and the layer's end may mix the results of all layers so far into the stream that goes on.  The norm
after a sublayer and the mixing are not kernels of their own: the delta that the sublayer hands on says what is to be
done with it, and the next norm's kernel does it on its way (the layer's last delta reaches the next layer's first
norm, or the final norm).
"""
from __future__ import annotations

from dataclasses import replace

import torch

from ..kernels import api
from .base import ARRANGEMENTS, Arrangement, Delta, DepthStep, StreamStep


@ARRANGEMENTS.register("pre_norm")
class PreNorm(Arrangement):
    """A layer without a feed-forward leaves out ``ffn_norm`` and ``ffn``: its mixer's output is then what the next
    layer's norm adds.  ``side`` (optional): a side input at the layer's end, which reads the stream with the last
    sublayer's output added and hands on what it adds itself.  ``scale`` (a constant) and ``mixer_scale`` / ``ffn_scale`` (factors
    per channel) multiply a sublayer's output before the stream takes it.  ``mixer_streams`` / ``ffn_streams``: the stream comes in
    several copies (the model's ``streams``), which each sublayer reads and writes with weights of its own."""

    roles = {"mixer_norm": "norm", "mixer": "mixer", "mixer_scale": "scale", "mixer_streams": "streams", "ffn_norm": "norm", "ffn": "ffn",
             "ffn_scale": "scale", "ffn_streams": "streams", "side": "side"}
    optional = ("mixer_scale", "mixer_streams", "ffn_norm", "ffn", "ffn_scale", "ffn_streams", "side")

    def __init__(self, parts, scale: float = 1.0):
        super().__init__(parts)
        if ("ffn" in parts) != ("ffn_norm" in parts):
            raise ValueError("a pre-norm layer has a feed-forward and its norm, or neither")
        if "ffn" not in parts and ("ffn_scale" in parts or "ffn_streams" in parts):
            raise ValueError("a scale or stream weights of a feed-forward go with one")
        if "ffn" in parts and ("mixer_streams" in parts) != ("ffn_streams" in parts):
            raise ValueError("both sublayers read and write the streams with weights of their own, or neither does")
        self.scale = float(scale)
        self.plain = self.scale == 1.0 and not {"mixer_scale", "mixer_streams", "ffn_scale", "ffn_streams"} & set(parts)
        if "side" in parts and not self.plain:
            raise ValueError("a side input goes with a single stream and unscaled sublayers")

    def mixers(self):
        return [self.parts["mixer"]]

    def device_driven(self) -> bool:
        return all(part.device_driven() for part in self.parts.values())

    def run(self, ctx, residual, pending: Delta | None, caches, states) -> Delta:
        hidden = residual.shape[-1]
        # Between a part's output and the norm that follows nothing else reads the stream, so a part
        # may add its output into it directly instead of handing it on (not one that is scaled or mixed on its way).
        ctx.residual = residual if self.plain else None
        normed = ctx.scratch("block.normed", (ctx.n_tokens, hidden))
        self.parts["mixer_norm"].forward(ctx, residual, self.reading("mixer", pending), normed)
        last = self.written("mixer", self.parts["mixer"].forward(ctx, normed, caches[0], states[0]))
        if "ffn" in self.parts:
            self.parts["ffn_norm"].forward(ctx, residual, self.reading("ffn", last), normed)
            last = self.written("ffn", self.parts["ffn"].forward(ctx, normed))
        if "side" in self.parts:
            last = self.parts["side"].forward(ctx, residual, last)
        return last

    def reading(self, sublayer: str, pending: Delta | None) -> Delta | None:
        """The pending delta with the weights with which this sublayer's norm reads the streams."""
        streams = self.parts.get(sublayer + "_streams")
        if streams is None:
            return pending
        pending = pending or Delta(None)
        return replace(pending, streams=replace(pending.streams or StreamStep(), read=streams.read))

    def written(self, sublayer: str, delta: Delta) -> Delta:
        """The sublayer's output with its factors and the weights with which the streams take it."""
        if self.plain:
            return delta
        scale, streams = self.parts.get(sublayer + "_scale"), self.parts.get(sublayer + "_streams")
        return Delta(delta.tensor, scale=self.scale, gain=None if scale is None else scale.weight,
                     streams=None if streams is None else StreamStep(streams.mix, streams.write))


@ARRANGEMENTS.register("pre_norm_pair")
class PreNormPair(Arrangement):
    """Two mixers side by side on the same normed input, ``h += left_scale * left(norm(h)) + right_scale *
    right(norm(h))``, then the feed-forward sublayer (if the layer has one).  Each mixer has a cache and states of
    its own.  The weighted sum is formed in float32 from the two output projections' partial sums."""

    roles = {"mixer_norm": "norm", "left": "mixer", "right": "mixer", "ffn_norm": "norm", "ffn": "ffn"}
    optional = ("ffn_norm", "ffn")

    def __init__(self, parts, left_scale: float = 1.0, right_scale: float = 1.0):
        super().__init__(parts)
        if ("ffn" in parts) != ("ffn_norm" in parts):
            raise ValueError("a pre-norm layer has a feed-forward and its norm, or neither")
        self.left_scale, self.right_scale = float(left_scale), float(right_scale)

    def mixers(self):
        return [self.parts["left"], self.parts["right"]]

    def device_driven(self) -> bool:
        return all(part.device_driven() for part in self.parts.values())

    def run(self, ctx, residual, pending: Delta | None, caches, states) -> Delta:
        hidden = residual.shape[-1]
        normed = ctx.scratch("block.normed", (ctx.n_tokens, hidden))
        self.parts["mixer_norm"].forward(ctx, residual, pending, normed)
        ctx.residual = None                 # the branches' outputs are weighted before they reach the stream
        left = self.parts["left"].forward(ctx, normed, caches[0], states[0])
        right = self.parts["right"].forward(ctx, normed, caches[1], states[1])
        both = ctx.scratch("block.pair", (1, ctx.n_tokens, hidden), torch.float32)
        api.weighted_pair(left.tensor, self.left_scale, right.tensor, self.right_scale, both)
        mixed = Delta(both)
        if "ffn" not in self.parts:
            return mixed
        ctx.residual = residual
        self.parts["ffn_norm"].forward(ctx, residual, mixed, normed)
        return self.parts["ffn"].forward(ctx, normed)


@ARRANGEMENTS.register("parallel")
class Parallel(Arrangement):
    """Both sublayers read the same stream: ``h = norm(x); x += scale * (mixer(shift(h)) + ffn(h))``.  ``shift`` (an input
    shift, optional) stands between the norm and the mixer only; the feed-forward (optional) reads ``h`` as it is, or, with
    an ``ffn_norm``, the stream through a norm of its own (the two norms are then one kernel where their kinds allow).  The
    shift's per-sequence state is the arrangement's own."""

    roles = {"norm": "norm", "shift": "shift", "mixer": "mixer", "ffn_norm": "norm", "ffn": "ffn"}
    optional = ("shift", "ffn_norm", "ffn")

    def __init__(self, parts, scale: float = 1.0):
        super().__init__(parts)
        if "ffn_norm" in parts and "ffn" not in parts:
            raise ValueError("a parallel layer's second norm belongs to its feed-forward")
        self.scale = float(scale)

    def mixers(self):
        return [self.parts["mixer"]]

    def state_needs(self):
        return list(self.parts["shift"].state_needs()) if "shift" in self.parts else []

    def device_driven(self) -> bool:
        return all(part.device_driven() for part in self.parts.values())

    def run(self, ctx, residual, pending: Delta | None, caches, states) -> Delta:
        hidden = residual.shape[-1]
        normed = ctx.scratch("block.normed", (ctx.n_tokens, hidden))
        ffn_in = normed
        if "ffn_norm" in self.parts:
            ffn_in = ctx.scratch("block.ffn_normed", (ctx.n_tokens, hidden))
            self.parts["norm"].forward_pair(ctx, residual, pending, normed, self.parts["ffn_norm"], ffn_in)
        else:
            self.parts["norm"].forward(ctx, residual, pending, normed)
        # both sublayers read normed rows and nothing reads the stream before the next norm, so either may add into it
        # (not where the sum has a factor)
        ctx.residual = residual if self.scale == 1.0 else None
        mixer_in = self.parts["shift"].forward(ctx, normed, states[1]) if "shift" in self.parts else normed
        mixed = self.parts["mixer"].forward(ctx, mixer_in, caches[0], states[0])
        if "ffn" not in self.parts:
            return Delta(mixed.tensor, scale=self.scale)
        fed = self.parts["ffn"].forward(ctx, ffn_in)
        if mixed.tensor is None:
            return Delta(fed.tensor, scale=self.scale)
        return Delta(mixed.tensor, second=fed.tensor, scale=self.scale)       # the next norm's kernel adds the two


@ARRANGEMENTS.register("sandwich")
class Sandwich(Arrangement):
    """``h += post(mixer(pre(h))); h += post'(ffn(pre'(h)))`` with four norms (the feed-forward and its two may be left
    out).  With a ``depth`` part the stream at the layer's end is kept as result ``result_index`` of ``results`` (the
    embedding's output is result 0, kept by the first layer before its first norm) and replaced by the weighted sum of
    results ``0 .. result_index``.  A sublayer's output is normalised before the stream takes it, so no part may add
    into the stream itself."""

    roles = {"mixer_norm": "norm", "mixer": "mixer", "mixer_post_norm": "norm", "ffn_norm": "norm", "ffn": "ffn", "ffn_post_norm": "norm",
             "depth": "depth"}
    optional = ("ffn_norm", "ffn", "ffn_post_norm", "depth")

    def __init__(self, parts, result_index: int = 0, results: int = 0):
        super().__init__(parts)
        present = [role in parts for role in ("ffn_norm", "ffn", "ffn_post_norm")]
        if any(present) and not all(present):
            raise ValueError("a sandwich layer has a feed-forward and both of its norms, or none of the three")
        self.result_index, self.results = int(result_index), int(results)
        if "depth" in parts and not 1 <= self.result_index < self.results:
            raise ValueError(f"a layer that mixes results needs its place among them, got {result_index} of {results}")

    def mixers(self):
        return [self.parts["mixer"]]

    def device_driven(self) -> bool:
        return all(part.device_driven() for part in self.parts.values())

    def run(self, ctx, residual, pending: Delta | None, caches, states) -> Delta:
        hidden = residual.shape[-1]
        ctx.residual = None                     # outputs pass a norm before the stream takes them
        depth = self.parts.get("depth")
        kept = None
        if depth is not None:
            kept = ctx.scratch("model.results", (self.results, ctx.n_tokens, hidden), torch.float32)
            if pending is None:                 # the first layer: the embedding's output is result 0
                pending = Delta(None, depth=DepthStep(kept, 0, None))
        normed = ctx.scratch("block.normed", (ctx.n_tokens, hidden))
        self.parts["mixer_norm"].forward(ctx, residual, pending, normed)
        last = self.parts["mixer"].forward(ctx, normed, caches[0], states[0])
        last = Delta(last.tensor, post=self.parts["mixer_post_norm"].after())
        if "ffn" in self.parts:
            self.parts["ffn_norm"].forward(ctx, residual, last, normed)
            last = self.parts["ffn"].forward(ctx, normed)
            last = Delta(last.tensor, post=self.parts["ffn_post_norm"].after())
        if depth is not None:
            last.depth = DepthStep(kept, self.result_index, depth.weight)
        return last
