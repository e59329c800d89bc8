"""Recurrent token mixers: a state of fixed size per sequence instead of keys and values.

Both mixers here share one skeleton.  One matrix product makes everything that is linear in the
normed hidden state; a short causal convolution over time with silu follows on part of it; a
recurrence walks each sequence's tokens and reads out one vector per head; the read-out is gated
and divided by its root mean square in groups; the output projection follows.  What a sequence
carries from step to step are the recurrence's matrix per head (float32) and the last ``conv - 1``
inputs of the convolution (float32), both declared as states, so the cache hands them out per slot,
zeroed for a new sequence, and prompts cut into steps, decoding and batches all continue from them.

``mamba2``: the state-space recurrence of Mamba-2 (Dao and Gu, "Transformers are SSMs").  The input
projection is laid out [z | x | B | C | dt] (z and x ``heads * head_dim`` wide, B and C ``groups *
state`` wide, dt one number per head); x, B and C pass the convolution (with bias) and silu;
``dt = softplus(dt + dt_bias)``; per head, with S of shape state x head_dim,
``S <- exp(-exp(A_log) dt) S + dt B x^T`` and ``y = S^T C + D x``; then ``y * silu(z)`` is divided by
its root mean square in ``norm_groups`` equal parts and multiplied by the norm weight.

``gated_delta``: the gated delta rule (Yang, Kautz and Hatamizadeh, "Gated Delta Networks").  Queries
and keys (``qk_heads`` heads of ``key_dim``) and values (``heads`` heads of ``value_dim``) pass
convolutions of their own (no bias) and silu; q and k become unit vectors per head
(``x / sqrt(sum x^2 + 1e-6)``, q also times ``key_dim ** -0.5``); per head, with S of shape key_dim x
value_dim, ``S <- g S``, ``u = beta (v - S^T k)``, ``S <- S + k u^T``, ``o = S^T q`` with
``beta = sigmoid(W_b h)`` and ``g = exp(-exp(A_log) softplus(W_a h + dt_bias))``; each head's o is
divided by its root mean square, multiplied by a weight of ``value_dim`` numbers that the heads
share, and by ``silu(W_g h)``.  Options: a decay for every head and key channel from a product of low rank
(``channel_decay``), ``g = exp(-exp(A_log) softplus(W_a2 (W_a1 h) + dt_bias))`` with ``dt_bias`` and g laid out heads x key_dim
and A_log still one number per head, g multiplying the rows of S; a gate from a product of low rank (``low_rank_gate``),
``W_g2 (W_g1 h)``, and ``sigmoid`` instead of silu on it (``gate``).  The ranks are the checkpoint's.

``decay_linear_attention``: linear attention with a fixed decay per head and neither softmax nor
denominator: per head, with S of shape key_dim x value_dim, ``S <- decay_h S + k v^T`` and ``o = S^T q``.
Two published forms are parameter sets of it.  Lightning attention: ``activation="silu"`` on q, k and v,
the read-out of all heads RMS-normed together with a weight (``norm="all"``) and gated by
``sigmoid(W_g h)``.  Retention: q and k rotated by the position (``position``), k times
``key_dim ** -0.5`` (``key_scale``), every head's read-out divided by its own root mean square without a
weight (``norm="head"``) and gated by ``silu(W_g h)``.  With ``channel_decay`` the decay is not fixed but comes from the
token, one number per head and key channel, ``S <- diag(a) S + k v^T`` with ``a = sigmoid(W_a2 (W_a1 h) + b) ** (1 / tau)``: gated
linear attention (Yang, Wang, Shen, Panda and Kim, "Gated Linear Attention Transformers with Hardware-Efficient Training"),
q times ``query_scale``.  There is no convolution; the only state is S.

Decays, step sizes, gates of the recurrence, unit norms and the states are float32 whatever the
model's dtype; only the normed read-out that feeds the output projection is narrowed.
"""
from __future__ import annotations

import torch

from ..kernels import api
from .base import MIXERS, POSITION_ENCODINGS, Delta, Mixer, RotaryTable, StateNeed, WeightDecl
from .linear import Linear
from .spec import PartSpec


def _f32(t: torch.Tensor) -> torch.Tensor:
    return t.to(torch.float32).contiguous()


def _low_rank_decls(down: str, up: str, inputs: int, rank: int, outputs: int) -> dict[str, WeightDecl]:
    """A product of low rank, ``W_up (W_down h)``; the rank is the checkpoint's."""
    return {down: WeightDecl((rank, inputs), free=(0,)), up: WeightDecl((outputs, rank), free=(1,))}


class LowRankProduct:
    """The second half of a product of low rank, ``W_up`` on columns ``col ..`` of an input product (which ends with the ``W_down``
    rows), and what is made of it: nothing (``plain``), a ``delta_decay``, a ``sigmoid_root`` or an ``exp_decay`` (see
    :class:`api.LowRank`).  ``tanh``: the columns pass tanh first.  Few
    tokens run one kernel that does all of it in float32 for up to two such products of one layer; for many the columns become
    a matrix of the activation dtype and the product one like any other."""

    FEW_TOKENS = 128

    def __init__(self, tensors, down: str, up: str, col: int, name: str, kind: str = "plain", bias: torch.Tensor | None = None,
                 a_log: torch.Tensor | None = None, per_head: int = 1, tau: float = 1.0, tanh: bool = False):
        self.tanh = bool(tanh)
        if tensors[down].shape[0] != tensors[up].shape[1]:
            raise ValueError(f"{down!r} makes {tensors[down].shape[0]} numbers, {up!r} takes {tensors[up].shape[1]}")
        self.up = Linear(tensors[up])
        self.transposed = tensors[up].t().contiguous()          # as the kernel for few tokens reads it
        self.col, self.rank, self.cols = int(col), tensors[up].shape[1], tensors[up].shape[0]
        self.name, self.kind, self.bias, self.a_log, self.per_head, self.tau = name, kind, bias, a_log, int(per_head), float(tau)

    @staticmethod
    def run(ctx, proj: torch.Tensor, products: "list[LowRankProduct]") -> list[torch.Tensor]:
        """One float32 tensor of partial sums ``[slices, tokens, cols]`` for each product (one slice where something is made of it)."""
        tokens = proj.shape[1]
        if tokens <= LowRankProduct.FEW_TOKENS:
            out = [ctx.scratch(p.name, (1, tokens, p.cols), torch.float32) for p in products]
            jobs = [api.LowRank(p.col, p.transposed, o[0], p.kind, p.bias, p.a_log, p.per_head, p.tau, p.tanh) for p, o in zip(products, out)]
            if len({p.transposed.dtype for p in products}) == 1:
                api.low_rank(proj, jobs)
            else:
                for job in jobs:
                    api.low_rank(proj, [job])
            return out
        inputs = [ctx.scratch(p.name + ".in", (tokens, p.rank)) for p in products]
        api.low_rank_inputs(proj, [(p.col, x, p.tanh) for p, x in zip(products, inputs)])
        out = []
        for p, x in zip(products, inputs):
            z = p.up(ctx, x, p.name)
            if p.kind != "plain":
                api.low_rank_finish(z, p.kind, p.bias, z[0], p.a_log, p.per_head, p.tau)
                z = z[:1]
            out.append(z)
        return out


def in_blocks(ctx) -> bool:
    """Whether a recurrence with decays per channel takes its tokens four at a time: prompts do (decided by the step's
    shape alone, so a replayed step and the step it was captured from agree)."""
    return not ctx.decode and ctx.n_tokens >= 4 * ctx.sequences


@MIXERS.register("mamba2")
class Mamba2(Mixer):
    NAMES = {"in": "in_proj.weight", "conv": "conv1d.weight", "conv_bias": "conv1d.bias", "dt_bias": "dt_bias", "A_log": "A_log",
             "D": "D", "norm": "norm.weight", "out": "out_proj.weight"}

    def __init__(self, hidden: int, heads: int, head_dim: int, state: int, groups: int = 1, norm_groups: int = 1, conv: int = 4,
                 eps: float = 1e-6, names: dict | None = None):
        self.hidden, self.heads, self.head_dim, self.state = int(hidden), int(heads), int(head_dim), int(state)
        self.groups, self.norm_groups, self.conv, self.eps = int(groups), int(norm_groups), int(conv), float(eps)
        self.inner = self.heads * self.head_dim
        self.channels = self.inner + 2 * self.groups * self.state          # what passes the convolution: x, B, C
        if self.heads % self.groups:
            raise ValueError(f"{heads} heads are not a multiple of {groups} groups")
        if self.inner % self.norm_groups:
            raise ValueError(f"the inner width {self.inner} is not a multiple of {norm_groups} norm groups")
        if not 1 <= self.conv <= 8 or not 1 <= self.state <= 256:
            raise ValueError("the recurrent kernels take 1 to 8 convolution taps and states of up to 256")
        self.names = {**self.NAMES, **(names or {})}
        self.proj: Linear | None = None
        self.out: Linear | None = None

    def weights(self) -> dict[str, WeightDecl]:
        n = self.names
        return {
            n["in"]: WeightDecl((2 * self.inner + 2 * self.groups * self.state + self.heads, self.hidden)),
            n["conv"]: WeightDecl((self.channels, self.conv)),
            n["conv_bias"]: WeightDecl((self.channels,)),
            n["dt_bias"]: WeightDecl((self.heads,)),
            n["A_log"]: WeightDecl((self.heads,)),
            n["D"]: WeightDecl((self.heads,), init="norm"),
            n["norm"]: WeightDecl((self.inner,), init="norm"),
            n["out"]: WeightDecl((self.hidden, self.inner)),
        }

    def state_needs(self) -> list[StateNeed]:
        return [StateNeed((self.heads, self.head_dim, self.state), torch.float32),
                StateNeed((self.conv - 1, self.channels), torch.float32)]

    def bind(self, tensors, dtype, device) -> None:
        n = self.names
        self.proj = Linear(tensors[n["in"]])
        self.out = Linear(tensors[n["out"]])
        self.conv_weight, self.conv_bias = _f32(tensors[n["conv"]]), _f32(tensors[n["conv_bias"]])
        self.dt_bias, self.a_log, self.d_skip = _f32(tensors[n["dt_bias"]]), _f32(tensors[n["A_log"]]), _f32(tensors[n["D"]])
        self.norm = _f32(tensors[n["norm"]])

    def projections(self) -> list:
        return [self.proj, self.out]

    def vectors(self) -> list[torch.Tensor]:
        return [self.conv_weight, self.conv_bias, self.dt_bias, self.a_log, self.d_skip, self.norm]

    def device_driven(self) -> bool:
        return True

    def forward(self, ctx, x, cache, states) -> Delta:
        recurrent, tail = states
        tokens = ctx.n_tokens
        proj = self.proj(ctx, x, "mamba2.in")
        xbc = ctx.scratch("mamba2.xbc", (tokens, self.channels), torch.float32)
        api.causal_conv(proj, self.inner, self.channels, self.conv_weight, self.conv_bias, True, tail, xbc, ctx.cu, ctx.slots,
                        ctx.sequences, tokens, ctx.decode)
        y = ctx.scratch("mamba2.y", (tokens, self.inner), torch.float32)
        api.mamba2_scan(xbc, proj, self.inner + self.channels, self.dt_bias, self.a_log, self.d_skip, recurrent, y, ctx.cu, ctx.slots,
                        ctx.sequences, self.heads, self.head_dim, self.state, self.groups)
        gated = ctx.scratch("mamba2.gated", (tokens, self.inner))
        api.gated_group_norm(y, self.inner // self.norm_groups, proj, 0, self.norm, self.eps, True, gated)
        return self.out.delta(ctx, gated, "mamba2.out")


@MIXERS.register("gated_delta")
class GatedDelta(Mixer):
    NAMES = {"q": "q_proj.weight", "k": "k_proj.weight", "v": "v_proj.weight", "q_conv": "q_conv1d.weight", "k_conv": "k_conv1d.weight",
             "v_conv": "v_conv1d.weight", "b": "b_proj.weight", "a": "a_proj.weight", "g": "g_proj.weight", "dt_bias": "dt_bias",
             "A_log": "A_log", "norm": "o_norm.weight", "out": "o_proj.weight", "a1": "a1_proj.weight", "a2": "a2_proj.weight",
             "g1": "g1_proj.weight", "g2": "g2_proj.weight"}

    def __init__(self, hidden: int, heads: int, qk_heads: int, key_dim: int, value_dim: int, conv: int = 4, eps: float = 1e-6,
                 names: dict | None = None, channel_decay: int | None = None, low_rank_gate: int | None = None, gate: str = "silu"):
        """``channel_decay`` and ``low_rank_gate``: the rank with which random weights are drawn (a checkpoint may bring
        another), or None for the forms of full rank."""
        self.hidden, self.heads, self.qk_heads = int(hidden), int(heads), int(qk_heads)
        self.key_dim, self.value_dim, self.conv, self.eps = int(key_dim), int(value_dim), int(conv), float(eps)
        if self.heads % self.qk_heads:
            raise ValueError(f"{heads} heads are not a multiple of {qk_heads} query/key heads")
        if not 1 <= self.conv <= 8 or not 1 <= self.key_dim <= 256:
            raise ValueError("the recurrent kernels take 1 to 8 convolution taps and key sizes of up to 256")
        self.qk, self.v = self.qk_heads * self.key_dim, self.heads * self.value_dim
        self.channels = 2 * self.qk + self.v                               # what passes the convolutions: q, k, v
        self.channel_decay = None if channel_decay is None else int(channel_decay)
        self.low_rank_gate = None if low_rank_gate is None else int(low_rank_gate)
        if gate not in api.NORM_GATES:
            raise ValueError(f"the gate is one of {sorted(api.NORM_GATES)}, not {gate!r}")
        self.gate = gate
        self.low_rank: list[LowRankProduct] = []       # the decay's, then the gate's
        self.names = {**self.NAMES, **(names or {})}
        self.proj: Linear | None = None
        self.out: Linear | None = None

    def weights(self) -> dict[str, WeightDecl]:
        n = self.names
        return {
            n["q"]: WeightDecl((self.qk, self.hidden)),
            n["q_conv"]: WeightDecl((self.qk, self.conv)),
            n["k"]: WeightDecl((self.qk, self.hidden)),
            n["k_conv"]: WeightDecl((self.qk, self.conv)),
            n["v"]: WeightDecl((self.v, self.hidden)),
            n["v_conv"]: WeightDecl((self.v, self.conv)),
            n["b"]: WeightDecl((self.heads, self.hidden)),
            n["A_log"]: WeightDecl((self.heads,)),
            n["norm"]: WeightDecl((self.value_dim,), init="norm"),
            **(_low_rank_decls(n["a1"], n["a2"], self.hidden, self.channel_decay, self.heads * self.key_dim) if self.channel_decay
               else {n["a"]: WeightDecl((self.heads, self.hidden))}),
            n["dt_bias"]: WeightDecl((self.heads * self.key_dim if self.channel_decay else self.heads,)),
            **(_low_rank_decls(n["g1"], n["g2"], self.hidden, self.low_rank_gate, self.v) if self.low_rank_gate
               else {n["g"]: WeightDecl((self.v, self.hidden))}),
            n["out"]: WeightDecl((self.hidden, self.v)),
        }

    def state_needs(self) -> list[StateNeed]:
        return [StateNeed((self.heads, self.value_dim, self.key_dim), torch.float32),
                StateNeed((self.conv - 1, self.channels), torch.float32)]

    def bind(self, tensors, dtype, device) -> None:
        n = self.names
        # one product for everything linear in the input: [q | k | v | gate | b | a], gate and a down to their ranks only where
        # they are products of low rank
        gate, decay = "g1" if self.low_rank_gate else "g", "a1" if self.channel_decay else "a"
        self.proj = Linear(torch.cat([tensors[n[key]] for key in ("q", "k", "v", gate, "b", decay)], dim=0))
        self.out = Linear(tensors[n["out"]])
        self.b_col = self.channels + tensors[n[gate]].shape[0]
        self.a_col = self.b_col + self.heads
        self.conv_weight = torch.cat([_f32(tensors[n[key]]) for key in ("q_conv", "k_conv", "v_conv")], dim=0).contiguous()
        self.dt_bias, self.a_log, self.norm = _f32(tensors[n["dt_bias"]]), _f32(tensors[n["A_log"]]), _f32(tensors[n["norm"]])
        self.low_rank = []
        if self.channel_decay:
            self.low_rank.append(LowRankProduct(tensors, n["a1"], n["a2"], self.a_col, "delta.decay", "delta_decay", self.dt_bias, self.a_log,
                                                self.key_dim))
        if self.low_rank_gate:
            self.low_rank.append(LowRankProduct(tensors, n["g1"], n["g2"], self.channels, "delta.gates"))

    def projections(self) -> list:
        return [self.proj, self.out] + [p.up for p in self.low_rank]

    def vectors(self) -> list[torch.Tensor]:
        return [self.conv_weight, self.dt_bias, self.a_log, self.norm]

    def device_driven(self) -> bool:
        return True

    def forward(self, ctx, x, cache, states) -> Delta:
        recurrent, tail = states
        tokens = ctx.n_tokens
        proj = self.proj(ctx, x, "delta.in")
        decay, gate_source, gate_col = None, proj, self.channels
        if self.low_rank:
            made = LowRankProduct.run(ctx, proj, self.low_rank)
            if self.channel_decay:
                decay = made[0][0]
            if self.low_rank_gate:
                gate_source, gate_col = made[-1], 0
        qkv = ctx.scratch("delta.qkv", (tokens, self.channels), torch.float32)
        api.causal_conv(proj, 0, self.channels, self.conv_weight, None, True, tail, qkv, ctx.cu, ctx.slots, ctx.sequences, tokens, ctx.decode)
        read = ctx.scratch("delta.read", (tokens, self.v), torch.float32)
        if decay is not None and in_blocks(ctx):
            api.row_decay_blocks(qkv[:, :self.qk], qkv[:, self.qk: 2 * self.qk], qkv[:, 2 * self.qk:], decay, recurrent, read, ctx.cu, ctx.slots,
                                 ctx.sequences, self.heads, self.qk_heads, self.key_dim, self.value_dim, self.key_dim ** -0.5, (proj, self.b_col))
        else:
            api.delta_scan(qkv, proj, self.b_col, self.a_col, self.dt_bias, self.a_log, recurrent, read, ctx.cu,
                           ctx.slots, ctx.sequences, self.heads, self.qk_heads, self.key_dim, self.value_dim, row_decay=decay)
        gated = ctx.scratch("delta.gated", (tokens, self.v))
        api.gated_group_norm(read, self.value_dim, gate_source, gate_col, self.norm, self.eps, False, gated, self.gate)
        return self.out.delta(ctx, gated, "delta.out")


@MIXERS.register("decay_linear_attention")
class DecayLinearAttention(Mixer):
    NAMES = {"q": "q_proj.weight", "k": "k_proj.weight", "v": "v_proj.weight", "g": "g_proj.weight", "norm": "norm.weight",
             "out": "o_proj.weight", "a1": "a1_proj.weight", "a2": "a2_proj.weight", "a_bias": "a2_proj.bias"}

    def __init__(self, hidden: int, heads: int, key_dim: int, value_dim: int, decay=None, activation: str | None = None,
                 position: PartSpec | None = None, key_scale: float = 1.0, norm: str = "head", norm_weight: bool = False,
                 gate: str = "silu", eps: float = 1e-6, names: dict | None = None, channel_decay: dict | None = None,
                 query_scale: float = 1.0):
        """``channel_decay``: ``{"tau": the root, "rank": the rank with which random weights are drawn}``, instead of ``decay``."""
        self.hidden, self.heads, self.key_dim, self.value_dim = int(hidden), int(heads), int(key_dim), int(value_dim)
        if (decay is None) == (channel_decay is None):
            raise ValueError("linear attention has a fixed decay per head or one per key channel from the token")
        self.decay = None if decay is None else tuple(float(d) for d in decay)
        if self.decay is not None and len(self.decay) != self.heads:
            raise ValueError(f"{len(self.decay)} decays for {self.heads} heads")
        self.rank = None if channel_decay is None else int(channel_decay["rank"])
        self.tau = None if channel_decay is None else float(channel_decay["tau"])
        self.query_scale = float(query_scale)
        self.low_rank: LowRankProduct | None = None
        if activation not in (None, "silu"):
            raise ValueError(f"q, k and v pass silu or nothing, not {activation!r}")
        if norm not in ("head", "all"):
            raise ValueError(f"the read-out is normed per head or over all heads, not {norm!r}")
        if gate not in api.NORM_GATES:
            raise ValueError(f"the gate is one of {sorted(api.NORM_GATES)}, not {gate!r}")
        if not 1 <= self.key_dim <= 256:
            raise ValueError("the recurrent kernels take key sizes of up to 256")
        self.activation, self.key_scale, self.norm, self.norm_weight = activation, float(key_scale), norm, bool(norm_weight)
        self.gate, self.eps = gate, float(eps)
        self.qk, self.v = self.heads * self.key_dim, self.heads * self.value_dim
        self.names = {**self.NAMES, **(names or {})}
        position = position or PartSpec("none", {"head_dim": self.key_dim})
        self.position = POSITION_ENCODINGS.build(position.kind, dict(position.params))
        if self.position.kind not in ("rotary", "none"):
            raise ValueError(f"linear attention applies rotary position encodings or none, not one of kind {self.position.kind!r}")
        self.rot: RotaryTable | None = None
        self.proj: Linear | None = None
        self.out: Linear | None = None

    def weights(self) -> dict[str, WeightDecl]:
        n = self.names
        out = {
            n["q"]: WeightDecl((self.qk, self.hidden)),
            n["k"]: WeightDecl((self.qk, self.hidden)),
            n["v"]: WeightDecl((self.v, self.hidden)),
            n["g"]: WeightDecl((self.v, self.hidden)),
            n["out"]: WeightDecl((self.hidden, self.v)),
        }
        if self.rank is not None:
            out.update(_low_rank_decls(n["a1"], n["a2"], self.hidden, self.rank, self.qk))
            out[n["a_bias"]] = WeightDecl((self.qk,))
        if self.norm_weight:
            out[n["norm"]] = WeightDecl((self.v if self.norm == "all" else self.value_dim,), init="norm")
        return out

    def state_needs(self) -> list[StateNeed]:
        return [StateNeed((self.heads, self.value_dim, self.key_dim), torch.float32)]

    def bind(self, tensors, dtype, device) -> None:
        n = self.names
        self.position.bind({}, dtype, device)
        self.rot = None
        if self.position.kind == "rotary":
            self.rot = self.position.rotary()
            if self.rot.interleaved or self.rot.attention_scaling != 1.0 or self.rot.rotary_dim % 2 or self.rot.rotary_dim > self.key_dim:
                raise ValueError("linear attention rotates halves of an even part of the head and does not scale the rotation")
        # one product for everything linear in the input: [q | k | v | gate], then the first half of the decays' product
        keys = ("q", "k", "v", "g") + (("a1",) if self.rank is not None else ())
        self.proj = Linear(torch.cat([tensors[n[key]] for key in keys], dim=0))
        self.out = Linear(tensors[n["out"]])
        self.decays = None
        if self.rank is not None:
            self.low_rank = LowRankProduct(tensors, n["a1"], n["a2"], 2 * self.qk + 2 * self.v, "linear_attention.decay", "sigmoid_root",
                                           _f32(tensors[n["a_bias"]]), tau=self.tau)
        else:
            self.decays = torch.tensor(self.decay, dtype=torch.float32, device=device)
        count = self.v if self.norm == "all" else self.value_dim
        self.norm_w = _f32(tensors[n["norm"]]) if self.norm_weight else torch.ones(count, dtype=torch.float32, device=device)

    def projections(self) -> list:
        return [self.proj, self.out] + ([self.low_rank.up] if self.low_rank is not None else [])

    def vectors(self) -> list[torch.Tensor]:
        return ([self.norm_w] if self.norm_weight else []) + ([self.low_rank.bias] if self.low_rank is not None else [])

    def device_driven(self) -> bool:
        return True

    def forward(self, ctx, x, cache, states) -> Delta:
        (recurrent,) = states
        tokens = ctx.n_tokens
        proj = self.proj(ctx, x, "linear_attention.in")
        rotary_dim = self.rot.rotary_dim if self.rot is not None else 0
        read = ctx.scratch("linear_attention.read", (tokens, self.v), torch.float32)
        decay = None
        if self.low_rank is not None:
            decay = LowRankProduct.run(ctx, proj, [self.low_rank])[0][0]
        blocks = decay is not None and in_blocks(ctx)
        if blocks and proj.shape[0] == 1 and not rotary_dim and self.activation is None and self.key_scale == 1.0:
            q, k, v = proj[0].split((self.qk, self.qk, self.v, proj.shape[2] - 2 * self.qk - self.v), dim=1)[:3]     # the product as it is
            api.row_decay_blocks(q, k, v, decay, recurrent, read, ctx.cu, ctx.slots, ctx.sequences, self.heads, self.heads, self.key_dim,
                                 self.value_dim, self.query_scale)
            return self.finish(ctx, proj, read)
        vkq = ctx.scratch("linear_attention.vkq", (tokens, self.v + 2 * self.qk), torch.float32)
        api.linear_attention_prepare(proj, self.heads, self.key_dim, self.value_dim, self.activation == "silu",
                                     self.rot.inv_freq if rotary_dim else None, rotary_dim, self.key_scale, vkq, ctx.cu, ctx.len_before,
                                     ctx.sequences, tokens, self.query_scale)
        if blocks:
            v, k, q = vkq.split((self.v, self.qk, self.qk), dim=1)
            api.row_decay_blocks(q, k, v, decay, recurrent, read, ctx.cu, ctx.slots, ctx.sequences, self.heads, self.heads, self.key_dim,
                                 self.value_dim, 1.0)
        elif decay is not None:
            api.row_decay_scan(vkq, decay, recurrent, read, ctx.cu, ctx.slots, ctx.sequences, self.heads, self.key_dim, self.value_dim)
        else:
            api.decay_scan(vkq, self.decays, recurrent, read, ctx.cu, ctx.slots, ctx.sequences, self.heads, self.key_dim, self.value_dim)
        return self.finish(ctx, proj, read)

    def finish(self, ctx, proj, read) -> Delta:
        """Norm and gate of the read-out, output projection."""
        gated = ctx.scratch("linear_attention.gated", (ctx.n_tokens, self.v))
        api.gated_group_norm(read, self.v if self.norm == "all" else self.value_dim, proj, 2 * self.qk + self.v, self.norm_w, self.eps,
                             False, gated, self.gate)
        return self.out.delta(ctx, gated, "linear_attention.out")
