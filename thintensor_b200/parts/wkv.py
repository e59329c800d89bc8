"""Time mixing with a decay per key channel, a bonus for the current token, and shifted inputs.

The form of RWKV-6 (Peng et al., "Eagle and Finch: RWKV with Matrix-Valued States and Dynamic Recurrence") without its
token-dependent shifts: each of the five projections reads a blend of its own of the token's row h and the row h' before it (zeros
before a sequence's first token), ``h + (h' - h) * mu``.  ``r``, ``k``, ``v`` are ``heads * dim`` numbers each; the decay of head and key
channel is ``a = exp(-exp(W_2 tanh(W_1 h_w) + w_0))``.  Per head, with S of shape key x value, ``o = (S + diag(u) k v^T)^T r`` and then
``S <- diag(a) S + k v^T``.  Every head's o is divided by its root mean square; the heads together are multiplied by a weight and by
``silu(W_g h_g)``, and the output projection follows.

All five blends are one kernel and the five projections one product whose output features read the blend of their group.  What
comes after runs the kernels of linear attention with a decay per key channel (token by token for few tokens, four at a time for
prompts), which take the bonus as an option.  A sequence carries S per head and the last row h, both float32.
"""
from __future__ import annotations

import torch

from ..kernels import api
from .base import MIXERS, Delta, Mixer, StateNeed, WeightDecl
from .linear import GroupedLinear, Linear
from .recurrent import LowRankProduct, in_blocks


@MIXERS.register("wkv")
class Wkv(Mixer):
    NAMES = {"r": "receptance.weight", "k": "key.weight", "v": "value.weight", "g": "gate.weight", "w1": "decay_a.weight", "w2": "decay_b.weight",
             "w0": "decay", "u": "bonus", "mu": "mix_{}", "norm": "norm.weight", "out": "output.weight"}
    INPUTS = ("r", "k", "v", "g", "w")

    def __init__(self, hidden: int, heads: int, dim: int, rank: int = 64, eps: float = 1e-6, names: dict | None = None):
        """``rank``: that of the decays' product with which random weights are drawn; a checkpoint may bring another."""
        self.hidden, self.heads, self.dim, self.rank, self.eps = int(hidden), int(heads), int(dim), int(rank), float(eps)
        if not 1 <= self.dim <= 256:
            raise ValueError("the recurrent kernels take heads of up to 256 numbers")
        self.inner = self.heads * self.dim
        self.names = {**self.NAMES, **(names or {})}
        self.proj: GroupedLinear | None = None
        self.out: Linear | None = None

    def weights(self) -> dict[str, WeightDecl]:
        n = self.names
        return {
            **{n["mu"].format(key): WeightDecl((self.hidden,), init="small") for key in self.INPUTS},
            **{n[key]: WeightDecl((self.inner, self.hidden)) for key in ("r", "k", "v", "g")},
            n["w1"]: WeightDecl((self.rank, self.hidden), free=(0,)),
            n["w2"]: WeightDecl((self.inner, self.rank), free=(1,)),
            n["w0"]: WeightDecl((self.inner,), init="small"),
            n["u"]: WeightDecl((self.heads, self.dim), init="small"),
            n["norm"]: WeightDecl((self.inner,), init="norm"),
            n["out"]: WeightDecl((self.hidden, self.inner)),
        }

    def state_needs(self) -> list[StateNeed]:
        return [StateNeed((self.heads, self.dim, self.dim), torch.float32), StateNeed((self.hidden,), torch.float32)]

    def bind(self, tensors, dtype, device) -> None:
        n = self.names
        f32 = lambda key: tensors[n[key]].to(torch.float32).contiguous()
        self.mix = torch.stack([tensors[n["mu"].format(key)].to(torch.float32) for key in self.INPUTS]).contiguous()
        self.proj = GroupedLinear([tensors[n[key]] for key in ("r", "k", "v", "g", "w1")])       # [r | k | v | gate | decay input]
        self.decay = LowRankProduct(tensors, n["w1"], n["w2"], 4 * self.inner, "wkv.decay", "exp_decay", f32("w0"), tanh=True)
        self.bonus, self.norm = f32("u").reshape(-1), f32("norm")
        self.out = Linear(tensors[n["out"]])

    def projections(self) -> list:
        return [self.proj.fused, self.decay.up, self.out]

    def vectors(self) -> list[torch.Tensor]:
        return [self.mix, self.decay.bias, self.bonus, self.norm]

    def device_driven(self) -> bool:
        return True

    def forward(self, ctx, x, cache, states) -> Delta:
        recurrent, before = states
        tokens, inner = ctx.n_tokens, self.inner
        blends = ctx.scratch("wkv.blends", (len(self.INPUTS), tokens, self.hidden))
        api.token_shifts(x, self.mix, before, blends, ctx.cu, ctx.slots, ctx.sequences)
        proj = self.proj(ctx, blends, "wkv.in")
        decay = LowRankProduct.run(ctx, proj, [self.decay])[0][0]
        read = ctx.scratch("wkv.read", (tokens, inner), torch.float32)
        blocks = in_blocks(ctx)
        if blocks and proj.shape[0] == 1:                       # the product as it is
            r, k, v = (proj[0, :, i * inner:(i + 1) * inner] for i in range(3))
        else:
            vkr = ctx.scratch("wkv.vkr", (tokens, 3 * inner), torch.float32)
            api.linear_attention_prepare(proj, self.heads, self.dim, self.dim, False, None, 0, 1.0, vkr, ctx.cu, ctx.len_before, ctx.sequences, tokens)
            v, k, r = vkr.split(inner, dim=1)
        if blocks:
            api.row_decay_blocks(r, k, v, decay, recurrent, read, ctx.cu, ctx.slots, ctx.sequences, self.heads, self.heads, self.dim, self.dim, 1.0,
                                 bonus=self.bonus)
        else:
            api.row_decay_scan(vkr, decay, recurrent, read, ctx.cu, ctx.slots, ctx.sequences, self.heads, self.dim, self.dim, bonus=self.bonus)
        gated = ctx.scratch("wkv.gated", (tokens, inner))
        api.gated_group_norm(read, self.dim, proj, 3 * inner, self.norm, self.eps, False, gated)
        return self.out.delta(ctx, gated, "wkv.out")
