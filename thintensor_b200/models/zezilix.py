"""The Zezilix decoder as a description: which parts each layer has, with what numbers, and what the
checkpoint calls their tensors.

The residual stream comes in ``streams`` copies.  Layers are pre-norm with RMS norms (``l<i>.norm1``, ``l<i>.norm2``); each sublayer has
weights with which it reads the copies and is written back to them (``l<i>.hc1.in`` / ``out`` / ``mix``, ``l<i>.hc2...``) and a scale per
channel (``l<i>.ls1``, ``l<i>.ls2``).  The mixer's tensors lie under ``l<i>.mix.``, the feed-forward's under ``l<i>.mlp.`` (``gate`` / ``up`` /
``down``, or ``e<k>.up`` / ``down`` and ``router``).  The token table is ``embed`` with the norm ``embed.norm``, the last norm
``final.norm``, the output matrix ``head``.  A stretch of layers may run several times with the same weights (``loop``): each pass is a
run of the schedule with a cache and states of its own.

What the design fixes lives here: the rotation pairs neighbours, the dense unit uses ``sigmoid(1.702 g)``, experts are ungated with the
square of relu, routing weights are the softmax's scores times a factor, not renormalised.
"""
from __future__ import annotations

from ..config.registry import Architecture, register_architecture
from ..config.zezilix import ARCHITECTURE, DenseSizes, LatentAttentionSizes, MoeSizes, WkvSizes, ZezilixConfig
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, Run

LATENT_NAMES = {"q": "q", "dq": "dq", "dq_norm": "dq.norm", "uq": "uq", "dkv": "dkv", "dkv_norm": "dkv.norm", "uk": "uk", "uv": "uv", "g": "g", "o": "o"}
WKV_NAMES = {"r": "r", "k": "k", "v": "v", "g": "g", "w1": "w1", "w2": "w2", "w0": "w0", "u": "u", "mu": "mu.{}", "norm": "norm", "out": "o"}
FFN_NAMES = {"gate": "gate", "up": "up", "down": "down"}
MOE_NAMES = {"router": "router", "expert": "e{}.", "up": "up", "down": "down"}
UNIT_ALPHA = 1.702
DRAWN_RANK = 64             # the decays' rank in random weights; a checkpoint's tensors bring their own


def latent_attention_part(config: ZezilixConfig, sizes: LatentAttentionSizes, prefix: str) -> PartSpec:
    position = None
    if sizes.rot is not None:
        position = PartSpec("rope", {"head_dim": sizes.rot_dim, "theta": sizes.rot.base, "rotary_dim": sizes.rot.dims, "interleaved": True,
                                     "table_precision": "float64"})
    return PartSpec("latent_attention", {
        "hidden": config.width, "heads": sizes.heads, "dim": sizes.dim, "rot_dim": sizes.rot_dim, "value_dim": sizes.vdim,
        "q_rank": sizes.q_rank, "kv_rank": sizes.kv_rank, "scale": sizes.scale, "eps": config.eps, "position": position,
        "gate": "elementwise" if sizes.q_rank is None else None, "names": LATENT_NAMES}, prefix)


def wkv_part(config: ZezilixConfig, sizes: WkvSizes, prefix: str) -> PartSpec:
    return PartSpec("wkv", {"hidden": config.width, "heads": sizes.heads, "dim": sizes.dim, "rank": DRAWN_RANK, "eps": config.eps,
                            "names": WKV_NAMES}, prefix)


def feed_forward_part(config: ZezilixConfig, sizes, prefix: str) -> PartSpec:
    if isinstance(sizes, DenseSizes):
        return PartSpec("swiglu", {"hidden": config.width, "inter": sizes.ff, "activation": "clamped", "limit": sizes.limit, "alpha": UNIT_ALPHA,
                                   "names": FFN_NAMES}, prefix)
    assert isinstance(sizes, MoeSizes)
    return PartSpec("moe", {"hidden": config.width, "experts": sizes.experts, "top": sizes.top, "inter": sizes.ff, "gated": False,
                            "activation": "relu2", "renormalize": False, "weight_scale": sizes.scale, "names": MOE_NAMES}, prefix)


def describe_zezilix(config: ZezilixConfig) -> ModelSpec:
    def norm(prefix: str, name: str) -> PartSpec:
        return PartSpec("rmsnorm", {"dim": config.width, "eps": config.eps, "name": name}, prefix)

    def streams(prefix: str) -> PartSpec:
        return PartSpec("hyper", {"streams": config.streams, "names": {"read": "in", "write": "out", "mix": "mix"}}, prefix)

    def scale(prefix: str, name: str) -> PartSpec:
        return PartSpec("channel", {"dim": config.width, "name": name}, prefix)

    layers = []
    for index, layer in enumerate(config.layers):
        prefix = f"l{index}."
        mixer = wkv_part if layer.type == "wkv" else latent_attention_part
        parts = {"mixer_norm": norm(prefix, "norm1"), "mixer": mixer(config, layer.mixer, prefix + "mix."),
                 "mixer_scale": scale(prefix, "ls1"), "mixer_streams": streams(prefix + "hc1.")}
        if layer.mlp is not None:
            parts.update({"ffn_norm": norm(prefix, "norm2"), "ffn": feed_forward_part(config, layer.mlp, prefix + "mlp."),
                          "ffn_scale": scale(prefix, "ls2"), "ffn_streams": streams(prefix + "hc2.")})
        layers.append(LayerSpec("pre_norm", parts, {"scale": config.residual_mult}))
    schedule = [Run(i) for i in range(len(layers))]
    if config.loop is not None:
        stretch = schedule[config.loop.start:config.loop.stop]
        schedule[config.loop.start:config.loop.stop] = stretch * config.loop.times
    return ModelSpec(
        hidden_size=config.width,
        vocab_size=config.vocab,
        embedding=PartSpec("table", {"vocab": config.vocab, "hidden": config.width, "name": "embed", "norm_eps": config.eps,
                                     "norm_name": "embed.norm"}, ""),
        layers=tuple(layers),
        schedule=tuple(schedule),
        final_norm=norm("final.", "norm"),
        head=PartSpec("linear", {"hidden": config.width, "vocab": config.vocab, "name": "head"}, ""),
        streams=config.streams,
    )


register_architecture(Architecture(
    name=ARCHITECTURE,
    model_types=("zezilix",),
    config_class=ZezilixConfig,
    describe=describe_zezilix,
))
