"""The Zuvepel decoder as a description: which parts each layer has, with what numbers, and what the
checkpoint calls their tensors.

Layers are parallel with two layer norms (``l<i>.norm1`` for the mixer, ``l<i>.norm2`` for the feed-forward, biases under the
same names with ``.b`` added), both sublayers' sum times ``residual_mult``.  The mixer's tensors lie under ``l<i>.mix.``, the
feed-forward's under ``l<i>.mlp.``.  The token table is ``embed``, the last norm ``final.norm`` and the output matrix ``head``.  A
stretch of layers may run several times with the same weights (``loop``): each pass is a run of the schedule with a cache and
states of its own, and each pass but the first starts by adding the embedding's output.

``channel_delta`` is the gated delta rule with a decay per key channel and a sigmoid gate, both from products of low rank;
``gla`` is linear attention with a decay per key channel; ``attention`` has biases on q, k and v, chunks, one added to the
softmax denominator and a gate per head.
"""
from __future__ import annotations

from ..config.registry import Architecture, register_architecture
from ..config.zuvepel import ARCHITECTURE, AttentionSizes, ChannelDeltaSizes, GlaSizes, ZuvepelConfig
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, Run

ATTENTION_NAMES = {"q": "q", "k": "k", "v": "v", "o": "o", "g": "g", "q_bias": "q.b", "k_bias": "k.b", "v_bias": "v.b"}
DELTA_NAMES = {"q": "q", "k": "k", "v": "v", "q_conv": "q.conv", "k_conv": "k.conv", "v_conv": "v.conv", "b": "b", "a1": "a1", "a2": "a2",
               "g1": "g1", "g2": "g2", "dt_bias": "dt_bias", "A_log": "A_log", "norm": "norm", "out": "o"}
GLA_NAMES = {"q": "q", "k": "k", "v": "v", "g": "g", "a1": "a1", "a2": "a2", "a_bias": "a2.b", "norm": "norm", "out": "o"}
FFN_NAMES = {"gate": "gate", "up": "up", "down": "down"}
GLA_DRAWN_RANK = 16         # the rank of random weights; a checkpoint's tensors bring their own


def attention_part(config: ZuvepelConfig, sizes: AttentionSizes, prefix: str) -> PartSpec:
    position = None
    if sizes.rot is not None:
        position = PartSpec("rope", {"head_dim": sizes.dim, "theta": sizes.rot.base, "rotary_dim": sizes.rot.dims, "table_precision": "float64"})
    return PartSpec("attention", {
        "hidden": config.width, "heads": sizes.heads, "kv_heads": sizes.kv_heads, "head_dim": sizes.dim, "value_dim": sizes.vdim,
        "position": position, "scale": sizes.scale, "chunk": sizes.chunk, "bias": "qkv", "null_score": 0.0, "gate": "head",
        "names": ATTENTION_NAMES}, prefix)


def channel_delta_part(config: ZuvepelConfig, sizes: ChannelDeltaSizes, prefix: str) -> PartSpec:
    return PartSpec("gated_delta", {
        "hidden": config.width, "heads": sizes.heads, "qk_heads": sizes.kv_heads, "key_dim": sizes.dim, "value_dim": sizes.vdim,
        "conv": sizes.conv, "eps": config.eps, "channel_decay": sizes.dim, "low_rank_gate": sizes.vdim, "gate": "sigmoid",
        "names": DELTA_NAMES}, prefix)


def gla_part(config: ZuvepelConfig, sizes: GlaSizes, prefix: str) -> PartSpec:
    return PartSpec("decay_linear_attention", {
        "hidden": config.width, "heads": sizes.heads, "key_dim": sizes.dim, "value_dim": sizes.vdim,
        "channel_decay": {"tau": sizes.tau, "rank": GLA_DRAWN_RANK}, "query_scale": sizes.dim ** -0.5, "norm": "head", "norm_weight": True,
        "gate": "silu", "eps": config.eps, "names": GLA_NAMES}, prefix)


MIXER_PARTS = {"attention": attention_part, "channel_delta": channel_delta_part, "gla": gla_part}


def describe_zuvepel(config: ZuvepelConfig) -> ModelSpec:
    def norm(prefix: str, name: str) -> PartSpec:
        return PartSpec("layernorm", {"dim": config.width, "eps": config.eps, "bias": True, "name": name, "bias_name": name + ".b"}, prefix)

    layers = []
    for index, layer in enumerate(config.layers):
        prefix = f"l{index}."
        parts = {"norm": norm(prefix, "norm1"), "mixer": MIXER_PARTS[layer.type](config, layer.mixer, prefix + "mix.")}
        if layer.mlp is not None:
            parts["ffn_norm"] = norm(prefix, "norm2")
            parts["ffn"] = PartSpec("swiglu", {"hidden": config.width, "inter": layer.mlp.ff, "activation": "gelu_tanh", "names": FFN_NAMES},
                                    prefix + "mlp.")
        layers.append(LayerSpec("parallel", parts, {"scale": config.residual_mult}))
    schedule = [Run(i) for i in range(len(layers))]
    if config.loop is not None:
        passes = [Run(i, add_embedding=turn > 0 and i == config.loop.start) for turn in range(config.loop.times)
                  for i in range(config.loop.start, config.loop.stop)]
        schedule[config.loop.start:config.loop.stop] = passes
    return ModelSpec(
        hidden_size=config.width,
        vocab_size=config.vocab,
        embedding=PartSpec("table", {"vocab": config.vocab, "hidden": config.width, "scale": config.embedding_scale, "name": "embed"}, ""),
        layers=tuple(layers),
        schedule=tuple(schedule),
        final_norm=norm("final.", "norm"),
        head=PartSpec("linear", {"hidden": config.width, "vocab": config.vocab, "name": "head"}, ""),
    )


register_architecture(Architecture(
    name=ARCHITECTURE,
    model_types=("zuvepel",),
    config_class=ZuvepelConfig,
    describe=describe_zuvepel,
))
