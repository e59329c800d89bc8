"""Plain, slow implementation of the Zuvepel decoder, used only as the test oracle.

Zuvepel is a decoder of parallel layers with two layer norms, ``x += m * (mixer(norm1(x)) + ff(norm2(x)))``, both sublayers
reading the same stream.  A stretch of layers is run several times with the same weights, every pass with a cache and
states of its own, and each pass but the first starts by adding the embedding's output to the stream.  The mixer is one of
three, in an order config.json lists.  *Attention*: grouped heads with biases on q, k and v, half-rotated positions,
keys of the query's own chunk of the sequence only, one added to the softmax denominator, one sigmoid gate per head.
*channel_delta*: the gated delta rule with a decay for every head and key channel, made by a product of low rank, behind short
convolutions; the read-out RMS-normed per head and gated by another product of low rank.  *gla*: linear attention whose state
decays per key channel, the read-out RMS-normed per head and gated by silu.  The feed-forward is gated by the tanh form of
gelu.

Everything here works on one whole sequence at a time, token by token where there is a state, with no cache and no
batching.  It shares no code with the package under test: own config reading, own safetensors reader, one function per
mechanism.  Arithmetic is float64 except for the rotation's angles, which are float32 products of float32 factors like an
engine's.
"""
from __future__ import annotations

import json
import math
import struct
from pathlib import Path

import numpy as np
import torch

# What stands in for the narrowing of activations: None (exact), or a function applied wherever an engine that
# multiplies bfloat16 matrices narrows its operand.  ``forward(..., narrow=f)`` sets it.
_narrow = None


def nar(x):
    return x if _narrow is None else _narrow(x)


_NP = {"F32": np.float32, "F64": np.float64, "F16": np.float16, "I32": np.int32, "I64": np.int64}


def read_safetensors(path) -> dict[str, torch.Tensor]:
    """name -> float64 (or int64) tensor; bfloat16 is widened exactly."""
    data = Path(path).read_bytes()
    (n,) = struct.unpack("<Q", data[:8])
    header = json.loads(data[8:8 + n].decode("utf-8"))
    out = {}
    for name, meta in header.items():
        if name == "__metadata__":
            continue
        lo, hi = meta["data_offsets"]
        raw = data[8 + n + lo:8 + n + hi]
        shape = tuple(meta["shape"])
        if meta["dtype"] == "BF16":
            words = np.frombuffer(raw, dtype="<u2").astype(np.uint32) << 16
            array = words.view(np.float32).astype(np.float64)
        else:
            array = np.frombuffer(raw, dtype=np.dtype(_NP[meta["dtype"]]).newbyteorder("<"))
            array = array.astype(np.int64 if meta["dtype"].startswith("I") else np.float64)
        out[name] = torch.from_numpy(array.reshape(shape).copy())
    return out


def read_model(folder):
    folder = Path(folder)
    return json.loads((folder / "config.json").read_text()), read_safetensors(folder / "model.safetensors")


# ------------------------------------------------------------------------- small pieces
def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return torch.clamp(x, min=0.0) + torch.log1p(torch.exp(-x.abs()))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def layer_norm(x, w, b, eps):
    """(x - mean) / sqrt(mean((x - mean)^2) + eps) * w + b over the last axis."""
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def short_convolution(u, w):
    """u [T, C], w [C, taps]: y_t = sum_j w[:, j] * u_(t - taps + 1 + j), zeros before the sequence's start; then silu."""
    taps = w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=u.dtype), u], dim=0)
    y = torch.zeros_like(u)
    for j in range(taps):
        y = y + padded[j:j + u.shape[0]] * w[:, j]
    return silu(y)


def low_rank(h, w, p, a, b):
    return nar(h @ w[p + a].T) @ w[p + b].T


def rotate_halves(x, positions, rot):
    """Rotate the first ``dims`` numbers of the last axis of x [T, heads, n], i paired with i + dims / 2."""
    dims = rot["dims"]
    f = (float(rot["base"]) ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims)).to(torch.float32)
    angle = (positions.to(torch.float32)[:, None] * f[None, :]).to(torch.float64)
    cos, sin = torch.cos(angle)[:, None, :], torch.sin(angle)[:, None, :]
    u, v = x[..., :dims // 2], x[..., dims // 2:dims]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., dims:]], dim=-1)


# ------------------------------------------------------------------------------- mixers
def attention(h, w, p, m, eps):
    T = h.shape[0]
    H, D, V = m["heads"], m["dim"], m["vdim"]
    G = m.get("kv_heads") or H
    h = nar(h)
    q, k, v = ((h @ w[p + n].T + w[p + n + ".b"]) for n in "qkv")
    q, k, v = q.reshape(T, H, D), k.reshape(T, G, D), v.reshape(T, G, V)
    if m.get("rot"):
        q, k = rotate_halves(q, torch.arange(T), m["rot"]), rotate_halves(k, torch.arange(T), m["rot"])
    q, k, v = nar(q), nar(k), nar(v)
    chunk = (m.get("mask") or {}).get("size")
    out = torch.zeros(T, H, V, dtype=h.dtype)
    for t in range(T):
        lo = 0 if not chunk else t // chunk * chunk
        for g in range(G):
            mine = slice(g * (H // G), (g + 1) * (H // G))
            s = (q[t, mine] @ k[lo:t + 1, g].T) * m["scale"]
            top = torch.clamp(s.max(dim=-1, keepdim=True).values, min=0.0)
            e = torch.exp(s - top)
            out[t, mine] = (e / (torch.exp(-top) + e.sum(-1, keepdim=True))) @ v[lo:t + 1, g]
    out = out * sigmoid(h @ w[p + "g"].T)[:, :, None]
    return nar(out.reshape(T, H * V)) @ w[p + "o"].T


def delta_rule(q, k, v, beta, g):
    """q, k, g [T, H, D], v [T, H, V], beta [T, H] -> o [T, H, V]: per head S (D x V) from zero, S <- g S (rows),
    u = beta (v - S^T k), S <- S + k u^T, o = S^T q."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=q.dtype)
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out


def linear_attention(q, k, v, alpha):
    """S <- diag(alpha_t) S + k_t v_t^T, o_t = S^T q_t, per head; alpha [T, H, D]."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=q.dtype)
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out


def channel_delta(h, w, p, m, eps):
    T = h.shape[0]
    H, D, V = m["heads"], m["dim"], m["vdim"]
    G = m.get("kv_heads") or H
    h = nar(h)
    q, k, v = (short_convolution(h @ w[p + n].T, w[p + n + ".conv"]) for n in "qkv")
    q = (unit(q.reshape(T, G, D)) * D ** -0.5).repeat_interleave(H // G, dim=1)
    k = unit(k.reshape(T, G, D)).repeat_interleave(H // G, dim=1)
    beta = sigmoid(h @ w[p + "b"].T)
    z = (low_rank(h, w, p, "a1", "a2") + w[p + "dt_bias"]).reshape(T, H, D)
    g = torch.exp(-torch.exp(w[p + "A_log"])[None, :, None] * softplus(z))
    o = delta_rule(q, k, v.reshape(T, H, V), beta, g)
    o = rms(o, eps) * w[p + "norm"] * sigmoid(low_rank(h, w, p, "g1", "g2")).reshape(T, H, V)
    return nar(o.reshape(T, H * V)) @ w[p + "o"].T


def gla(h, w, p, m, eps):
    T = h.shape[0]
    H, D, V = m["heads"], m["dim"], m["vdim"]
    h = nar(h)
    q, k, v = (h @ w[p + "q"].T * D ** -0.5).reshape(T, H, D), (h @ w[p + "k"].T).reshape(T, H, D), (h @ w[p + "v"].T).reshape(T, H, V)
    z = (low_rank(h, w, p, "a1", "a2") + w[p + "a2.b"]).reshape(T, H, D)
    o = linear_attention(q, k, v, torch.exp(-softplus(-z) / m["tau"]))
    o = (rms(o, eps) * w[p + "norm"]).reshape(T, H * V) * silu(h @ w[p + "g"].T)
    return nar(o) @ w[p + "o"].T


MIXERS = {"attention": attention, "channel_delta": channel_delta, "gla": gla}


def dense(h, w, p):
    h = nar(h)
    return nar(gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


# -------------------------------------------------------------------------------- model
def schedule(config):
    """(layer, whether the embedding's output is added first) in the order of the runs."""
    n = len(config["layers"])
    loop = config.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    start, stop, times = loop["start"], loop["stop"], loop["times"]
    runs = [(i, False) for i in range(start)]
    for turn in range(times):
        runs += [(i, turn > 0 and i == start) for i in range(start, stop)]
    return runs + [(i, False) for i in range(stop, n)]


def forward(config, w, tokens, dtype=torch.float64, layers_out=None, narrow=None):
    """Logits [tokens, vocab] of one whole sequence.  ``layers_out``: a list that receives the stream after each layer run."""
    global _narrow
    _narrow = narrow
    try:
        return _forward(config, w, tokens, dtype, layers_out)
    finally:
        _narrow = None


def _forward(config, w, tokens, dtype, layers_out):
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in w.items()}
    eps, m = config["norm"]["eps"], config["residual_mult"]
    embedded = w["embed"][torch.as_tensor(tokens, dtype=torch.int64)] * config["embedding"]["scale"]
    x = embedded
    for i, again in schedule(config):
        layer, p = config["layers"][i], f"l{i}."
        if again:
            x = x + embedded
        add = MIXERS[layer["type"]](layer_norm(x, w[p + "norm1"], w[p + "norm1.b"], eps), w, p + "mix.", layer["mixer"], eps)
        if layer.get("mlp") is not None:
            add = add + dense(layer_norm(x, w[p + "norm2"], w[p + "norm2.b"], eps), w, p + "mlp.")
        x = x + m * add
        if layers_out is not None:
            layers_out.append(x.clone())
    return nar(layer_norm(x, w["final.norm"], w["final.norm.b"], eps)) @ w["head"].T
