"""Plain, slow implementation of the Zezilix decoder, used only as the test oracle.

Zezilix is a pre-norm decoder with RMS norms whose residual stream comes in several copies ("hyper-connections"): a sublayer
reads a weighted sum of the copies, and afterwards every copy becomes a weighted sum of the old copies plus its own multiple of
the sublayer's output.  A sublayer's output passes a scale per channel and the model's residual factor first.  The token
embedding is normed.  A stretch of layers runs several times with the same weights, every pass with a cache and states of
its own.  The mixer is one of three, in an order config.json lists: latent attention with a low-rank query path, latent
attention with direct queries and a sigmoid gate on every number of the concatenated heads, and *wkv*, a recurrence with a decay
per key channel and token, a bonus for the current token and a token shift of its own on each of its five inputs.  The
feed-forward is dense with a clamped gated unit, or a mixture of ungated experts (squared relu) with softmax routing.

Everything here works on one whole sequence at a time, token by token where there is a state, with no cache and no
batching.  It shares no code with the package under test: own config reading, own safetensors reader, one function per
mechanism.  Arithmetic is float64 except for the rotation's angles, which are float32 products of float32 factors like an
engine's.
"""
from __future__ import annotations

import json
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


def rms(x, eps):
    """x over the root of its mean square on the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rotate_pairs(x, positions, rot):
    """Rotate the first ``dims`` numbers of the last axis of x [T, heads, n], 2i paired with 2i + 1."""
    dims = rot["dims"]
    f = (float(rot["base"]) ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims)).to(torch.float32)
    angle = (positions.to(torch.float32)[:, None] * f[None, :]).to(torch.float64)
    cos, sin = torch.cos(angle)[:, None, :], torch.sin(angle)[:, None, :]
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * cos - v * sin
    out[..., 1:dims:2] = v * cos + u * sin
    return out


def shifted(h, mu):
    """h_t + (h_(t-1) - h_t) * mu, zeros before the sequence's start."""
    before = torch.cat([torch.zeros(1, h.shape[1], dtype=h.dtype), h[:-1]], dim=0)
    return h + (before - h) * mu


# ------------------------------------------------------------------------------- mixers
def latent_attention(h, w, p, m, eps, low_rank_queries, gated):
    T = h.shape[0]
    H, D, R, V, C = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    h = nar(h)
    if low_rank_queries:
        q = nar(rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]) @ w[p + "uq"].T
    else:
        q = h @ w[p + "q"].T
    q = q.reshape(T, H, D + R)
    down = h @ w[p + "dkv"].T
    c = nar(rms(down[:, :C], eps) * w[p + "dkv.norm"])
    k_rot = nar(rotate_pairs(down[:, None, C:], torch.arange(T), m["rot"])[:, 0])
    q_rot = nar(rotate_pairs(q[..., D:], torch.arange(T), m["rot"]))
    q = nar(q)
    k = nar(c @ w[p + "uk"].T).reshape(T, H, D)
    v = nar(c @ w[p + "uv"].T).reshape(T, H, V)
    out = torch.zeros(T, H, V, dtype=h.dtype)
    for t in range(T):
        s = (torch.einsum("hd,jhd->hj", q[t, :, :D], k[:t + 1]) + q_rot[t] @ k_rot[:t + 1].T) * m["scale"]
        e = torch.exp(s - s.max(dim=-1, keepdim=True).values)
        out[t] = torch.einsum("hj,jhv->hv", e / e.sum(-1, keepdim=True), v[:t + 1])
    out = out.reshape(T, H * V)
    if gated:
        out = nar(out) * sigmoid(h @ w[p + "g"].T)
    return nar(out) @ w[p + "o"].T


def bonus_recurrence(r, k, v, decay, u):
    """r, k, v, decay [T, H, D], u [H, D] -> o [T, H, D]: per head, with S (key x value) from zero,
    o_t = (S + diag(u) k_t v_t^T)^T r_t, then S <- diag(decay_t) S + k_t v_t^T."""
    T, H, D = r.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=r.dtype)
    out = torch.zeros(T, H, v.shape[-1], dtype=r.dtype)
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S + u[:, :, None] * kv, r[t])
        S = decay[t][:, :, None] * S + kv
    return out


def wkv(h, w, p, m, eps):
    T = h.shape[0]
    H, D = m["heads"], m["dim"]
    mixed = {s: nar(shifted(h, w[p + "mu." + s])) for s in "rkvgw"}
    r, k, v = ((mixed[s] @ w[p + s].T).reshape(T, H, D) for s in "rkv")
    gate = silu(mixed["g"] @ w[p + "g"].T)
    decay = torch.exp(-torch.exp(nar(torch.tanh(mixed["w"] @ w[p + "w1"].T)) @ w[p + "w2"].T + w[p + "w0"])).reshape(T, H, D)
    o = rms(bonus_recurrence(r, k, v, decay, w[p + "u"]), eps).reshape(T, H * D)
    return nar(o * w[p + "norm"] * gate) @ w[p + "o"].T


def mixer(kind, h, w, p, m, eps):
    if kind == "latent_attention":
        return latent_attention(h, w, p, m, eps, True, False)
    if kind == "latent_attention_2":
        return latent_attention(h, w, p, m, eps, False, True)
    assert kind == "wkv", kind
    return wkv(h, w, p, m, eps)


# ------------------------------------------------------------------------- feed-forward
def dense(h, w, p, m):
    h = nar(h)
    g = torch.clamp(h @ w[p + "gate"].T, max=m["limit"])
    u = torch.clamp(h @ w[p + "up"].T, -m["limit"], m["limit"])
    return nar(g * sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def experts(h, w, p, m):
    h = nar(h)
    router = m["router"]
    z = h @ w[p + "router"].T
    s = torch.exp(z - z.max(-1, keepdim=True).values)
    s = s / s.sum(-1, keepdim=True)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in torch.topk(s[t], router["top"]).indices.tolist():
            a = torch.clamp(w[f"{p}e{e}.up"] @ h[t], min=0.0) ** 2
            out[t] += w[f"{p}e{e}.down"] @ nar(s[t, e] * router["scale"] * a)
    return out


def feed_forward(h, w, p, m):
    return dense(h, w, p, m) if m["kind"] == "dense" else experts(h, w, p, m)


# -------------------------------------------------------------------------------- model
def schedule(config):
    """The layers in the order in which they run."""
    order = list(range(len(config["layers"])))
    loop = config.get("loop")
    if loop:
        order[loop["start"]:loop["stop"]] = order[loop["start"]:loop["stop"]] * loop["times"]
    return order


def hyper_read(streams, a):
    """streams [S, T, n], a [S]: what the sublayer's norm reads."""
    return torch.einsum("stn,s->tn", streams, a)


def hyper_write(streams, mix, out, y):
    """New stream t = sum over s of mix[s, t] * (old stream s), plus out[t] * y."""
    return torch.einsum("stn,sz->ztn", streams, mix) + out[:, None, None] * y


def forward(config, w, tokens, dtype=torch.float64, layers_out=None, narrow=None):
    """Logits [tokens, vocab] of one whole sequence.  ``layers_out``: a list that receives the streams' sum after each layer run."""
    global _narrow
    _narrow = narrow
    try:
        return _forward(config, w, tokens, dtype, layers_out)
    finally:
        _narrow = None


def _forward(config, w, tokens, dtype, layers_out):
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in w.items()}
    eps = config["norm"]["eps"]
    factor = 1.0 if config.get("residual_mult") is None else config["residual_mult"]
    count = config.get("streams") or 1
    x = rms(w["embed"][torch.as_tensor(tokens, dtype=torch.int64)], eps) * w["embed.norm"]
    streams = x[None].repeat(count, 1, 1)
    for i in schedule(config):
        layer, p = config["layers"][i], f"l{i}."
        for q, run in ((1, lambda h: mixer(layer["type"], h, w, p + "mix.", layer["mixer"], eps)),
                       (2, lambda h: feed_forward(h, w, p + "mlp.", layer["mlp"]))):
            if q == 2 and layer.get("mlp") is None:
                continue
            hc = f"{p}hc{q}."
            h = rms(hyper_read(streams, w[hc + "in"]), eps) * w[f"{p}norm{q}"]
            y = factor * w[f"{p}ls{q}"] * run(h)
            streams = hyper_write(streams, w[hc + "mix"], w[hc + "out"], y)
        if layers_out is not None:
            layers_out.append(streams.sum(0))
    return nar(rms(streams.sum(0), eps) * w["final.norm"]) @ w["head"].T
