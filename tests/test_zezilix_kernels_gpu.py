"""The kernels that the Zezilix decoder brought, each alone against a restatement in float64: the norm of a stream in several
copies; several blends of shifted rows; the normed embedding; the recurrences with a bonus in every form; decays from a product of
low rank with tanh in front; products with activations of their own for groups of features; ungated experts as a pass and as a
product's epilogue; routing with a factor; the dense clamped unit; latent attention with a gate per output number, and prompts in the
expanded form with heads that are padded, one far key made to dominate."""
from __future__ import annotations

import pytest
import torch

pytestmark = pytest.mark.gpu

DEV = "cuda"
DTYPES = [torch.float32, torch.bfloat16]


def i32(values):
    return torch.tensor(values, dtype=torch.int32, device=DEV)


def rand(*shape, seed=0, scale=1.0):
    g = torch.Generator().manual_seed(seed)
    return torch.randn(*shape, generator=g) * scale


def status():
    return torch.zeros(1, dtype=torch.int32, device=DEV)


def close(got, want, tol, what=""):
    got, want = got.double().cpu(), want.double().cpu()
    assert got.shape == want.shape and torch.isfinite(got).all(), what
    scale = max(1.0, float(want.abs().max()))
    err = float((got - want).abs().max())
    assert err <= tol * scale, f"{what}: {err:.3e} with numbers up to {scale:.3f}"


# ------------------------------------------------------------------------------ streams
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("copies,hidden,tokens,splits", [
    (copies, *size) for copies in (1, 2, 3, 4) for size in ((128, 5, 1), (96, 3, 9), (250, 4, 2), (2056, 7, 3), (4096, 2, 16), (512, 1100, 1), (9000, 2, 1))
] + [(2, 3072, 1024, 1), (3, 6000, 1030, 2), (6, 128, 5, 1), (6, 250, 4, 9), (16, 2056, 3, 2), (5, 512, 1100, 1)])
def test_stream_norm(dtype, copies, hidden, tokens, splits):
    """Mixing, writing and reading all at once from the old copies; several slices; the spread of the first copy; wanted rows leave
    the copies alone."""
    from thintensor_b200.kernels import api

    x = rand(copies, tokens, hidden, seed=1)
    delta, gain, weight = rand(splits, tokens, hidden, seed=2), 1.0 + rand(hidden, seed=3, scale=0.3), 1.0 + rand(hidden, seed=4, scale=0.3)
    mix, write, read = rand(copies, copies, seed=5), rand(copies, seed=6), rand(copies, seed=7)
    eps, tol = 1e-5, 2e-6 if dtype == torch.float32 else 8e-3
    cuda = lambda t: t.to(DEV)

    def want(old, d, scale, gain, mix, write, read):
        old = old.double()
        y = torch.zeros(tokens, hidden, dtype=torch.float64) if d is None else scale * d.double().sum(0)
        if gain is not None:
            y = y * gain.double()
        m = torch.eye(copies, dtype=torch.float64) if mix is None else mix.double()
        w = torch.ones(copies, dtype=torch.float64) if write is None else write.double()
        r = torch.ones(copies, dtype=torch.float64) if read is None else read.double()
        new = torch.einsum("stn,sz->ztn", old, m) + w[:, None, None] * y
        u = torch.einsum("stn,s->tn", new, r)
        return new, u / torch.sqrt((u * u).mean(-1, keepdim=True) + eps) * weight.double()

    out = torch.empty(tokens, hidden, dtype=dtype, device=DEV)
    for spread, d, g, m, w, r in ((False, delta, gain, mix, write, read), (False, delta, None, None, None, None), (True, None, None, None, None, read),
                                  (True, delta, gain, mix, write, None)):
        streams = cuda(x).clone()
        opt = lambda t: None if t is None else cuda(t)
        api.stream_norm(streams, opt(d), 0.6, opt(g), opt(m), opt(w), opt(r), spread, cuda(weight), 0.0, eps, out)
        old = x[:1].expand(copies, -1, -1) if spread else x
        new, normed = want(old, d, 0.6, g, m, w, r)
        close(streams, new, 2e-6, "copies")
        close(out, normed, tol, "norm")
    rows = i32([tokens - 1, 0])
    streams = cuda(x).clone()
    picked = torch.empty(2, hidden, dtype=dtype, device=DEV)
    api.stream_norm(streams, cuda(delta), 0.6, cuda(gain), cuda(mix), cuda(write), None, False, cuda(weight), 0.0, eps, picked, rows)
    _, normed = want(x, delta, 0.6, gain, mix, write, None)
    assert torch.equal(streams.cpu(), x)
    close(picked, normed[[tokens - 1, 0]], tol, "wanted rows")


def test_stream_norm_without_a_stream_axis():
    from thintensor_b200.kernels import api

    x, d, gain, w = rand(4, 64, seed=1), rand(2, 4, 64, seed=2), rand(64, seed=3), rand(64, seed=4)
    stream = x.to(DEV).clone()
    out = torch.empty(4, 64, device=DEV)
    api.stream_norm(stream, d.to(DEV), 0.5, gain.to(DEV), None, None, None, False, w.to(DEV), 1.0, 1e-6, out)
    new = x.double() + 0.5 * gain.double() * d.double().sum(0)
    close(stream, new, 1e-6)
    close(out, new / torch.sqrt((new * new).mean(-1, keepdim=True) + 1e-6) * (w.double() + 1.0), 2e-6)
    with pytest.raises(api.KernelError):
        api.stream_norm(torch.zeros(17, 4, 64, device=DEV), None, 1.0, None, None, None, None, False, w.to(DEV), 0.0, 1e-6, out)


# ------------------------------------------------------------------- embedding and shifts
@pytest.mark.parametrize("stored", DTYPES)
@pytest.mark.parametrize("hidden", [33, 128, 2048])
def test_normed_embedding(stored, hidden):
    from thintensor_b200.kernels import api

    table, weight = rand(50, hidden, seed=1, scale=0.02).to(stored), 1.0 + rand(hidden, seed=2, scale=0.2)
    tokens = [3, 49, 0, 3]
    out, flag = torch.empty(4, hidden, device=DEV), status()
    api.embed_norm_gather(table.to(DEV), i32(tokens), weight.to(DEV), 1e-5, out, 1.5, flag)
    e = table.double()[tokens] * 1.5
    close(out, e / torch.sqrt((e * e).mean(-1, keepdim=True) + 1e-5) * weight.double(), 2e-6)
    assert int(flag) == 0
    api.embed_norm_gather(table.to(DEV), i32([3, 50]), weight.to(DEV), 1e-5, out[:2], 1.5, flag)
    assert int(flag) == api.STATUS_BAD_TOKEN and not out[1].any()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden,blends", [(64, 5), (50, 3), (2048, 5), (136, 8)])
def test_several_shifts(dtype, hidden, blends):
    """Steps of several sequences in shuffled slots, down to one token each, against whole sequences; more than 1,024 tokens take
    tiles of eight, which cross from one sequence into the next."""
    from thintensor_b200.kernels import api

    mix = torch.rand(blends, hidden, generator=torch.Generator().manual_seed(3))
    steps = [[3, 1, 700], [1, 2, 600], [1, 1, 1], [400, 5, 800]]
    rows = [rand(sum(s[b] for s in steps), hidden, seed=10 + b).to(dtype) for b in range(3)]
    state = torch.zeros(5, hidden, device=DEV)
    slots, at, got = [4, 0, 2], [0, 0, 0], [[], [], []]
    for step in steps:
        x = torch.cat([rows[b][at[b]: at[b] + n] for b, n in enumerate(step)]).to(DEV)
        cu = [0, step[0], step[0] + step[1], sum(step)]
        out = torch.empty(blends, len(x), hidden, dtype=dtype, device=DEV)
        api.token_shifts(x, mix.to(DEV), state, out, i32(cu), i32(slots), 3)
        for b in range(3):
            got[b].append(out[:, cu[b]: cu[b + 1]].cpu())
            at[b] += step[b]
    for b in range(3):
        x = rows[b].double()
        before = torch.cat([torch.zeros(1, hidden, dtype=torch.float64), x[:-1]])
        want = x[None] + (before - x)[None] * mix.double()[:, None]
        close(torch.cat(got[b], dim=1), want, 1e-6 if dtype == torch.float32 else 8e-3, f"sequence {b}")
        assert torch.equal(state[slots[b]].cpu(), rows[b][-1].float())
    assert not state[[1, 3]].any()


# --------------------------------------------------------------------------- recurrences
def bonus_reference(r, k, v, a, u, S):
    T, H, D = r.shape
    out = torch.zeros(T, H, v.shape[-1], dtype=torch.float64)
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S + u[:, :, None] * kv, r[t])
        S = a[t][:, :, None] * S + kv
    return out, S


@pytest.mark.parametrize("form", ["narrow", "wide", "blocks"])
@pytest.mark.parametrize("heads,dim,value", [(3, 24, 24), (2, 64, 40), (2, 65, 70), (1, 128, 128), (2, 200, 16), (4, 3, 5)])
def test_recurrence_with_a_bonus(form, heads, dim, value):
    """From states that are not zero, in shuffled slots, sequences of unequal lengths down to one token; the state it leaves is the
    one after the last token (the token's own update, without the bonus)."""
    from thintensor_b200.kernels import api

    lengths = [1, 2, 5, 37, 4]
    tokens, qk, vw = sum(lengths), heads * dim, heads * value
    r, k, v = rand(tokens, heads, dim, seed=1), rand(tokens, heads, dim, seed=2), rand(tokens, heads, value, seed=3)
    a = torch.rand(tokens, heads, dim, generator=torch.Generator().manual_seed(4)) * 0.6 + 0.4
    u = rand(heads, dim, seed=5)
    first = rand(7, heads, value, dim, seed=6)
    slots = [5, 0, 3, 6, 1]
    cu = [0]
    for n in lengths:
        cu.append(cu[-1] + n)
    state = first.to(DEV).clone()
    out = torch.empty(tokens, vw, device=DEV)
    vkq = torch.cat([v.reshape(tokens, vw), k.reshape(tokens, qk), r.reshape(tokens, qk)], dim=1).to(DEV).contiguous()
    decay, bonus = a.reshape(tokens, qk).to(DEV), u.reshape(-1).to(DEV)
    if form == "blocks":
        api.row_decay_blocks(vkq[:, vw + qk:], vkq[:, vw:vw + qk], vkq[:, :vw], decay, state, out, i32(cu), i32(slots), len(lengths), heads, heads, dim,
                             value, 1.0, bonus=bonus)
    else:
        api.row_decay_scan(vkq, decay, state, out, i32(cu), i32(slots), len(lengths), heads, dim, value, form, bonus=bonus)
    for b, n in enumerate(lengths):
        part = slice(cu[b], cu[b + 1])
        want, S = bonus_reference(r[part].double(), k[part].double(), v[part].double(), a[part].double(), u.double(),
                                  first[slots[b]].double().transpose(1, 2))
        close(out[part].reshape(n, heads, value), want, 3e-6, f"sequence {b}")
        close(state[slots[b]].transpose(1, 2), S, 3e-6, f"state {b}")
    for slot in (2, 4):
        assert torch.equal(state[slot].cpu(), first[slot])


@pytest.mark.parametrize("tokens", [3, 200])
@pytest.mark.parametrize("rank,cols", [(16, 96), (13, 40), (200, 64)])
def test_decays_of_low_rank(tokens, rank, cols):
    """``exp(-exp(W tanh(x) + b))`` in the kernel for few tokens, and as inputs and finish around a product of its own."""
    from thintensor_b200.kernels import api

    proj, w, bias = rand(3, tokens, rank + 11, seed=1, scale=0.7), rand(cols, rank, seed=2, scale=0.4), rand(cols, seed=3)
    x = torch.tanh(proj.double().sum(0)[:, 7:7 + rank])
    want = torch.exp(-torch.exp(x @ w.double().T + bias.double()))
    out = torch.empty(tokens, cols, device=DEV)
    api.low_rank(proj.to(DEV), [api.LowRank(7, w.t().contiguous().to(DEV), out, "exp_decay", bias.to(DEV), tanh=True)])
    close(out, want, 3e-6)
    inputs = torch.empty(tokens, rank, device=DEV)
    api.low_rank_inputs(proj.to(DEV), [(7, inputs, True)])
    close(inputs, x, 2e-6)
    z = torch.empty(1, tokens, cols, device=DEV)
    api.gemm_simt(inputs, w.to(DEV), None, z)
    api.low_rank_finish(z, "exp_decay", bias.to(DEV), z[0])
    close(z[0], want, 3e-6)


# ------------------------------------------------------------------------------ products
@pytest.mark.parametrize("tokens,k,rows,last", [(1, 128, 128, 16), (8, 2048, 256, 40), (40, 136, 384, 384), (130, 256, 256, 24), (300, 512, 512, 64),
                                                (700, 1024, 512, 8), (2100, 192, 256, 100)])
def test_grouped_product(tokens, k, rows, last):
    """Every group of features reads rows of its own, at token counts that are no multiple of a tile, so that a group's last tile
    of rows runs into the next group's."""
    from thintensor_b200.engine.context import StepContext, Workspace
    from thintensor_b200.kernels import api
    from thintensor_b200.parts.linear import GroupedLinear

    groups = 4
    x = rand(groups, tokens, k, seed=1).to(torch.bfloat16)
    weights = [rand(n, k, seed=2 + i, scale=k ** -0.5).to(torch.bfloat16) for i, n in enumerate([rows] * (groups - 1) + [last])]
    flag = status()
    ctx = StepContext(tokens, 1, False, tokens, tokens, None, None, None, None, [], torch.bfloat16, Workspace(torch.device(DEV)), flag)
    linear = GroupedLinear([w.to(DEV) for w in weights])
    assert api.gemm_tcgen05_groups_takes(x.to(DEV), linear.fused.weight, rows)
    for _ in range(2):                                  # the second call finds the flags of shared tiles as the first left them
        got = linear(ctx, x.to(DEV), "grouped").sum(0)
        want = torch.cat([x[i].double() @ w.double().T for i, w in enumerate(weights)], dim=1)
        close(got, want, 2e-5)
    assert int(flag) == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens,k,rows,last", [(5, 520, 100, 7), (33, 72, 192, 40), (150, 128, 96, 16), (600, 64, 320, 400), (20, 50, 30, 5)])
def test_grouped_product_group_by_group(dtype, tokens, k, rows, last):
    """Groups that no tile fits, float32, and a last group larger than the others: a product for each, into its columns."""
    from thintensor_b200.engine.context import StepContext, Workspace
    from thintensor_b200.kernels import api
    from thintensor_b200.parts.linear import GroupedLinear

    x = rand(3, tokens, k, seed=1).to(dtype)
    weights = [rand(n, k, seed=2 + i, scale=k ** -0.5).to(dtype) for i, n in enumerate([rows, rows, last])]
    flag = status()
    ctx = StepContext(tokens, 1, False, tokens, tokens, None, None, None, None, [], dtype, Workspace(torch.device(DEV)), flag)
    linear = GroupedLinear([w.to(DEV) for w in weights])
    assert not api.gemm_tcgen05_groups_takes(x.to(DEV), linear.fused.weight, rows)
    got = linear(ctx, x.to(DEV), "grouped")
    close(got.sum(0), torch.cat([x[i].double() @ w.double().T for i, w in enumerate(weights)], dim=1), 2e-5)
    assert int(flag) == 0


UNARY = {"relu2": lambda z: torch.clamp(z, min=0.0) ** 2, "relu": lambda z: torch.clamp(z, min=0.0), "silu": lambda z: z / (1.0 + torch.exp(-z)),
         "gelu_tanh": lambda z: 0.5 * z * (1.0 + torch.tanh((2.0 / torch.pi) ** 0.5 * (z + 0.044715 * z ** 3)))}


@pytest.mark.parametrize("activation", list(UNARY))
@pytest.mark.parametrize("tokens,k,experts,width", [(300, 128, 8, 128), (129, 256, 4, 256), (530, 512, 2, 384), (2100, 192, 16, 128), (1025, 64, 6, 256)])
def test_ungated_experts_in_the_product(activation, tokens, k, experts, width):
    """The activation and the routing weights as the product's epilogue against the pass over the float32 product, and both
    against the restatement; nothing is written behind the output."""
    from thintensor_b200.kernels import api

    x, w = rand(tokens, k, seed=1).to(torch.bfloat16), rand(experts * width, k, seed=2, scale=k ** -0.5).to(torch.bfloat16)
    gates = torch.rand(tokens, experts + 1, generator=torch.Generator().manual_seed(3)) * (torch.rand(tokens, experts + 1) < 0.5)
    flag = status()
    assert api.gemm_tcgen05_unary_takes(x.to(DEV), w.to(DEV), width, activation)
    buffer = torch.full((tokens + 3, experts * width), 7.0, dtype=torch.bfloat16, device=DEV)
    act = buffer[:tokens]
    api.gemm_tcgen05_unary(x.to(DEV), w.to(DEV), act, flag, activation, gates.to(DEV), width)
    z = x.double() @ w.double().T
    want = UNARY[activation](z) * gates.double()[:, :experts].repeat_interleave(width, dim=1)
    close(act, want, 6e-3)
    assert bool((buffer[tokens:] == 7.0).all()) and int(flag) == 0
    passed = torch.empty_like(act)
    up = torch.stack([z * 0.25, z * 0.75]).float().to(DEV)
    api.expert_unary_activation(up, passed, width, activation, gates.to(DEV))
    close(passed, want, 6e-3)
    api.gemm_tcgen05_unary(x.to(DEV), w.to(DEV), act, flag, activation)                   # without factors
    close(act, UNARY[activation](z), 6e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens,experts,width", [(1, 3, 7), (9, 5, 40), (33, 1, 12)])
def test_ungated_experts_pass(dtype, tokens, experts, width):
    from thintensor_b200.kernels import api

    up = rand(3, tokens, experts * width, seed=1)
    gates = torch.rand(tokens, experts, generator=torch.Generator().manual_seed(3))
    gates[0, 0] = 0.0
    for activation in UNARY:
        act = torch.empty(tokens, experts * width, dtype=dtype, device=DEV)
        api.expert_unary_activation(up.to(DEV), act, width, activation, gates.to(DEV))
        close(act, UNARY[activation](up.double().sum(0)) * gates.double().repeat_interleave(width, dim=1), 2e-6 if dtype == torch.float32 else 6e-3)
    act = torch.empty(tokens, experts * width, dtype=dtype, device=DEV)
    api.activation(up.to(DEV), act, "relu2")
    close(act, UNARY["relu2"](up.double().sum(0)), 2e-6 if dtype == torch.float32 else 6e-3)


@pytest.mark.parametrize("experts,top,scale", [(9, 4, 2.2), (5, 5, 0.4), (40, 1, 1.0)])
def test_routing_with_a_factor(experts, top, scale):
    """Weights are the softmax's scores over all experts times the factor, not renormalised; both kernels."""
    from thintensor_b200.kernels import api

    x, w = rand(21, 96, seed=1), rand(experts, 96, seed=2, scale=0.3)
    s = torch.softmax(x.double() @ w.double().T, dim=-1)
    best = torch.topk(s, top)
    dense = torch.zeros(21, experts, dtype=torch.float64).scatter(1, best.indices, best.values * scale)
    gates, chosen, weights = torch.empty(21, experts, device=DEV), torch.empty(21, top, dtype=torch.int32, device=DEV), torch.empty(21, top, device=DEV)
    api.route_rows(x.to(DEV), w.to(DEV), top, 1, 1, gates, chosen, weights, renormalize=False, weight_scale=scale)
    close(gates, dense, 3e-6)
    close(weights, best.values * scale, 3e-6)
    logits = (x @ w.T)[None].to(DEV).contiguous()
    api.route_topk(logits, top, 1, 1, gates, chosen, weights, renormalize=False, weight_scale=scale)
    close(gates, dense, 3e-6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens", [1, 20, 200, 600])
def test_dense_clamped_unit(dtype, tokens):
    """The clamp on both sides of both factors, as a pass and as a product's epilogue."""
    from thintensor_b200.engine.context import StepContext, Workspace
    from thintensor_b200.parts.linear import GatedLinear

    x = rand(tokens, 128, seed=1).to(dtype)
    gate, up = rand(512, 128, seed=2, scale=0.15).to(dtype), rand(512, 128, seed=3, scale=0.15).to(dtype)
    ctx = StepContext(tokens, 1, False, tokens, tokens, None, None, None, None, [], dtype, Workspace(torch.device(DEV)), status())
    linear = GatedLinear(gate.to(DEV), up.to(DEV), None, None, "clamped", 1.2, 1.702)
    g, u = (x.double() @ gate.double().T).clamp(max=1.2), (x.double() @ up.double().T).clamp(-1.2, 1.2)
    assert bool((g == 1.2).any()) and bool((u == 1.2).any()) and bool((u == -1.2).any())
    close(linear(ctx, x.to(DEV), "unit"), g / (1.0 + torch.exp(-1.702 * g)) * (u + 1.0), 1e-5 if dtype == torch.float32 else 8e-3)


# --------------------------------------------------------------------- latent attention
def latent_case(dtype, totals, heads, dim, rot, vdim, rank, q_rank, gate, seed, dominate):
    """A latent attention part with random weights, a cache for it and input rows for sequences of ``totals`` tokens.  ``dominate``:
    (sequence, position) of a row that is longer than the others, so that the keys' rotated part there (which no norm shortens) makes
    one score of every query stand out."""
    from thintensor_b200.cache.cache import SequenceCache
    from thintensor_b200.parts.base import MIXERS
    from thintensor_b200.parts.spec import PartSpec

    hidden = 96
    part = MIXERS.build("latent_attention", {
        "hidden": hidden, "heads": heads, "dim": dim, "rot_dim": rot, "value_dim": vdim, "q_rank": q_rank, "kv_rank": rank, "scale": 0.3,
        "eps": 1e-5, "gate": gate, "position": PartSpec("rope", {"head_dim": rot, "theta": 1000.0, "interleaved": True, "table_precision": "float64"})})
    w = {}
    for i, (name, decl) in enumerate(part.weights().items()):
        w[name] = (1.0 + rand(*decl.shape, seed=seed + i, scale=0.2)) if "norm" in name else rand(*decl.shape, seed=seed + i, scale=decl.shape[-1] ** -0.5)
        w[name] = w[name].to(dtype)
    part.bind({k: v.to(DEV) for k, v in w.items()}, dtype, torch.device(DEV))
    cache = SequenceCache([part.cache_need()], [[]], [None], 32, 4, dtype, torch.device(DEV))
    rows = [rand(n, hidden, seed=seed + 50 + i) for i, n in enumerate(totals)]
    rows[dominate[0]][dominate[1]] = rand(hidden, seed=seed + 99) * 4.0
    rows = [x.to(dtype) for x in rows]
    return part, w, cache, rows


def plain_latent(x, w, heads, dim, rot, vdim, rank, q_rank, gate):
    import plain_zezilix as plain

    n = {"q_a_proj.weight": "dq", "q_a_norm.weight": "dq.norm", "q_b_proj.weight": "uq", "kv_a_proj.weight": "dkv", "kv_a_norm.weight": "dkv.norm",
         "k_b_proj.weight": "uk", "v_b_proj.weight": "uv", "o_proj.weight": "o", "q_proj.weight": "q", "g_proj.weight": "g"}
    named = {n[k]: v.double() for k, v in w.items()}
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": 0.3, "rot": {"dims": rot, "base": 1000.0}}
    return plain.latent_attention(x.double(), named, "", m, 1e-5, q_rank is not None, gate is not None)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,rot,vdim,rank,q_rank,gate", [
    (3, 20, 12, 40, 48, None, "elementwise"), (4, 72, 32, 100, 64, None, "elementwise"), (2, 64, 64, 128, 64, 40, None), (2, 32, 32, 64, 32, None, "elementwise"),
    (5, 100, 60, 24, 40, 24, "elementwise"), (2, 30, 6, 7, 24, 16, "elementwise")])
def test_latent_attention_part(dtype, heads, dim, rot, vdim, rank, q_rank, gate):
    """The part through a cache, in portions (expanded ones and small ones) and token by token, beside a second sequence, with one far
    key that dominates: bfloat16 prompts run the padded heads on the tensor cores."""
    from thintensor_b200.engine.context import StepContext, Workspace

    new_tokens = [[150, 3], [140, 60], [1, 1], [1, 1], [2, 130]]
    part, w, cache, rows = latent_case(dtype, [sum(s[b] for s in new_tokens) for b in range(2)], heads, dim, rot, vdim, rank, q_rank, gate, 700 + heads,
                                       (0, 3))
    workspace, flag = Workspace(torch.device(DEV)), status()
    slots = [cache.alloc_slot() for _ in range(2)]
    at, got = [0, 0], [[], []]
    for step in new_tokens:
        for b in range(2):
            cache.reserve(slots[b], at[b] + step[b])
        table = torch.tensor(cache.table_rows(0, slots, 8), dtype=torch.int32, device=DEV)
        x = torch.cat([rows[b][at[b]: at[b] + n] for b, n in enumerate(step)]).to(DEV)
        cu, tokens = [0, step[0], sum(step)], sum(step)
        ctx = StepContext(tokens, 2, step == [1, 1], max(step), max(a + n for a, n in zip(at, step)), None, i32(cu), i32(at), i32(slots), [table],
                          dtype, workspace, flag)
        out = part.forward(ctx, x.contiguous(), cache.run_cache(0), [])
        out = out.tensor.sum(0).cpu()
        for b in range(2):
            got[b].append(out[cu[b]: cu[b + 1]])
            cache.advance(slots[b], step[b])
            at[b] += step[b]
    assert int(flag) == 0
    for b in range(2):
        want = plain_latent(rows[b], w, heads, dim, rot, vdim, rank, q_rank, gate)
        result = torch.cat(got[b]).double()
        if dtype == torch.float32:
            close(result, want, 2e-5, f"sequence {b}")
        else:
            cos = torch.nn.functional.cosine_similarity(result, want, dim=-1)
            assert float(cos.min()) > 0.99 and float(cos.mean()) > 0.9995, f"sequence {b}: cosine {float(cos.min())}, mean {float(cos.mean())}"
