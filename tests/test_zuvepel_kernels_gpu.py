"""The kernels behind the Zuvepel parts, each alone against a plain float64 restatement written here, at other sizes than
the engine tests': two scaled branches and an addend added into the stream with two norms of the sum; products of low rank
and what is made of them; both recurrences with decays per key channel, token by token and four tokens at a time, from
states that are not zero, with unequal sequences, scrambled slots and sequences that end anywhere in a block; linear
attention's preparation with scaled queries; attention over the query's own chunk with a constant null score, one key made
to dominate at a chunk's first place and at the last place of the chunk before, in prompts and in decoding, keys in one slice
and in several, on the exact and on the tensor-core kernels."""
from __future__ import annotations

import math

import pytest
import torch

from test_kerepel_kernels_gpu import fill_pools, i32, scrambled_pools, status

pytestmark = pytest.mark.gpu

DEV = "cuda"


def randn(*shape, seed, scale=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=torch.float32) * scale


def slices(x: torch.Tensor, n: int, seed: int) -> torch.Tensor:
    """x as n partial sums [n, ...]."""
    parts = [randn(*x.shape, seed=seed + i) for i in range(n - 1)]
    return torch.stack(parts + [x - sum(parts)] if parts else [x])


# ---------------------------------------------------------------------------------- norms
def norm_plain(x, w, b, eps, centered, offset=0.0):
    if centered:
        x = x - x.mean(-1, keepdim=True)
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * (w + offset)
    return y if b is None else y + b


@pytest.mark.parametrize("rows,hidden", [(5, 72), (3, 333), (4, 4100), (1100, 256), (2, 2048)])
@pytest.mark.parametrize("out_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("a_splits,b_splits,addend,two,centered", [(1, 1, True, True, True), (3, 10, False, True, True), (0, 0, True, True, True),
                                                                   (2, 0, False, False, True), (1, 2, True, True, False), (9, 1, True, False, False)])
def test_branches_addend_and_two_norms(rows, hidden, out_dtype, a_splits, b_splits, addend, two, centered):
    from thintensor_b200.kernels import api

    residual = randn(rows, hidden, seed=1) + 2.0                # a mean far from zero: forgetting to take it off shows
    a = randn(a_splits, rows, hidden, seed=2) if a_splits else None
    b = randn(b_splits, rows, hidden, seed=3) if b_splits else None
    more = randn(rows, hidden, seed=4) if addend else None
    w1, w2, b1, b2 = 1.0 + randn(hidden, seed=5, scale=0.2), randn(hidden, seed=6), randn(hidden, seed=7), randn(hidden, seed=8)
    if not centered:
        b1 = b2 = None
    offset = 0.0 if centered else 1.0
    scale, eps = 0.37, 1e-5
    x = residual.double()
    for branch in (a, b):
        if branch is not None:
            x = x + scale * branch.double().sum(0)
    if addend:
        x = x + more.double()
    dev = lambda t: None if t is None else t.to(DEV)
    for pick in (None, [rows - 1, 0, rows - 1]):
        n = rows if pick is None else len(pick)
        res = residual.clone().to(DEV)
        out1 = torch.empty(n, hidden, dtype=out_dtype, device=DEV)
        out2 = torch.empty(n, hidden, dtype=out_dtype, device=DEV)
        api.add_norms(res, dev(a), dev(b), scale, dev(more), dev(w1), dev(b1), out1, eps, centered, offset, (dev(w2), dev(b2), out2) if two else None,
                      None if pick is None else i32(pick))
        rows_x = x if pick is None else x[pick]
        tol = 3e-5 if out_dtype == torch.float32 else 2e-2
        for out, w, shift in ((out1, w1, b1),) + (((out2, w2, b2),) if two else ()):
            want = norm_plain(rows_x, w.double(), None if shift is None else shift.double(), eps, centered, offset)
            assert float((out.double().cpu() - want).abs().max()) <= tol * float(want.abs().max())
        kept = x if pick is None else residual.double()
        assert float((res.double().cpu() - kept).abs().max()) <= 1e-5 * float(kept.abs().max())


# ------------------------------------------------------------------------------- low rank
@pytest.mark.parametrize("tokens", [1, 7, 9, 128, 300])
@pytest.mark.parametrize("weights", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("splits,rank_a,heads,dim,rank_b,n_b", [(1, 16, 4, 24, 130, 66), (3, 5, 3, 7, 24, 77), (2, 129, 2, 136, 1, 600)])
def test_low_rank_products(tokens, weights, splits, rank_a, heads, dim, rank_b, n_b):
    """A decay and a plain product from neighbouring and from separate columns of one projection, in one launch and alone."""
    from thintensor_b200.kernels import api

    n_a, off = heads * dim, 3
    cols = off + rank_a + 2 + rank_b + 1
    x = randn(tokens, cols, seed=10)
    proj = slices(x, splits, 20).to(DEV)
    x = proj.double().sum(0).cpu()
    w_a, w_b = randn(n_a, rank_a, seed=11, scale=1.5 / math.sqrt(rank_a)).to(weights), randn(n_b, rank_b, seed=12).to(weights)
    bias, a_log, tau = randn(n_a, seed=13), randn(heads, seed=14), 7.0
    z = x[:, off: off + rank_a] @ w_a.double().T + bias.double()
    want_b = x[:, off + rank_a + 2: off + rank_a + 2 + rank_b] @ w_b.double().T
    delta = torch.exp(-torch.exp(a_log.double()).repeat_interleave(dim) * torch.nn.functional.softplus(z))
    root = torch.sigmoid(z) ** (1.0 / tau)
    up_a, up_b = w_a.t().contiguous().to(DEV), w_b.t().contiguous().to(DEV)
    out_a = torch.full((tokens, n_a), float("nan"), device=DEV)
    out_b = torch.full((tokens, n_b), float("nan"), device=DEV)
    second = api.LowRank(off + rank_a + 2, up_b, out_b)
    api.low_rank(proj, [api.LowRank(off, up_a, out_a, "delta_decay", bias.to(DEV), a_log.to(DEV), dim), second])
    assert float((out_a.double().cpu() - delta).abs().max()) <= 2e-5
    assert float((out_b.double().cpu() - want_b).abs().max()) <= 2e-5 * float(want_b.abs().max())
    out_a.fill_(float("nan"))
    api.low_rank(proj, [api.LowRank(off, up_a, out_a, "sigmoid_root", bias.to(DEV), tau=tau)])
    assert float((out_a.double().cpu() - root).abs().max()) <= 2e-5
    # the pieces of the form for many tokens
    for dtype in (torch.float32, torch.bfloat16):
        in_a, in_b = (torch.empty(tokens, n, dtype=dtype, device=DEV) for n in (rank_a, rank_b))
        api.low_rank_inputs(proj, [(off, in_a, False), (off + rank_a + 2, in_b, False)])
        for got, lo in ((in_a, off), (in_b, off + rank_a + 2)):
            want = x[:, lo: lo + got.shape[1]]
            assert float((got.double().cpu() - want).abs().max()) <= (1e-5 if dtype == torch.float32 else 5e-3) * float(want.abs().max())
    product = slices((z - bias.double()).float(), splits, 30).to(DEV)
    api.low_rank_finish(product, "delta_decay", bias.to(DEV), out_a, a_log.to(DEV), dim)
    assert float((out_a.double().cpu() - delta).abs().max()) <= 2e-5
    api.low_rank_finish(product, "sigmoid_root", bias.to(DEV), product[0], tau=tau)         # in place
    assert float((product[0].double().cpu() - root).abs().max()) <= 2e-5


# ---------------------------------------------------------------------------- recurrences
def delta_plain(q, k, v, beta, decay, S):
    """q, k [T, G, D], v [T, H, V], beta [T, H], decay [T, H, D], S [H, D, V] -> read-outs [T, H, V], S."""
    T, G, D = q.shape
    H = v.shape[1]
    unit = lambda x: x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)
    q, k = unit(q) * D ** -0.5, unit(k)
    S, out = S.clone(), torch.zeros_like(v)
    for t in range(T):
        for h in range(H):
            g = h // (H // G)
            S[h] = decay[t, h][:, None] * S[h]
            S[h] += torch.outer(k[t, g], beta[t, h] * (v[t, h] - S[h].T @ k[t, g]))
            out[t, h] = S[h].T @ q[t, g]
    return out, S


def linear_plain(q, k, v, decay, S):
    S, out = S.clone(), torch.zeros_like(v)
    for t in range(q.shape[0]):
        S = decay[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out, S


NEWS = [[1, 1, 1], [3, 17, 4], [33, 2, 21], [16, 5, 48]]
SIZES = [(4, 2, 24, 40), (3, 1, 136, 8), (2, 2, 64, 33), (6, 3, 5, 17), (1, 1, 128, 16), (2, 1, 256, 20), (3, 3, 3, 1)]


def decays(T, H, D, seed):
    """Between almost nothing kept and almost everything, and the two ends themselves."""
    a = torch.rand(T, H, D, generator=torch.Generator().manual_seed(seed), dtype=torch.float32) ** 0.2
    a[::3, :, 0] = 1.0
    a[1::5, :, -1] = 0.0
    return a


@pytest.mark.parametrize("form", ["narrow", "wide", "blocks"])
@pytest.mark.parametrize("heads,qk_heads,D,V", SIZES)
def test_delta_rule_with_channel_decays(heads, qk_heads, D, V, form):
    """Steps that continue one another, sequences of unequal lengths in scrambled slots; a wrong order of decay, read and
    write, or a state that a step leaves behind wrong, shows in the next step's read-outs."""
    from thintensor_b200.kernels import api

    if form == "wide" and D > 128:
        pytest.skip("the wide form holds up to 128 rows")
    slot_ids = [4, 0, 2]
    state = torch.zeros(6, heads, V, D, dtype=torch.float32, device=DEV)
    kept = {s: randn(heads, D, V, seed=50 + s).double() for s in slot_ids}
    for s in slot_ids:
        state[s] = kept[s].transpose(1, 2).float().to(DEV)
    qk, hv, b_col = qk_heads * D, heads * V, 5
    for step, news in enumerate(NEWS):
        tokens = sum(news)
        qkv = randn(tokens, 2 * qk + hv, seed=60 + step)
        proj = slices(randn(tokens, b_col + heads + 2, seed=70 + step), 1 + step % 3, 80)
        raw = proj.double().sum(0)[:, b_col: b_col + heads]
        g = decays(tokens, heads, D, 90 + step)
        out = torch.full((tokens, hv), float("nan"), device=DEV)
        cu = i32([0] + torch.tensor(news).cumsum(0).tolist())
        dev = qkv.to(DEV)
        if form == "blocks":
            api.row_decay_blocks(dev[:, :qk], dev[:, qk: 2 * qk], dev[:, 2 * qk:], g.reshape(tokens, -1).to(DEV), state, out, cu, i32(slot_ids), len(news),
                                 heads, qk_heads, D, V, D ** -0.5, (proj.to(DEV), b_col))
        else:
            api.delta_scan(dev, proj.to(DEV), b_col, 0, None, None, state, out, cu, i32(slot_ids), len(news), heads, qk_heads, D, V, form,
                           g.reshape(tokens, -1).to(DEV))
        at = 0
        for s, n in zip(slot_ids, news):
            x = qkv[at: at + n].double()
            want, kept[s] = delta_plain(x[:, :qk].reshape(n, qk_heads, D), x[:, qk: 2 * qk].reshape(n, qk_heads, D), x[:, 2 * qk:].reshape(n, heads, V),
                                        torch.sigmoid(raw[at: at + n]), g[at: at + n].double(), kept[s])
            got = out[at: at + n].double().cpu().reshape(n, heads, V)
            assert float((got - want).abs().max()) <= 2e-5 * max(1.0, float(want.abs().max())), (step, s)
            held = state[s].double().cpu().transpose(1, 2)
            assert float((held - kept[s]).abs().max()) <= 2e-5 * max(1.0, float(kept[s].abs().max())), (step, s)
            at += n
    assert float(state[[1, 3, 5]].abs().max()) == 0.0           # other slots are not touched


@pytest.mark.parametrize("form", ["narrow", "wide", "blocks"])
@pytest.mark.parametrize("heads,D,V", [(h, d, v) for h, _, d, v in SIZES])
def test_linear_attention_with_channel_decays(heads, D, V, form):
    from thintensor_b200.kernels import api

    if form == "wide" and D > 128:
        pytest.skip("the wide form holds up to 128 rows")
    slot_ids = [1, 5, 0]
    state = torch.zeros(6, heads, V, D, dtype=torch.float32, device=DEV)
    kept = {s: randn(heads, D, V, seed=150 + s).double() for s in slot_ids}
    for s in slot_ids:
        state[s] = kept[s].transpose(1, 2).float().to(DEV)
    qk, hv = heads * D, heads * V
    for step, news in enumerate(NEWS):
        tokens = sum(news)
        vkq = randn(tokens, hv + 2 * qk, seed=160 + step)
        g = decays(tokens, heads, D, 190 + step)
        out = torch.full((tokens, hv), float("nan"), device=DEV)
        cu = i32([0] + torch.tensor(news).cumsum(0).tolist())
        dev, scale = vkq.to(DEV), 1.0
        if form == "blocks":
            scale = 0.6
            api.row_decay_blocks(dev[:, hv + qk:], dev[:, hv: hv + qk], dev[:, :hv], g.reshape(tokens, -1).to(DEV), state, out, cu, i32(slot_ids), len(news),
                                 heads, heads, D, V, scale)
        else:
            api.row_decay_scan(dev, g.reshape(tokens, -1).to(DEV), state, out, cu, i32(slot_ids), len(news), heads, D, V, form)
        at = 0
        for s, n in zip(slot_ids, news):
            x = vkq[at: at + n].double()
            want, kept[s] = linear_plain(x[:, hv + qk:].reshape(n, heads, D) * scale, x[:, hv: hv + qk].reshape(n, heads, D),
                                         x[:, :hv].reshape(n, heads, V), g[at: at + n].double(), kept[s])
            got = out[at: at + n].double().cpu().reshape(n, heads, V)
            assert float((got - want).abs().max()) <= 2e-5 * max(1.0, float(want.abs().max())), (step, s)
            held = state[s].double().cpu().transpose(1, 2)
            assert float((held - kept[s]).abs().max()) <= 2e-5 * max(1.0, float(kept[s].abs().max())), (step, s)
            at += n
    assert float(state[[2, 3, 4]].abs().max()) == 0.0


def test_forms_agree_over_a_long_sequence():
    """600 tokens of one sequence: four at a time in two steps that are cut inside a block, against token by token."""
    from thintensor_b200.kernels import api

    heads, D, V, T = 2, 48, 24, 600
    qkv, beta = randn(T, heads * (2 * D + V), seed=200).to(DEV), randn(1, T, heads, seed=201).to(DEV)
    g = decays(T, heads, D, 202).reshape(T, -1).to(DEV)
    one, two = (torch.zeros(1, heads, V, D, device=DEV) for _ in range(2))
    a, b = (torch.empty(T, heads * V, device=DEV) for _ in range(2))
    api.delta_scan(qkv, beta, 0, 0, None, None, one, a, i32([0, T]), i32([0]), 1, heads, heads, D, V, "narrow", g)
    for lo, hi in ((0, 333), (333, T)):
        x = qkv[lo:hi]
        api.row_decay_blocks(x[:, :heads * D], x[:, heads * D: 2 * heads * D], x[:, 2 * heads * D:], g[lo:hi].contiguous(), two, b[lo:hi],
                             i32([0, hi - lo]), i32([0]), 1, heads, heads, D, V, D ** -0.5, (beta[:, lo:hi].contiguous(), 0))
    assert float((a - b).abs().max()) <= 1e-5 * max(1.0, float(a.abs().max()))
    assert float((one - two).abs().max()) <= 1e-5 * max(1.0, float(one.abs().max()))


def test_linear_attention_preparation_scales_queries_and_keys():
    from thintensor_b200.kernels import api

    heads, D, V, tokens = 3, 10, 7, 5
    proj = slices(randn(tokens, heads * (2 * D + V) + 4, seed=210), 2, 211).to(DEV)
    vkq = torch.empty(tokens, heads * (2 * D + V), device=DEV)
    api.linear_attention_prepare(proj, heads, D, V, False, None, 0, 0.5, vkq, i32([0, tokens]), i32([3]), 1, tokens, 0.25)
    x, qk = proj.double().sum(0).cpu(), heads * D
    want = torch.cat([x[:, 2 * qk: 2 * qk + heads * V], 0.5 * x[:, qk: 2 * qk], 0.25 * x[:, :qk]], dim=1)
    assert float((vkq.double().cpu() - want).abs().max()) <= 1e-5


# ------------------------------------------------------------------------------ attention
def chunk_plain(q, keys, values, pos, heads, kv_heads, scale, chunk, null):
    lo = 0 if not chunk else pos // chunk * chunk
    out = []
    for h in range(heads):
        g = h // (heads // kv_heads)
        s = torch.cat([(keys[lo:pos + 1, g] @ q[h]) * scale, torch.tensor([null], dtype=torch.float64)])
        out.append(torch.softmax(s, dim=0)[:-1] @ values[lo:pos + 1, g])
    return torch.cat(out)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,chunk,null", [
    (4, 2, 64, 64, 90, 0.0), (6, 2, 16, 24, 21, 0.0), (3, 3, 20, 36, 64, 2.5), (4, 1, 128, 128, 65, 0.0), (2, 2, 32, 32, 1, 0.0),
    (8, 2, 64, 64, 7, 0.0), (5, 1, 96, 96, 129, -1.0), (4, 4, 64, 64, 0, 0.0), (14, 2, 128, 128, 1000, 0.0), (2, 1, 48, 80, 150, 0.0)])
def test_chunks_and_null_score(dtype, heads, kv_heads, dim, vdim, chunk, null):
    """Sequences of unequal lengths, prompts over several chunks and decoding, through a scrambled table.  In every sequence
    a key is lined up with the last query of head 0: the first key of its chunk for two sequences, the last key of the chunk
    before for the other two.  Seen or not, it decides that token's output.  Another token's scores are all far below the
    null score, which then takes nearly all the weight."""
    from thintensor_b200.kernels import api

    g = torch.Generator().manual_seed(heads * 100 + dim + chunk)
    scale = 0.3 / math.sqrt(dim)
    totals, new = [300, 411, 200, 131], [120, 1, 200, 1]
    k_pool, v_pool, table = scrambled_pools(totals, kv_heads, dim, vdim, dtype, 13)
    cached, queries = [], []
    moved = 0
    for b, n in enumerate(totals):
        keys = torch.randn(n, kv_heads, dim, generator=g, dtype=torch.float64)
        values = torch.randn(n, kv_heads, vdim, generator=g, dtype=torch.float64) + 1.0
        q = torch.randn(new[b], heads, dim, generator=g, dtype=torch.float64).to(dtype).double()
        last = n - 1
        start = last // chunk * chunk if chunk else 0
        marked = start if b in (0, 3) else max(start - 1, 0)
        if new[b] > 1:                      # every key of head 0 leans away from one query, whose scores are all about -30
            keys[:, 0] -= q[-2, 0] / q[-2, 0].norm() ** 2 * 30.0 / scale
        keys[marked, 0] = q[-1, 0] / q[-1, 0].norm() ** 2 * 30.0 / scale
        cached.append(fill_pools(k_pool, v_pool, table, b, keys, values))
        queries.append(q)
    q_all, cu = torch.cat(queries), [0]
    for n in new:
        cu.append(cu[-1] + n)
    tokens, before = q_all.shape[0], [t - n for t, n in zip(totals, new)]
    want = torch.stack([chunk_plain(queries[b][i], *cached[b], before[b] + i, heads, kv_heads, scale, chunk, null) for b in range(4) for i in range(new[b])])
    if 1 < chunk < 300:                     # planted in the oracle: without chunks a marked token's output is another
        for b in range(4):
            other = chunk_plain(queries[b][-1], cached[b][0], cached[b][1], totals[b] - 1, heads, kv_heads, scale, 0, null)
            moved += float((other - want[cu[b + 1] - 1]).abs().max()) > 0.2
        assert moved >= 1
    sinks = torch.full((heads,), null, dtype=torch.float32, device=DEV)
    top = max(1.0, float(want.abs().max()))
    decoding = [b for b in range(4) if new[b] == 1]
    for splits in (1, 3):
        pick = decoding if splits > 1 else list(range(4))
        rows_of = [r for b in pick for r in range(cu[b], cu[b + 1])]
        cu_step = [0]
        for b in pick:
            cu_step.append(cu_step[-1] + new[b])
        out = torch.zeros(len(rows_of), heads * vdim, dtype=dtype, device=DEV)
        parts = [torch.zeros(len(rows_of) * heads * splits * n, dtype=torch.float32, device=DEV) for n in (vdim, 2)]
        word = status()
        api.attention(q_all[rows_of].reshape(len(rows_of), -1).to(dtype).to(DEV), k_pool, v_pool, table[pick].contiguous(), i32(cu_step),
                      i32([before[b] for b in pick]), len(pick), len(rows_of), heads, kv_heads, dim, scale, -chunk, splits, out, *parts, word,
                      value_dim=vdim, sinks=sinks)
        assert int(word.item()) == 0
        assert float((out.double().cpu() - want[rows_of]).abs().max()) <= (2e-5 if dtype == torch.float32 else 0.03) * top, splits
    if dtype != torch.bfloat16 or dim != vdim:
        return
    if api.attention_tcgen05_supports(dtype, heads, kv_heads, dim):
        out = torch.zeros(tokens, heads * vdim, dtype=dtype, device=DEV)
        word = status()
        api.attention_tcgen05(q_all.reshape(tokens, -1).to(dtype).to(DEV), k_pool, v_pool, table, i32(cu), i32(before), 4, tokens, heads, kv_heads, dim,
                              scale, -chunk, out, word, sinks=sinks)
        assert int(word.item()) == 0
        assert float((out.double().cpu() - want).abs().max()) <= 0.04 * top
    if api.attention_mma_supports(dtype, heads, kv_heads, dim):
        rows_of = [cu[b] for b in decoding]
        for splits in (1, 2, 11):
            out = torch.zeros(len(decoding), heads * vdim, dtype=dtype, device=DEV)
            parts = [torch.zeros(len(decoding) * heads * splits * n, dtype=torch.float32, device=DEV) for n in (vdim, 2)]
            word = status()
            api.attention_mma(q_all[rows_of].reshape(len(decoding), -1).to(dtype).to(DEV), k_pool, v_pool, table[decoding].contiguous(),
                              i32(list(range(len(decoding) + 1))), i32([before[b] for b in decoding]), len(decoding), len(decoding), heads, kv_heads, dim,
                              scale, -chunk, splits, out, *parts, word, one_token_each=True, sinks=sinks)
            assert int(word.item()) == 0
            assert float((out.double().cpu() - want[rows_of]).abs().max()) <= 0.04 * top, splits
        # the prompt kernel of the same file, which takes no null score
        plain_rows = torch.stack([chunk_plain(queries[b][i], *cached[b], before[b] + i, heads, kv_heads, scale, chunk, -1e30) for b in range(4) for i in range(new[b])])
        out = torch.zeros(tokens, heads * vdim, dtype=dtype, device=DEV)
        word = status()
        api.attention_mma(q_all.reshape(tokens, -1).to(dtype).to(DEV), k_pool, v_pool, table, i32(cu), i32(before), 4, tokens, heads, kv_heads, dim, scale,
                          -chunk, 1, out, None, None, word)
        assert int(word.item()) == 0
        assert float((out.double().cpu() - plain_rows).abs().max()) <= 0.04 * max(1.0, float(plain_rows.abs().max()))
