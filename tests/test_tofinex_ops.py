"""Operators of stacks with output norms (row norms, query / key / value preparation, grouped-query attention with capped scores,
experts), one mechanism at a time, against the plain restatement (``oracles/tofinex_plain.py``)."""

import math
import zlib

import pytest
import torch

from oracles import tofinex_plain as plain
from stack_testing import PLACES
from verl_b200.ops import functional as F
from verl_b200.ops import mixers as X

GEN = torch.Generator().manual_seed(11)


@pytest.fixture(params=PLACES)
def place(request):
    GEN.manual_seed(zlib.crc32(request.node.name.split("[")[0].encode()))     # the same inputs whatever ran before
    return request.param


def rand(*shape, scale=1.0):
    """Random values that bf16 holds exactly, so every path starts from the same numbers."""
    return (torch.randn(*shape, generator=GEN) * scale).bfloat16().float()


def put(t, place):
    return t.to(place[0], place[1])


def close(got, want, place, rel32=2e-5, rel16=8e-3):
    got, want = got.detach().cpu().double(), want.double()
    err = float((got - want).pow(2).mean().sqrt() / want.pow(2).mean().sqrt().clamp_min(1e-6))
    assert math.isfinite(err) and err < (rel32 if place[1] == torch.float32 else rel16), err


def i32(v, place):
    return torch.tensor(v, dtype=torch.int32, device=place[0])


# ---------------------------------------------------------------------------------------------- norms and products
@pytest.mark.parametrize("width", [24, 65, 1088, 4104])
def test_normed_embedding(place, width):
    table, w = rand(11, width, scale=0.02), 1 + rand(width, scale=0.2)
    ids = torch.tensor([3, 0, 10, 3, 7])
    x, h = X.embed_rms(ids.to(place[0]), put(table, place), 1.0, put(w, place), 3e-4)
    want = plain.rms_norm(table[ids].double(), w.bfloat16().double() if place[1] == torch.bfloat16 else w.double(), 3e-4)
    assert x.dtype == torch.float32
    close(x, want, (place[0], torch.float32))
    close(h, want, place, rel16=4e-3)


@pytest.mark.parametrize("t,width", [(1, 16), (5, 33), (7, 264), (3, 2048), (2, 4104), (2, 9000)])
@pytest.mark.parametrize("form", ["rows", "parts", "experts", "both"])
def test_residual_add_of_a_normed_output(place, t, width, form):
    """Rows, partial products, chosen experts' rows with and without a gated shared part; with and without the next norm."""
    x0, w, nxt = torch.randn(t, width, generator=GEN), rand(width), rand(width)
    y, gate, eps = None, None, 1e-3
    total = torch.zeros(t, width).double()
    if form == "parts":
        parts = torch.randn(3, t, width, generator=GEN)
        y, total = parts.to(place[0]), parts.double().sum(0)
    elif form in ("rows", "both"):
        rows = rand(t, width)
        y, total = put(rows, place), rows.double()
    if form == "both":
        tail = torch.randn(t, 5, generator=GEN)
        gate, total = tail.to(place[0])[:, 3], total * plain.sigmoid(tail[:, 3:4].double())
    experts = None
    if form in ("experts", "both"):
        slot, outs = torch.randint(0, 9, (t, 2), generator=GEN), rand(9, width)
        experts = (put(outs, place), slot.int().to(place[0]) if place[0] == "cuda" else slot)
        total = total + outs.double()[slot].sum(1)
    for next_w in (None, nxt):
        x = x0.to(place[0]).clone()
        h = X.residual_rms_(x, y, put(w, place), eps, 0.7, None if next_w is None else put(next_w, place), experts, gate)
        want = x0.double() + 0.7 * plain.rms_norm(total, w.double(), eps)
        close(x, want, (place[0], torch.float32))
        close(h, want if next_w is None else plain.rms_norm(want, next_w.double(), eps), place, rel16=4e-3)
        assert h.dtype == place[1]


@pytest.mark.parametrize("m,n,k", [(1, 8, 16), (5, 24, 40), (37, 130, 72), (64, 10, 30), (8, 640, 2176), (1100, 392, 136), (200, 256, 4096)])
def test_products_for_row_kernels_and_capped_logits(place, m, n, k):
    a, w = rand(m, k), rand(n, k, scale=3 * k ** -0.5)
    want = a.double() @ w.double().t()
    y = X.linear_partial(put(a, place), put(w, place))
    close(y.float().sum(0) if y.dim() == 3 else y, want, place, rel16=4e-3)
    for cap in (2.5, 30.0):
        close(X.linear_softcap(put(a, place), put(w, place), cap), plain.soft_cap(want, cap), place, rel16=4e-3)
    close(X.linear_softcap(put(a, place), put(w, place), 0.0), want, place, rel16=4e-3)


@pytest.mark.parametrize("m,ff,k", [(3, 24, 40), (9, 11, 30), (70, 136, 64), (1100, 72, 88), (1030, 20, 24)])
def test_gated_up_projection(place, m, ff, k):
    h, wg, wu, wt = rand(m, k), rand(ff, k, scale=2 * k ** -0.5), rand(ff, k, scale=k ** -0.5), rand(8, k)
    want = plain.silu(h.double() @ wg.double().t()) * (h.double() @ wu.double().t())
    close(X.gated_up(put(h, place), put(torch.cat([wg, wu]), place)), want, place)
    act, tail = X.gated_up_split(put(h, place), put(torch.cat([wg, wu, wt]), place), 2 * ff)
    close(act, want, place)
    assert tail.dtype == torch.float32
    close(tail, h.double() @ wt.double().t(), (place[0], torch.float32))
    none, tail = X.gated_up_split(put(h, place), put(wt, place), 0)
    assert none is None
    close(tail, h.double() @ wt.double().t(), (place[0], torch.float32))


# ---------------------------------------------------------------------------------------------- experts
def separated_logits(t, n, experts):
    """[t, n] random logits without close calls among the first ``experts`` columns."""
    z = torch.stack([torch.randperm(experts, generator=GEN) for _ in range(t)]).float() * (6.0 / experts) - 3.0
    return torch.cat([z + 0.01 * torch.randn(t, experts, generator=GEN) / experts, 50.0 * torch.ones(t, n - experts)], 1)


@pytest.mark.parametrize("t,experts,top,width,ff", [(1, 1, 1, 16, 8), (6, 4, 1, 24, 40), (50, 7, 3, 33, 13), (40, 9, 9, 40, 24), (300, 5, 2, 64, 72), (700, 130, 6, 72, 16),
                                                    (33, 40, 34, 32, 8), (1500, 8, 2, 136, 264)])
def test_experts(place, t, experts, top, width, ff):
    h, z = rand(t, width), separated_logits(t, experts + 3, experts)
    wg, wu, wd = rand(experts, ff, width, scale=3 * width ** -0.5), rand(experts, ff, width, scale=2 * width ** -0.5), rand(experts, width, ff, scale=ff ** -0.5)
    for renorm in (False, True):
        plan = X.expert_dispatch(put(h, place), z.to(place[0]), experts, top, renorm)
        act = X.expert_up(plan, put(torch.cat([wg, wu], 1).flatten(0, 1), place), ff)
        rows = X.expert_down(act, put(wd.flatten(0, 1), place), plan)
        got = rows.float()[plan.slot.long()].sum(1)
        score, which = plain.choose_experts(z[:, :experts].double(), torch.eye(experts).double(), top)
        if renorm:
            score = score / score.sum(-1, keepdim=True)
        x = h.double()[:, None, :] * score[..., None]                             # [t, top, width]
        want = torch.zeros(t, width).double()
        for e in range(experts):
            at, j = torch.nonzero(which == e, as_tuple=True)
            w = {"gate": wg[e].double(), "up": wu[e].double(), "down": wd[e].double()}
            want.index_add_(0, at, plain.gated_mlp(x[at, j], w))
        close(got, want, place, rel16=1.2e-2)
        assert len(set(plan.slot.flatten().tolist())) == t * top


def test_experts_when_all_tokens_choose_the_same(place):
    """One expert gets every token (its rows pass several tiles), the others none."""
    t, width, ff = 391, 48, 24
    h, z = rand(t, width), torch.full((t, 6), -4.0)
    z[:, 2] = 3.0
    wg, wu, wd = rand(6, ff, width), rand(6, ff, width, scale=0.2), rand(6, width, ff, scale=0.2)
    plan = X.expert_dispatch(put(h, place), z.to(place[0]), 6, 1)
    rows = X.expert_down(X.expert_up(plan, put(torch.cat([wg, wu], 1).flatten(0, 1), place), ff), put(wd.flatten(0, 1), place), plan)
    want = plain.gated_mlp(h.double() * plain.sigmoid(torch.tensor(3.0).double()), {"gate": wg[2].double(), "up": wu[2].double(), "down": wd[2].double()})
    close(rows.float()[plan.slot.long()].sum(1), want, place, rel16=1.2e-2)


# ---------------------------------------------------------------------------------------------- query / key / value preparation
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,rot", [(4, 2, 24, 40, 24), (3, 1, 10, 14, 6), (5, 5, 72, 16, 20), (2, 1, 136, 264, 8), (1, 1, 2, 1, 2), (6, 2, 16, 8, 16)])
@pytest.mark.parametrize("mixed", [False, True])
def test_query_key_value_preparation(place, heads, kv_heads, dim, vdim, rot, mixed):
    T, bs, a, b = 13, 4, heads * dim, (heads + kv_heads) * dim
    pad = -(b + kv_heads * vdim) % 8
    p, qn, kn, first, lam = rand(T, b + kv_heads * vdim + pad), 1 + rand(dim, scale=0.3), rand(dim), rand(T, kv_heads * vdim + 5), torch.tensor([0.375])
    qn = qn.bfloat16().float()
    pos = torch.tensor([0, 1, 2, 3, 100, 101, 7, 900, 5, 6, 7, 8, 9])
    spec = {"dims": rot, "base": 700.0}
    cos, sin = F.rope_table(1024, rot, 700.0, place[0])
    width = kv_heads * (dim + vdim)
    pages = torch.zeros(6, bs * width + 16, dtype=place[1], device=place[0])[:, : bs * width].view(6, bs, width)   # blocks with room for other layers
    slots = torch.tensor([5, 4, 23, 0, 1, 2, 3, -1, 8, 9, 10, 11, 12])
    vf = put(first, place)[:, : kv_heads * vdim] if mixed else None
    q, rows = X.qkv_prep(put(p, place), put(qn, place), put(kn, place), 2e-3, pos.int().to(place[0]), cos, sin, heads, kv_heads, vdim, vf,
                         put(lam, place) if mixed else None, pages, slots.to(place[0]), True)
    turn = lambda x: plain.rotate_pairs(x, pos, spec)
    close(q, turn(plain.rms_norm(p[:, :a].double().view(T, heads, dim), qn.double(), 2e-3)), place, rel16=4e-3)
    k = turn(plain.rms_norm(p[:, a:b].double().view(T, kv_heads, dim), kn.double(), 2e-3)).flatten(1)
    v = p[:, b : b + kv_heads * vdim].double()
    v = plain.mix_values(v, first[:, : kv_heads * vdim].double(), 0.375) if mixed else v
    close(rows[:, : kv_heads * dim], k, place, rel16=4e-3)
    close(rows[:, kv_heads * dim :], v, place, rel16=4e-3)
    flat = pages.reshape(-1, width).cpu()
    for t, s in enumerate(slots.tolist()):
        if s >= 0:
            assert torch.equal(flat[s], rows[t].cpu())
    assert not flat[[i for i in range(24) if i not in slots.tolist()]].any()


# ---------------------------------------------------------------------------------------------- attention
SHAPES = [(4, 2, 24, 40), (3, 1, 10, 14), (5, 5, 72, 16), (20, 1, 64, 64), (6, 3, 136, 200), (2, 1, 200, 136), (8, 2, 128, 128), (34, 2, 16, 72)]


def stored_rows(k, v, block_size, blocks, tables, place):
    """Keys and values of every sequence in pages of a pool full of other numbers."""
    G, d, e = k[0].shape[1], k[0].shape[2], v[0].shape[2]
    width = G * (d + e)
    extra = -(block_size * width) % 8 + 8
    pool = put(rand(blocks, block_size * width + extra, scale=3.0), place)
    pages = pool[:, : block_size * width].view(blocks, block_size, width)
    for kk, vv, table in zip(k, v, tables):
        row = put(torch.cat([kk.flatten(1), vv.flatten(1)], 1), place)
        for t in range(row.shape[0]):
            pages[table[t // block_size], t % block_size] = row[t]
    return pages


@pytest.mark.parametrize("heads,kv_heads,dim,vdim", SHAPES)
@pytest.mark.parametrize("cap", [0.0, 1.5, 40.0])
def test_prompt_attention(place, heads, kv_heads, dim, vdim, cap):
    lens, past = [1, 70, 19, 200], [0, 0, 64, 77]
    q = [rand(n, heads, dim) for n in lens]
    k, v = [rand(n + m, kv_heads, dim) for n, m in zip(lens, past)], [rand(n + m, kv_heads, vdim) for n, m in zip(lens, past)]
    cu = lambda ns: i32([0] + torch.tensor(ns).cumsum(0).tolist(), place)
    row = put(torch.cat([torch.cat([a.flatten(1), b.flatten(1)], 1) for a, b in zip(k, v)]), place)     # keys and values share their rows
    K, V = row[:, : kv_heads * dim].unflatten(1, (kv_heads, dim)), row[:, kv_heads * dim :].unflatten(1, (kv_heads, vdim))
    scale = 1.7 * dim ** -0.5
    sink = torch.zeros(heads, device=place[0], dtype=place[1])
    got = X.grouped_attention_prefill(put(torch.cat(q), place), K, V, cu(lens), cu([n + m for n, m in zip(lens, past)]), 0, scale, cap, sink)
    at = 0
    for i, n in enumerate(lens):
        qq = torch.cat([torch.zeros(past[i], heads, dim), q[i]]).double()
        want = plain.attention_core(qq, k[i].double(), v[i].double(), scale, cap if cap > 0 else 1e9)[past[i] :]
        close(got[at : at + n], want, place, rel16=1.2e-2)
        at += n


@pytest.mark.parametrize("heads,kv_heads,dim,vdim", SHAPES)
@pytest.mark.parametrize("block_size", [8, 16, 64, 128, 12])
def test_decode_attention_over_pages(place, heads, kv_heads, dim, vdim, block_size):
    cap, scale = 2.0, 2.0 * dim ** -0.5
    ctx = [1, 0, 63, 64, 65, 200, 129]
    per = -(-max(ctx) // block_size) + 1
    tables = torch.randperm(len(ctx) * per, generator=GEN).view(len(ctx), per)
    k, v = [rand(n, kv_heads, dim) for n in ctx], [rand(n, kv_heads, vdim) for n in ctx]
    pages = stored_rows(k, v, block_size, len(ctx) * per, tables.tolist(), place)
    q = rand(len(ctx), heads, dim)
    sink = torch.zeros(heads, device=place[0], dtype=place[1])
    for rows in (slice(None), slice(5, 6)):      # a batch, and one sequence alone (split over its keys)
        got = X.grouped_attention_decode(put(q, place)[rows], pages, tables.int().to(place[0])[rows].contiguous(), i32(ctx, place)[rows].contiguous(), kv_heads, vdim, 0, scale,
                                         cap, sink)
        for j, i in enumerate(range(len(ctx))[rows]):
            if ctx[i] == 0:
                assert not got[j].any()
                continue
            qq = torch.cat([torch.zeros(ctx[i] - 1, heads, dim), q[i : i + 1]]).double()
            close(got[j], plain.attention_core(qq, k[i].double(), v[i].double(), scale, cap)[-1], place, rel16=1.2e-2)


@pytest.mark.parametrize("n", [1, 2, 64, 65, 500])
@pytest.mark.parametrize("level", [-9.0, 0.0, 9.0, 60.0])
def test_one_in_the_denominator(place, n, level):
    """All scores equal: the weights sum to n e^s / (1 + n e^s), far from 1 for low scores; high scores run into the cap."""
    cap, d = 12.0, 16
    q, k, v = torch.zeros(n, 2, d), torch.zeros(n, 1, d), torch.ones(n, 1, 8)
    q[..., 0], k[..., 0] = 1.0, 1.0
    s = plain.soft_cap(torch.tensor(level).double(), cap)
    count = torch.arange(1, n + 1).double()
    want = (count * s.exp() / (1 + count * s.exp()))[:, None, None].expand(n, 2, 8)
    sink = torch.zeros(2, device=place[0], dtype=place[1])
    cu = i32([0, n], place)
    got = X.grouped_attention_prefill(put(q, place), put(k, place), put(v, place), cu, cu, 0, level, cap, sink)
    close(got, want, place)
    tables = torch.arange(8)[None]
    pages = stored_rows([k], [v], 64, 8, tables.tolist(), place)
    got = X.grouped_attention_decode(put(q[:1], place), pages, tables.int().to(place[0]), i32([n], place), 1, 8, 0, level, cap, sink)
    close(got[0], want[-1], place)


@pytest.mark.parametrize("far", [0, 1, 15, 16, 63, 64, 127, 128, 299])
def test_one_key_that_stands_out(place, far):
    """One key among 300 has a score far above the rest; its value alone must come out, wherever its page begins."""
    n, heads, d, cap, scale = 300, 4, 32, 30.0, 1.0
    q, k, v = rand(n, heads, d, scale=0.1), rand(n, 2, d, scale=0.1), rand(n, 2, 24)
    q[-1] = 0.0
    q[-1, :, 5], k[:, :, 5] = 5.0, -2.0
    k[far, :, 5] = 5.0                     # 25 against -10 before the cap
    cu, sink = i32([0, n], place), torch.zeros(heads, device=place[0], dtype=place[1])
    scores: list = []
    want = plain.attention_core(q.double(), k.double(), v.double(), scale, cap, scores)
    assert float((want[-1, 3] - v[far, 1].double()).abs().max()) < 1e-4 and float(scores[0][-1, far]) < 21.0
    got = X.grouped_attention_prefill(put(q, place), put(k, place), put(v, place), cu, cu, 0, scale, cap, sink)
    close(got[-1], want[-1], place)
    close(got, want, place, rel16=1.2e-2)
    for bs in (16, 64):
        per = -(-n // bs)
        tables = torch.randperm(per, generator=GEN)[None]
        pages = stored_rows([k], [v], bs, per, tables.tolist(), place)
        got = X.grouped_attention_decode(put(q[-1:], place), pages, tables.int().to(place[0]), i32([n], place), 2, 24, 0, scale, cap, sink)
        close(got[0], want[-1], place)


@pytest.mark.parametrize("window", [1, 5, 64, 65])
def test_windows_of_grouped_attention(place, window):
    n, heads, kv_heads, d, e, cap = 150, 4, 2, 40, 24, 3.0
    q, k, v = rand(n, heads, d), rand(n, kv_heads, d), rand(n, kv_heads, e)
    dist = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    want = []
    for h in range(heads):
        s = plain.soft_cap(q[:, h].double() @ k[:, h // 2].double().t() * 0.3, cap).masked_fill((dist < 0) | (dist >= window), float("-inf"))
        want.append(plain.one_plus_softmax(s) @ v[:, h // 2].double())
    want = torch.stack(want, 1)
    cu, sink = i32([0, n], place), torch.zeros(heads, device=place[0], dtype=place[1])
    close(X.grouped_attention_prefill(put(q, place), put(k, place), put(v, place), cu, cu, window, 0.3, cap, sink), want, place, rel16=1.2e-2)
    tables = torch.arange(10).flip(0)[None]
    pages = stored_rows([k], [v], 16, 10, tables.tolist(), place)
    got = X.grouped_attention_decode(put(q[-1:], place), pages, tables.int().to(place[0]), i32([n], place), kv_heads, e, window, 0.3, cap, sink)
    close(got[0], want[-1], place, rel16=1.2e-2)
