"""Operators of stacks with Dynamic Tanh on both sides of the sublayers (norms in GEMM epilogues, convolved query / key / value
preparation, attention that keeps the first tokens, lightning recurrence, grouped routing, clipped experts), one mechanism at a time,
against the plain restatement (``oracles/luzitar_plain.py``)."""

import math
import zlib

import pytest
import torch

from oracles import luzitar_plain as plain
from stack_testing import PLACES
from verl_b200.ops import functional as F
from verl_b200.ops import mixers as X

GEN = torch.Generator().manual_seed(5)


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
    assert got.shape == want.shape
    err = float((got - want).pow(2).mean().sqrt() / want.pow(2).mean().sqrt().clamp_min(1e-6))
    assert math.isfinite(err) and err < (rel32 if place[1] == torch.float32 else rel16), err


def i32(v, place):
    return torch.tensor(v, dtype=torch.int32, device=place[0])


def norm_of(width, alpha):
    return {"n.alpha": torch.tensor(alpha), "n": rand(width), "n.b": rand(width, scale=0.2)}


def norm_args(n, place):
    return tuple(put(n[k].reshape(-1), place) for k in ("n.alpha", "n", "n.b"))


def dyt(x, n):
    return plain.dynamic_tanh(x.double(), {k: v.double() for k, v in n.items()}, "n")


# ---------------------------------------------------------------------------------------------- norms and products
@pytest.mark.parametrize("width", [24, 65, 1088])
def test_normed_embedding(place, width):
    table, a, b = rand(11, width), norm_of(width, 0.75), norm_of(width, 1.5)
    ids = torch.tensor([3, 0, 10, 3, 7])
    x, h = X.embed_dyt2(ids.to(place[0]), put(table, place), norm_args(a, place), norm_args(b, place))
    want = dyt(table[ids], a)
    assert x.dtype == torch.float32
    close(x, want, (place[0], torch.float32))
    close(h, dyt(want, b), place, rel16=4e-3)


SHAPES = [(1, 16, 24), (5, 30, 22), (7, 264, 200), (300, 96, 72), (260, 512, 1024), (1500, 136, 80), (3, 2048, 2048), (2500, 320, 256)]


@pytest.mark.parametrize("m,n,k", SHAPES)
def test_product_with_bias_and_with_silu_on_leading_columns(place, m, n, k):
    a, w, b = rand(m, k), rand(n, k, scale=k ** -0.5), rand(n)
    y = a.double() @ w.double().t()
    close(X.linear_bias(put(a, place), put(w, place), put(b, place)), y + b.double(), place, rel16=4e-3)
    for n0 in (n, n // 2 // 8 * 8 or 1, 5):
        want = torch.cat([plain.silu(y[:, :n0]), y[:, n0:]], -1)
        close(X.linear_silu(put(a, place), put(w, place), n0), want, place, rel16=4e-3)


@pytest.mark.parametrize("m,n,k", SHAPES)
@pytest.mark.parametrize("following", [True, False])
def test_residual_add_of_a_normed_product(place, m, n, k, following):
    a, w, x0 = rand(m, k), rand(n, k, scale=2 * k ** -0.5), torch.randn(m, n, generator=GEN)
    post, nxt = norm_of(n, 0.875), norm_of(n, 0.5)
    x = x0.to(place[0]).clone()
    h = X.linear_residual_(put(a, place), put(w, place), x, norm_args(nxt, place) if following else None, norm_args(post, place))
    want = x0.double() + dyt(a.double() @ w.double().t(), post)
    close(x, want, (place[0], torch.float32))
    if following:
        close(h, dyt(want, nxt), place, rel16=4e-3)
    else:
        assert h is None


@pytest.mark.parametrize("t,width,top", [(1, 16, 1), (5, 33, 3), (300, 264, 5), (3, 2048, 9)])
def test_residual_add_of_normed_expert_rows(place, t, width, top):
    x0, rows, slot = torch.randn(t, width, generator=GEN), rand(t * top + 7, width, scale=0.4), torch.randperm(t * top + 7, generator=GEN)[: t * top].view(t, top)
    post, nxt = norm_of(width, 0.875), norm_of(width, 0.5)
    x = x0.to(place[0]).clone()
    h = X.residual_dyt_(x, put(rows, place), slot.int().to(place[0]), norm_args(post, place), norm_args(nxt, place))
    want = x0.double() + dyt(rows.double()[slot].sum(1), post)
    close(x, want, (place[0], torch.float32))
    close(h, dyt(want, nxt), place, rel16=4e-3)


@pytest.mark.parametrize("t,width", [(1, 16), (5, 35), (40, 264), (3, 4096), (2, 9000)])
def test_gated_norm_of_whole_rows(place, t, width):
    both, w = rand(t, 2 * width + 8), rand(width)
    view = put(both, place)
    got = X.gated_rms(put(both[:, :width].contiguous(), place), view[:, width + 8 :], put(w, place), 3e-2)
    o, g = both[:, :width].double(), both[:, width + 8 :].double()
    close(got, plain.unit_rms(o, 3e-2) * w.double() * plain.sigmoid(g), place)


# ---------------------------------------------------------------------------------------------- convolution, rotation, norm
def table_of(rot, place):
    s = rot.get("scaling")
    scaling = s and {"rope_type": "yarn", "factor": s["factor"], "original_max_position_embeddings": s["original"], "beta_fast": s["fast"], "beta_slow": s["slow"],
                     "attention_factor": 0.1 * math.log(s["factor"]) + 1.0}
    return F.rope_table(512, rot["dims"], rot["base"], place[0], scaling)


def prepared(p, conv, H, G, d, e, rot, halves, eps, start=0):
    u = plain.short_conv(p.double(), conv.double()) if conv is not None else p.double()
    T, pos = p.shape[0], torch.arange(start, start + p.shape[0])
    q = plain.unit_rms(plain.rotate(u[:, : H * d].view(T, H, d), pos, rot, halves), eps)
    k = plain.unit_rms(plain.rotate(u[:, H * d : (H + G) * d].view(T, G, d), pos, rot, halves), eps)
    return q, torch.cat([k.flatten(1), u[:, (H + G) * d : (H + G) * d + G * e]], -1)


YARN = {"factor": 6.0, "original": 300, "fast": 20.0, "slow": 2.0}
PREP = [  # heads, key heads, size, value size, rotation, taps
    (4, 2, 16, 24, {"dims": 16, "base": 700.0}, 3), (3, 1, 48, 16, {"dims": 32, "base": 900.0, "scaling": YARN}, 4), (2, 2, 24, 40, {"dims": 8, "base": 50.0}, 2),
    (6, 3, 10, 7, {"dims": 6, "base": 90.0, "scaling": YARN}, 3), (2, 1, 136, 72, {"dims": 128, "base": 5e3, "scaling": YARN}, 4), (1, 1, 8, 8, {"dims": 2, "base": 30.0}, 1),
    (2, 1, 16, 16, {"dims": 16, "base": 700.0}, 6), (4, 4, 32, 32, {"dims": 32, "base": 1e4}, None)]


@pytest.mark.parametrize("halves", [True, False])
@pytest.mark.parametrize("H,G,d,e,rot,taps", PREP)
def test_convolved_preparation(place, H, G, d, e, rot, taps, halves):
    """Prompts without a cache, portions down to one and two tokens beside other sequences, steps, and rows in pages."""
    C, eps, bs = (H + G) * d + G * e, 1e-3, 8
    conv = rand(C, taps, scale=taps ** -0.5) if taps else None
    lens = (1, 2, 37, 60)
    ps = [rand(n, C + 3 if C % 8 else C) for n in lens]
    tab = table_of(rot, place)
    args = (H, G, d, e, halves)
    dev_conv = put(conv, place) if conv is not None else None
    cum = lambda ns: i32([sum(ns[:i]) for i in range(len(ns) + 1)], place)
    want = [prepared(p[:, :C], conv, H, G, d, e, rot, halves, eps) for p in ps]
    pos = torch.cat([torch.arange(n, dtype=torch.int32) for n in lens]).to(place[0])
    q, rows = X.conv_qkv_prep(put(torch.cat(ps), place), dev_conv, eps, pos, *tab, *args, cu=cum(lens), want_rows=True)
    close(q, torch.cat([w[0] for w in want]), place)
    close(rows, torch.cat([w[1] for w in want]), place)
    # portions of unequal sizes, then steps, through state rows 4, 1, 0, 2 and one page pool; what the rows held before must not show
    past = max((taps or 1) - 1, 0)
    state = torch.full((5, past * C), 7.0, device=place[0])[:, : past * C]
    pages = torch.zeros(60, bs, G * (d + e), dtype=place[1], device=place[0])
    slots, at, got, new = [3, 1, 0, 2], [0] * 4, [[] for _ in lens], True
    page_row = lambda b, t: (b * 8 + t // bs) * bs + t % bs if b < 3 else (24 + t // bs) * bs + t % bs
    for sizes in ([1, 1, 2, 5], [0, 1, 1, 2], [0, 0, 17, 2], [0, 0, 2, 21]):
        live = [b for b in range(4) if sizes[b]]
        part = [ps[b][at[b] : at[b] + sizes[b]] for b in live]
        pos = torch.cat([torch.arange(at[b], at[b] + sizes[b], dtype=torch.int32) for b in live]).to(place[0])
        where = torch.tensor([page_row(b, t) for b in live for t in range(at[b], at[b] + sizes[b])], device=place[0])
        kept = dict(state=state, slots=i32([slots[b] for b in live], place), fresh=i32([int(at[b] == 0) for b in live], place)) if past else {}
        q, rows = X.conv_qkv_prep(put(torch.cat(part), place), dev_conv, eps, pos, *tab, *args, cu=cum([sizes[b] for b in live]), pages=pages, page_slots=where, **kept)
        assert rows.numel() == 0
        for b, x in zip(live, q.split([sizes[b] for b in live])):
            got[b].append(x)
            at[b] += sizes[b]
    untouched = state[4].clone()
    for _ in range(12):                    # sequences 2 and 3 go on token by token; row s of a step is slot s
        p, pos, act, where = torch.zeros(5, ps[0].shape[1]), torch.zeros(5, dtype=torch.int32), torch.zeros(5, dtype=torch.bool), torch.full((5,), -1, dtype=torch.int64)
        for b in (2, 3):
            s = slots[b]
            p[s], pos[s], act[s], where[s] = ps[b][at[b]], at[b], True, page_row(b, at[b])
        before = state[[slots[0], slots[1]]].clone()
        kept = dict(state=state) if past else {}
        q, _ = X.conv_qkv_prep(put(p, place), dev_conv, eps, pos.to(place[0]), *tab, *args, active=act.to(place[0]), pages=pages, page_slots=where.to(place[0]), **kept)
        assert torch.equal(state[[slots[0], slots[1]]], before)
        for b in (2, 3):
            got[b].append(q[slots[b]][None])
            at[b] += 1
    assert torch.equal(state[4], untouched)
    for b in range(4):
        n = at[b]
        close(torch.cat(got[b]), want[b][0][:n], place)
        flat = pages.view(-1, pages.shape[2])[[page_row(b, t) for t in range(n)]]
        close(flat, want[b][1][:n], place)


@pytest.mark.parametrize("taps", [2, 3, 4])
def test_convolution_of_many_portions_at_once(place, taps):
    """Thousands of tokens in portions of one to a few hundred, some behind kept inputs."""
    H, G, d, e, eps, rot = 6, 2, 32, 24, 1e-3, {"dims": 16, "base": 500.0}
    C = (H + G) * d + G * e
    lens = [1, 2, 3, 4, 5, 7, 1, 1, 300, 2, 259, 3] * 11 + [1900]
    starts = [i % 3 * 2 for i in range(len(lens))]            # 0, 2 or 4 tokens came before
    conv, tab = rand(C, taps, scale=taps ** -0.5), F.rope_table(2048, rot["dims"], rot["base"], place[0])
    ps = [rand(n + a, C) for n, a in zip(lens, starts)]
    state = torch.zeros(len(lens), (taps - 1) * C)
    for b, (p, a) in enumerate(zip(ps, starts)):
        before = torch.cat([torch.zeros(taps - 1, C), p[:a]])[-(taps - 1):]
        state[b] = before.flatten() if a else 9.0
    state = state.to(place[0])
    part = torch.cat([p[a:] for p, a in zip(ps, starts)])
    pos = torch.cat([torch.arange(a, a + n, dtype=torch.int32) for n, a in zip(lens, starts)]).to(place[0])
    cu = i32([sum(lens[:i]) for i in range(len(lens) + 1)], place)
    q, rows = X.conv_qkv_prep(put(part, place), put(conv, place), eps, pos, *tab, H, G, d, e, True, cu, state, i32(range(len(lens)), place),
                              i32([int(a == 0) for a in starts], place), want_rows=True)
    want = [prepared(p, conv, H, G, d, e, rot, True, eps) for p in ps]
    at = 0
    for n, a, (wq, wr), p, st in zip(lens, starts, want, ps, state.cpu()):
        close(q[at : at + n], wq[a:], place)
        close(rows[at : at + n], wr[a:], place)
        assert torch.equal(st.view(taps - 1, C), torch.cat([torch.zeros(taps - 1, C), p])[-(taps - 1):])
        at += n


def test_convolution_reaches_over_every_portion_edge(place):
    """One loud input: the outputs of the next taps - 1 tokens show it wherever the portions are cut."""
    taps, H, d = 4, 1, 8
    C = 3 * d
    conv, tab = rand(C, taps), F.rope_table(64, 2, 100.0, place[0])
    for loud in range(6):
        p = rand(12, C, scale=0.05)
        p[loud] = rand(C, scale=20.0)
        want = prepared(p, conv, 1, 1, d, d, {"dims": 2, "base": 100.0}, True, 1e-6)
        for cuts in ([12], [1] * 12, [2] * 6, [3] * 4, [5, 1, 6]):
            state, at, rows = torch.zeros(1, (taps - 1) * C, device=place[0]), 0, []
            for n in cuts:
                pos = torch.arange(at, at + n, dtype=torch.int32, device=place[0])
                rows.append(X.conv_qkv_prep(put(p[at : at + n], place), put(conv, place), 1e-6, pos, *tab, 1, 1, d, d, True, i32([0, n], place), state, i32([0], place),
                                            i32([int(at == 0)], place), want_rows=True)[1])
                at += n
            close(torch.cat(rows), want[1], place)


# ---------------------------------------------------------------------------------------------- attention that keeps the first tokens
MASKS = [(1, 0), (1, 1), (5, 3), (64, 1), (64, 64), (70, 65), (33, 130), (130, 20), (400, 9), (0, 0)]


def loud_pair(q, k, i, j):
    """Query ``i`` finds key ``j`` before all others."""
    q[i] = k[j] * 2.0


@pytest.mark.parametrize("H,G,d,e", [(4, 2, 32, 16), (20, 1, 64, 72), (3, 1, 10, 7), (2, 2, 136, 136)])
@pytest.mark.parametrize("window,keep", MASKS)
def test_grouped_attention_with_window_and_kept_tokens(place, H, G, d, e, window, keep):
    T, scale = 300, d ** -0.5
    lens = (T, 40, 1)
    mask = {"size": window, "keep_first": keep} if window else None
    q, k, v = rand(sum(lens), H, d), rand(sum(lens), G, d), rand(sum(lens), G, e)
    for i in range(20, T, 7):      # keys just inside and just outside every edge, at block borders, far away
        js = [i - window, i - window + 1, i - window - 1, keep - 1, keep, keep + 1, 0, 63, 64, i - 1]
        j = js[(i // 7) % len(js)]
        if 0 <= j <= i:
            for h in range(H):
                q[i, h] = k[j, h // (H // G)] * 1.5
    cu, out, at = i32([0, T, T + 40, T + 41], place), [], 0
    for n in lens:
        s = slice(at, at + n)
        out.append(torch.stack([plain.weighted_values(q[s, h].double() @ k[s, h // (H // G)].double().t() * scale, plain.sees(n, mask), v[s, h // (H // G)].double())
                                for h in range(H)], 1))
        at += n
    want = torch.cat(out)
    rows = torch.cat([k.flatten(1), v.flatten(1)], -1)
    kv = put(rows, place)
    kd, vd = kv[:, : G * d].unflatten(1, (G, d)), kv[:, G * d :].unflatten(1, (G, e))
    close(X.grouped_attention_prefill(put(q, place), kd, vd, cu, cu, window, scale, 0.0, None, keep), want, place)
    # the last 90 queries of the first sequence alone, all keys
    close(X.grouped_attention_prefill(put(q[T - 90 : T], place), kd[:T], vd[:T], i32([0, 90], place), i32([0, T], place), window, scale, 0.0, None, keep),
          want[T - 90 : T], place)
    # single queries over pages, at several places of the first sequence
    for bs in (16, 64):
        blocks = -(-T // bs)
        pages = torch.zeros(blocks + 3, bs, rows.shape[1], dtype=place[1], device=place[0])
        order = torch.randperm(blocks + 3, generator=GEN)[:blocks]
        for t in range(T):
            pages[order[t // bs], t % bs] = kv[t]
        at = [0, 1, 15, 62, 63, 64, 65, 127, 128, 129, 200, 255, 256, 298, 299]
        ctx = [a + 1 for a in at] + [0]
        table = order.int()[None].expand(len(ctx), -1).contiguous().to(place[0])
        got = X.grouped_attention_decode(put(q[at + [0]], place), pages, table, i32(ctx, place), G, e, window, scale, 0.0, None, keep)
        close(got[:-1], want[at], place)
        assert float(got[-1].abs().max()) == 0


@pytest.mark.parametrize("H,du,dr,rank,e", [(4, 16, 8, 40, 24), (20, 32, 16, 64, 32), (3, 9, 6, 13, 7)])
@pytest.mark.parametrize("window,keep", [(0, 0), (50, 0), (50, 7), (64, 64), (20, 100)])
def test_latent_attention_without_sink_and_gate(place, H, du, dr, rank, e, window, keep):
    T, scale = 200, (du + dr) ** -0.5
    mask = {"size": window, "keep_first": keep} if window else None
    q, row, uk, uv = rand(T, H, du + dr), rand(T, rank + dr), rand(H, du, rank, scale=rank ** -0.5), rand(H, e, rank, scale=rank ** -0.5)
    ku, v = torch.einsum("tr,hdr->thd", row[:, :rank], uk).bfloat16().float(), torch.einsum("tr,her->the", row[:, :rank], uv).bfloat16().float()

    def reference(kk, vv):
        s = [(q[:, h, :du].double() @ kk[:, h].double().t() + q[:, h, du:].double() @ row[:, rank:].double().t()) * scale for h in range(H)]
        return torch.stack([plain.weighted_values(s[h], plain.sees(T, mask), vv[:, h].double()) for h in range(H)], 1)

    cu = i32([0, T], place)
    got = X.latent_attention_prefill(put(q, place), put(ku, place), put(row[:, rank:].contiguous(), place), put(v, place), cu, cu, window, scale, None, None, keep)
    close(got, reference(ku, v), place)
    # the latents as keys and values of one head size: what decoding reads
    qa = torch.cat([torch.einsum("thd,hdr->thr", q[..., :du], uk), q[..., du:]], -1).bfloat16().float()
    s = [qa[:, h].double() @ row.double().t() * scale for h in range(H)]
    want = torch.stack([plain.weighted_values(x, plain.sees(T, mask), row[:, :rank].double()) for x in s], 1)
    bs = 16
    order = torch.randperm(15, generator=GEN)[: -(-T // bs)]
    pages = torch.zeros(15, bs, rank + dr, dtype=place[1], device=place[0])
    for t in range(T):
        pages[order[t // bs], t % bs] = put(row[t], place)
    at = [0, 7, 31, 32, 49, 50, 51, 63, 64, 99, 100, 101, 150, 199]
    table = order.int()[None].expand(len(at), -1).contiguous().to(place[0])
    close(X.latent_attention_decode(put(qa[at], place), pages, table, i32([a + 1 for a in at], place), rank, window, scale, None, keep), want[at], place)


def test_latent_rows_without_a_query_latent(place):
    rank, dr, T = 40, 8, 30
    p, w, tab = rand(T, 16 + rank + dr), rand(rank), F.rope_table(64, dr, 300.0, place[0])
    pos = torch.arange(T, dtype=torch.int32, device=place[0])
    cq, rows = X.latent_prep(put(p, place)[:, 16:], None, put(w, place), 1e-3, pos, *tab, None, None, True)
    z = p[:, 16:].double()
    want = torch.cat([plain.unit_rms(z[:, :rank], 1e-3) * w.double(), plain.rotate(z[:, None, rank:], torch.arange(T), {"dims": dr, "base": 300.0}, False)[:, 0]], -1)
    assert cq.shape == (T, 0)
    close(rows, want, place)


# ---------------------------------------------------------------------------------------------- lightning recurrence
DECAYS = (0.97, 0.3, 1.0, 0.999, 0.0, 0.75)
RECUR = [(2, 64, 64), (3, 16, 8), (1, 128, 128), (2, 136, 200), (3, 5, 7), (2, 128, 72), (1, 24, 264), (6, 8, 16), (1, 256, 64)]


def recurrence(q, k, v, decay):
    return torch.stack([plain.decayed_memory(q[:, h].double(), k[:, h].double(), v[:, h].double(), decay[h]) for h in range(q.shape[1])], 1)


@pytest.mark.parametrize("H,d,e", RECUR)
def test_lightning_recurrence(place, H, d, e):
    """Prompts without state, portions beside other sequences, steps; slots that held something else before."""
    decay = [float(torch.tensor(x)) for x in DECAYS[:H]]
    lens = (1, 2, 70, 139)
    ps = [rand(n, H * (2 * d + e) + 8, scale=0.7) for n in lens]
    cut = lambda p: (p[:, : H * d].view(-1, H, d), p[:, H * d : 2 * H * d].view(-1, H, d), p[:, 2 * H * d : H * (2 * d + e)].view(-1, H, e))
    want = [recurrence(*cut(p), decay).flatten(1) for p in ps]
    dec = torch.tensor(decay, device=place[0])
    cum = lambda ns: i32([sum(ns[:i]) for i in range(len(ns) + 1)], place)
    close(X.lightning_prefill(put(torch.cat(ps), place), dec, d, e, cum(lens), all_fresh=True), torch.cat(want), place)
    slots, at, got = [3, 1, 0, 2], [0] * 4, [[] for _ in lens]
    state = torch.full((5, H * d * e), 3.0, device=place[0])
    for sizes in ([1, 1, 2, 64], [0, 1, 1, 2], [0, 0, 57, 61]):
        live = [b for b in range(4) if sizes[b]]
        part = put(torch.cat([ps[b][at[b] : at[b] + sizes[b]] for b in live]), place)
        o = X.lightning_prefill(part, dec, d, e, cum([sizes[b] for b in live]), state, i32([slots[b] for b in live], place), i32([int(at[b] == 0) for b in live], place),
                                all(at[b] == 0 for b in live))
        for b, x in zip(live, o.split([sizes[b] for b in live])):
            got[b].append(x)
            at[b] += sizes[b]
    for _ in range(10):
        p, act = torch.zeros(5, ps[0].shape[1]), torch.zeros(5, dtype=torch.bool)
        for b in (2, 3):
            p[slots[b]], act[slots[b]] = ps[b][at[b]], True
        before = state[[1, 3, 4]].clone()
        o = X.lightning_decode(put(p, place), dec, d, e, state, act.to(place[0]))
        assert torch.equal(state[[1, 3, 4]], before) and float(o[[1, 3, 4]].abs().max()) == 0
        for b in (2, 3):
            got[b].append(o[slots[b]][None])
            at[b] += 1
    for b in range(4):
        close(torch.cat(got[b]), want[b][: at[b]], place)
    final = torch.zeros(H, d, e).double()
    for t in range(at[3]):
        q, k, v = (x[t].double() for x in cut(ps[3]))
        final = torch.tensor(decay).double()[:, None, None] * final + k[:, :, None] * v[:, None, :]
    close(state[slots[3]].view(H, d, e), final, place, rel16=1e-4)


@pytest.mark.parametrize("H,d,e,lens", [(2, 64, 64, (1500, 700, 3)), (1, 128, 128, (2100,)), (3, 32, 136, (513, 64, 128, 1))])
def test_lightning_over_long_prompts(place, H, d, e, lens):
    """Few long sequences (cut into segments on the GPU); one early token stands out and is still read at the end."""
    decay = [float(torch.tensor(x)) for x in (0.9995, 1.0, 0.9)[:H]]
    p = rand(sum(lens), H * (2 * d + e), scale=0.5)
    p[3, H * d :] *= 8.0
    want, at = [], 0
    for n in lens:
        x = p[at : at + n]
        want.append(recurrence(x[:, : H * d].view(n, H, d), x[:, H * d : 2 * H * d].view(n, H, d), x[:, 2 * H * d :].view(n, H, e), decay).flatten(1))
        at += n
    cu = i32([sum(lens[:i]) for i in range(len(lens) + 1)], place)
    state = torch.full((len(lens), H * d * e), 5.0, device=place[0])
    ids = list(range(len(lens)))
    got = X.lightning_prefill(put(p, place), torch.tensor(decay, device=place[0]), d, e, cu, state, i32(ids, place), i32([1] * len(lens), place), True)
    close(got, torch.cat(want), place)
    nxt = rand(len(lens), H * (2 * d + e), scale=0.5)
    more = X.lightning_decode(put(nxt, place), torch.tensor(decay, device=place[0]), d, e, state, torch.ones(len(lens), dtype=torch.bool, device=place[0]))
    at = 0
    for b, n in enumerate(lens):
        x = torch.cat([p[at : at + n], nxt[b : b + 1]])
        w = recurrence(x[:, : H * d].view(n + 1, H, d), x[:, H * d : 2 * H * d].view(n + 1, H, d), x[:, 2 * H * d :].view(n + 1, H, e), decay)[-1].flatten()
        close(more[b], w, place)
        at += n


# ---------------------------------------------------------------------------------------------- experts
ROUTES = [  # experts, top, groups, kept groups
    (6, 2, 3, 1), (8, 3, 4, 2), (5, 5, 1, 1), (12, 4, 12, 5), (1, 1, 1, 1), (16, 6, 2, 2), (72, 5, 9, 4), (160, 9, 8, 3), (300, 4, 50, 40)]


@pytest.mark.parametrize("E,top,groups,keep", ROUTES)
@pytest.mark.parametrize("t", [1, 9, 150])
def test_grouped_routing_and_clipped_experts(place, E, top, groups, keep, t):
    """Router, copies in expert order, both products and the sum of the rows, against the token-by-token mixture."""
    W, ff, limit = 24, 16, 0.8
    h, z = rand(t, W), torch.randn(t, -(-E // 8) * 8, generator=GEN)
    corr = (rand(E, scale=0.7) - 0.6).bfloat16().float()     # many choice scores are negative
    gate, up, down = rand(E, ff, W, scale=0.4), rand(E, ff, W, scale=0.4), rand(E, W, ff, scale=0.3)
    s = plain.sigmoid(z[:, :E].double())
    want = torch.zeros(t, W).double()
    for i in range(t):
        chosen = plain.choose_experts(s[i], corr.double(), top, groups, keep)
        assert len(set(chosen)) == top
        total = s[i][chosen].sum() + 1e-20
        for e in chosen:
            want[i] += s[i, e] / total * plain.clipped_expert(h[i].double(), gate[e].double(), up[e].double(), down[e].double(), limit)
    plan = X.expert_dispatch(put(h, place), z.to(place[0]), E, top, True, put(corr, place), groups, keep)
    w_in = put(torch.cat([gate, up], 1).reshape(-1, W), place)
    rows = X.expert_down(X.expert_up(plan, w_in, ff, "clipped", limit), put(down.reshape(-1, ff), place), plan)
    close(rows[plan.slot.long()].float().sum(1), want, place, rel16=1.2e-2)
    sums = plan.scale[plan.slot.long()].sum(1)
    assert float((sums - 1).abs().max()) < 1e-5


def test_hidden_groups_stay_hidden_when_all_choices_are_negative(place):
    """The best expert of a dropped group must not be taken, and a dropped group counts below every negative score."""
    z = torch.tensor([[0.0, 0.0, 9.0, -9.0, 0.5, 0.4, 0.0, 0.0]])
    corr = torch.tensor([-2.0, -2.0, -2.0, -2.0, -2.0, -2.0, -2.0, -2.0])
    plan = X.expert_dispatch(put(torch.ones(1, 8), place), z.to(place[0]), 8, 2, True, put(corr, place), 4, 1)
    s = torch.sigmoid(torch.tensor([0.5, 0.4]))       # group 2 (0.62 + 0.60) beats group 1 (0.9999 + 0.0001)
    close(plan.scale[plan.slot.long()].flatten(), s / s.sum(), (place[0], torch.float32))


@pytest.mark.parametrize("t,ff", [(3, 16), (200, 72), (40, 11), (600, 128)])
def test_clipped_activation_clips_only_what_it_should(place, t, ff):
    W, limit = 32, 1.25
    h, w = rand(t, W, scale=2.0), rand(2 * ff, W, scale=0.5)
    plan = X.expert_dispatch(put(h, place), torch.zeros(t, 8, device=place[0]), 1, 1, True)
    y = h.double() @ w.double().t()
    g, u = y[:, :ff].clamp(max=limit), y[:, ff:].clamp(-limit, limit)
    assert float(y[:, :ff].min()) < -2 * limit and float((y.abs() > limit).double().mean()) > 0.3     # low gates stay, both kinds occur
    got = X.expert_up(plan, put(w, place), ff, "clipped", limit)[plan.slot.long()[:, 0]]
    close(got, g * plain.sigmoid(1.702 * g) * (u + 1), place, rel16=6e-3)
