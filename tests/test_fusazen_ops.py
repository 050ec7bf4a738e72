"""Operators of stacks with RMS norms in front of the sublayers (normed rows with a convolution over time, norms over whole projections,
chunked and differential attention, generalized delta rule, epilogues with bias, squared relu and tanh), one mechanism at a time, against the plain
restatement (``oracles/fusazen_plain.py``)."""

import math
import zlib

import pytest
import torch

from oracles import fusazen_plain as plain
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


def fp32(place):
    return (place[0], torch.float32)


def i32(v, place):
    return torch.tensor(v, dtype=torch.int32, device=place[0])


def offsets(lens):
    return [0] + torch.tensor(lens).cumsum(0).tolist()


# ---------------------------------------------------------------------------------------------- embedding, norm, convolution
@pytest.mark.parametrize("width,scale", [(24, 3.0), (65, 0.25), (1088, 1.0)])
def test_scaled_embedding(place, width, scale):
    table, ids = rand(11, width), torch.tensor([3, 0, 10, 3, 7])
    x = X.embed_rows(ids.to(place[0]), put(table, place), scale)
    assert x.dtype == torch.float32
    close(x, table[ids] * scale, fp32(place))


@pytest.mark.parametrize("t,width", [(1, 16), (5, 35), (40, 264), (3, 4096), (2, 9000)])
@pytest.mark.parametrize("parts", [0, 1, 3])
@pytest.mark.parametrize("with_bias", [False, True])
def test_norm_of_the_stream_with_what_a_product_leaves(place, t, width, parts, with_bias):
    x0, w, y = torch.randn(t, width, generator=GEN), rand(width), rand(max(parts, 1), t, width)
    b = rand(width) if with_bias else None
    x = x0.to(place[0]).clone()
    given = None if parts == 0 else put(y[0], place) if parts == 1 else y.to(place[0])
    h = X.rms_conv(x, put(w, place), 3e-2, given, put(b, place) if with_bias else None)
    want = x0.double() + (y.double().sum(0) if parts else 0) + (b.double() if with_bias else 0)
    close(x, want, fp32(place))
    close(h, plain.unit_rms(want, 3e-2) * w.double(), place, rel16=4e-3)


CONV = [(24, 3), (1088, 4), (40, 2), (35, 3), (16, 1), (72, 6), (264, 3)]


@pytest.mark.parametrize("width,taps", CONV)
@pytest.mark.parametrize("lens", [[1], [50], [3, 1, 17, 2, 30], [15, 16, 17], [100, 1, 1]])
def test_convolution_of_normed_prompts(place, width, taps, lens):
    x, w, c = torch.randn(sum(lens), width, generator=GEN), rand(width), rand(width, taps, scale=0.6)
    cu = offsets(lens)
    h = X.rms_conv(x.to(place[0]), put(w, place), 1e-2, conv=put(c, place), cu=i32(cu, place))
    n = plain.unit_rms(x.double(), 1e-2) * w.double()
    want = torch.cat([plain.with_past(n[a:b], c.double()) for a, b in zip(cu, cu[1:])])
    close(h, want, place, rel16=4e-3)


@pytest.mark.parametrize("width,taps", CONV)
def test_convolution_goes_on_from_what_a_sequence_kept(place, width, taps):
    """Portions of two sequences in turn, one of them shorter than the taps, then single tokens; a third slot stays untouched."""
    lens = {2: 41, 0: 38}
    x = {s: torch.randn(n, width, generator=GEN) for s, n in lens.items()}
    w, c = rand(width), rand(width, taps, scale=0.6)
    state = torch.full((4, (taps - 1) * width), 7.0, device=place[0])
    args = (put(w, place), 1e-2)
    out, at = {s: [] for s in x}, {s: 0 for s in x}
    for n in (1, 2, 17, 3, 1):
        rows = torch.cat([x[s][at[s] : at[s] + n] for s in x])
        h = X.rms_conv(rows.to(place[0]), *args, conv=put(c, place), cu=i32(offsets([n] * 2), place), state=state if taps > 1 else None,
                       slots=i32(list(x), place), fresh=i32([int(at[s] == 0) for s in x], place))
        for s, part in zip(x, h.split(n)):
            out[s].append(part.cpu())
            at[s] += n
    while any(at[s] < lens[s] for s in x):
        active = torch.zeros(4, dtype=torch.bool)
        rows = torch.randn(4, width, generator=GEN)
        for s in x:
            if at[s] < lens[s]:
                active[s], rows[s] = True, x[s][at[s]]
        h = X.rms_conv(rows.to(place[0]), *args, conv=put(c, place), state=state, active=active.to(place[0]))
        for s in x:
            if active[s]:
                out[s].append(h[s : s + 1].cpu())
                at[s] += 1
    for s in x:
        close(torch.cat(out[s]), plain.with_past(plain.unit_rms(x[s].double(), 1e-2) * w.double(), c.double()), place, rel16=4e-3)
    assert bool((state[[1, 3]] == 7.0).all())


# ---------------------------------------------------------------------------------------------- products
SHAPES = [(1, 16, 24), (5, 30, 22), (7, 264, 200), (300, 96, 72), (260, 512, 1024), (1500, 136, 80), (3, 2048, 2048), (2500, 320, 256)]


@pytest.mark.parametrize("m,n,k", SHAPES)
def test_products_with_bias_squared_relu_tanh_and_residual(place, m, n, k):
    a, w, b = rand(m, k), rand(n, k, scale=k ** -0.5), rand(n)
    y = a.double() @ w.double().t()
    z = (y + b.double()).clamp(min=0)
    close(X.linear_bias(put(a, place), put(w, place), put(b, place), "relu2"), z * z, place, rel16=4e-3)
    for n0 in (n, n // 2 // 8 * 8, 5, 0):
        close(X.linear_tanh(put(a, place), put(w, place), n0), torch.cat([y[:, :n0], torch.tanh(y[:, n0:])], -1), place, rel16=4e-3)
    x0 = torch.randn(m, n, generator=GEN)
    x = x0.to(place[0]).clone()
    assert X.linear_residual_(put(a, place), put(w, place), x, bias=put(b, place)) is None
    close(x, x0.double() + y + b.double(), fp32(place))


def test_product_with_a_slice_of_few_columns(place):
    """The second factor of a low-rank projection reads a slice of the first one's rows."""
    for rank in (8, 12, 16, 96):
        p, w = rand(70, 264), rand(48, rank)
        close(X.linear_act(put(p, place)[:, 120 : 120 + rank], put(w, place)), p[:, 120 : 120 + rank].double() @ w.double().t(), place, rel16=4e-3)


# ---------------------------------------------------------------------------------------------- query / key / value preparation
PREP = [(4, 2, 16, 24), (3, 1, 48, 16), (1, 1, 8, 8), (6, 3, 10, 7), (20, 2, 136, 72), (8, 8, 64, 128)]


@pytest.mark.parametrize("H,G,d,e", PREP)
@pytest.mark.parametrize("paged", [False, True])
def test_norms_over_whole_projections(place, H, G, d, e, paged):
    T = 9
    p, qn, kn, temp = rand(T, (H + G) * d + G * e + 8), rand(H * d), rand(G * d), rand(H)
    pages = torch.full((4, 8, G * (d + e)), 5.0, dtype=place[1], device=place[0])
    slots = torch.tensor([17, 3, -1, 0, 31, 8, 9, -1, 16])
    q, rows = X.whole_norm_prep(put(p, place), put(qn, place), put(kn, place), put(temp, place), 2e-2, H, G, e, pages if paged else None,
                                slots.to(place[0]) if paged else None, not paged)
    f = p.double()
    want_q = (plain.unit_rms(f[:, : H * d], 2e-2) * qn.double()).view(T, H, d) * temp.double()[:, None]
    want = torch.cat([plain.unit_rms(f[:, H * d : (H + G) * d], 2e-2) * kn.double(), f[:, (H + G) * d : (H + G) * d + G * e]], -1)
    close(q, want_q, place, rel16=4e-3)
    if not paged:
        close(rows, want, place, rel16=4e-3)
        return
    assert rows.shape[0] == 0
    flat = pages.view(32, -1).cpu().float()
    close(flat[slots[slots >= 0]], want[slots >= 0], place, rel16=4e-3)
    left = [i for i in range(32) if i not in slots.tolist()]
    assert bool((flat[left] == 5.0).all())


@pytest.mark.parametrize("H,G,GV,d,e,dims", [(8, 4, 2, 16, 24, 16), (4, 0, 0, 48, 16, 32), (2, 2, 1, 24, 40, 6), (12, 4, 2, 10, 14, 10), (4, 2, 1, 64, 128, 64)])
def test_rotation_in_halves_without_norms(place, H, G, GV, d, e, dims):
    """Query and key maps rotated, values as they are; fewer value heads than key maps, or queries alone."""
    T, rot = 21, {"dims": dims, "base": 300.0}
    p = rand(T, (H + G) * d + GV * e)
    cos, sin = F.rope_table(64, dims, 300.0, place[0], None)
    q, rows = X.conv_qkv_prep(put(p, place), None, 0.0, torch.arange(T, dtype=torch.int32, device=place[0]), cos, sin, H, G, d, e, True, cu=i32([0, T], place),
                              want_rows=True, norm=False, v_heads=GV)
    turned = [plain.turn_halves(p[:, i * d : (i + 1) * d].double(), rot) for i in range(H + G)]
    close(q, torch.stack(turned[:H], 1), place, rel16=4e-3)
    if G:
        close(rows, torch.cat([*turned[H:], p[:, (H + G) * d :].double()], -1), place, rel16=4e-3)


# ---------------------------------------------------------------------------------------------- attention
def difference(a, vec, diff, eps):
    """[.., 2 H, e] -> [.., H, e]"""
    x = vec.double().chunk(4)
    lam = plain.difference_weight({"lq1": x[0], "lk1": x[1], "lq2": x[2], "lk2": x[3]}, diff)
    return plain.unit_rms(a[:, 0::2] - lam * a[:, 1::2], eps) * (1.0 - diff)


def plain_attention(q, k, v, scale, chunk, maps):
    """One sequence, the queries on its last keys: [T, H, e]."""
    n, H, visible = q.shape[0], q.shape[1], plain.same_chunk(k.shape[0], {"size": chunk} if chunk else None)[-q.shape[0] :]
    share, out = H // k.shape[1], []
    for h in range(H):
        g = h // maps // share
        out.append(plain.attend(q[:, h].double(), k[:, g * maps + h % maps].double(), v[:, g].double(), scale, visible))
    return torch.stack(out, 1)


ATTENTION = [  # heads, key heads, size, value size
    (4, 2, 16, 24), (3, 3, 48, 96), (2, 1, 72, 40), (1, 1, 8, 8), (6, 2, 10, 14), (9, 1, 40, 128), (4, 4, 64, 128), (2, 1, 128, 72), (2, 2, 128, 256), (20, 1, 24, 136)]


@pytest.mark.parametrize("H,G,d,e", ATTENTION)
@pytest.mark.parametrize("chunk", [0, 1, 20, 64, 100, 128, 333])
@pytest.mark.parametrize("maps", [1, 2])
def test_chunked_and_differential_prompts(place, H, G, d, e, chunk, maps):
    lens, past = [150, 1, 5, 64, 290], [0, 0, 40, 200, 130]    # keys in front of the first query, from a chunk's start on
    past = [n // chunk * chunk if chunk else n for n in past]
    q = [rand(n, H * maps, d) for n in lens]
    k, v = ([rand(n + m, G * r, w) for n, m in zip(lens, past)] for r, w in ((maps, d), (1, e)))
    vec, scale = rand(4 * d, scale=0.3 * d ** -0.5), 1.3 * d ** -0.5
    diff = (put(vec, place), 0.35, 1e-3) if maps == 2 else None
    got = X.grouped_attention_prefill(*(put(torch.cat(z), place) for z in (q, k, v)), i32(offsets(lens), place), i32(offsets([a + b for a, b in zip(lens, past)]), place),
                                      0, scale, chunk=chunk, diff=diff)
    want = torch.cat([plain_attention(*z, scale, chunk, maps) for z in zip(q, k, v)])
    close(got, difference(want, vec, 0.35, 1e-3) if maps == 2 else want, place, rel16=1.5e-2)


@pytest.mark.parametrize("H,G,d,e", ATTENTION)
@pytest.mark.parametrize("chunk", [0, 1, 20, 64, 128, 333])
@pytest.mark.parametrize("maps", [1, 2])
@pytest.mark.parametrize("bs", [8, 64])
def test_chunked_and_differential_steps(place, H, G, d, e, chunk, maps, bs):
    lens, width = [0, 1, 20, 21, 64, 65, 128, 129, 700], G * (maps * d + e)
    q = rand(len(lens), H * maps, d)
    rows = [rand(n, width) for n in lens]
    blocks = 800 // bs
    pages = torch.full((len(lens) * blocks, bs, width), 9.0)
    table = torch.randperm(len(lens) * blocks, generator=GEN).view(len(lens), blocks)
    for s, r in enumerate(rows):
        for i in range(0, len(r), bs):
            pages[table[s, i // bs], : len(r[i : i + bs])] = r[i : i + bs]
    vec, scale = rand(4 * d, scale=0.3 * d ** -0.5), 1.3 * d ** -0.5
    diff = (put(vec, place), 0.35, 1e-3) if maps == 2 else None
    got = X.grouped_attention_decode(put(q, place), put(pages, place), table.int().to(place[0]), i32(lens, place), G, e, 0, scale, chunk=chunk, diff=diff)
    assert got.shape == (len(lens), H, e) and bool((got[0] == 0).all())
    for s, r in enumerate(rows[1:], 1):
        k, v = r[:, : G * maps * d].view(-1, G * maps, d), r[:, G * maps * d :].view(-1, G, e)
        want = plain_attention(q[s : s + 1], k, v, scale, chunk, maps)
        close(got[s : s + 1], difference(want, vec, 0.35, 1e-3) if maps == 2 else want, place, rel16=2e-2)


@pytest.mark.parametrize("maps", [1, 2])
@pytest.mark.parametrize("chunk", [64, 50, 100])
def test_one_loud_key_at_the_edge_of_a_chunk(place, chunk, maps):
    """A key that outweighs all others: seen from its chunk's start on and never from the next chunk, in prompts and in steps."""
    T, d, e, at = 260, 16, 16, chunk
    for loud in (at - 1, at, at + 1, 2 * chunk - 1):
        q, k, v = rand(T, maps, d, scale=0.1), rand(T, maps, d, scale=0.1), rand(T, 1, e)
        q[:, 0, 0], k[loud, 0, 0], v[loud] = 4.0, 16.0, 8.0
        vec = torch.zeros(4 * d)
        diff = (put(vec, place), 0.5, 1e-3) if maps == 2 else None
        want = plain_attention(q, k, v, 1.0, chunk, maps)
        assert float(want[loud, 0].min()) > 7.9 and float(want[loud // chunk * chunk + chunk, 0].abs().max()) < 4.0
        want = difference(want, vec, 0.5, 1e-3) if maps == 2 else want
        got = X.grouped_attention_prefill(put(q, place), put(k, place), put(v, place), i32([0, T], place), i32([0, T], place), 0, 1.0, chunk=chunk, diff=diff)
        close(got, want, place, rel16=1.5e-2)
        rows = torch.cat([k.flatten(1), v.flatten(1)], -1)
        pages = put(torch.cat([rows, torch.zeros(60, rows.shape[1])]).view(20, 16, -1), place)
        steps = [loud, loud + 1, loud // chunk * chunk + chunk - 1, loud // chunk * chunk + chunk]
        table = torch.arange(20, dtype=torch.int32).repeat(len(steps), 1).to(place[0])
        got = X.grouped_attention_decode(put(q[steps], place), pages, table, i32([s + 1 for s in steps], place), 1, e, 0, 1.0, chunk=chunk, diff=diff)
        close(got, want[steps], place, rel16=1.5e-2)


# ---------------------------------------------------------------------------------------------- generalized delta rule
def delta_inputs(T, H, d, same_keys=False):
    n = H * d
    p, zw = rand(T, 5 * n + 8), rand(T, n, scale=1.5)
    if same_keys:                                  # every token writes at the same place: the removals matter most
        p[:, n : 2 * n] = p[:1, n : 2 * n]
    return p, zw, rand(n) + 1.0, rand(n)


def plain_delta(p, zw, ab, w0, H):
    n = ab.numel()
    d = n // H
    part = lambda z: z.double().view(-1, H, d)
    w, a = plain.decay_and_rate(zw.double(), w0.double(), p[:, 3 * n : 4 * n].double(), ab.double())
    r, k, v, w, a = (part(z) for z in (p[:, :n], p[:, n : 2 * n], p[:, 2 * n : 3 * n], w, a))
    return torch.cat([plain.delta_rule(r[:, h], k[:, h], v[:, h], w[:, h], a[:, h]) for h in range(H)], -1)


DELTA = [(2, 8), (3, 32), (1, 40), (4, 64), (2, 96), (2, 128), (3, 10), (2, 7), (1, 136), (1, 250), (1, 260), (1, 1)]


@pytest.mark.parametrize("H,d", DELTA)
@pytest.mark.parametrize("same_keys", [False, True])
def test_delta_rule_over_prompts(place, H, d, same_keys):
    lens = [1, 16, 90, 17, 15, 33]
    p, zw, ab, w0 = delta_inputs(sum(lens), H, d, same_keys)
    cu = offsets(lens)
    got = X.delta_prefill(put(p, place), put(zw, place), put(ab, place), put(w0, place), H, i32(cu, place))
    want = torch.cat([plain_delta(p[a:b], zw[a:b], ab, w0, H) for a, b in zip(cu, cu[1:])])
    close(got, want, place, rel16=4e-3)


@pytest.mark.parametrize("H,d", DELTA)
def test_delta_rule_in_portions_and_steps(place, H, d):
    """Portions of two slots, then steps with the output norm and the gate; the states agree and other slots stay as they are."""
    n, lens, eps = H * d, {1: 70, 3: 61}, 1e-2
    data = {s: delta_inputs(T, H, d) for s, T in lens.items()}
    ab, w0, norm = data[1][2], data[1][3], rand(n)
    state = torch.full((5, n * d), 3.0, device=place[0])
    want = {s: plain_delta(data[s][0], data[s][1], ab, w0, H) for s in lens}
    at = 0
    for c in (2, 16, 1, 29, 7):
        p, zw = (torch.cat([data[s][i][at : at + c] for s in lens]) for i in (0, 1))
        got = X.delta_prefill(put(p, place), put(zw, place), put(ab, place), put(w0, place), H, i32([0, c, 2 * c], place), state, i32([1, 3], place), i32([int(at == 0)] * 2, place))
        close(got, torch.cat([want[s][at : at + c] for s in lens]), place, rel16=4e-3)
        at += c
    while at < 70:
        p, zw = rand(5, 5 * n + 8), rand(5, n)
        active = torch.tensor([False, True, False, at < 61, False])
        for s in lens:
            if active[s]:
                p[s], zw[s] = data[s][0][at], data[s][1][at]
        got = X.delta_decode(put(p, place), put(zw, place), put(ab, place), put(w0, place), H, put(norm, place), eps, state, active.to(place[0])).cpu()
        for s in lens:
            if active[s]:
                o = plain.unit_rms(want[s][at].view(H, d), eps).flatten() * norm.double() * plain.sigmoid(p[s, 4 * n : 5 * n].double())
                close(got[s], o, place, rel16=4e-3)
        at += 1
    assert bool((state[[0, 2, 4]] == 3.0).all())


@pytest.mark.gpu
@pytest.mark.parametrize("d,lens", [(32, [2500, 2100]), (64, [4200]), (96, [2100, 2200]), (128, [4100])])
def test_delta_rule_over_long_prompts_in_segments(d, lens):
    """Few long prompts are cut into segments that run side by side, also behind a state that was kept."""
    place, H = ("cuda", torch.bfloat16), 2
    GEN.manual_seed(d)
    p, zw, ab, w0 = delta_inputs(sum(lens), H, d)
    cu, n = offsets(lens), H * d
    want = X.delta_prefill(p, zw, ab, w0, H, torch.tensor(cu))
    args = (put(p, place), put(zw, place), put(ab, place), put(w0, place), H)
    close(X.delta_prefill(*args, i32(cu, place)), want, place, rel16=4e-3)
    state, slots = torch.zeros(len(lens), n * d, device="cuda"), i32(list(range(len(lens))), place)
    first = 40                                       # a short portion leaves a state, the long rest starts from it
    at = [torch.arange(a, a + first) for a in cu[:-1]], [torch.arange(a + first, b) for a, b in zip(cu, cu[1:])]
    for part, fresh in zip(at, (1, 0)):
        idx = torch.cat(part)
        got = X.delta_prefill(put(p[idx], place), put(zw[idx], place), *args[2:], i32(offsets([len(a) for a in part]), place), state, slots, i32([fresh] * len(lens), place))
        close(got, want[idx], place, rel16=4e-3)


@pytest.mark.parametrize("t,heads,size", [(1, 2, 16), (5, 3, 35), (40, 4, 64), (3, 2, 264), (70, 32, 64)])
def test_gated_norm_of_every_head(place, t, heads, size):
    width = heads * size
    both, w = rand(t, 2 * width + 8), rand(width)
    got = X.gated_rms(put(both[:, :width].contiguous(), place), put(both, place)[:, width + 8 :], put(w, place), 3e-2, heads)
    o, g = both[:, :width].double(), both[:, width + 8 :].double()
    close(got, plain.unit_rms(o.view(t, heads, size), 3e-2).flatten(1) * w.double() * plain.sigmoid(g), place)
