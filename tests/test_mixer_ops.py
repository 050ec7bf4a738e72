"""Operators of the mixer stacks, one mechanism at a time, against the plain restatement (``oracles/mixer_stack_plain.py``)."""

import math
import zlib

import pytest
import torch

from oracles import mixer_stack_plain as plain
from verl_b200.models.mixer_stack_config import _rotary
from verl_b200.ops import functional as F
from verl_b200.ops import mixers as X

PLACES = [pytest.param(("cpu", torch.float32), id="cpu-fp32"),
          pytest.param(("cuda", torch.float32), id="cuda-fp32", marks=pytest.mark.gpu),
          pytest.param(("cuda", torch.bfloat16), id="cuda-bf16", marks=pytest.mark.gpu)]
GEN = torch.Generator().manual_seed(7)


@pytest.fixture(params=PLACES)
def place(request):
    GEN.manual_seed(zlib.crc32(request.node.name.split("[")[0].encode()))     # the same inputs whatever ran before
    return request.param


def rand(*shape, scale=1.0):
    """Random values that bf16 holds exactly, so every path starts from the same numbers."""
    return (torch.randn(*shape, generator=GEN) * scale).bfloat16().float()


def put(t, place):
    return t.to(place[0], place[1])


def close(got, want, place, rel32=2e-5, rel16=1.2e-2):
    got, want = got.detach().cpu().double(), want.double()
    err = float((got - want).pow(2).mean().sqrt() / want.pow(2).mean().sqrt().clamp_min(1e-6))
    assert math.isfinite(err) and err < (rel32 if place[1] == torch.float32 else rel16), err


def i32(v, place):
    return torch.tensor(v, dtype=torch.int32, device=place[0])


# ---------------------------------------------------------------------------------------------- norm, embedding, GEMM epilogues
@pytest.mark.parametrize("width", [24, 65, 1088])
def test_dynamic_tanh_and_scaled_embedding(place, width):
    table, w, b, alpha = rand(11, width), rand(width), rand(width), torch.tensor([0.75])
    ids = torch.tensor([3, 0, 10, 3, 7])
    x, h = X.embed_dyt(ids.to(place[0]), put(table, place), 1.7, *(put(t, place) for t in (alpha, w, b)))
    assert x.dtype == torch.float32
    close(x, table[ids].double() * 1.7, (place[0], torch.float32), rel32=1e-6)
    close(h, plain.dynamic_tanh(table[ids].double() * 1.7, 0.75, w.double(), b.double()), place, rel16=4e-3)
    tiny = rand(4, width, scale=1e-4)   # the linear range of tanh, and its saturation
    for z in (tiny, tiny * 3e5):
        close(X.dynamic_tanh(z.to(place[0]), *(put(t, place) for t in (alpha, w, torch.zeros(width)))),
              plain.dynamic_tanh(z.double(), 0.75, w.double(), torch.zeros(width).double()), place, rel16=4e-3)


@pytest.mark.parametrize("m,n,k", [(1, 8, 16), (5, 24, 40), (37, 130, 72), (64, 10, 30), (300, 264, 576), (1100, 392, 136), (8, 640, 2176)])
def test_linear_epilogues(place, m, n, k):
    a, w = rand(m, k), rand(n, k, scale=k ** -0.5)
    want = a.double() @ w.double().t()
    A, W = put(a, place), put(w, place)
    close(X.linear_act(A, W), want, place, rel16=4e-3)
    close(X.linear_act(A, W, out_f32=True), want, (place[0], torch.float32))
    close(X.linear_act(A, W, "gelu_erf"), plain.gelu_erf(want), place, rel16=4e-3)
    n0 = n // 16 * 8 if n >= 16 else n // 2
    lo, hi = X.linear_split(A, W, n0)
    assert hi.dtype == torch.float32 and lo.dtype == place[1]
    close(lo, want[:, :n0], place, rel16=4e-3)
    close(hi, want[:, n0:], (place[0], torch.float32))
    x0, nw, nb, alpha = torch.randn(m, n, generator=GEN), rand(n), rand(n), torch.tensor([0.625])
    x = x0.to(place[0]).clone()
    h = X.linear_residual_(A, W, x, tuple(put(t, place) for t in (alpha, nw, nb)))
    close(x, x0.double() + want, (place[0], torch.float32))
    close(h, plain.dynamic_tanh(x0.double() + want, 0.625, nw.double(), nb.double()), place, rel16=4e-3)
    assert X.linear_residual_(A, W, x) is None
    close(x, x0.double() + 2 * want, (place[0], torch.float32))


@pytest.mark.parametrize("m,h,k,n", [(3, 2, 24, 40), (33, 5, 10, 14), (70, 3, 128, 192), (130, 2, 320, 72)])
def test_headwise_linear(place, m, h, k, n):
    wide = rand(m, h, k + 8)
    a, w, wt, gate = wide[..., :k], rand(h, n, k, scale=k ** -0.5), rand(h, k, n, scale=k ** -0.5), torch.randn(m, h + 3, generator=GEN)
    A = put(wide, place)[..., :k]
    close(X.headwise_linear(A, put(w, place), False), torch.einsum("mhk,hnk->mhn", a.double(), w.double()), place, rel16=4e-3)
    got = X.headwise_linear(A, put(wt, place), True, gate.to(place[0]))
    close(got, torch.einsum("mhk,hkn->mhn", a.double(), wt.double()) * torch.sigmoid(gate[:, :h].double()).unsqueeze(-1), place, rel16=4e-3)


# ---------------------------------------------------------------------------------------------- rotation
ROTS = [dict(dims=16, base=10000.0), dict(dims=12, base=500.0, scaling=dict(factor=8.0, original=64, fast=32.0, slow=1.0)),
        dict(dims=8, base=50000.0, scaling=dict(factor=2.0, original=4096, fast=4.0, slow=2.0)),
        dict(dims=6, base=30.0, scaling=dict(factor=16.0, original=100000, fast=3.0, slow=2.9))]


@pytest.mark.parametrize("rot", ROTS)
def test_rotation_of_pairs(place, rot):
    spec = _rotary(rot)
    cos, sin = F.rope_table(700, spec.dims, spec.base, place[0], spec.scaling)
    pos = torch.tensor([0, 1, 2, 63, 64, 65, 300, 699])
    x = rand(8, 3, rot["dims"] + 10)
    want = x.clone().double()
    want[..., 4:] = plain.rotate_pairs(want[..., 4:], pos, rot)
    got = put(x, place)
    X.rope_pairs_(got, pos.to(place[0], torch.int32), cos, sin, 4)
    close(got, want, place, rel16=4e-3)


@pytest.mark.parametrize("q_rank,kv_rank,rot_dim,bs", [(40, 64, 16, 16), (10, 14, 6, 4), (136, 512, 64, 64)])
def test_latent_preparation_appends_to_pages(place, q_rank, kv_rank, rot_dim, bs):
    rot = dict(dims=rot_dim, base=3000.0, scaling=dict(factor=4.0, original=256, fast=16.0, slow=1.0))
    spec, T, eps = _rotary(rot), 9, 1e-5
    cos, sin = F.rope_table(256, spec.dims, spec.base, place[0], spec.scaling)
    p, qn, kn = rand(T, q_rank + kv_rank + rot_dim, scale=0.02), rand(q_rank), rand(kv_rank)
    pos = torch.tensor([0, 3, 15, 16, 17, 31, 32, 100, 200])
    slots = torch.tensor([5, 0, -1, 3 * bs - 1, 2 * bs, bs, bs - 1, -1, 4 * bs + 2])
    pages = torch.zeros(5, bs, kv_rank + rot_dim).to(*place)
    cq, rows = X.latent_prep(put(p, place), put(qn, place), put(kn, place), eps, i32(pos.tolist(), place), cos, sin, pages, slots.to(place[0]), True)
    d = p.double()
    close(cq, plain.unit_rms(d[:, :q_rank], eps) * qn.double(), place, rel16=4e-3)
    want = torch.cat([plain.unit_rms(d[:, q_rank : q_rank + kv_rank], eps) * kn.double(), plain.rotate_pairs(d[:, q_rank + kv_rank :], pos, rot)], -1)
    close(rows[:, :kv_rank], want[:, :kv_rank], place, rel16=4e-3)
    close(rows[:, kv_rank:], want[:, kv_rank:], place, rel16=4e-3)
    flat = pages.cpu().reshape(5 * bs, -1)
    for t, s in enumerate(slots.tolist()):
        if s >= 0:
            assert torch.equal(flat[s], rows[t].cpu())
    untouched = torch.ones(5 * bs, dtype=torch.bool)
    untouched[slots[slots >= 0]] = False
    assert not flat[untouched].any()


# ---------------------------------------------------------------------------------------------- attention
def attention_want(q, ku, kr, v, window, scale, sink, gate):
    """One sequence, fp64; the last query sits on the last key."""
    nq, nk, du = q.shape[0], ku.shape[0], ku.shape[2]
    s = (torch.einsum("qhd,khd->hqk", q[..., :du], ku) + torch.einsum("qhd,kd->hqk", q[..., du:], kr)) * scale
    seen = plain.window_mask(nk, window or None)[nk - nq :]
    o = torch.einsum("hqk,khd->qhd", plain.softmax_with_sink(s, seen, sink), v)
    return o * torch.sigmoid(gate)[:, :, None]


ATT_SIZES = [(3, 16, 8, 24), (2, 128, 64, 128), (5, 40, 24, 48), (2, 10, 6, 12), (1, 64, 48, 64), (5, 48, 16, 128), (2, 128, 128, 128), (2, 64, 16, 192)]


@pytest.mark.parametrize("heads,du,dr,dv", ATT_SIZES)
@pytest.mark.parametrize("window", [0, 1, 7, 64, 100, 129, 1000])
def test_prompt_attention(place, heads, du, dr, dv, window):
    lens, past = [1, 2, 70, 300, 128, 65], [0, 5, 0, 0, 33, 200]
    scale, sink = (du + dr) ** -0.5, rand(heads)
    qs, ks, vs, rs, gs, want = [], [], [], [], [], []
    for n, m in zip(lens, past):
        q, ku, kr, v, g = rand(n, heads, du + dr), rand(n + m, heads, du), rand(n + m, dr), rand(n + m, heads, dv), torch.randn(n, heads, generator=GEN)
        if window and n > window:
            # one key that outweighs everything for the queries just inside and just outside its window
            j = (n + m) - window - 1
            for i in (n - 1, n - 2):
                q[i, :, :du] = ku[j] * 4.0
        want.append(attention_want(*(t.double() for t in (q, ku, kr, v)), window, scale, sink.double(), g.double()))
        qs.append(q), ks.append(ku), rs.append(kr), vs.append(v), gs.append(g)
    cu = lambda c: i32([0] + torch.tensor(c).cumsum(0).tolist(), place)
    kv = put(torch.cat([torch.cat(ks).flatten(1), torch.cat(vs).flatten(1)], 1), place)      # one matrix, as the model has it
    got = X.latent_attention_prefill(put(torch.cat(qs), place), kv[:, : heads * du].unflatten(1, (heads, du)), put(torch.cat(rs), place),
                                     kv[:, heads * du :].unflatten(1, (heads, dv)), cu(lens), cu([n + m for n, m in zip(lens, past)]), window, scale,
                                     put(sink, place), torch.cat(gs).to(place[0]))
    row = 0
    for n, w in zip(lens, want):
        close(got[row : row + n], w, place)
        close(got[row + n - 1], w[-1], place, rel16=2e-2)
        row += n


def test_sink_takes_its_share(place):
    """A large sink empties the output, a very negative one leaves the plain softmax; it does not scale with the scores."""
    h, du, dr, dv, n = 2, 16, 8, 16, 40
    q, ku, kr, v = rand(n, h, du + dr), rand(n, h, du), rand(n, dr), rand(n, h, dv)
    gate = torch.full((n, h), 30.0)
    for sink in (torch.tensor([20.0, -60.0]), torch.tensor([2.0, 0.5])):
        want = attention_want(*(t.double() for t in (q, ku, kr, v)), 9, 0.01, sink.double(), gate.double())
        got = X.latent_attention_prefill(put(q, place), put(ku, place), put(kr, place), put(v, place), i32([0, n], place), i32([0, n], place), 9, 0.01,
                                         put(sink, place), gate.to(place[0]))
        for i in range(h):
            close(got[:, i], want[:, i], place)


@pytest.mark.parametrize("heads,rank,dr,bs", [(6, 120, 40, 16), (3, 20, 6, 8), (16, 512, 64, 64), (20, 256, 64, 32), (2, 72, 24, 64), (1, 64, 16, 16)])
@pytest.mark.parametrize("window", [0, 1, 16, 33, 64, 200])
def test_decode_attention_over_pages(place, heads, rank, dr, bs, window):
    ctx = [1, 0, 2, 15, 16, 17, 33, 64, 65, 200, 201, 500]
    S, per = len(ctx), -(-max(ctx) // bs)
    pages = put(rand(S * per + 3, bs, rank + dr), place)
    table = torch.randperm(S * per + 3, generator=GEN)[: S * per].view(S, per).to(torch.int32)
    q, sink, scale = rand(S, heads, rank + dr), rand(heads), (rank + dr) ** -0.5
    rows_of = lambda b, n: pages.cpu().float()[table[b].long()].reshape(per * bs, -1)[:n]
    for b, n in enumerate(ctx):
        if window and n > window:
            q[b] = rows_of(b, n)[n - window - (b % 2)] * 2.0       # the key on the window's edge, inside or outside
        elif n > 1:
            q[b] = rows_of(b, n)[0] * 2.0                          # the farthest key
    got = X.latent_attention_decode(put(q, place), pages, table.to(place[0]), i32(ctx, place), rank, window, scale, put(sink, place))
    for b, n in enumerate(ctx):
        if n == 0:
            assert not got[b].any()
            continue
        r = rows_of(b, n).double()
        s = torch.einsum("hd,kd->hk", q[b].double(), r)[:, None] * scale
        p = plain.softmax_with_sink(s, plain.window_mask(n, window or None)[-1:], sink.double())[:, 0]
        close(got[b], p @ r[:, :rank], place)


# ---------------------------------------------------------------------------------------------- mLSTM
def mlstm_inputs(T, H, d, e, gate_scale=2.0, f_bias=1.0):
    p = rand(T, 2 * H * (d + e))
    gates = torch.randn(T, 2 * H + 5, generator=GEN) * gate_scale
    return p, gates, rand(H), (rand(H) + f_bias).bfloat16().float(), rand(H * e)


def mlstm_want(p, gates, ib, fb, norm, cap, eps, H, d, e):
    p, gates, ib, fb, norm = (t.double() for t in (p, gates, ib, fb, norm))
    T = p.shape[0]
    il = cap * torch.tanh((gates[:, :H] + ib) / cap)
    fl = torch.nn.functional.logsigmoid(cap * torch.tanh((gates[:, H : 2 * H] + fb) / cap))
    q, k, v = p[:, : H * d].view(T, H, d) * d ** -0.5, p[:, H * d : 2 * H * d].view(T, H, d), p[:, 2 * H * d : 2 * H * d + H * e].view(T, H, e)
    o = plain.unit_rms(plain.mlstm_recurrence(q, k, v, il, fl), eps).reshape(T, -1)
    return o * norm * torch.sigmoid(p[:, 2 * H * d + H * e :])


MLSTM_SIZES = [(2, 16, 24), (3, 40, 16), (1, 128, 256), (2, 64, 64), (2, 10, 14), (1, 256, 96), (2, 72, 320), (1, 64, 32)]


@pytest.mark.parametrize("all_fresh", [False, True])
@pytest.mark.parametrize("H,d,e", MLSTM_SIZES)
def test_mlstm_prompts_and_steps(place, H, d, e, all_fresh):
    """Prompts of unequal length, portions and single steps give what the token-by-token recurrence gives; slots are reused."""
    cap, eps, slots_n = 9.0, 1e-6, 6
    size = H * (d * e + d + 1)
    state = torch.full((slots_n, -(-size // 4) * 4 + 8), 3.0, device=place[0])[:, :size]       # stale content of an earlier user
    lens = [1, 2, 63, 64, 65, 150 if not all_fresh else 900]
    parts = [mlstm_inputs(n + 12, H, d, e) for n in lens]
    want = [mlstm_want(p, g, parts[0][2], parts[0][3], parts[0][4], cap, eps, H, d, e) for p, g, *_ in parts]
    ib, fb, norm = (put(t, place) for t in parts[0][2:])
    slots = [3, 0, 5, 1, 4, 2]
    cut = lambda lo, hi: (put(torch.cat([p[a:b] for (p, *_), a, b in zip(parts, lo, hi)]), place),
                          torch.cat([g[a:b] for (_, g, *_), a, b in zip(parts, lo, hi)]).to(place[0]))
    cu = lambda n: i32([0] + torch.tensor(n).cumsum(0).tolist(), place)
    p, g = cut([0] * 6, lens)
    got = X.mlstm_prefill(p, g, ib, fb, cap, norm, eps, d, cu(lens), state, i32(slots, place), i32([1] * 6, place), all_fresh)
    row = 0
    for n, w in zip(lens, want):
        close(got[row : row + n], w[:n], place)
        row += n
    alone = X.mlstm_prefill(p, g, ib, fb, cap, norm, eps, d, cu(lens))
    close(alone, torch.cat([w[:n] for n, w in zip(lens, want)]), place)
    p, g = cut(lens, [n + 7 for n in lens])                                                     # a portion that goes on
    got = X.mlstm_prefill(p, g, ib, fb, cap, norm, eps, d, cu([7] * 6), state, i32(slots, place), i32([0] * 6, place))
    for j, (n, w) in enumerate(zip(lens, want)):
        close(got[j * 7 : j * 7 + 7], w[n : n + 7], place)
    active = torch.tensor([True, True, True, False, True, True], device=place[0])               # slot 3 rests
    frozen = state[3].clone()
    for t in range(7, 12):
        order = [slots.index(s) for s in range(slots_n)]
        P = put(torch.stack([parts[j][0][lens[j] + t] for j in order]), place)
        G = torch.stack([parts[j][1][lens[j] + t] for j in order]).to(place[0])
        got = X.mlstm_decode(P, G, ib, fb, cap, norm, eps, d, state, active)
        for s, j in enumerate(order):
            if s != 3:
                close(got[s], want[j][lens[j] + t], place)
    assert torch.equal(state[3], frozen)


@pytest.mark.parametrize("gate_scale,f_bias", [(0.3, 6.0), (8.0, 0.0), (1.0, -8.0)])
def test_mlstm_gate_extremes(place, gate_scale, f_bias):
    """Almost no forgetting over a long prompt, gates at their cap, and almost immediate forgetting."""
    H, d, e, T = 2, 32, 48, 700
    p, g, ib, fb, norm = mlstm_inputs(T, H, d, e, gate_scale, f_bias)
    p[5, H * d : 2 * H * d] *= 6.0                                                               # an early key that must still count
    want = mlstm_want(p, g, ib, fb, norm, 15.0, 1e-6, H, d, e)
    got = X.mlstm_prefill(put(p, place), g.to(place[0]), put(ib, place), put(fb, place), 15.0, put(norm, place), 1e-6, d, i32([0, T], place))
    close(got[-100:], want[-100:], place, rel32=1e-4)
    close(got, want, place, rel32=1e-4)


def test_mlstm_starts_from_zero_maximum(place):
    """The running maximum starts at 0: with strongly negative gates the denominator is exp(-m), not the key product."""
    H, d, e, T = 1, 16, 16, 3
    p, g, _, _, norm = mlstm_inputs(T, H, d, e, 0.0)
    ib, fb = torch.tensor([-6.0]), torch.tensor([8.0])
    want = mlstm_want(p, g, ib, fb, norm, 10.0, 1e-2, H, d, e)
    got = X.mlstm_prefill(put(p, place), g.to(place[0]), put(ib, place), put(fb, place), 10.0, put(norm, place), 1e-2, d, i32([0, T], place))
    close(got, want, place)


@pytest.mark.parametrize("m,h,dim,rank,rot_dim", [(3, 2, 24, 40, 8), (33, 5, 10, 14, 6), (70, 3, 128, 512, 64), (20, 17, 64, 136, 32)])
def test_absorbed_query(place, m, h, dim, rank, rot_dim):
    rot = dict(dims=rot_dim - 2, base=700.0)
    spec = _rotary(rot)
    cos, sin = F.rope_table(64, spec.dims, spec.base, place[0], spec.scaling)
    q, uk, pos = rand(m, h, dim + rot_dim), rand(h, dim, rank, scale=dim ** -0.5), torch.randint(0, 64, (m,), generator=GEN)
    got = X.latent_absorb(put(q, place), put(uk, place), pos.to(place[0], torch.int32), cos, sin)
    close(got[..., :rank], torch.einsum("mhd,hdr->mhr", q[..., :dim].double(), uk.double()), place, rel16=4e-3)
    close(got[..., rank:], plain.rotate_pairs(q[..., dim:].double(), pos, rot), place, rel16=4e-3)
