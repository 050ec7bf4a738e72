"""Operators of the mixer stacks (``models/mixer_stack.py``): norms, GEMMs with fused epilogues, latent attention over expanded
keys (prompts) and over the paged latents (decoding), grouped-query attention with capped scores over cached keys and values,
differential attention, mixtures of experts, short convolutions, and the mLSTM, lightning and delta-rule recurrences.

As in ``functional``: CUDA tensors go to the hand-written kernels (bf16 or true fp32; nothing falls back silently), CPU
tensors take a plain PyTorch path. The residual stream, gates, statistics and recurrent state are fp32 on every path.
"""

from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Optional

import torch
import torch.nn.functional as TF

from . import native

__all__ = ["embed_dyt", "dynamic_tanh", "linear_act", "linear_split", "linear_residual_", "rope_pairs_", "latent_prep", "gather_pages",
           "headwise_linear", "latent_absorb", "latent_attention_prefill", "latent_attention_decode", "mlstm_prefill", "mlstm_decode",
           "embed_rms", "linear_partial", "linear_softcap", "residual_rms_", "gated_silu", "gated_up", "gated_up_split", "ExpertPlan", "expert_dispatch",
           "expert_up", "expert_down", "qkv_prep", "grouped_attention_prefill", "grouped_attention_decode", "embed_dyt2", "linear_bias",
           "linear_silu", "residual_dyt_", "conv_qkv_prep", "lightning_prefill", "lightning_decode", "gated_rms",
           "embed_rows", "rms_conv", "linear_tanh", "whole_norm_prep", "delta_prefill", "delta_decode"]


def _ops():
    return native.ops()


def _mm(a: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    return a.float() @ w.float().t()


# ----------------------------------------------------------------------------------------------- norm, embedding, GEMMs
def dynamic_tanh(x: torch.Tensor, alpha: torch.Tensor, weight: torch.Tensor, bias: torch.Tensor) -> torch.Tensor:
    """``tanh(alpha x) * weight + bias`` of the fp32 stream, in the weights' type (no statistics over the row)."""
    if x.is_cuda:
        return _ops().dynamic_tanh(x, alpha, weight, bias)
    return (torch.tanh(alpha.float() * x) * weight.float() + bias.float()).to(weight.dtype)


def embed_dyt(ids, weight, scale: float, alpha, nw, nb):
    """(fp32 residual stream ``weight[ids] * scale``, its first Dynamic Tanh)."""
    if weight.is_cuda:
        return _ops().embed_dyt(ids.reshape(-1).contiguous(), weight, float(scale), alpha, nw, nb)
    x = weight[ids.reshape(-1)].float() * scale
    return x, dynamic_tanh(x, alpha, nw, nb)


def embed_dyt2(ids, weight, embed_norm, first_norm):
    """(fp32 residual stream: the Dynamic Tanh ``embed_norm`` of ``weight[ids]``, the Dynamic Tanh ``first_norm`` of that stream)."""
    if weight.is_cuda:
        return _ops().embed_dyt2(ids.reshape(-1).contiguous(), weight, *embed_norm, *first_norm)
    x = dynamic_tanh_f32(weight[ids.reshape(-1)].float(), *embed_norm)
    return x, dynamic_tanh(x, *first_norm)


def dynamic_tanh_f32(x: torch.Tensor, alpha: torch.Tensor, weight: torch.Tensor, bias: torch.Tensor) -> torch.Tensor:
    return torch.tanh(alpha.float() * x) * weight.float() + bias.float()


def linear_act(a: torch.Tensor, w: torch.Tensor, act: Optional[str] = None, out_f32: bool = False) -> torch.Tensor:
    """``a w^T`` with an optional activation (``gelu_erf``) in the epilogue."""
    assert act in (None, "gelu_erf")
    if a.is_cuda:
        return _ops().linear_act(a, w, act == "gelu_erf", bool(out_f32))
    y = _mm(a, w)
    y = TF.gelu(y) if act == "gelu_erf" else y
    return y if out_f32 else y.to(a.dtype)


def linear_split(a: torch.Tensor, w: torch.Tensor, n0: int):
    """``a w^T`` whose first ``n0`` columns come in ``a``'s type and the rest as fp32 (gates that must not be rounded)."""
    if a.is_cuda:
        return _ops().linear_split(a, w, int(n0))
    y = _mm(a, w)
    return y[:, :n0].to(a.dtype).contiguous(), y[:, n0:].contiguous()


def linear_bias(a: torch.Tensor, w: torch.Tensor, b: torch.Tensor, act: Optional[str] = None) -> torch.Tensor:
    """``a w^T + b`` with an optional activation (``relu2``: the square of relu) in the epilogue."""
    assert act in (None, "relu2")
    if a.is_cuda:
        return _ops().linear_bias(a, w, b, act == "relu2")
    y = _mm(a, w) + b.float()
    return (y if act is None else y.clamp(min=0).square()).to(a.dtype)


def linear_tanh(a: torch.Tensor, w: torch.Tensor, n0: int) -> torch.Tensor:
    """``a w^T`` with a tanh on the columns from ``n0`` on."""
    if a.is_cuda:
        return _ops().linear_tanh(a, w, int(n0))
    y = _mm(a, w)
    return torch.cat([y[:, :n0], torch.tanh(y[:, n0:])], -1).to(a.dtype)


def linear_silu(a: torch.Tensor, w: torch.Tensor, n0: int) -> torch.Tensor:
    """``a w^T`` with a silu on the first ``n0`` columns."""
    if a.is_cuda:
        return _ops().linear_silu(a, w, int(n0))
    y = _mm(a, w)
    return torch.cat([TF.silu(y[:, :n0]), y[:, n0:]], -1).to(a.dtype)


def linear_residual_(a: torch.Tensor, w: torch.Tensor, x: torch.Tensor, norm=None, post=None, bias=None) -> Optional[torch.Tensor]:
    """``x += a w^T (+ bias)`` on the fp32 residual stream, or with ``post = (alpha, weight, bias)`` the Dynamic Tanh of that product; with
    ``norm`` (likewise) also returns the Dynamic Tanh of the new stream, computed in the same epilogue."""
    none = (None, None, None)
    if a.is_cuda:
        h = _ops().linear_residual_(a, w, x, *(norm if norm is not None else none), *(post if post is not None else none), bias)
        return h if norm is not None else None
    y = _mm(a, w) if bias is None else _mm(a, w) + bias.float()
    x += y if post is None else dynamic_tanh_f32(y, *post)
    return dynamic_tanh(x, *norm) if norm is not None else None


def residual_dyt_(x, rows, slot, post, norm) -> torch.Tensor:
    """``x += post(Y)`` on the fp32 residual stream with Y[t] the sum of the expert rows ``rows[slot[t, j]]``; returns ``norm`` of the
    new stream (both Dynamic Tanh ``(alpha, weight, bias)``)."""
    if x.is_cuda:
        return _ops().residual_dyt_(x, rows, slot, *post, *norm)
    x += dynamic_tanh_f32(rows[slot.long()].float().sum(1), *post)
    return dynamic_tanh(x, *norm)


# ----------------------------------------------------------------------------------------------- RMS norms on sublayer outputs
def _rms(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps) * w.float()


def embed_rms(ids, weight, scale: float, nw, eps: float):
    """(fp32 residual stream ``rms_norm(weight[ids] * scale) * nw``, the same in the weights' type)."""
    if weight.is_cuda:
        return _ops().embed_rms(ids.reshape(-1).contiguous(), weight, float(scale), nw, float(eps))
    x = _rms(weight[ids.reshape(-1)].float() * scale, nw, eps)
    return x, x.to(weight.dtype)


def embed_rows(ids, weight, scale: float) -> torch.Tensor:
    """fp32 residual stream ``weight[ids] * scale``."""
    if weight.is_cuda:
        return _ops().embed_rows(ids.reshape(-1).contiguous(), weight, float(scale))
    return weight[ids.reshape(-1)].float() * scale


def rms_conv(x: torch.Tensor, nw: torch.Tensor, eps: float, y=None, bias=None, conv=None, cu=None, state=None, slots=None, fresh=None, active=None) -> torch.Tensor:
    """``h = rms_norm(x) * nw`` of the fp32 residual stream in the weights' type, or with ``conv`` [width, taps] ``h`` plus its causal
    convolution over time (last tap: the token itself, zeros before a sequence's first token). ``y`` ([T, W], or partial products
    [splits, T, W]) and ``bias`` are added to ``x`` first (not with ``cu``). Portions (``cu``), steps (``active``) and ``state`` as in
    ``conv_qkv_prep``: what is kept are the last taps - 1 rows ``h`` (fp32) of a sequence."""
    assert y is None or cu is None, "rms_conv: portions take the stream as it is"
    if x.is_cuda:
        return _ops().rms_conv(x, y, bias, nw, float(eps), conv, cu, state, slots, fresh, active)
    if y is not None:
        x += y.float().sum(0) if y.dim() == 3 else y.float()
    if bias is not None:
        x += bias.float()
    h = _rms(x, nw, eps)
    if conv is not None:
        h = h + _conv_rows(h, conv, cu, state, slots, fresh, active)
    return h.to(nw.dtype)


def linear_partial(a: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """``a w^T`` for a consumer that reads whole rows (``residual_rms_``): [M, N] in ``a``'s type, or, where few tokens make the
    GEMM split its depth, the fp32 partial products [splits, M, N] for the consumer to add up."""
    if a.is_cuda:
        return _ops().linear_partial(a, w)
    return _mm(a, w).to(a.dtype)


def residual_rms_(x, y: Optional[torch.Tensor], nw, eps: float, mult: float, next_nw=None, experts=None, gate: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``x += mult * rms_norm(Y) * nw`` on the fp32 residual stream. ``Y`` is ``y`` ([T, W], or partial products [splits, T, W];
    multiplied by ``sigmoid(gate[t])`` when a gate is given) plus, with ``experts = (rows, slot)``, the rows ``slot[t, j]`` of the
    expert outputs. Returns the new stream in the weights' type, or its RMS norm with ``next_nw``."""
    rows, slot = experts if experts is not None else (None, None)
    if x.is_cuda:
        return _ops().residual_rms_(x, y, nw, float(eps), float(mult), next_nw, rows, slot, gate)
    total = torch.zeros_like(x)
    if y is not None:
        total = y.float().sum(0) if y.dim() == 3 else y.float()
        if gate is not None:
            total = total * torch.sigmoid(gate)[:, None]
    if rows is not None:
        total = total + rows[slot.long()].float().sum(1)
    x += mult * _rms(total, nw, eps)
    return (x if next_nw is None else _rms(x, next_nw, eps)).to(nw.dtype)


def linear_softcap(a: torch.Tensor, w: torch.Tensor, cap: float) -> torch.Tensor:
    """``cap * tanh(a w^T / cap)`` in ``a``'s type (``cap`` 0: the plain product)."""
    if cap <= 0:
        return linear_act(a, w)
    if a.is_cuda:
        return _ops().linear_softcap(a, w, float(cap))
    return (cap * torch.tanh(_mm(a, w) / cap)).to(a.dtype)


# ----------------------------------------------------------------------------------------------- gated feed-forward, experts
def gated_silu(gu: torch.Tensor) -> torch.Tensor:
    """``silu(g) * u`` of rows [g | u]."""
    if gu.is_cuda:
        return _ops().gated_silu(gu)
    g, u = gu.float().chunk(2, -1)
    return (TF.silu(g) * u).to(gu.dtype)


def gated_up(h: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """``silu(h W_g^T) * (h W_u^T)`` for the stacked rows ``w = [W_g; W_u]``: in the GEMM's epilogue for prompts."""
    if h.is_cuda and h.dtype == torch.bfloat16 and h.shape[0] > 1024 and w.shape[0] % 16 == 0 and w.shape[1] % 8 == 0 and w.data_ptr() % 16 == 0:
        return _ops().gemm_swiglu(h, w, False)[0]
    return gated_silu(linear_act(h, w))


def gated_up_split(h: torch.Tensor, w: torch.Tensor, n0: int):
    """(``gated_up`` of the first ``n0`` rows of ``w``, fp32 product with the rest); None in the first place when ``n0`` is 0."""
    if n0 == 0:
        return None, linear_act(h, w, out_f32=True)
    if h.shape[0] > 1024:
        return gated_up(h, w[:n0]), linear_act(h, w[n0:], out_f32=True)
    gu, tail = linear_split(h, w, n0)
    return gated_silu(gu), tail


@dataclass
class ExpertPlan:
    """Tokens grouped by expert: ``x`` [rows, width] copies of the tokens (every expert's rows start at a multiple of 128 on the
    GPU), ``slot`` [T, top] row of every copy, ``scale`` [rows] score of the copy's expert, and which expert owns which rows."""

    x: torch.Tensor
    slot: torch.Tensor
    scale: torch.Tensor
    tile_expert: torch.Tensor     # GPU: expert of every 128-row tile; CPU: first row of every expert [E + 1]
    num_tiles: torch.Tensor


def expert_dispatch(h: torch.Tensor, logits: torch.Tensor, experts: int, top: int, renormalize: bool = False, correction: Optional[torch.Tensor] = None,
                    groups: int = 1, keep: int = 1) -> ExpertPlan:
    """Router: the ``top`` experts with the largest ``sigmoid(logits)`` of every token (``logits`` fp32, columns past ``experts``
    ignored), and the tokens' copies in expert order. ``correction`` [experts] is added for the choice only. With ``groups`` > 1 only
    experts of the ``keep`` best groups of neighbours can be chosen; a group counts the sum of its two largest choice scores. No
    host synchronisation."""
    if h.is_cuda:
        return ExpertPlan(*_ops().expert_dispatch(h, logits, int(experts), int(top), bool(renormalize), correction, int(groups), int(keep)))
    score = torch.sigmoid(logits[:, :experts].float())
    choice = score if correction is None else score + correction.float()
    if groups > 1:
        g = choice.view(-1, groups, experts // groups)
        best = torch.topk(torch.topk(g, min(2, g.shape[2]), dim=-1).values.sum(-1), keep, dim=-1).indices
        hidden = torch.ones(g.shape[:2], dtype=torch.bool).scatter_(1, best, False)
        choice = g.masked_fill(hidden.unsqueeze(-1), float("-inf")).flatten(1)
    e = torch.topk(choice, top, dim=-1).indices
    s = score.gather(1, e)
    if renormalize:
        s = s / (s.sum(-1, keepdim=True) + 1e-20)
    order = torch.argsort(e.reshape(-1), stable=True)
    slot = torch.empty_like(order)
    slot[order] = torch.arange(order.numel())
    first = torch.zeros(experts + 1, dtype=torch.int64)
    first[1:] = torch.bincount(e.reshape(-1), minlength=experts).cumsum(0)
    return ExpertPlan(h[order // top], slot.view(-1, top), s.reshape(-1)[order], first, first[-1:])


def expert_up(plan: ExpertPlan, w: torch.Tensor, ff: int, act: str = "silu", limit: float = 0.0) -> torch.Tensor:
    """Per copy ``silu(s g) * (s u)`` with [g | u] = ``x w_e^T`` and the copy's score s (a factor on the expert's input), or with
    ``act`` "clipped" ``s g sigmoid(1.702 g) (u + 1)`` with g <= limit and -limit <= u <= limit; ``w`` [E * 2 ff, width]."""
    assert act in ("silu", "clipped") and (act == "silu" or limit > 0)
    w3 = w.view(-1, 2 * ff, w.shape[1])
    if w.is_cuda:
        return _ops().expert_up(plan.x, w3, plan.scale, plan.tile_expert, plan.num_tiles, float(limit) if act == "clipped" else 0.0)
    out = torch.empty(plan.x.shape[0], ff, dtype=plan.x.dtype)
    for e in range(w3.shape[0]):
        at = slice(int(plan.tile_expert[e]), int(plan.tile_expert[e + 1]))
        if act == "clipped":
            g, u = _mm(plan.x[at], w3[e]).chunk(2, -1)
            g, u = g.clamp(max=limit), u.clamp(-limit, limit)
            out[at] = (g * torch.sigmoid(1.702 * g) * (u + 1.0) * plan.scale[at, None]).to(out.dtype)
            continue
        g, u = (_mm(plan.x[at], w3[e]) * plan.scale[at, None]).chunk(2, -1)
        out[at] = (TF.silu(g) * u).to(out.dtype)
    return out


def expert_down(act: torch.Tensor, w: torch.Tensor, plan: ExpertPlan) -> torch.Tensor:
    """Per copy ``act w_e^T``; ``w`` [E * width, ff]. Rows without a copy hold anything."""
    w3 = w.view(-1, plan.x.shape[1], w.shape[1])
    if w.is_cuda:
        return _ops().expert_linear(act, w3, plan.tile_expert, plan.num_tiles)
    out = torch.empty(act.shape[0], w3.shape[1], dtype=act.dtype)
    for e in range(w3.shape[0]):
        at = slice(int(plan.tile_expert[e]), int(plan.tile_expert[e + 1]))
        out[at] = _mm(act[at], w3[e]).to(out.dtype)
    return out


# ----------------------------------------------------------------------------------------------- latent attention
def _rotate(x: torch.Tensor, pos: torch.Tensor, cos: torch.Tensor, sin: torch.Tensor) -> torch.Tensor:
    """``x`` [T, ..., n] fp32: pairs (2i, 2i + 1) of the first ``2 * cos.shape[1]`` dimensions are turned."""
    half = cos.shape[1]
    shape = (x.shape[0],) + (1,) * (x.dim() - 2) + (half,)
    c, s = cos[pos.long()].view(shape), sin[pos.long()].view(shape)
    pairs = x[..., : 2 * half].unflatten(-1, (half, 2))
    u, v = pairs[..., 0], pairs[..., 1]
    return torch.cat([torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2), x[..., 2 * half :]], -1)


def rope_pairs_(x: torch.Tensor, positions: torch.Tensor, cos: torch.Tensor, sin: torch.Tensor, offset: int = 0) -> torch.Tensor:
    """In-place interleaved rotation of ``x`` [T, heads, n] from dimension ``offset`` on (``2 * cos.shape[1]`` dimensions)."""
    if x.is_cuda:
        _ops().rope_pairs_(x, positions, cos, sin, int(offset), int(2 * cos.shape[1]))
        return x
    x[..., offset:] = _rotate(x[..., offset:].float(), positions, cos, sin).to(x.dtype)
    return x


def latent_prep(p, q_norm, kv_norm, eps: float, positions, cos, sin, pages=None, slots=None, want_rows: bool = False):
    """``p`` [T, q_rank + kv_rank + rot]: RMS-normed query latent (``q_norm`` None: there is none), and the row [normed latent |
    rotated shared key part], which is appended to ``pages`` [blocks, block_size, kv_rank + rot] at ``slots`` (negative: skipped) and / or returned."""
    if p.is_cuda:
        return _ops().latent_prep(p, q_norm, kv_norm, float(eps), positions, cos, sin, pages, slots, bool(want_rows))
    qr, kr = q_norm.numel() if q_norm is not None else 0, kv_norm.numel()
    rms = lambda z, w: z * torch.rsqrt(z.pow(2).mean(-1, keepdim=True) + eps) * w.float()
    f = p.float()
    cq = rms(f[:, :qr], q_norm).to(p.dtype) if qr else p[:, :0]
    row = torch.cat([rms(f[:, qr : qr + kr], kv_norm), _rotate(f[:, qr + kr :], positions, cos, sin)], -1).to(p.dtype)
    if pages is not None:
        ok = slots >= 0
        at, bs = slots[ok], pages.shape[1]
        pages[at // bs, at % bs] = row[ok]
    return cq, (row if want_rows else row[:0])


def gather_pages(pages, block_table, cu_k, k_start, total: int) -> torch.Tensor:
    """[total, width]: for every sequence the cached rows ``k_start[b] .. k_start[b] + cu_k[b + 1] - cu_k[b]`` in order."""
    if pages.is_cuda:
        return _ops().gather_pages(pages, block_table, cu_k, k_start, int(total))
    bs, out = pages.shape[1], []
    for b in range(block_table.shape[0]):
        at = int(k_start[b]) + torch.arange(int(cu_k[b + 1] - cu_k[b]))
        out.append(pages[block_table[b, at // bs].long(), at % bs])
    return torch.cat(out, 0)


def headwise_linear(a: torch.Tensor, w: torch.Tensor, transposed: bool, gate: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Per-head product: ``a`` [M, H, K] with ``w`` [H, N, K], or ``w`` [H, K, N] when ``transposed``; head h of row m is multiplied
    by ``sigmoid(gate[m, h])`` when a gate is given."""
    if a.is_cuda:
        return _ops().headwise_linear(a, w, bool(transposed), gate)
    y = torch.einsum("mhk,hkn->mhn" if transposed else "mhk,hnk->mhn", a.float(), w.float())
    if gate is not None:
        y = y * torch.sigmoid(gate[:, : a.shape[1]]).unsqueeze(-1)
    return y.to(a.dtype).contiguous()


def latent_absorb(q, uk, positions, cos, sin) -> torch.Tensor:
    """Decode query in the latent space: ``q`` [S, H, dim + rot] -> [q_unrotated uk | rotated part] [S, H, kv_rank + rot] with ``uk``
    [H, dim, kv_rank]."""
    if q.is_cuda:
        return _ops().latent_absorb(q, uk, positions, cos, sin)
    dim = uk.shape[1]
    return torch.cat([headwise_linear(q[..., :dim], uk, True), _rotate(q[..., dim:].float(), positions, cos, sin).to(q.dtype)], -1)


def _sink_softmax(s: torch.Tensor, sink: Optional[torch.Tensor]) -> torch.Tensor:
    """Softmax over the last dimension of ``s`` [H, ..., keys] with one extra score per head that has no value."""
    if sink is None:
        return torch.softmax(s, -1)
    extra = sink.float().view(-1, *([1] * (s.dim() - 1))).expand(*s.shape[:-1], 1)
    return torch.softmax(torch.cat([s, extra], -1), -1)[..., :-1]


def _hidden_keys(nq: int, nk: int, window: int, keep_first: int, chunk: int = 0) -> torch.Tensor:
    """[nq, nk]: keys a query does not see; the last query sits on the last key."""
    dist, key = torch.arange(nk - nq, nk)[:, None] - torch.arange(nk)[None, :], torch.arange(nk)[None, :]
    if chunk > 0:
        return (dist < 0) | ((dist + key) // chunk != key // chunk)
    return (dist < 0) | ((dist >= window) & (key >= keep_first) if window > 0 else torch.zeros_like(dist, dtype=torch.bool))


def _seen_keys(n: int, window: int, keep_first: int, chunk: int = 0) -> torch.Tensor:
    """Positions the last of ``n`` tokens sees."""
    key = torch.arange(n)
    if chunk > 0:
        return key[(n - 1) // chunk * chunk :]
    return key[(key >= n - window) | (key < keep_first)] if window > 0 else key


def latent_attention_prefill(q, k_unrot, k_rot, v, cu_q, cu_k, window: int, scale: float, sink=None, gate=None, keep_first: int = 0) -> torch.Tensor:
    """Causal windowed attention of packed prompts: ``q`` [T, H, du + dr] (rotated part last), ``k_unrot`` [Tk, H, du], ``k_rot``
    [Tk, dr] shared by the heads, ``v`` [Tk, H, dv]; the last query of a sequence sits on its last key (``cu_k`` may hold earlier
    keys). ``window`` > 0: a query sees that many keys, its own included, and the first ``keep_first`` keys of the sequence. Output
    times ``sigmoid(gate[t, h])``."""
    if q.is_cuda:
        return _ops().latent_attn_prefill(q, k_unrot, k_rot, v, cu_q, cu_k, sink, gate, int(window), float(scale), int(keep_first))
    out = torch.empty(q.shape[0], q.shape[1], v.shape[2], dtype=q.dtype)
    du = k_unrot.shape[2]
    cq, ck = cu_q.tolist(), cu_k.tolist()
    for b in range(len(cq) - 1):
        qs, ks = slice(cq[b], cq[b + 1]), slice(ck[b], ck[b + 1])
        nq, nk = cq[b + 1] - cq[b], ck[b + 1] - ck[b]
        qq = q[qs].float()
        s = torch.einsum("qhd,khd->hqk", qq[..., :du], k_unrot[ks].float()) + torch.einsum("qhd,kd->hqk", qq[..., du:], k_rot[ks].float())
        hide = _hidden_keys(nq, nk, window, keep_first)
        p = _sink_softmax((s * scale).masked_fill(hide, float("-inf")), sink)
        o = torch.einsum("hqk,khd->qhd", p, v[ks].float())
        if gate is not None:
            o = o * torch.sigmoid(gate[qs, : q.shape[1]])[:, :, None]
        out[qs] = o.to(q.dtype)
    return out


def latent_attention_decode(q, pages, block_table, ctx_len, kv_rank: int, window: int, scale: float, sink=None, keep_first: int = 0) -> torch.Tensor:
    """One query per sequence in the latent space: ``q`` [S, H, kv_rank + rot] against the cached rows, which are key (whole row)
    and value (first ``kv_rank``) of every head. Returns [S, H, kv_rank]; sequences with ``ctx_len`` 0 give zeros."""
    if q.is_cuda:
        return _ops().latent_attn_decode(q, pages, block_table, ctx_len, sink, int(kv_rank), int(window), float(scale), int(keep_first))
    out = torch.zeros(q.shape[0], q.shape[1], kv_rank, dtype=q.dtype)
    bs = pages.shape[1]
    for b, n in enumerate(ctx_len.tolist()):
        if n <= 0:
            continue
        at = _seen_keys(n, window, keep_first)
        rows = pages[block_table[b, at // bs].long(), at % bs].float()
        p = _sink_softmax(q[b].float() @ rows.t() * scale, sink)
        out[b] = (p @ rows[:, :kv_rank]).to(q.dtype)
    return out


# ----------------------------------------------------------------------------------------------- grouped-query attention
def qkv_prep(p, q_norm, k_norm, eps: float, positions, cos, sin, heads: int, kv_heads: int, vdim: int, v_first=None, vmix=None, pages=None, slots=None,
             want_rows: bool = False):
    """``p`` [T, q | k | v]: RMS norm per query and key head, rotation of their first ``2 * cos.shape[1]`` dimensions (pairs 2i,
    2i + 1), and values mixed as ``(1 - vmix) v + vmix v_first`` when ``v_first`` [T, kv_heads * vdim] is given. Returns the queries
    [T, heads, dim]; the row [keys | values] is appended to ``pages`` [blocks, block_size, kv_heads * (dim + vdim)] at ``slots``
    (negative: skipped) and / or returned."""
    dim = q_norm.numel()
    if p.is_cuda:
        return _ops().qkv_prep(p, q_norm, k_norm, float(eps), positions, cos, sin, int(heads), int(kv_heads), int(vdim), v_first, vmix, pages, slots,
                               bool(want_rows))
    T, a, b = p.shape[0], heads * dim, (heads + kv_heads) * dim
    f = p.float()
    q = _rotate(_rms(f[:, :a].view(T, heads, dim), q_norm, eps), positions, cos, sin).to(p.dtype)
    k = _rotate(_rms(f[:, a:b].view(T, kv_heads, dim), k_norm, eps), positions, cos, sin)
    v = f[:, b : b + kv_heads * vdim]
    if v_first is not None:
        v = (1.0 - vmix.float()) * v + vmix.float() * v_first.float()
    row = torch.cat([k.flatten(1), v], -1).to(p.dtype)
    if pages is not None:
        ok = slots >= 0
        at, bs = slots[ok], pages.shape[1]
        pages[at // bs, at % bs] = row[ok]
    return q, (row if want_rows else row[:0])


def _soft_cap(s: torch.Tensor, cap: float) -> torch.Tensor:
    return cap * torch.tanh(s / cap) if cap > 0 else s


def _difference(o: torch.Tensor, diff) -> torch.Tensor:
    """``o`` [..., 2 H, e] fp32, the two maps of a head behind each other -> [..., H, e]."""
    vectors, const, eps = diff
    q1, k1, q2, k2 = vectors.float().chunk(4)
    lam = torch.exp((q1 * k1).sum()) - torch.exp((q2 * k2).sum()) + const
    o = o.unflatten(-2, (-1, 2))
    o = o[..., 0, :] - lam * o[..., 1, :]
    return o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + eps) * (1.0 - const)


def _key_heads(heads: int, kv_heads: int, maps: int) -> torch.Tensor:
    """Key head of every query head; the maps of a head are neighbours."""
    h = torch.arange(heads)
    return h // maps // (heads // maps // kv_heads) * maps + h % maps


def grouped_attention_prefill(q, k, v, cu_q, cu_k, window: int, scale: float, softcap: float = 0.0, sink=None,
                              keep_first: int = 0, chunk: int = 0, diff=None) -> torch.Tensor:
    """Causal attention of packed prompts: ``q`` [T, H, d], ``k`` [Tk, G, d], ``v`` [Tk, G, e] (query head h reads key head h // (H / G));
    scores ``softcap * tanh(q k scale / softcap)``; ``cu_q`` / ``cu_k`` / ``window`` / ``keep_first`` / ``sink`` as in ``latent_attention_prefill``.
    ``chunk`` > 0: a query sees the keys of its own chunk of that many positions (the first key of every sequence starts a chunk).
    ``diff = (vectors, const, eps)``: differential attention, ``q`` [T, 2 H, d] and ``k`` [Tk, 2 G, d] hold the two maps of a head behind
    each other; the outputs a1, a2 become ``(1 - const) rms_norm(a1 - lambda a2)`` without weight, lambda = exp(x1 . x2) - exp(x3 . x4) +
    const with ``vectors`` = x1 | x2 | x3 | x4."""
    if q.is_cuda:
        return _ops().grouped_attn_prefill(q, k, v, cu_q, cu_k, sink, int(window), float(scale), float(softcap), int(keep_first), int(chunk),
                                           *(diff if diff is not None else (None, 0.0, 0.0)))
    maps = 1 if diff is None else 2
    H, G = q.shape[1], v.shape[1]
    out = torch.empty(q.shape[0], H // maps, v.shape[2], dtype=q.dtype)
    kh = _key_heads(H, G, maps)
    cq, ck = cu_q.tolist(), cu_k.tolist()
    for b in range(len(cq) - 1):
        qs, ks = slice(cq[b], cq[b + 1]), slice(ck[b], ck[b + 1])
        nq, nk = cq[b + 1] - cq[b], ck[b + 1] - ck[b]
        s = _soft_cap(torch.einsum("qhd,khd->hqk", q[qs].float(), k[ks].float()[:, kh]) * scale, softcap)
        hide = _hidden_keys(nq, nk, window, keep_first, chunk)
        w = _sink_softmax(s.masked_fill(hide, float("-inf")), sink)
        o = torch.einsum("hqk,khd->qhd", w, v[ks].float()[:, kh // maps])
        out[qs] = (o if diff is None else _difference(o, diff)).to(q.dtype)
    return out


def grouped_attention_decode(q, pages, block_table, ctx_len, kv_heads: int, vdim: int, window: int, scale: float, softcap: float = 0.0,
                             sink=None, keep_first: int = 0, chunk: int = 0, diff=None) -> torch.Tensor:
    """One query per sequence, ``q`` [S, H, d], against cached rows [keys | values] (``qkv_prep``). Returns [S, H, vdim]; sequences
    with ``ctx_len`` 0 give zeros. ``chunk`` and ``diff`` as in ``grouped_attention_prefill``."""
    if q.is_cuda:
        return _ops().grouped_attn_decode(q, pages, block_table, ctx_len, sink, int(kv_heads), int(vdim), int(window), float(scale), float(softcap),
                                          int(keep_first), int(chunk), *(diff if diff is not None else (None, 0.0, 0.0)))
    maps = 1 if diff is None else 2
    bs, G, d, H = pages.shape[1], kv_heads, q.shape[2], q.shape[1]
    out = torch.zeros(q.shape[0], H // maps, vdim, dtype=q.dtype)
    kh = _key_heads(H, G, maps)
    for b, n in enumerate(ctx_len.tolist()):
        if n <= 0:
            continue
        at = _seen_keys(n, window, keep_first, chunk)
        rows = pages[block_table[b, at // bs].long(), at % bs].float()
        k, v = rows[:, : G * maps * d].view(-1, G * maps, d), rows[:, G * maps * d :].view(-1, G, vdim)
        s = _soft_cap(torch.einsum("hd,khd->hk", q[b].float(), k[:, kh]) * scale, softcap)
        o = torch.einsum("hk,khe->he", _sink_softmax(s, sink), v[:, kh // maps])
        out[b] = (o if diff is None else _difference(o, diff)).to(q.dtype)
    return out


# ----------------------------------------------------------------------------------------------- short convolution in front of attention
def _rotate_halves(x: torch.Tensor, pos: torch.Tensor, cos: torch.Tensor, sin: torch.Tensor) -> torch.Tensor:
    """``x`` [T, heads, n] fp32: pairs (i, i + half) of the first ``2 * half`` dimensions are turned."""
    half = cos.shape[1]
    c, s = cos[pos.long()][:, None], sin[pos.long()][:, None]
    u, v = x[..., :half], x[..., half : 2 * half]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * half :]], -1)


def _conv_portion(u: torch.Tensor, w: torch.Tensor, past: torch.Tensor):
    """``u`` [n, C] behind ``past`` [taps - 1, C]: (outputs [n, C], the last taps - 1 inputs)."""
    taps = w.shape[1]
    row = torch.cat([past, u], 0)
    return sum(row[j : j + u.shape[0]] * w[:, j].float() for j in range(taps)), row[row.shape[0] - taps + 1 :]


def _conv_rows(u: torch.Tensor, conv: torch.Tensor, cu, state, slots, fresh, active) -> torch.Tensor:
    """Causal convolution of the rows ``u`` [T, C] of portions or steps (see ``conv_qkv_prep``); moves the kept inputs on."""
    (T, C), n = u.shape, conv.shape[1] - 1
    if n == 0:
        return u * conv[:, 0].float()
    f = torch.zeros(T, C)
    if cu is None:
        for s in torch.nonzero(active).flatten().tolist():
            past = state[s].view(n, C)
            f[s : s + 1], last = _conv_portion(u[s : s + 1], conv, past.clone())
            past.copy_(last)
        return f
    c = cu.tolist()
    for b in range(len(c) - 1):
        past = state[int(slots[b])].view(n, C) if slots is not None else None
        f[c[b] : c[b + 1]], last = _conv_portion(u[c[b] : c[b + 1]], conv, torch.zeros(n, C) if past is None or bool(fresh[b]) else past.clone())
        if past is not None:
            past.copy_(last)
    return f


def conv_qkv_prep(p, conv, eps: float, positions, cos, sin, heads: int, kv_heads: int, dim: int, vdim: int, halves: bool = True, cu=None, state=None, slots=None,
                  fresh=None, active=None, pages=None, page_slots=None, want_rows: bool = False, norm: bool = True, v_heads: Optional[int] = None):
    """``p`` [T, q | k | v]: causal convolution over time (``conv`` [channels, taps], None: none; zeros before a sequence's first
    token), rotation of the first ``2 * cos.shape[1]`` dimensions of every query and key head (pairs (i, i + half), or (2i, 2i + 1)
    without ``halves``), then with ``norm`` an RMS norm without weight over the head. There are ``kv_heads`` key heads (0: queries only) and
    ``v_heads`` value heads (default: as many). Portions (``cu`` given): sequence b goes on from the inputs in
    ``state[slots[b]]`` unless ``fresh[b]``, and leaves its last ones there; without ``slots`` every sequence starts from zeros and
    nothing is kept. Steps (``cu`` None): row s is the next token of ``state[s]`` where ``active[s]``. ``state`` rows: [taps - 1, channels]
    fp32, oldest first. Returns (queries [T, heads, dim], rows [keys | values]) as ``qkv_prep``."""
    v_heads = kv_heads if v_heads is None else v_heads
    if p.is_cuda:
        return _ops().conv_qkv_prep(p, conv, float(eps), positions, cos, sin, int(heads), int(kv_heads), int(v_heads), int(dim), int(vdim), bool(halves), bool(norm),
                                    cu, state, slots, fresh, active, pages, page_slots, bool(want_rows))
    T, C = p.shape[0], (heads + kv_heads) * dim + v_heads * vdim
    f = p[:, :C].float()
    if conv is not None:
        f = _conv_rows(f, conv, cu, state, slots, fresh, active)
    a, b = heads * dim, (heads + kv_heads) * dim
    turn = _rotate_halves if halves else _rotate
    unit = lambda z: z * torch.rsqrt(z.pow(2).mean(-1, keepdim=True) + eps) if norm else z
    q = unit(turn(f[:, :a].view(T, heads, dim), positions, cos, sin)).to(p.dtype)
    k = unit(turn(f[:, a:b].view(T, kv_heads, dim), positions, cos, sin))
    row = torch.cat([k.flatten(1), f[:, b:]], -1).to(p.dtype)
    _append(pages, page_slots, row)
    return q, (row if want_rows else row[:0])


def _append(pages, slots, row) -> None:
    if pages is not None:
        ok = slots >= 0
        at, bs = slots[ok], pages.shape[1]
        pages[at // bs, at % bs] = row[ok]


def whole_norm_prep(p, q_norm, k_norm, temp, eps: float, heads: int, kv_heads: int, vdim: int, pages=None, slots=None, want_rows: bool = False):
    """``p`` [T, q | k | v]: weighted RMS norms over all query and over all key columns, queries times their head's ``temp``. Returns
    (queries [T, heads, dim], rows [keys | values]) and appends the rows as ``qkv_prep`` does."""
    if p.is_cuda:
        return _ops().whole_norm_prep(p, q_norm, k_norm, temp, float(eps), int(heads), int(kv_heads), int(vdim), pages, slots, bool(want_rows))
    a, b = q_norm.numel(), q_norm.numel() + k_norm.numel()
    f = p.float()
    q = _rms(f[:, :a], q_norm, eps).view(-1, heads, a // heads) * temp.float()[:, None]
    row = torch.cat([_rms(f[:, a:b], k_norm, eps), f[:, b : b + kv_heads * vdim]], -1).to(p.dtype)
    _append(pages, slots, row)
    return q.to(p.dtype), (row if want_rows else row[:0])


# ----------------------------------------------------------------------------------------------- lightning recurrence
def _lightning_token(S, decay, q, k, v):
    """One token of one sequence, in place on S [H, d, e]; returns o [H, e]."""
    S.mul_(decay[:, None, None]).add_(k[:, :, None] * v[:, None, :])
    return torch.einsum("hde,hd->he", S, q)


def _lightning_parts(p, decay, dim: int, vdim: int):
    H, T, f = decay.numel(), p.shape[0], p.float()
    return f[:, : H * dim].view(T, H, dim), f[:, H * dim : 2 * H * dim].view(T, H, dim), f[:, 2 * H * dim : 2 * H * dim + H * vdim].view(T, H, vdim)


def lightning_prefill(p, decay, dim: int, vdim: int, cu, state=None, slots=None, fresh=None, all_fresh: bool = False) -> torch.Tensor:
    """``S = decay S + k v^T``, ``o = S^T q`` per head over packed portions; ``p`` [T, q | k | v | ...] (activated), ``decay`` [H] fp32.
    ``cu`` / ``state`` / ``slots`` / ``fresh`` / ``all_fresh`` as in ``mlstm_prefill`` with state rows [H, dim, vdim]. Returns [T, H vdim]."""
    if p.is_cuda:
        return _ops().lightning_prefill(p, decay, int(dim), int(vdim), cu, state, slots, fresh, bool(all_fresh))
    H = decay.numel()
    q, k, v = _lightning_parts(p, decay, dim, vdim)
    out = torch.empty(p.shape[0], H, vdim)
    c = cu.tolist()
    for b in range(len(c) - 1):
        S = torch.zeros(H, dim, vdim) if slots is None else state[int(slots[b])].view(H, dim, vdim)
        if slots is not None and bool(fresh[b]):
            S.zero_()
        for t in range(c[b], c[b + 1]):
            out[t] = _lightning_token(S, decay, q[t], k[t], v[t])
    return out.flatten(1).to(p.dtype)


def lightning_decode(p, decay, dim: int, vdim: int, state, active) -> torch.Tensor:
    """One token per slot: row s of ``p`` updates ``state[s]`` when ``active[s]`` (inactive slots keep theirs and give zeros)."""
    if p.is_cuda:
        return _ops().lightning_decode(p, decay, int(dim), int(vdim), state, active)
    H = decay.numel()
    q, k, v = _lightning_parts(p, decay, dim, vdim)
    out = torch.zeros(p.shape[0], H, vdim)
    for s in torch.nonzero(active).flatten().tolist():
        out[s] = _lightning_token(state[s].view(H, dim, vdim), decay, q[s], k[s], v[s])
    return out.flatten(1).to(p.dtype)


def gated_rms(o: torch.Tensor, gate: torch.Tensor, norm: torch.Tensor, eps: float, heads: int = 1) -> torch.Tensor:
    """``rms_norm(o) * norm * sigmoid(gate)``; the norm's statistics span whole rows, or each of ``heads`` equal parts."""
    if o.is_cuda:
        return _ops().gated_rms(o, gate, norm, float(eps), int(heads))
    n = o.float().unflatten(-1, (heads, -1))
    n = (n * torch.rsqrt(n.pow(2).mean(-1, keepdim=True) + eps)).flatten(-2)
    return (n * norm.float() * torch.sigmoid(gate.float())).to(norm.dtype)


# ----------------------------------------------------------------------------------------------- generalized delta rule
def _delta_parts(p, zw, ab, w0, heads: int):
    """(r, k, v, decay, removal rate) [T, heads, dim] and the unit keys, fp32."""
    n = ab.numel()
    f = lambda z: z.float().view(-1, heads, n // heads)
    r, k, v, za = (f(p[:, i * n : (i + 1) * n]) for i in range(4))
    w = torch.exp(-math.exp(-0.5) * torch.sigmoid(f(zw[:, :n]) + f(w0)))
    return r, k, v, w, torch.sigmoid(za + f(ab)), k * torch.rsqrt(k.pow(2).sum(-1, keepdim=True) + 1e-6)


def _delta_token(S, r, k, v, w, a, u):
    """One token of one sequence, in place on S [H, d, d]; returns o [H, d]."""
    held = torch.einsum("hd,hde->he", u, S)
    S.mul_(w[:, :, None]).sub_((a * u)[:, :, None] * held[:, None, :]).add_(k[:, :, None] * v[:, None, :])
    return torch.einsum("hde,hd->he", S, r)


def delta_prefill(p, zw, ab, w0, heads: int, cu, state=None, slots=None, fresh=None) -> torch.Tensor:
    """Generalized delta rule over packed portions: ``p`` [T, r | k | v | za | ...], ``zw`` [T, heads * dim], per head and key channel the decay
    ``w = exp(-exp(-1/2) sigmoid(zw + w0))`` and the removal rate ``a = sigmoid(za + ab)``; with the unit key u, ``S = diag(w) S - (a u)
    (u^T S) + k v^T``, ``o = S^T r``. ``cu`` / ``state`` / ``slots`` / ``fresh`` as in ``mlstm_prefill`` with state rows [heads, dim, dim]. Returns
    [T, heads * dim]."""
    if p.is_cuda:
        return _ops().delta_prefill(p, zw, ab, w0, int(heads), cu, state, slots, fresh)
    n = ab.numel()
    d = n // heads
    parts = _delta_parts(p, zw, ab, w0, heads)
    out = torch.empty(p.shape[0], heads, d)
    c = cu.tolist()
    for b in range(len(c) - 1):
        S = torch.zeros(heads, d, d) if slots is None else state[int(slots[b])].view(heads, d, d)
        if slots is not None and bool(fresh[b]):
            S.zero_()
        for t in range(c[b], c[b + 1]):
            out[t] = _delta_token(S, *(z[t] for z in parts))
    return out.flatten(1).to(p.dtype)


def delta_decode(p, zw, ab, w0, heads: int, norm, eps: float, state, active) -> torch.Tensor:
    """One token per slot: row s of ``p`` [S, r | k | v | za | g | ...] updates ``state[s]`` when ``active[s]`` (inactive slots keep theirs and give
    zeros). Returns the finished rows: per head ``rms_norm(o)``, times ``norm``, times ``sigmoid(g)``."""
    if p.is_cuda:
        return _ops().delta_decode(p, zw, ab, w0, int(heads), norm, float(eps), state, active)
    n = ab.numel()
    d = n // heads
    parts = _delta_parts(p, zw, ab, w0, heads)
    out = torch.zeros(p.shape[0], heads, d)
    for s in torch.nonzero(active).flatten().tolist():
        out[s] = _delta_token(state[s].view(heads, d, d), *(z[s] for z in parts))
    return gated_rms(out.flatten(1), p[:, 4 * n : 5 * n], norm, eps, heads)


# ----------------------------------------------------------------------------------------------- mLSTM
def _mlstm_parts(p, gates, ib, fb, cap: float, d: int, e: int):
    T, H = p.shape[0], ib.numel()
    f = p.float()
    q = f[:, : H * d].view(T, H, d) * d ** -0.5
    k = f[:, H * d : 2 * H * d].view(T, H, d)
    v = f[:, 2 * H * d : 2 * H * d + H * e].view(T, H, e)
    g = f[:, 2 * H * d + H * e : 2 * H * (d + e)].view(T, H, e)
    i_log = cap * torch.tanh((gates[:, :H] + ib.float()) / cap)
    f_log = TF.logsigmoid(cap * torch.tanh((gates[:, H : 2 * H] + fb.float()) / cap))
    return q, k, v, g, i_log, f_log


def _mlstm_finish(o, g, norm, eps: float, dtype):
    H, e = o.shape[1], o.shape[2]
    o = o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + eps) * norm.float().view(H, e) * torch.sigmoid(g)
    return o.reshape(o.shape[0], H * e).to(dtype)


def _state_views(row: torch.Tensor, H: int, d: int, e: int):
    return row[: H * d * e].view(H, d, e), row[H * d * e : H * d * e + H * d].view(H, d), row[H * d * e + H * d : H * (d * e + d + 1)]


def _mlstm_token(S, n, m, q, k, v, i_log, f_log):
    """One token of one sequence, in place on the state views; returns o [H, e]."""
    m_new = torch.maximum(f_log + m, i_log)
    keep, add = torch.exp(f_log + m - m_new), torch.exp(i_log - m_new)
    S.mul_(keep[:, None, None]).add_((add[:, None] * k)[:, :, None] * v[:, None, :])
    n.mul_(keep[:, None]).add_(add[:, None] * k)
    m.copy_(m_new)
    den = torch.maximum((n * q).sum(-1).abs(), torch.exp(-m)) + 1e-6
    return torch.einsum("hde,hd->he", S, q) / den[:, None]


def mlstm_prefill(p, gates, ib, fb, cap: float, norm, eps: float, dim: int, cu, state=None, slots=None, fresh=None,
                  all_fresh: bool = False) -> torch.Tensor:
    """Matrix-memory recurrence over packed portions. ``p`` [T, q | k | v | g] in the model's type, ``gates`` [T, i | f] fp32
    pre-activations. Sequence b starts from zero when ``fresh[b]`` (else from ``state[slots[b]]``) and leaves its final state in
    ``state[slots[b]]``; without ``slots`` every sequence starts from zero and nothing is kept. ``all_fresh``: the host knows that
    every sequence is fresh (long prompts may then be cut into segments that run side by side)."""
    if p.is_cuda:
        return _ops().mlstm_prefill(p, gates, ib, fb, float(cap), state, slots, fresh, cu, norm, float(eps), int(dim), bool(all_fresh))
    H = ib.numel()
    e = norm.numel() // H
    q, k, v, g, il, fl = _mlstm_parts(p, gates, ib, fb, cap, dim, e)
    out = torch.empty(p.shape[0], H, e)
    c = cu.tolist()
    for b in range(len(c) - 1):
        row = torch.zeros(H * (dim * e + dim + 1)) if slots is None else state[int(slots[b])]
        if slots is not None and bool(fresh[b]):
            row.zero_()
        S, n, m = _state_views(row, H, dim, e)
        for t in range(c[b], c[b + 1]):
            out[t] = _mlstm_token(S, n, m, q[t], k[t], v[t], il[t], fl[t])
    return _mlstm_finish(out, g, norm, eps, p.dtype)


def mlstm_decode(p, gates, ib, fb, cap: float, norm, eps: float, dim: int, state, active) -> torch.Tensor:
    """One token per slot: row s of ``p`` updates ``state[s]`` when ``active[s]`` (inactive slots keep theirs and give zeros)."""
    if p.is_cuda:
        return _ops().mlstm_decode(p, gates, ib, fb, float(cap), state, active, norm, float(eps), int(dim))
    H = ib.numel()
    e = norm.numel() // H
    q, k, v, g, il, fl = _mlstm_parts(p, gates, ib, fb, cap, dim, e)
    out = torch.zeros(p.shape[0], H, e)
    for s in torch.nonzero(active).flatten().tolist():
        S, n, m = _state_views(state[s], H, dim, e)
        out[s] = _mlstm_token(S, n, m, q[s], k[s], v[s], il[s], fl[s])
    return _mlstm_finish(out, g, norm, eps, p.dtype)
