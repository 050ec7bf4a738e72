"""Plain, slow restatement of the mixer-stack decoder (latent attention, mLSTM, Dynamic Tanh, dense MLP).

One function per mechanism, one sequence at a time, ordinary tensor arithmetic in the precision of its inputs (the tests
use fp64 or fp32). It reads the raw ``config.json`` dictionary and a name -> tensor dictionary with the checkpoint's own
names, and shares no code with the package.
"""

import math

import torch


def dynamic_tanh(x, alpha, weight, bias):
    return torch.tanh(alpha * x) * weight + bias


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def gelu_erf(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def rotary_frequencies(rot):
    """Angular frequency of every pair and the factor on cos and sin."""
    dims, base = rot["dims"], rot["base"]
    freq = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    scaling = rot.get("scaling")
    if not scaling:
        return torch.tensor(freq, dtype=torch.float64), 1.0
    factor, original = scaling["factor"], scaling["original"]

    def dim_of(turns):
        return dims * math.log(original / (2 * math.pi * turns)) / (2 * math.log(base))

    lo = max(math.floor(dim_of(scaling["fast"])), 0)
    hi = min(math.ceil(dim_of(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freq):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * ramp + f * (1.0 - ramp))
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(factor) + 1.0


def rotate_pairs(x, positions, rot):
    """``x`` [T, ..., n]: the first ``rot.dims`` entries are turned pair by pair (2i with 2i + 1), the rest stays."""
    freq, mag = rotary_frequencies(rot)
    ang = positions.double()[:, None] * freq[None, :]
    cos, sin = (torch.cos(ang) * mag).to(x.dtype), (torch.sin(ang) * mag).to(x.dtype)
    shape = (x.shape[0],) + (1,) * (x.dim() - 2) + (freq.numel(),)
    cos, sin = cos.view(shape), sin.view(shape)
    out = x.clone()
    d = rot["dims"]
    u, v = x[..., 0:d:2], x[..., 1:d:2]
    out[..., 0:d:2] = u * cos - v * sin
    out[..., 1:d:2] = v * cos + u * sin
    return out


def window_mask(n, size):
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    ok = j <= i
    return ok if size is None else ok & (i - j < size)


def softmax_with_sink(scores, visible, sink):
    """``scores`` [H, T, T], ``sink`` [H]: the sink adds exp(sink) to every denominator and has no key or value."""
    s = scores.masked_fill(~visible, float("-inf"))
    m = torch.maximum(s.max(-1, keepdim=True).values, sink[:, None, None])
    e = torch.exp(s - m)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink[:, None, None] - m))


def latent_attention(h, w, spec, eps, scores_out=None):
    """``h`` [T, width] of one sequence; ``w``: the mixer's tensors by their short names."""
    T, H, dim, rd, vd, r = h.shape[0], spec["heads"], spec["dim"], spec["rot_dim"], spec["vdim"], spec["kv_rank"]
    pos = torch.arange(T)
    cq = unit_rms(h @ w["dq"].t(), eps) * w["dq.norm"]
    q = (cq @ w["uq"].t()).view(T, H, dim + rd)
    q_plain, q_rot = q[..., :dim], rotate_pairs(q[..., dim:], pos, spec["rot"])
    down = h @ w["dkv"].t()
    c = unit_rms(down[:, :r], eps) * w["dkv.norm"]
    k_rot = rotate_pairs(down[:, r:], pos, spec["rot"])
    k_plain = (c @ w["uk"].t()).view(T, H, dim)
    v = (c @ w["uv"].t()).view(T, H, vd)
    scores = (torch.einsum("ihd,jhd->hij", q_plain, k_plain) + torch.einsum("ihd,jd->hij", q_rot, k_rot)) * spec["scale"]
    if scores_out is not None:
        scores_out.append(scores)
    p = softmax_with_sink(scores, window_mask(T, (spec.get("mask") or {}).get("size")), w["sink"])
    o = torch.einsum("hij,jhd->ihd", p, v)
    o = o * torch.sigmoid(h @ w["g"].t())[:, :, None]
    return o.reshape(T, H * vd) @ w["o"].t()


def mlstm_recurrence(q, k, v, i_log, f_log):
    """``q``/``k`` [T, H, d] (q already scaled), ``v`` [T, H, e], log gates [T, H] -> o [T, H, e]."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype)
    n = torch.zeros(H, d, dtype=q.dtype)
    m = torch.zeros(H, dtype=q.dtype)
    out = []
    for t in range(T):
        m_new = torch.maximum(f_log[t] + m, i_log[t])
        keep, add = torch.exp(f_log[t] + m - m_new), torch.exp(i_log[t] - m_new)
        S = keep[:, None, None] * S + add[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + add[:, None] * k[t]
        m = m_new
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out.append(torch.einsum("hde,hd->he", S, q[t]) / den[:, None])
    return torch.stack(out)


def mlstm(h, w, spec, eps):
    T, H, d, e, cap = h.shape[0], spec["heads"], spec["dim"], spec["vdim"], spec["gate_cap"]
    q = (h @ w["q"].t()).view(T, H, d) * d ** -0.5
    k = (h @ w["k"].t()).view(T, H, d)
    v = (h @ w["v"].t()).view(T, H, e)
    i_log = cap * torch.tanh((h @ w["i"].t() + w["i.b"]) / cap)
    f_log = torch.nn.functional.logsigmoid(cap * torch.tanh((h @ w["f"].t() + w["f.b"]) / cap))
    o = unit_rms(mlstm_recurrence(q, k, v, i_log, f_log), eps).reshape(T, H * e)
    return (o * w["norm"] * torch.sigmoid(h @ w["g"].t())) @ w["o"].t()


MIXERS = {"latent_attention": latent_attention, "mlstm": mlstm}


def owner_of(layers, i):
    while layers[i].get("weights_of") is not None:
        i = layers[i]["weights_of"]
    return i


def forward(config, tensors, tokens, dtype=torch.float64, layer_outputs=None):
    """Logits [T, vocab] of one token sequence."""
    t = {k: v.to(dtype) for k, v in tensors.items()}
    eps = config["norm"]["eps"]
    norm = lambda name, x: dynamic_tanh(x, t[name + ".alpha"], t[name], t[name + ".b"])
    x = t["embed"][torch.tensor(list(tokens))] * config["embedding"]["scale"]
    for i, layer in enumerate(config["layers"]):
        p = f"l{owner_of(config['layers'], i)}."
        w = {k[len(p) + 4:]: v for k, v in t.items() if k.startswith(p + "mix.")}
        x = x + MIXERS[layer["type"]](norm(p + "norm1", x), w, layer["mixer"], eps)
        if layer["mlp"] is not None:
            x = x + gelu_erf(norm(p + "norm2", x) @ t[p + "mlp.up"].t()) @ t[p + "mlp.down"].t()
        if layer_outputs is not None:
            layer_outputs.append(x)
    return norm("final.norm", x) @ t["head"].t()
