"""Plain, slow restatement of the Luzitar decoder (lightning recurrences, convolved grouped-query attention, latent attention with
shared latents, grouped mixture of experts, Dynamic Tanh around every sublayer).

One function per mechanism, one sequence at a time, ordinary tensor arithmetic in the precision of its inputs (the tests use
fp64 or fp32). It reads the raw ``config.json`` dictionary and a name -> tensor dictionary with the checkpoint's own names,
and shares no code with the package.
"""

import math

import torch


def dynamic_tanh(x, t, name):
    return torch.tanh(t[name + ".alpha"] * x) * t[name] + t[name + ".b"]


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def rotary_frequencies(rot):
    """Angular frequency of every pair and the factor on cos and sin."""
    n, base = rot["dims"], rot["base"]
    freq = [base ** (-2.0 * i / n) for i in range(n // 2)]
    ext = rot.get("scaling")
    if not ext:
        return freq, 1.0

    def turning_dim(turns):
        return n * math.log(ext["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

    lo, hi = max(math.floor(turning_dim(ext["fast"])), 0), min(math.ceil(turning_dim(ext["slow"])), n - 1)
    ramp = [min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(n // 2)]
    return [f / ext["factor"] * r + f * (1.0 - r) for f, r in zip(freq, ramp)], 0.1 * math.log(ext["factor"]) + 1.0


def rotate(x, positions, rot, halves):
    """``x`` [T, heads, n]: pairs of the first ``rot.dims`` entries are turned; a pair is (i, i + dims / 2) or (2i, 2i + 1)."""
    freq, size = rotary_frequencies(rot)
    n, out = rot["dims"], x.clone()
    for i, f in enumerate(freq):
        a, b = (i, i + n // 2) if halves else (2 * i, 2 * i + 1)
        ang = positions.double() * f
        c, s = (torch.cos(ang) * size).to(x.dtype)[:, None], (torch.sin(ang) * size).to(x.dtype)[:, None]
        out[..., a] = x[..., a] * c - x[..., b] * s
        out[..., b] = x[..., b] * c + x[..., a] * s
    return out


def short_conv(u, taps):
    """``u`` [T, channels], ``taps`` [channels, n]: the last tap meets the token itself, zeros stand before the first token."""
    n, y = taps.shape[1], torch.zeros_like(u)
    for j in range(n):
        back = n - 1 - j
        if back < u.shape[0]:
            y[back:] = y[back:] + u[: u.shape[0] - back] * taps[:, j]
    return y


def sees(T, mask):
    """[T, T] bool: query (row) sees key (column)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    ok = j <= i
    if mask:
        ok = ok & ((i - j < mask["size"]) | (j < mask.get("keep_first", 0)))
    return ok


def weighted_values(scores, visible, v):
    return torch.softmax(scores.masked_fill(~visible, float("-inf")), -1) @ v


def decayed_memory(q, k, v, decay):
    """``q`` / ``k`` [T, d], ``v`` [T, e] of one head: the memory fades by ``decay``, takes in k v^T, and is read with q."""
    S, out = torch.zeros(k.shape[1], v.shape[1], dtype=k.dtype), []
    for t in range(k.shape[0]):
        S = decay * S + torch.outer(k[t], v[t])
        out.append(q[t] @ S)
    return torch.stack(out)


def lightning(h, w, m, eps):
    T, H = h.shape[0], m["heads"]
    q, k = (silu(h @ w[n].t()).view(T, H, m["dim"]) for n in "qk")
    v = silu(h @ w["v"].t()).view(T, H, m["vdim"])
    o = torch.cat([decayed_memory(q[:, i], k[:, i], v[:, i], m["decay"][i]) for i in range(H)], -1)
    return (unit_rms(o, eps) * w["norm"] * sigmoid(h @ w["g"].t())) @ w["o"].t()


def attention(h, w, m, eps):
    T, H, G, pos = h.shape[0], m["heads"], m["kv_heads"], torch.arange(h.shape[0])
    part = {n: h @ w[n].t() + w[n + ".b"] for n in "qkv"}
    if m.get("conv"):
        part = {n: short_conv(u, w[n + ".conv"]) for n, u in part.items()}
    q = unit_rms(rotate(part["q"].view(T, H, m["dim"]), pos, m["rot"], True), eps)
    k = unit_rms(rotate(part["k"].view(T, G, m["dim"]), pos, m["rot"], True), eps)
    v, visible = part["v"].view(T, G, m["vdim"]), sees(T, m.get("mask"))
    o = [weighted_values(q[:, i] @ k[:, i // (H // G)].t() * m["scale"], visible, v[:, i // (H // G)]) for i in range(H)]
    return torch.cat(o, -1) @ w["o"].t()


def latent_rows(h, w, m, eps):
    """(normed latent, rotated shared key part) of every token."""
    z, n = h @ w["dkv"].t(), m["kv_rank"]
    return unit_rms(z[:, :n], eps) * w["dkv.norm"], rotate(z[:, None, n:], torch.arange(h.shape[0]), m["rot"], False)[:, 0]


def latent_attention(h, w, m, rows):
    T, H, du = h.shape[0], m["heads"], m["dim"]
    c, kr = rows
    q = (h @ w["q"].t()).view(T, H, du + m["rot_dim"])
    qr = rotate(q[..., du:], torch.arange(T), m["rot"], False)
    ku, v = (c @ w["uk"].t()).view(T, H, du), (c @ w["uv"].t()).view(T, H, m["vdim"])
    visible = sees(T, None)
    o = [weighted_values((q[:, i, :du] @ ku[:, i].t() + qr[:, i] @ kr.t()) * m["scale"], visible, v[:, i]) for i in range(H)]
    return torch.cat(o, -1) @ w["o"].t()


def clipped_expert(h, gate, up, down, limit):
    g, u = (h @ gate.t()).clamp(max=limit), (h @ up.t()).clamp(-limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ down.t()


def choose_experts(scores, correction, top, count, keep):
    """Experts of one token: the ``top`` best corrected scores inside the ``keep`` best groups of neighbours."""
    choice = scores + correction
    size = choice.numel() // count
    group = [float(torch.sort(choice[g * size : (g + 1) * size], descending=True).values[:2].sum()) for g in range(count)]
    best = sorted(range(count), key=lambda g: -group[g])[:keep]
    allowed = sorted((e for e in range(choice.numel()) if e // size in best), key=lambda e: -float(choice[e]))
    return allowed[:top]


def mixture(h, w, f, routes_out=None):
    r, rows = f["router"], []
    groups = r.get("groups") or {"count": 1, "keep": 1}
    s = sigmoid(h @ w["router"].t())
    for t in range(h.shape[0]):
        chosen = choose_experts(s[t], w["correction"], r["top"], groups["count"], groups["keep"])
        total = s[t][chosen].sum() + 1e-20
        rows.append(sum(s[t, e] / total * clipped_expert(h[t], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"], f["expert"]["limit"]) for e in chosen))
        if routes_out is not None:
            routes_out.append(chosen)
    return torch.stack(rows)


def forward(config, tensors, tokens, dtype=torch.float64, layer_outputs=None, routes_out=None):
    """Logits [T, vocab] of one token sequence."""
    t = {k: v.to(dtype) for k, v in tensors.items()}
    eps, latents = config["norm"]["eps"], {}
    x = dynamic_tanh(t["embed"][torch.tensor(list(tokens))], t, "embed.norm")
    for i, layer in enumerate(config["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer.get("mlp")
        part = lambda what: {k[len(p + what):]: v for k, v in t.items() if k.startswith(p + what)}
        h, w = dynamic_tanh(x, t, p + "norm1"), part("mix.")
        if layer["type"] == "lightning":
            y = lightning(h, w, m, eps)
        elif layer["type"] == "attention":
            y = attention(h, w, m, eps)
        else:
            latents[i] = latents[m["kv_from"]] if m.get("kv_from") is not None else latent_rows(h, w, m, eps)
            y = latent_attention(h, w, m, latents[i])
        x = x + dynamic_tanh(y, t, p + "norm1b")
        if f is not None:
            x = x + dynamic_tanh(mixture(dynamic_tanh(x, t, p + "norm2"), part("mlp."), f, routes_out), t, p + "norm2b")
        if layer_outputs is not None:
            layer_outputs.append(x)
    cap = config["logit_softcap"]
    return cap * torch.tanh(dynamic_tanh(x, t, "final.norm") @ t["head"].t() / cap)
