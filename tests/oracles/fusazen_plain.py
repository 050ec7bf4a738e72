"""Plain, slow restatement of the Fusazen decoder (generalized delta rule, chunked differential attention with shared keys, chunked
grouped-query attention with norms over whole projections, a short convolution in front of every mixer, biased squared-relu
feed-forwards).

One function per mechanism, one sequence at a time, ordinary tensor arithmetic in the precision of its inputs (the tests use
fp64 or fp32). It reads the raw ``config.json`` dictionary and a name -> tensor dictionary with the checkpoint's own names,
and shares no code with the package.
"""

import math

import torch


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def with_past(h, taps):
    """``h`` [T, channels] plus its causal convolution with ``taps`` [channels, n] (last tap: the token itself)."""
    T, n = h.shape[0], taps.shape[1]
    y = h.clone()
    for t in range(T):
        for j in range(n):
            s = t - (n - 1 - j)
            if s >= 0:
                y[t] = y[t] + taps[:, j] * h[s]
    return y


def turn_halves(x, rot):
    """``x`` [T, n], row t at position t: entries i and i + dims / 2 of the first ``dims`` are turned by t base^(-2 i / dims)."""
    half, out = rot["dims"] // 2, x.clone()
    t = torch.arange(x.shape[0], dtype=torch.float64)
    for i in range(half):
        ang = t * rot["base"] ** (-2.0 * i / rot["dims"])
        c, s = torch.cos(ang).to(x.dtype), torch.sin(ang).to(x.dtype)
        out[:, i], out[:, i + half] = x[:, i] * c - x[:, i + half] * s, x[:, i + half] * c + x[:, i] * s
    return out


def same_chunk(T, mask):
    """[T, T] bool: query (row) sees key (column)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    ok = j <= i
    return ok & (i // mask["size"] == j // mask["size"]) if mask else ok


def attend(q, k, v, scale, visible):
    return torch.softmax((q @ k.t() * scale).masked_fill(~visible, float("-inf")), -1) @ v


def decay_and_rate(zw, w0, za, a_b):
    """Decay and removal rate of every channel from their pre-activations."""
    return torch.exp(-math.exp(-0.5) * sigmoid(zw + w0)), sigmoid(za + a_b)


def delta_rule(r, k, v, w, a):
    """One head, ``r`` / ``k`` / ``w`` / ``a`` [T, d], ``v`` [T, e]: the memory decays per row, forgets what it holds along the unit
    key, takes in k v^T, and is read with r."""
    S, out = torch.zeros(k.shape[1], v.shape[1], dtype=k.dtype), []
    for t in range(k.shape[0]):
        u = k[t] / torch.sqrt((k[t] * k[t]).sum() + 1e-6)
        held = u @ S
        S = w[t][:, None] * S - torch.outer(a[t] * u, held) + torch.outer(k[t], v[t])
        out.append(r[t] @ S)
    return torch.stack(out)


def general_delta(h, p, m, eps):
    T, H, d = h.shape[0], m["heads"], m["dim"]
    heads = lambda z: z.view(T, H, d)
    w, a = decay_and_rate(torch.tanh(h @ p["w1"].t()) @ p["w2"].t(), p["w0"], h @ p["a"].t(), p["a.b"])
    r, k, v, w, a = (heads(z) for z in (h @ p["r"].t(), h @ p["k"].t(), h @ p["v"].t(), w, a))
    o = torch.cat([unit_rms(delta_rule(r[:, i], k[:, i], v[:, i], w[:, i], a[:, i]), eps) for i in range(H)], -1)
    return (o * p["norm"] * sigmoid(h @ p["g"].t())) @ p["o"].t()


def difference_weight(p, diff):
    return torch.exp((p["lq1"] * p["lk1"]).sum()) - torch.exp((p["lq2"] * p["lk2"]).sum()) + diff


def rotated_keys(h, p, m):
    """Per key head a pair of rotated key maps, and the values."""
    T, G, d = h.shape[0], m["kv_heads"], m["dim"]
    k = (h @ p["k"].t()).view(T, G, 2, d)
    return [[turn_halves(k[:, g, n], m["rot"]) for n in range(2)] for g in range(G)], (h @ p["v"].t()).view(T, G, m["vdim"])


def differential_attention(h, p, m, eps, keys, values):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q, lam, ok = (h @ p["q"].t()).view(T, H, 2, m["dim"]), difference_weight(p, m["diff"]), same_chunk(T, m.get("mask"))
    out = []
    for i in range(H):
        g = i // (H // G)
        a1, a2 = (attend(turn_halves(q[:, i, n], m["rot"]), keys[g][n], values[:, g], m["scale"], ok) for n in range(2))
        out.append(unit_rms(a1 - lam * a2, eps) * (1.0 - m["diff"]))
    return torch.cat(out, -1) @ p["o"].t()


def whole_norm_attention(h, p, m, eps):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = (unit_rms(h @ p["q"].t(), eps) * p["q.norm"]).view(T, H, m["dim"])
    k = (unit_rms(h @ p["k"].t(), eps) * p["k.norm"]).view(T, G, m["dim"])
    v, ok = (h @ p["v"].t()).view(T, G, m["vdim"]), same_chunk(T, m.get("mask"))
    o = [attend(q[:, i] * p["temp"][i], k[:, i // (H // G)], v[:, i // (H // G)], m["scale"], ok) for i in range(H)]
    return torch.cat(o, -1) @ p["o"].t()


def squared_relu_mlp(h, p):
    z = (h @ p["up"].t() + p["up.b"]).clamp(min=0)
    return (z * z) @ p["down"].t() + p["down.b"]


def forward(config, tensors, tokens, dtype=torch.float64, layer_outputs=None):
    """Logits [T, vocab] of one token sequence."""
    t = {k: v.to(dtype) for k, v in tensors.items()}
    eps, kept = config["norm"]["eps"], {}
    norm = lambda x, name: unit_rms(x, eps) * t[name]
    x = t["embed"][torch.tensor(list(tokens))] * config["embedding"]["scale"]
    for i, layer in enumerate(config["layers"]):
        pre, m = f"l{i}.", layer["mixer"]
        part = lambda what: {k[len(pre + what):]: v for k, v in t.items() if k.startswith(pre + what)}
        h, p = with_past(norm(x, pre + "norm1"), t[pre + "canon1"]), part("mix.")
        if layer["type"] == "general_delta":
            y = general_delta(h, p, m, eps)
        elif layer["type"] == "attention":
            kept[i] = kept[m["kv_from"]] if m.get("kv_from") is not None else rotated_keys(h, p, m)
            y = differential_attention(h, p, m, eps, *kept[i])
        else:
            y = whole_norm_attention(h, p, m, eps)
        x = x + y
        if layer.get("mlp") is not None:
            x = x + squared_relu_mlp(norm(x, pre + "norm2"), part("mlp."))
        if layer_outputs is not None:
            layer_outputs.append(x)
    return norm(x, "final.norm") @ t["head"].t()
