"""Plain, slow restatement of the Tofinex decoder (grouped-query attention with capped scores, mixture-of-experts layers).

One function per mechanism, one sequence at a time, ordinary tensor arithmetic in the precision of its inputs (the tests use
fp64 or fp32). It reads the raw ``config.json`` dictionary and a name -> tensor dictionary with the checkpoint's own names,
and shares no code with the package.
"""

import torch


def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def soft_cap(z, cap):
    return cap * torch.tanh(z / cap)


def rotate_pairs(x, positions, rot):
    """``x`` [T, heads, n]: the first ``rot.dims`` entries of a head are turned pair by pair (2i with 2i + 1), the rest stays."""
    d = rot["dims"]
    freq = torch.tensor([rot["base"] ** (-2.0 * i / d) for i in range(d // 2)], dtype=torch.float64)
    ang = positions.double()[:, None, None] * freq
    c, s = torch.cos(ang).to(x.dtype), torch.sin(ang).to(x.dtype)
    out = x.clone()
    out[..., 0:d:2] = x[..., 0:d:2] * c - x[..., 1:d:2] * s
    out[..., 1:d:2] = x[..., 1:d:2] * c + x[..., 0:d:2] * s
    return out


def one_plus_softmax(scores):
    """Weights exp(s) / (1 + sum exp(s)) over the last dimension; hidden scores are -inf."""
    top = scores.max(-1, keepdim=True).values.clamp_min(0.0)
    e = torch.exp(scores - top)
    return e / (torch.exp(-top) + e.sum(-1, keepdim=True))


def mix_values(v, first, lam):
    return (1.0 - lam) * v + lam * first


def attention_core(q, k, v, scale, softcap, scores_out=None):
    """``q`` [T, H, d], ``k`` [T, G, d], ``v`` [T, G, e] -> [T, H, e]; query head h reads key/value head h // (H / G)."""
    T, H = q.shape[:2]
    share = H // k.shape[1]
    seen = torch.arange(T)[None, :] <= torch.arange(T)[:, None]
    out = []
    for h in range(H):
        s = soft_cap(q[:, h] @ k[:, h // share].t() * scale, softcap)
        if scores_out is not None:
            scores_out.append(s)
        out.append(one_plus_softmax(s.masked_fill(~seen, float("-inf"))) @ v[:, h // share])
    return torch.stack(out, 1)


def attention(h, w, m, eps, first_values, scores_out=None):
    """``h`` [T, width], ``w``: the mixer's tensors by short name. Returns (output, this layer's own values)."""
    T, H, G, pos = h.shape[0], m["heads"], m["kv_heads"], torch.arange(h.shape[0])
    q = (h @ w["q"].t()).view(T, H, m["dim"])
    k = (h @ w["k"].t()).view(T, G, m["dim"])
    own = (h @ w["v"].t()).view(T, G, m["vdim"])
    q = rotate_pairs(rms_norm(q, w["q.norm"], eps), pos, m["rot"])
    k = rotate_pairs(rms_norm(k, w["k.norm"], eps), pos, m["rot"])
    v = own if first_values is None else mix_values(own, first_values, w["vmix"])
    o = attention_core(q, k, v, m["scale"], m["softcap"], scores_out)
    return o.reshape(T, H * m["vdim"]) @ w["o"].t(), own


def gated_mlp(h, w, prefix=""):
    return (silu(h @ w[prefix + "gate"].t()) * (h @ w[prefix + "up"].t())) @ w[prefix + "down"].t()


def choose_experts(h, router, top):
    """Sigmoid scores of the ``top`` best experts of every token, and which they are."""
    best = torch.sort(sigmoid(h @ router.t()), -1, descending=True)
    return best.values[:, :top], best.indices[:, :top]


def mixture(h, w, top, shared, routes_out=None):
    """Token by token: the weight of a chosen expert scales that expert's input; a gated shared expert is added."""
    score, which = choose_experts(h, w["router"], top)
    if routes_out is not None:
        routes_out.append(which)
    rows = []
    for t in range(h.shape[0]):
        y = torch.zeros_like(h[t])
        for s, e in zip(score[t], which[t].tolist()):
            y = y + gated_mlp(s * h[t], w, f"e{e}.")
        rows.append(y)
    y = torch.stack(rows)
    if shared:
        y = y + gated_mlp(h, w, "shared.") * sigmoid(h @ w["shared.sg"].t())
    return y


def forward(config, tensors, tokens, dtype=torch.float64, layer_outputs=None, routes_out=None):
    """Logits [T, vocab] of one token sequence."""
    t = {k: v.to(dtype) for k, v in tensors.items()}
    eps, mult = config["norm"]["eps"], config["residual_mult"]
    x = rms_norm(t["embed"][torch.tensor(list(tokens))], t["embed.norm"], eps)
    first = None
    for i, layer in enumerate(config["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer.get("mlp")
        part = lambda what: {k[len(p + what):]: v for k, v in t.items() if k.startswith(p + what)}
        y, own = attention(x, part("mix."), m, eps, first if m.get("v_mix") else None)
        if m.get("v_mix") and first is None:
            first = own
        x = x + mult * rms_norm(y, t[p + "norm1"], eps)
        if f is not None:
            w = part("mlp.")
            y = gated_mlp(x, w) if f["kind"] == "dense" else mixture(x, w, f["router"]["top"], f.get("shared"), routes_out)
            x = x + mult * rms_norm(y, t[p + "norm2"], eps)
        if layer_outputs is not None:
            layer_outputs.append(x)
    return soft_cap(rms_norm(x, t["final.norm"], eps) @ t["embed"].t(), config["logit_softcap"])
