"""Luzitar models through the rollout engine: prompts, decoding, portions, batches, reused slots and pages, window edges, generation.

Routers make choices, and a choice between two experts (or groups) of nearly equal scores may fall differently in bf16. The models
that choose therefore keep a few dimensions of the stream for their routers: they come from the embedding, the sublayers add
nothing to them, and every token's choices are clear (``settle_routers``).
"""

import json
import os
import subprocess
import sys

import pytest
import torch

from oracles import luzitar_plain as plain
from stack_testing import PLACES, feed_all, position_errors, tokens
from verl_b200.models import FlatParams, ModelConfig, PackedBatch, build_decoder
from verl_b200.utils.model import load_hf_weights_into, save_hf_weights
from verl_b200.workers.rollout.native.engine import RolloutEngine, SamplingParams

torch.set_num_threads(min(4, torch.get_num_threads()))
REPO = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.fixture(params=PLACES)
def place(request):
    return request.param


YARN = {"factor": 5.0, "original": 120, "fast": 16.0, "slow": 2.0}


def moe(experts=6, top=2, groups=(3, 2), ff=24, limit=1.1):
    r = {"experts": experts, "top": top}
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {**r, "groups": {"count": groups[0], "keep": groups[1]}} if groups else r}


def lightning(mlp=None, decay=(0.9, 0.995), dim=16, vdim=24):
    return {"type": "lightning", "mlp": mlp, "mixer": {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay)}}


def attention(mlp=None, heads=4, kv_heads=2, dim=24, vdim=16, rot=16, base=600.0, scaling=YARN, conv=3, mask=(20, 3), scale=0.9):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": rot}, "scale": scale}
    if conv:
        m["conv"] = conv
    if scaling:
        m["rot"]["scaling"] = scaling
    if mask:
        m["mask"] = {"size": mask[0], "keep_first": mask[1]}
    return {"type": "attention", "mlp": mlp, "mixer": m}


def latent(mlp=None, heads=3, dim=16, rot=8, vdim=24, kv_rank=40, base=2e3, scale=0.5, kv_from=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": kv_rank, "rot": {"base": base, "dims": rot}, "scale": scale}
    return {"type": "latent_attention", "mlp": mlp, "mixer": m if kv_from is None else {**m, "kv_from": kv_from}}


def config(layers, width=72, vocab=88, eps=1e-3, cap=9.0):
    return {"architecture": "Luzitar", "layers": layers, "logit_softcap": cap, "norm": {"eps": eps}, "vocab": vocab, "width": width}


CONFIGS = {
    # every kind of layer, in an order of its own; two latents, one of them read by two later layers, masks of several forms
    "mixed": config([attention(moe()), latent(moe(8, 3, (4, 2), 16, 0.7)), lightning(None), latent(moe(4, 4, (2, 2)), heads=5, dim=8, vdim=16, kv_from=1),
                     attention(None, heads=6, kv_heads=2, dim=16, vdim=32, conv=2, mask=None, rot=16), latent(None, kv_rank=24, rot=16, heads=2),
                     lightning(moe(5, 2, None), decay=(0.0, 1.0, 0.6), dim=24, vdim=8), latent(moe(), kv_from=1), latent(None, kv_rank=24, rot=16, heads=4, dim=24, kv_from=5)]),
    # sizes that are no multiple of 8, rotation over a part of a head
    "odd": config([lightning(moe(5, 3, None, 11), decay=(0.8, 0.99, 0.3), dim=5, vdim=7), latent(None, heads=2, dim=9, rot=6, vdim=11, kv_rank=13),
                   attention(moe(6, 2, (2, 1), 10), heads=3, kv_heads=1, dim=10, vdim=14, rot=6, conv=4, mask=(9, 1)), latent(moe(3, 3, (1, 1), 9), heads=3, dim=7, rot=6, vdim=5,
                                                                                                                             kv_rank=13, kv_from=1)],
                  width=42, vocab=61, eps=2e-2, cap=4.0),
    # all experts of every layer are used; more than 16 query heads per key head, sizes of two and three panels, wide states
    "wide": config([latent(moe(3, 3, None, 72), heads=20, dim=72, rot=32, vdim=40, kv_rank=136, scale=0.1), lightning(moe(2, 2, (2, 2), 64), decay=(0.99, 0.9), dim=136, vdim=200),
                    attention(moe(3, 3, (3, 3), 40), heads=20, kv_heads=1, dim=72, vdim=136, rot=64, conv=4, mask=(70, 66), scale=0.3),
                    latent(None, heads=17, dim=40, rot=32, vdim=72, kv_rank=136, scale=0.1, kv_from=0), attention(None, heads=2, kv_heads=2, dim=64, vdim=64, rot=64, conv=1, mask=(64, 0))],
                   width=200, vocab=264),
    # no second sublayer anywhere, no convolution, no context extension, a window of one token
    "bare": config([attention(heads=2, kv_heads=2, scaling=None, conv=None, mask=(1, 0)), lightning(), latent(), attention(conv=None, scaling=None, mask=(30, 40))]),
    # one of everything
    "ones": config([attention(moe(1, 1, (1, 1), 8), heads=1, kv_heads=1, dim=8, vdim=8, rot=2, conv=1, mask=(5, 1)), latent(moe(1, 1, None, 8), heads=1, dim=8, rot=2, vdim=8, kv_rank=8),
                    lightning(moe(1, 1, None, 8), decay=(0.9,), dim=8, vdim=8), latent(None, heads=1, dim=8, rot=2, vdim=8, kv_rank=8, kv_from=1)], width=16, vocab=24),
}


def expected_tensors(cfg):
    """Checkpoint names and shapes, written from the format (not from the package)."""
    D, out = cfg["width"], {"embed": (cfg["vocab"], cfg["width"]), "head": (cfg["vocab"], cfg["width"])}

    def norm(name):
        out.update({name: (D,), name + ".b": (D,), name + ".alpha": ()})

    norm("embed.norm")
    norm("final.norm")
    for i, l in enumerate(cfg["layers"]):
        m, f, p = l["mixer"], l["mlp"], f"l{i}."
        H, d, e = m["heads"], m["dim"], m["vdim"]
        norm(p + "norm1")
        norm(p + "norm1b")
        out[p + "mix.o"] = (D, H * e)
        if l["type"] == "lightning":
            out.update({p + "mix.q": (H * d, D), p + "mix.k": (H * d, D), p + "mix.v": (H * e, D), p + "mix.g": (H * e, D), p + "mix.norm": (H * e,)})
        elif l["type"] == "attention":
            G = m["kv_heads"]
            for n, rows in (("q", H * d), ("k", G * d), ("v", G * e)):
                out.update({p + "mix." + n: (rows, D), p + f"mix.{n}.b": (rows,)})
                if m.get("conv"):
                    out[p + f"mix.{n}.conv"] = (rows, m["conv"])
        else:
            out.update({p + "mix.q": (H * (d + m["rot_dim"]), D), p + "mix.uk": (H * d, m["kv_rank"]), p + "mix.uv": (H * e, m["kv_rank"])})
            if m.get("kv_from") is None:
                out.update({p + "mix.dkv": (m["kv_rank"] + m["rot_dim"], D), p + "mix.dkv.norm": (m["kv_rank"],)})
        if f is None:
            continue
        norm(p + "norm2")
        norm(p + "norm2b")
        E, ff = f["router"]["experts"], f["expert"]["ff"]
        out.update({p + "mlp.router": (E, D), p + "mlp.correction": (E,)})
        for j in range(E):
            out.update({p + f"mlp.e{j}.gate": (ff, D), p + f"mlp.e{j}.up": (ff, D), p + f"mlp.e{j}.down": (D, ff)})
    return out


def random_tensors(cfg, seed=0):
    g, t = torch.Generator().manual_seed(seed), {}
    for name, shape in expected_tensors(cfg).items():
        x = torch.randn(shape, generator=g)
        if name.endswith(".alpha"):
            x = 0.6 + 0.2 * x.abs()
        elif name.endswith("norm") or "norm1" in name or "norm2" in name:
            x = 0.2 * x if name.endswith(".b") else 1.0 + 0.3 * x
        elif name.endswith(".correction"):
            x = -1.0 + 0.5 * x
        elif name.endswith(".conv"):
            x = x * shape[1] ** -0.5 + 0.5
        elif name.endswith(".b"):
            x = 0.3 * x
        elif name != "embed":
            x = x * (2.0 if "router" in name else 1.3) * shape[-1] ** -0.5
        t[name] = x.bfloat16().float()
    if any(chosen(l) for l in cfg["layers"]):
        settle_routers(cfg, t, g)
    return {k: v.bfloat16().float() for k, v in t.items()}


def chosen(l):
    """(experts, top, groups, kept groups) of a layer whose tokens leave some experts out."""
    r = (l["mlp"] or {}).get("router")
    if r is None or r["top"] == r["experts"]:
        return None
    groups = r.get("groups") or {"count": 1, "keep": 1}
    return r["experts"], r["top"], groups["count"], groups["keep"]


def choice_gap(choice, top, groups, keep):
    """How far the choice of experts is from another one."""
    size = len(choice) // groups
    best = torch.stack([torch.sort(choice[g * size : (g + 1) * size], descending=True).values[:2].sum() for g in range(groups)])
    order = torch.sort(best, descending=True)
    gap = 9.0 if keep == groups else float(order.values[keep - 1] - order.values[keep])
    left = torch.sort(torch.cat([choice[g * size : (g + 1) * size] for g in order.indices[:keep].tolist()]), descending=True).values
    return gap if top == len(left) else min(gap, float(left[top - 1] - left[top]))


def settle_routers(cfg, t, g, own=8):
    """The last ``own`` dimensions decide: nothing is added there, large router weights there, and embedding rows drawn until every
    choice in every layer is clear."""
    for name in t:
        if name.startswith("l") and ("norm1" in name or "norm2" in name) and not name.endswith(".alpha"):
            t[name][-own:] = 1.0 if name.endswith("norm2") else 0.0
        if name.endswith("router"):
            t[name][:, :-own] *= 0.02
            t[name][:, -own:] = (1.5 * torch.randn(t[name].shape[0], own, generator=g)).bfloat16().float()
    t["embed.norm"][-own:], t["embed.norm.b"][-own:] = 1.0, 0.0
    left = range(cfg["vocab"])
    for _ in range(3000):
        bad = []
        for v in left:
            x = torch.tanh(t["embed.norm.alpha"] * t["embed"][v, -own:])
            for i, l in enumerate(cfg["layers"]):
                if chosen(l):
                    _, top, groups, keep = chosen(l)
                    z = t[f"l{i}.mlp.router"][:, -own:] @ torch.tanh(t[f"l{i}.norm2.alpha"] * x)
                    if choice_gap(plain.sigmoid(z) + t[f"l{i}.mlp.correction"], top, groups, keep) < 0.03:
                        bad.append(v)
                        break
        if not bad:
            return
        left = bad
        t["embed"][left, -own:] = torch.randn(len(left), own, generator=g).bfloat16().float()
    raise AssertionError("no clear choices found")


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """name -> (config, tensors, directory with config.json and safetensors)"""
    from safetensors.torch import save_file

    out = {}
    for i, (name, cfg) in enumerate(CONFIGS.items()):
        d = tmp_path_factory.mktemp(name)
        t = random_tensors(cfg, seed=i)
        (d / "config.json").write_text(json.dumps(cfg))
        save_file({k: v.bfloat16().contiguous() for k, v in t.items()}, str(d / "model.safetensors"))
        out[name] = (cfg, t, str(d))
    return out


_WANT = {}


def want_logits(models, name, toks):
    key = (name, tuple(toks))
    if key not in _WANT:
        _WANT[key] = plain.forward(models[name][0], models[name][1], toks)
    return _WANT[key]


def close(got, want, place, name="", what=""):
    """fp32: every position; bf16: a position in a hundred may round badly (the memories' read-outs cancel here and there), within twice the limit."""
    err = position_errors(got, want)
    limit = 1e-4 if place[1] == torch.float32 else 0.08
    most = limit if place[1] == torch.float32 else 2 * limit
    assert float(err.max()) < most and int((err > limit).sum()) <= max(1, len(err) // 100), (name, what, float(err.max()), int(err.argmax()))


def load(models, name, place):
    arch = ModelConfig.from_pretrained(models[name][2])
    P = FlatParams(arch, dtype=place[1], device=place[0])
    assert load_hf_weights_into(P, models[name][2], strict=True) == []
    return arch, P


def engine(models, name, place, **kw):
    arch, P = load(models, name, place)
    args = dict(max_num_seqs=5, max_model_len=400, block_size=16, num_blocks=100, sync_interval=3, eos_token_id=-1)
    args.update(kw)
    return RolloutEngine(arch, P, **args)


# ---------------------------------------------------------------------------------------------- configuration and weights
@pytest.mark.parametrize("name", list(CONFIGS))
def test_checkpoint_names_and_round_trip(models, name, tmp_path):
    cfg, t, _ = models[name]
    arch, P = load(models, name, ("cpu", torch.float32))
    sd = P.hf_state_dict()
    assert {k: tuple(v.shape) for k, v in sd.items()} == expected_tensors(cfg)
    assert all(torch.equal(sd[k], t[k]) for k in t)
    assert arch.is_stack and arch.hidden_size == cfg["width"] and arch.to_hf_dict() == cfg and arch.num_parameters() >= sum(v.numel() for v in t.values())
    save_hf_weights(P, str(tmp_path))
    again = FlatParams(ModelConfig.from_pretrained(str(tmp_path)), dtype=torch.float32)
    load_hf_weights_into(again, str(tmp_path), strict=True)
    assert all(torch.equal(again.hf_state_dict()[k], t[k]) for k in t)


def test_missing_tensors_and_bad_configurations_are_errors(models):
    cfg, t, _ = models["mixed"]
    P = FlatParams(ModelConfig.from_hf_dict(cfg), dtype=torch.float32)
    for gone in ("l1.mlp.e3.up", "l0.mix.k.conv", "l0.mix.v.b", "l1.mlp.correction", "embed.norm", "l2.norm1b.alpha", "l1.mix.dkv.norm"):
        with pytest.raises(KeyError):
            P.load_hf_state_dict({k: v for k, v in t.items() if k != gone})
    for change in (lambda c: c["layers"][1].update(type="mlstm"), lambda c: c["layers"][0]["mlp"].update(kind="other")):
        bad = json.loads(json.dumps(cfg))
        change(bad)
        with pytest.raises(NotImplementedError):
            ModelConfig.from_hf_dict(bad)
    for change in (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), lambda c: c["layers"][3]["mixer"].update(kv_rank=48), lambda c: c["layers"][3]["mixer"].update(kv_from=2),
                   lambda c: c["layers"][3]["mixer"].update(kv_from=5), lambda c: c["layers"][2]["mixer"].update(decay=[0.5]),
                   lambda c: c["layers"][0]["mlp"]["router"].update(top=5), lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=4)):
        bad = json.loads(json.dumps(cfg))
        change(bad)
        with pytest.raises(ValueError):
            ModelConfig.from_hf_dict(bad)
    with pytest.raises(NotImplementedError):
        build_decoder(P.cfg, P).forward_logprobs(PackedBatch.from_lengths(torch.tensor([1, 2]), [2]), torch.tensor([1, 2]), need_grad=True)


def test_layers_that_read_other_rows_have_no_pages(models):
    eng = engine(models, "mixed", ("cpu", torch.float32))
    width = {i: eng.cache.pages(i).shape[2] for i in range(9) if i in eng.cache._page_off}
    assert width == {0: 2 * 40, 1: 48, 4: 2 * 48, 5: 40}
    assert {i: eng.cache.state(i).shape[1] for i in eng.cache._state_off} == {0: 2 * (6 * 24 + 2 * 16), 2: 2 * 16 * 24, 4: 8 * 16 + 2 * 32, 6: 3 * 24 * 8}


# ---------------------------------------------------------------------------------------------- logits
@pytest.mark.parametrize("name", list(CONFIGS))
def test_packed_prompts_without_cache(models, name, place):
    arch, P = load(models, name, place)
    seqs = [tokens(n, n, arch.vocab_size) for n in (1, 2, 30, 131)]
    model = build_decoder(arch, P)
    batch = PackedBatch.from_lengths(torch.tensor(sum(seqs, [])), [len(s) for s in seqs], device=place[0])
    want = torch.cat([want_logits(models, name, s) for s in seqs])
    close(model.forward_logits(batch), want, place, name)
    labels = torch.randint(0, arch.vocab_size, (want.shape[0],), generator=torch.Generator().manual_seed(1))
    lp, ent = model.forward_logprobs(batch, labels.to(place[0]), 1.0, need_grad=False)
    ref = torch.log_softmax(want, -1)
    d_lp, d_ent = (lp.cpu() - ref.gather(-1, labels[:, None])[:, 0]).abs(), (ent.cpu() + (ref.exp() * ref).sum(-1)).abs()
    tol = 1e-3 if place[1] == torch.float32 else 0.35
    assert float(d_lp.max()) < tol and float(d_ent.max()) < tol


@pytest.mark.parametrize("name", list(CONFIGS))
def test_stream_after_every_layer(models, name, place):
    arch, P = load(models, name, place)
    seen, model, toks = [], build_decoder(arch, P), tokens(23, 2, arch.vocab_size)
    model.stats_hook = lambda what, x: seen.append(x.cpu().double())
    model.forward_hidden(PackedBatch.from_lengths(torch.tensor(toks), [23], device=place[0]))
    want: list = []
    plain.forward(models[name][0], models[name][1], toks, layer_outputs=want)
    for got, ref in zip(seen, want, strict=True):
        err = (got - ref).pow(2).mean(-1).sqrt() / ref.pow(2).mean().sqrt()
        assert float(err.max()) < (1e-5 if place[1] == torch.float32 else 0.08)


@pytest.mark.parametrize("name", list(CONFIGS))
def test_token_by_token_equals_prompt(models, name, place):
    eng = engine(models, name, place)
    t = tokens(90, 3, eng.cfg.vocab_size)
    want = want_logits(models, name, t)
    for cuts in ([90], [1], [40, 1], [2, 1]):
        close(feed_all(eng, {"a": t}, cuts)["a"], want, place, name, cuts)


@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("cuts", [[2], [3, 2], [16], [17], [33, 1, 16], [64, 5]])
def test_portions(models, name, place, cuts):
    eng = engine(models, name, place)
    seqs = {"a": tokens(100, 5, eng.cfg.vocab_size), "b": tokens(71, 6, eng.cfg.vocab_size)}
    got = feed_all(eng, seqs, cuts)
    for k, t in seqs.items():
        close(got[k], want_logits(models, name, t), place, name, cuts)


@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
def test_unequal_batches_equal_each_alone(models, name, place):
    eng = engine(models, name, place)
    seqs = {str(n): tokens(n, 10 + n, eng.cfg.vocab_size) for n in (1, 2, 17, 64, 80)}
    for cuts in ([200], [30, 1]):
        together = feed_all(eng, seqs, cuts)
        for k, t in seqs.items():
            alone = feed_all(eng, {k: t}, cuts)[k]
            close(together[k], want_logits(models, name, t), place, name, (k, cuts))
            close(together[k], alone.double(), place, name, (k, cuts))


@pytest.mark.parametrize("name", ["mixed", "wide"])
@pytest.mark.parametrize("block_size", [8, 64])
def test_slots_and_pages_used_again(models, name, place, block_size):
    """A cache with no room to spare: finished sequences leave full pages and states behind, the next ones must not see them."""
    blocks = 192 // block_size
    eng = engine(models, name, place, max_num_seqs=2, num_blocks=blocks, max_model_len=104, block_size=block_size)
    for round_ in range(4):
        seqs = {f"{round_}a": tokens(83 - 9 * round_, round_, eng.cfg.vocab_size), f"{round_}b": tokens(20 + 13 * round_, 50 + round_, eng.cfg.vocab_size)}
        got = feed_all(eng, seqs, [[200], [1], [20, 1], [7]][round_])
        for k, t in seqs.items():
            close(got[k], want_logits(models, name, t), place, name, k)
    assert len(eng.free_blocks) == blocks and len(eng.free_slots) == 2
    with pytest.raises(AssertionError):
        feed_all(eng, {"x": tokens(103, 1, eng.cfg.vocab_size), "y": tokens(102, 2, eng.cfg.vocab_size)}, [200])


# ---------------------------------------------------------------------------------------------- keys that must (not) be found
N = 32


def question_model(layers, answers, T):
    """A model of sign patterns: token T + p carries pattern p as its content, token p asks for it. Queries read the question,
    keys and values the content; a question that meets its token moves the logits by their whole size."""
    cfg = config(layers, width=2 * N, vocab=2 * T, eps=1e-4, cap=30.0)
    t = random_tensors(cfg, 9)
    signs = torch.randn(T, N, generator=torch.Generator().manual_seed(3)).sign()
    signs[:, :2] = 0                                        # nothing in the rotated pair: scores do not depend on the distance
    t["embed"].zero_()
    t["embed"][:T, :N], t["embed"][T:, N:] = signs, signs
    for name in t:
        if name.endswith(".alpha"):
            t[name] = torch.tensor(3.0 if "norm1b" not in name else 0.7)
        elif name.endswith("norm.b") or ".norm1" in name and name.endswith(".b"):
            t[name].zero_()
        elif name in ("embed.norm", "final.norm") or name.endswith(("norm1", "norm1b")):
            t[name] = torch.ones(2 * N)
    t["final.norm.alpha"] = torch.tensor(0.5)
    eye, none = torch.eye(N), torch.zeros(N, N)
    ask, content, back = torch.cat([eye, none], 1), torch.cat([none, eye], 1), torch.cat([eye, none])
    for i, l in enumerate(layers):
        p, m = f"l{i}.mix.", l["mixer"]
        t[p + "o"] = torch.cat([back] * m["heads"], 1) / m["heads"]
        if l["type"] == "attention":
            t[p + "q"], t[p + "k"], t[p + "v"] = torch.cat([ask] * m["heads"]), content.clone(), content.clone()
            for n in "qkv":
                t[p + n + ".b"].zero_()
                if m.get("conv"):
                    t[p + n + ".conv"].zero_()
                    t[p + n + ".conv"][:, -1] = 1.0
        else:
            t[p + "q"] = torch.cat([torch.cat([ask, torch.zeros(2, 2 * N)])] * m["heads"])
            t[p + "uk"], t[p + "uv"] = torch.cat([eye] * m["heads"]), torch.cat([eye] * m["heads"])
            if m.get("kv_from") is None:
                t[p + "dkv"], t[p + "dkv.norm"] = torch.cat([content, torch.zeros(2, 2 * N)]), torch.ones(N)
    ids = [T + p for p in range(T)]
    for p, far in answers.items():
        if 0 <= far < p and ids[far] >= T:
            ids[p] = ids[far] - T
    return cfg, {k: v.bfloat16().float() for k, v in t.items()}, ids


def run_questions(cfg, t, ids, place, name, seen):
    """``seen`` / unseen places: the plain logits tell whether the answer was found, and the engine gives the same ones."""
    want = plain.forward(cfg, t, ids)
    T = len(ids)
    moved = 0
    for p, far in seen.items():
        if ids[p] < T and ids[p] == far:
            gone = list(ids)
            gone[far] = T + (far + 7) % T
            moved += float((plain.forward(cfg, t, gone[: p + 1])[-1] - want[p]).abs().max()) > 0.5
            if moved >= 6:
                break
    assert moved >= 6, moved
    arch = ModelConfig.from_hf_dict(cfg)
    P = FlatParams(arch, dtype=place[1], device=place[0])
    P.load_hf_state_dict(t)
    for bs in (16, 64):
        eng = RolloutEngine(arch, P, max_num_seqs=2, max_model_len=320, block_size=bs, num_blocks=640 // bs)
        for cuts in ([T], [1], [50, 1], [16], [63, 65, 2]):
            close(feed_all(eng, {"a": ids}, cuts)["a"], want, place, name, (bs, cuts))


@pytest.mark.parametrize("size,keep", [(50, 5), (64, 64), (70, 66), (17, 1), (40, 0)])
def test_questions_at_the_edges_of_the_window(place, size, keep):
    """Tokens that ask for the oldest key of their window, the one behind it, the last kept token and the next one, and keys at page
    borders: in prompts, portions and steps."""
    T = 230
    layers = [attention(None, heads=2, kv_heads=1, dim=N, vdim=N, rot=2, base=1e9, scaling=None, conv=3, mask=(size, keep), scale=1.0)]
    answers = {}
    for n, p in enumerate(range(25, T, 2)):
        answers[p] = [p - size + 1, p - size, keep - 1, keep, p - 1, 0, p - size + 2, p - size - 1, keep - 2, keep + 1, p // 16 * 16 - 1, p // 16 * 16][n % 12]
    cfg, t, ids = question_model(layers, answers, T)
    run_questions(cfg, t, ids, place, "window", {p: far for p, far in answers.items() if far >= 0 and (p - far < size or far < keep)})


def test_far_questions_to_latents_of_another_layer(place):
    """A latent layer and a layer that reads its rows: the second finds what the first one's cache holds."""
    T = 200
    layers = [latent(None, heads=2, dim=N, rot=2, vdim=N, kv_rank=N, base=1e9, scale=1.0), latent(None, heads=3, dim=N, rot=2, vdim=N, kv_rank=N, base=1e9, scale=1.0, kv_from=0)]
    answers = {p: [0, 1, 15, 16, 17, 31, 32, 63, 64, 65, p - 1, p - 16, p - 17][(p // 3) % 13] for p in range(40, T, 3)}
    cfg, t, ids = question_model(layers, answers, T)
    run_questions(cfg, t, ids, place, "latents", answers)


def test_long_decoding(models, place):
    eng = engine(models, "mixed", place)
    t = tokens(390, 21, eng.cfg.vocab_size)
    got = feed_all(eng, {"a": t, "b": t[:200]}, [5, 1])
    want = want_logits(models, "mixed", t)
    close(got["a"], want, place, "mixed")
    close(got["b"], want[:200], place, "mixed")


# ---------------------------------------------------------------------------------------------- generation
def check_greedy(models, name, prompt, generated, place):
    """Every generated token is the plain model's argmax for its prefix (bf16: within rounding of it)."""
    want = want_logits(models, name, list(prompt) + list(generated))[len(prompt) - 1 : -1]
    gap = want.max(-1).values - want.gather(-1, torch.tensor(generated)[:, None])[:, 0]
    assert float(gap.max()) < (1e-3 if place[1] == torch.float32 else 0.5), gap


@pytest.mark.parametrize("name", ["mixed", "odd", "wide", "bare"])
def test_greedy_generation_with_the_scheduler(models, name, place):
    """More requests than slots, unequal prompts and lengths, repeated prompts (prefilled once), slots and pages used again."""
    eng = engine(models, name, place, max_num_seqs=3, num_blocks=40, enable_prefix_caching=True)
    V = eng.cfg.vocab_size
    prompts = [tokens(n, 60 + n, V) for n in (5, 40, 17, 1, 33)]
    prompts += [prompts[1], prompts[1], prompts[0]]
    params = [SamplingParams(temperature=0.0, max_tokens=m) for m in (20, 12, 31, 40, 3, 12, 25, 20)]
    for _ in range(2):
        outs = eng.generate(prompts, params)
        assert [len(o.token_ids) for o in outs] == [p.max_tokens for p in params]
        for p, o in zip(prompts, outs):
            check_greedy(models, name, p, o.token_ids, place)
    assert len(eng.free_slots) == 3 and len(eng.free_blocks) == 40


def test_sampled_generation_and_log_probs(models, place):
    eng = engine(models, "wide", place)
    prompt = tokens(21, 4, eng.cfg.vocab_size)
    outs = eng.generate([prompt] * 4, [SamplingParams(temperature=1.0, max_tokens=15, seed=s) for s in (1, 2, 3, 1)])
    assert outs[0].token_ids == outs[3].token_ids and outs[0].token_ids != outs[1].token_ids
    for o in outs:
        want = torch.log_softmax(want_logits(models, "wide", prompt + o.token_ids)[len(prompt) - 1 : -1], -1)
        lp = want.gather(-1, torch.tensor(o.token_ids)[:, None])[:, 0]
        assert float((lp - torch.tensor(o.log_probs)).abs().max()) < (1e-3 if place[1] == torch.float32 else 0.5)


def test_prefill_decode_handoff(models, place):
    pre, dec = engine(models, "mixed", place), engine(models, "mixed", place)
    prompts = [tokens(n, n, pre.cfg.vocab_size) for n in (9, 34)]
    sp = SamplingParams(temperature=0.0, max_tokens=14)
    for i, h in enumerate(pre.prefill_only(prompts, sp)):
        dec.add_prefilled(h, sp, f"r{i}")
    got = {}
    while len(got) < 2:
        got.update({o.request_id: o.token_ids for o in dec.step()})
    for i, p in enumerate(prompts):
        check_greedy(models, "mixed", p, got[f"r{i}"], place)


def test_generation_command_line(models, tmp_path, monkeypatch):
    """``main_generation_server`` on a checkpoint directory: token-id prompts in, token-id responses out."""
    pd = pytest.importorskip("pandas")
    from verl_b200.trainer import main_generation_server as cli

    monkeypatch.setenv("VERL_ENGINE_DEVICE", "cpu")
    cfg, _, path = models["mixed"]
    prompts = [tokens(n, n, cfg["vocab"]) for n in (6, 19)]
    src, dst = str(tmp_path / "in.parquet"), str(tmp_path / "out.parquet")
    pd.DataFrame({"prompt": prompts}).to_parquet(src)
    cli.main([f"data.path={src}", f"data.output_path={dst}", "data.n_samples=1", f"actor_rollout_ref.model.path={path}", "trainer.device=cpu",
              "actor_rollout_ref.rollout.temperature=0.0", "actor_rollout_ref.rollout.prompt_length=32", "actor_rollout_ref.rollout.response_length=11",
              "actor_rollout_ref.rollout.max_num_seqs=2", "actor_rollout_ref.rollout.block_size=16"])
    for p, r in zip(prompts, pd.read_parquet(dst)["responses"]):
        out = [int(t) for t in r[0]]
        assert len(out) == 11
        check_greedy(models, "mixed", p, out, ("cpu", torch.float32))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_runner(models, tmp_path, dtype):
    """The program replays unequal requests, decodes them together, ends them one by one and writes only what is wanted."""
    import numpy as np

    name = "wide"
    cfg, _, path = models[name]
    seqs = {"a": tokens(30, 1, cfg["vocab"]), "b": tokens(12, 2, cfg["vocab"])}
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": seqs["a"][:20], "want": [0, 19]}, {"id": "b", "tokens": seqs["b"][:9], "want": []}], "end": []}]
    for n in range(10):
        e = [{"id": k, "tokens": [t[c + n]], "want": [0] if n % 2 else []} for k, t, c in (("a", seqs["a"], 20), ("b", seqs["b"], 9)) if c + n < len(t)]
        steps.append({"step": n + 1, "entries": e, "end": [k for k, c in (("a", 20), ("b", 9)) if c + n + 1 == len(seqs[k])]})
    run = subprocess.run([sys.executable, os.path.join(REPO, "bin", "trace_run"), "--model", path, "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "64",
                          "--device", "cpu"], input="\n".join(map(json.dumps, steps)) + "\n", capture_output=True, text=True, timeout=300)
    assert run.returncode == 0, run.stderr[-2000:]
    assert [l for l in run.stdout.splitlines() if l.startswith("done")] == [f"done {n}" for n in range(11)]
    read = lambda n: torch.from_numpy(np.fromfile(tmp_path / f"{n}.f32", dtype="<f4")).view(-1, cfg["vocab"])
    place = ("cpu", getattr(torch, dtype))
    a, b = want_logits(models, name, seqs["a"]), want_logits(models, name, seqs["b"])
    close(read(0), a[[0, 19]], place, name)
    assert not (tmp_path / "1.f32").exists()
    close(read(2), torch.stack([a[21], b[10]]), place, name)
    close(read(10), a[[29]], place, name)
