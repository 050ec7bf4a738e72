"""Fusazen models through the rollout engine: prompts, decoding, portions, batches, reused slots and pages, chunk edges, generation."""

import json
import os
import subprocess
import sys

import pytest
import torch

from oracles import fusazen_plain as plain
from stack_testing import PLACES, feed_all, position_errors, tokens
from verl_b200.models import FlatParams, ModelConfig, PackedBatch, build_decoder
from verl_b200.utils.model import load_hf_weights_into, save_hf_weights
from verl_b200.workers.rollout.native.engine import RolloutEngine, SamplingParams

torch.set_num_threads(min(4, torch.get_num_threads()))
REPO = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.fixture(params=PLACES)
def place(request):
    return request.param


def dense(ff=40):
    return {"kind": "dense", "ff": ff}


def delta(mlp=None, heads=2, dim=24):
    return {"type": "general_delta", "mlp": mlp, "mixer": {"heads": heads, "dim": dim}}


def differential(mlp=None, heads=4, kv_heads=2, dim=16, vdim=24, rot=8, base=500.0, chunk=20, scale=0.4, diff=0.45, kv_from=None):
    m = {"diff": diff, "dim": dim, "heads": heads, "kv_heads": kv_heads, "mask": {"size": chunk}, "rot": {"base": base, "dims": rot}, "scale": scale, "vdim": vdim}
    return {"type": "attention", "mlp": mlp, "mixer": m if kv_from is None else {**m, "kv_from": kv_from}}


def whole(mlp=None, heads=6, kv_heads=3, dim=16, vdim=32, chunk=33, scale=0.3):
    return {"type": "attention_2", "mlp": mlp, "mixer": {"dim": dim, "heads": heads, "kv_heads": kv_heads, "mask": {"size": chunk}, "scale": scale, "vdim": vdim}}


def config(layers, width=72, vocab=88, eps=1e-4, taps=4, scale=5.0):
    return {"architecture": "Fusazen", "canon": {"taps": taps}, "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


CONFIGS = {
    # every kind of layer, in an order of its own; two layers with keys that others read, one of them twice and with other chunks
    "mixed": config([differential(dense()), whole(dense(24)), delta(None), differential(dense(), chunk=50, scale=0.6, diff=0.2, kv_from=0), differential(None, heads=3, kv_heads=3, vdim=40, rot=16, chunk=64),
                     delta(dense(56), heads=3, dim=32), differential(dense(), chunk=7, kv_from=0), differential(dense(), heads=3, kv_heads=3, vdim=40, rot=16, chunk=16, kv_from=4), whole(None, chunk=16)]),
    # sizes that are no multiple of 8, rotation over a part of a head
    "odd": config([delta(dense(18), heads=3, dim=7), differential(dense(30), heads=3, kv_heads=1, dim=10, vdim=14, rot=6, chunk=9), whole(dense(21), heads=3, kv_heads=1, dim=9, vdim=5, chunk=31),
                   differential(dense(10), heads=3, kv_heads=1, dim=10, vdim=14, rot=6, chunk=40, kv_from=1), delta(None, heads=1, dim=30)], width=42, vocab=61, eps=2e-2, taps=2, scale=1.0),
    # more than 16 maps per key head, sizes of two and three panels, large heads
    "wide": config([whole(dense(136), heads=20, kv_heads=1, dim=72, vdim=136, chunk=70, scale=0.1), delta(dense(264), heads=2, dim=128), differential(dense(72), heads=9, kv_heads=1, dim=72, vdim=128, rot=64,
                                                                                                                                                chunk=65, scale=0.1),
                    delta(dense(), heads=1, dim=136), differential(None, heads=2, kv_heads=1, dim=64, vdim=200, rot=64, base=1e4, chunk=128, scale=0.1)], width=200, vocab=264, taps=3),
    # no second sublayer anywhere, one tap, chunks of one token
    "bare": config([whole(chunk=1), delta(), differential(chunk=1, kv_heads=4), delta(dim=16)], taps=1, scale=0.5),
    # one of everything
    "ones": config([delta(dense(8), heads=1, dim=8), differential(dense(8), heads=1, kv_heads=1, dim=8, vdim=8, rot=2, chunk=5), whole(dense(8), heads=1, kv_heads=1, dim=8, vdim=8, chunk=6),
                    differential(None, heads=1, kv_heads=1, dim=8, vdim=8, rot=2, chunk=3, kv_from=1)], width=16, vocab=24, taps=6),
}
RANK = {"mixed": 16, "odd": 5, "wide": 24, "bare": 3, "ones": 1}


def expected_tensors(cfg, rank):
    """Checkpoint names and shapes, written from the format (not from the package)."""
    D, out = cfg["width"], {"embed": (cfg["vocab"], cfg["width"]), "head": (cfg["vocab"], cfg["width"]), "final.norm": (cfg["width"],)}
    for i, l in enumerate(cfg["layers"]):
        m, f, p = l["mixer"], l["mlp"], f"l{i}."
        H, d = m["heads"], m["dim"]
        out.update({p + "norm1": (D,), p + "canon1": (D, cfg["canon"]["taps"])})
        if l["type"] == "general_delta":
            n = H * d
            out.update({p + "mix." + k: (n, D) for k in "rkvga"})
            out.update({p + "mix.a.b": (n,), p + "mix.w1": (rank, D), p + "mix.w2": (n, rank), p + "mix.w0": (n,), p + "mix.norm": (n,), p + "mix.o": (D, n)})
        else:
            G, e, maps = m["kv_heads"], m["vdim"], 2 if l["type"] == "attention" else 1
            out.update({p + "mix.q": (H * maps * d, D), p + "mix.o": (D, H * e)})
            if m.get("kv_from") is None:
                out.update({p + "mix.k": (G * maps * d, D), p + "mix.v": (G * e, D)})
            if maps == 2:
                out.update({p + "mix." + k: (d,) for k in ("lq1", "lk1", "lq2", "lk2")})
            else:
                out.update({p + "mix.q.norm": (H * d,), p + "mix.k.norm": (G * d,), p + "mix.temp": (H,)})
        if f is not None:
            out.update({p + "norm2": (D,), p + "mlp.up": (f["ff"], D), p + "mlp.up.b": (f["ff"],), p + "mlp.down": (D, f["ff"]), p + "mlp.down.b": (D,)})
    return out


def random_tensors(cfg, rank, seed=0):
    g, t = torch.Generator().manual_seed(seed), {}
    for name, shape in expected_tensors(cfg, rank).items():
        x, last = torch.randn(shape, generator=g), name.rsplit(".", 1)[-1]
        if last in ("norm", "norm1", "norm2", "temp"):
            x = 1.0 + 0.3 * x
        elif last == "canon1":
            x = 0.6 * x * shape[1] ** -0.5
        elif last in ("lq1", "lk1", "lq2", "lk2"):
            x = x * 0.5 * shape[0] ** -0.25
        elif last in ("b", "w0"):
            x = 0.3 * x + (1.0 if name.endswith("a.b") else 0.0)
        elif name != "embed":
            x = x * 1.3 * shape[-1] ** -0.5
        t[name] = x.bfloat16().float()
    return t


def with_rank(cfg, rank):
    """The configuration as it is when the weights have been looked at."""
    return {**cfg, "layers": [{**l, "mixer": {**l["mixer"], "decay_rank": rank}} if l["type"] == "general_delta" else l for l in cfg["layers"]]}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """name -> (config, tensors, directory with config.json and safetensors)"""
    from safetensors.torch import save_file

    out = {}
    for i, (name, cfg) in enumerate(CONFIGS.items()):
        d = tmp_path_factory.mktemp(name)
        t = random_tensors(cfg, RANK[name], seed=i)
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
    """fp32: every position; bf16: a position in a hundred may round badly (differences of maps and read-outs cancel here and there), within twice
    the limit."""
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
    assert {k: tuple(v.shape) for k, v in sd.items()} == expected_tensors(cfg, RANK[name])
    assert all(torch.equal(sd[k], t[k]) for k in t)
    assert arch.is_stack and arch.hidden_size == cfg["width"] and arch.to_hf_dict() == with_rank(cfg, RANK[name])
    assert arch.num_parameters() >= sum(v.numel() for v in t.values())
    save_hf_weights(P, str(tmp_path))
    again = FlatParams(ModelConfig.from_pretrained(str(tmp_path)), dtype=torch.float32)
    load_hf_weights_into(again, str(tmp_path), strict=True)
    assert all(torch.equal(again.hf_state_dict()[k], t[k]) for k in t)


def test_ranks_of_layers_may_differ(tmp_path):
    """The decay's inner size is known from the weights alone, layer by layer."""
    from safetensors.torch import save_file

    cfg = config([delta(heads=1, dim=8), delta(heads=2, dim=8)], width=16, vocab=24, taps=2)
    t = random_tensors(cfg, 5, 1)
    t["l1.mix.w1"], t["l1.mix.w2"] = torch.randn(11, 16).bfloat16().float(), torch.randn(16, 11).bfloat16().float()
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_file({k: v.bfloat16() for k, v in t.items()}, str(tmp_path / "model.safetensors"))
    P = FlatParams(ModelConfig.from_pretrained(str(tmp_path)), dtype=torch.float32)
    load_hf_weights_into(P, str(tmp_path), strict=True)
    toks = tokens(20, 1, 24)
    got = build_decoder(P.cfg, P).forward_logits(PackedBatch.from_lengths(torch.tensor(toks), [20]))
    close(got, plain.forward(cfg, t, toks), ("cpu", torch.float32))
    with pytest.raises(ValueError):
        ModelConfig.from_hf_dict(cfg)
    save_file({k: v.bfloat16() for k, v in t.items() if k != "l1.mix.w1"}, str(tmp_path / "model.safetensors"))
    with pytest.raises(KeyError):
        ModelConfig.from_pretrained(str(tmp_path))


def test_missing_tensors_and_bad_configurations_are_errors(models):
    cfg, t = with_rank(models["mixed"][0], RANK["mixed"]), models["mixed"][1]
    P = FlatParams(ModelConfig.from_hf_dict(cfg), dtype=torch.float32)
    for gone in ("l2.mix.w2", "l0.mix.lk2", "l0.mix.v", "l1.mix.temp", "l1.mix.k.norm", "l4.canon1", "l0.mlp.up.b", "l5.mix.a.b", "final.norm"):
        with pytest.raises(KeyError):
            P.load_hf_state_dict({k: v for k, v in t.items() if k != gone})
    for change in (lambda c: c["layers"][1].update(type="mlstm"), lambda c: c["layers"][0]["mlp"].update(kind="other")):
        bad = json.loads(json.dumps(cfg))
        change(bad)
        with pytest.raises(NotImplementedError):
            ModelConfig.from_hf_dict(bad)
    for change in (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), lambda c: c["layers"][3]["mixer"].update(dim=24), lambda c: c["layers"][3]["mixer"].update(kv_from=2),
                   lambda c: c["layers"][3]["mixer"].update(kv_from=4), lambda c: c["layers"][3]["mixer"].update(kv_from=1), lambda c: c["layers"][3]["mixer"]["rot"].update(base=3.0),
                   lambda c: c["layers"][6]["mixer"].update(kv_from=3), lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), lambda c: c["canon"].update(taps=0)):
        bad = json.loads(json.dumps(cfg))
        change(bad)
        with pytest.raises(ValueError):
            ModelConfig.from_hf_dict(bad)
    with pytest.raises(NotImplementedError):
        build_decoder(P.cfg, P).forward_logprobs(PackedBatch.from_lengths(torch.tensor([1, 2]), [2]), torch.tensor([1, 2]), need_grad=True)


def test_pages_and_states_of_the_layers(models):
    """Layers that read other rows have no pages; every layer keeps its convolution's past."""
    eng = engine(models, "mixed", ("cpu", torch.float32))
    width = {i: eng.cache.pages(i).shape[2] for i in range(9) if i in eng.cache._page_off}
    assert width == {0: 2 * (32 + 24), 1: 3 * 48, 4: 3 * (32 + 40), 8: 3 * 48}
    assert {i: eng.cache.state(i).shape[1] for i in (2, 5)} == {2: 2 * 24 * 24, 5: 3 * 32 * 32}
    assert all(eng.cache.input_state(i).shape[1] == 3 * 72 for i in range(9))
    assert engine(models, "bare", ("cpu", torch.float32)).cache.input_state(0) is None


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
    tol = 1e-3 if place[1] == torch.float32 else 0.5
    assert float(d_lp.max()) < tol and float(d_ent.max()) < tol


@pytest.mark.parametrize("name", list(CONFIGS))
def test_stream_after_every_layer(models, name, place):
    """Of a prompt, and of steps (whose last addition is still to come when a layer ends)."""
    toks, want = tokens(23, 2, models[name][0]["vocab"]), []
    plain.forward(models[name][0], models[name][1], toks, layer_outputs=want)
    eng, seen = engine(models, name, place), []
    eng.model.stats_hook = lambda what, x: seen.append(x.cpu().double())
    eng.open_sequence("a")
    eng.feed([("a", toks[:20], [])])
    prompt, slot = list(seen), eng.sequences["a"].slot
    steps = [[] for _ in want]
    for n in range(20, 23):
        seen.clear()
        eng.feed([("a", toks[n : n + 1], [])])
        for rows, x in zip(steps, seen, strict=True):
            rows.append(x[slot])
    for got, step, ref in zip(prompt, steps, want, strict=True):
        err = (torch.cat([got, torch.stack(step)]) - ref).pow(2).mean(-1).sqrt() / ref.pow(2).mean().sqrt()
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


def test_first_tokens_of_a_sequence(models, place):
    """The convolutions and memories start from nothing, whatever the slot held before."""
    for name in ("mixed", "ones"):
        eng = engine(models, name, place, max_num_seqs=1)
        for n, cuts in ((40, [40]), (3, [1]), (5, [2, 1]), (1, [1]), (7, [7]), (2, [1])):
            t = tokens(n, 70 + n, eng.cfg.vocab_size)
            close(feed_all(eng, {"a": t}, cuts)["a"], want_logits(models, name, t), place, name, (n, cuts))


def test_weights_that_change_in_place_are_seen(models, place):
    """The weight of a map's difference is taken from the weights at every call."""
    eng = engine(models, "ones", place)
    cfg, t, _ = models["ones"]
    toks, new = tokens(20, 8, cfg["vocab"]), dict(t)
    new["l1.mix.lq1"], new["l1.mix.lk1"] = torch.full((8,), 0.5), torch.full((8,), 0.375)
    eng.params.load_hf_state_dict(new)
    want = plain.forward(cfg, new, toks)
    assert float(position_errors(want_logits(models, "ones", toks), want).max()) > 0.2
    for cuts in ([20], [1]):
        close(feed_all(eng, {"a": toks}, cuts)["a"], want, place)


# ---------------------------------------------------------------------------------------------- keys that must (not) be found
N = 32


def question_model(layers, answers, T):
    """A model of sign patterns: token T + p carries pattern p as its content, token p asks for it. Queries read the question,
    keys and values the content; a question that meets its token moves the logits by their whole size."""
    cfg = config(layers, width=2 * N, vocab=2 * T, taps=3, scale=1.0)
    t = random_tensors(cfg, 4, 9)
    signs = torch.randn(T, N, generator=torch.Generator().manual_seed(3)).sign()
    signs[:, :2] = 0                                        # nothing in the rotated pair: scores do not depend on the distance
    t["embed"].zero_()
    t["embed"][:T, :N], t["embed"][T:, N:] = signs, signs
    for name in t:
        if name.endswith("norm") or name.endswith("norm1") or name.endswith("temp"):
            t[name] = torch.ones_like(t[name])
        elif name.endswith("canon1"):
            t[name].zero_()
    eye, none = torch.eye(N), torch.zeros(N, N)
    ask, content, back = torch.cat([eye, none], 1), torch.cat([none, eye], 1), torch.cat([eye, none])
    for i, l in enumerate(layers):
        p, m = f"l{i}.mix.", l["mixer"]
        two = l["type"] == "attention"                      # the second map asks nothing
        t[p + "o"] = torch.cat([back] * m["heads"], 1) / m["heads"]
        t[p + "q"] = torch.cat([torch.cat([ask, 0 * ask]) if two else ask] * m["heads"])
        if m.get("kv_from") is None:
            t[p + "k"], t[p + "v"] = torch.cat([torch.cat([content] * (2 if two else 1))] * m["kv_heads"]), torch.cat([content] * m["kv_heads"])
    ids = [T + p for p in range(T)]
    for p, far in answers.items():
        if 0 <= far < p and ids[far] >= T:
            ids[p] = ids[far] - T
    return cfg, with_rank(cfg, 4), {k: v.bfloat16().float() for k, v in t.items()}, ids


def run_questions(cfg, full, t, ids, place, name, seen):
    """``seen`` / unseen places: the plain logits tell whether the answer was found, and the engine gives the same ones."""
    want = plain.forward(cfg, t, ids)
    T, moved = len(ids), 0
    for p, far in seen.items():
        if ids[p] < T and ids[p] == far:
            gone = list(ids)
            gone[far] = T + (far + 7) % T
            moved += float((plain.forward(cfg, t, gone[: p + 1])[-1] - want[p]).abs().max()) > 0.5
            if moved >= 6:
                break
    assert moved >= 6, moved
    arch = ModelConfig.from_hf_dict(full)
    P = FlatParams(arch, dtype=place[1], device=place[0])
    P.load_hf_state_dict(t)
    for bs in (16, 64):
        eng = RolloutEngine(arch, P, max_num_seqs=2, max_model_len=320, block_size=bs, num_blocks=640 // bs)
        for cuts in ([T], [1], [50, 1], [16], [63, 65, 2]):
            close(feed_all(eng, {"a": ids}, cuts)["a"], want, place, name, (bs, cuts))


@pytest.mark.parametrize("kind", ["differential", "whole"])
@pytest.mark.parametrize("size", [50, 64, 17, 100, 128])
def test_questions_at_the_edges_of_chunks(place, kind, size):
    """Tokens that ask for the first key of their chunk, the last one of the chunk before, and keys at page borders: in prompts, portions and
    steps."""
    T = 230
    one = dict(heads=2, kv_heads=1, dim=N, vdim=N, chunk=size, scale=0.5)
    layers = [differential(None, rot=2, base=1e9, diff=0.25, **one) if kind == "differential" else whole(None, **one)]
    answers = {}
    for n, p in enumerate(range(9, T, 2)):
        first = p // size * size
        answers[p] = [first, first - 1, first + 1, p - 1, 0, first - 2, p // 16 * 16 - 1, p // 16 * 16, first - size, first + 2][n % 10]
    cfg, full, t, ids = question_model(layers, answers, T)
    run_questions(cfg, full, t, ids, place, kind, {p: far for p, far in answers.items() if 0 <= far and p // size == far // size})


def test_questions_to_keys_of_another_layer(place):
    """A layer that reads another one's rows finds them within its own chunks, which are longer or shorter than the owner's."""
    T = 200
    one = dict(heads=2, kv_heads=2, dim=N, vdim=N, rot=2, base=1e9, diff=0.25, scale=0.5)
    layers = [differential(None, chunk=24, **one), differential(None, chunk=150, kv_from=0, **one), differential(None, chunk=10, kv_from=0, **one)]
    answers = {p: [p // 150 * 150, p // 24 * 24, p // 24 * 24 - 1, p // 150 * 150 - 1, p // 10 * 10, p - 1, 63, 64, p - 16, p - 17][(p // 3) % 10] for p in range(40, T, 3)}
    cfg, full, t, ids = question_model(layers, answers, T)
    run_questions(cfg, full, t, ids, place, "rows", {p: far for p, far in answers.items() if 0 <= far < p and p // 150 == far // 150})


def test_memory_recalls_far_keys_and_forgets_on_request(place):
    """A delta-rule layer whose decays are as slow as they get and whose removals are switched by the token: what was written long ago is read
    again, and a removal of the same key takes it away."""
    heads, d, V = 1, 16, 40
    cfg = config([delta(None, heads=heads, dim=d)], width=64, vocab=V, taps=2, scale=1.0)
    t = random_tensors(cfg, 3, 4)
    t["embed"] = torch.zeros(V, 64)
    keys = torch.eye(16)
    for v in range(16):
        t["embed"][v, :16] = 4.0 * keys[v]                                      # reads key v
        t["embed"][16 + v, 16:32], t["embed"][16 + v, 32:48] = 4.0 * keys[v], 4.0 * keys[(5 * v + 3) % 16]   # writes value 5 v + 3 under key v
    t["embed"][32:, 48:] = torch.randn(8, 16, generator=torch.Generator().manual_seed(1)).bfloat16().float()
    t["l0.norm1"], t["l0.canon1"] = torch.ones(64), torch.zeros(64, 2)
    put = lambda at: torch.cat([torch.zeros(16, at), torch.eye(16), torch.zeros(16, 48 - at)], 1)
    t["l0.mix.r"], t["l0.mix.k"], t["l0.mix.v"] = put(0), put(16), put(32)
    t["l0.mix.w2"].zero_()
    t["l0.mix.w0"] = torch.full((16,), -12.0)                                   # decay exp(-0.6 sigmoid(-12))
    t["l0.mix.a"] = 8.0 * put(16)
    t["l0.mix.a.b"] = torch.full((16,), -6.0)
    t = {k: v.bfloat16().float() for k, v in t.items()}
    ids = [16 + 2, 16 + 7, *([33, 38, 35] * 20), 2, 7, 16 + 2, 2, 7, *([34] * 40), 7, 2, 9]
    want = plain.forward(cfg, t, ids)
    alone = plain.forward(cfg, t, [7])
    assert float((want[-3] - alone[0]).abs().max()) > 0.5                       # still there after 100 tokens
    arch = ModelConfig.from_hf_dict(with_rank(cfg, 3))
    P = FlatParams(arch, dtype=place[1], device=place[0])
    P.load_hf_state_dict(t)
    eng = RolloutEngine(arch, P, max_num_seqs=2, max_model_len=320, block_size=16, num_blocks=40)
    for cuts in ([len(ids)], [1], [50, 1], [16], [17, 2]):
        close(feed_all(eng, {"a": ids}, cuts)["a"], want, place, "memory", cuts)


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
