"""Tofinex models through the rollout engine: prompts, decoding, portions, batches, reused slots and pages, far keys, generation.

Routers make choices, and a choice between two experts of nearly equal scores may fall differently in bf16. The models that
choose therefore keep a few dimensions of the stream for their routers: they come from the embedding, the sublayers add nothing
to them, and every token's choice is clear (``settle_routers``).
"""

import json
import os
import subprocess
import sys

import pytest
import torch

from oracles import tofinex_plain as plain
from stack_testing import PLACES, feed_all, position_errors, tokens
from verl_b200.models import FlatParams, ModelConfig, PackedBatch, build_decoder
from verl_b200.utils.model import load_hf_weights_into, save_hf_weights
from verl_b200.workers.rollout.native.engine import RolloutEngine, SamplingParams

torch.set_num_threads(min(4, torch.get_num_threads()))
REPO = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.fixture(params=PLACES)
def place(request):
    return request.param


def layer(mlp=None, heads=4, kv_heads=2, dim=24, vdim=16, rot=16, base=800.0, scale=0.35, cap=6.0, mix=True):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": rot}, "scale": scale, "softcap": cap, "v_mix": mix}}


def dense(ff=40):
    return {"kind": "dense", "ff": ff}


def moe(experts=5, top=2, ff=24, shared=32):
    f = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    return f if shared is None else {**f, "shared": {"ff": shared}}


def config(layers, width=72, vocab=88, mult=0.6, eps=1e-4, cap=9.0):
    return {"architecture": "Tofinex", "layers": layers, "logit_softcap": cap, "norm": {"eps": eps}, "residual_mult": mult, "vocab": vocab, "width": width}


CONFIGS = {
    # every kind of layer; values are mixed from the second layer on, other sizes where they may differ
    "mixed": config([layer(dense(), mix=False, heads=3, kv_heads=3, dim=32, vdim=24, rot=32), layer(moe()), layer(None), layer(moe(7, 1, 16, None), heads=6, dim=16, rot=8),
                     layer(dense(56), mix=False, heads=8, kv_heads=1, scale=0.2, cap=20.0), layer(moe(4, 3), heads=2)]),
    # sizes that are no multiple of 8, one pair of rotated dimensions
    "odd": config([layer(dense(22), heads=3, kv_heads=1, dim=10, vdim=14, rot=6), layer(moe(5, 3, 11, 13), heads=6, kv_heads=1, dim=7, vdim=14, rot=2),
                   layer(moe(3, 3, 10, 6), heads=1, kv_heads=1, dim=12, vdim=14, rot=12)], width=42, vocab=61, mult=1.0, eps=3e-3, cap=4.0),
    # all experts of every layer are used; more than 16 query heads per key head, sizes of two and three panels
    "wide": config([layer(moe(3, 3, 72, 40), heads=20, kv_heads=1, dim=72, vdim=136, rot=64, scale=0.1), layer(moe(2, 2, 64, 64), heads=4, kv_heads=1, dim=136, vdim=136, rot=120),
                    layer(dense(200), heads=2, kv_heads=2, dim=64, vdim=68, rot=64, mix=False)], width=200, vocab=264, mult=0.3),
    # no mixing, no second sublayer at the end
    "plain": config([layer(dense(72), mix=False), layer(dense(48), mix=False, heads=6, kv_heads=3, vdim=40), layer(None, mix=False)], mult=1.3),
    # one of everything
    "ones": config([layer(moe(1, 1, 8, 8), heads=1, kv_heads=1, dim=8, vdim=8, rot=2)], width=16, vocab=24),
}


def expected_tensors(cfg):
    """Checkpoint names and shapes, written from the format (not from the package)."""
    D = cfg["width"]
    out = {"embed": (cfg["vocab"], D), "embed.norm": (D,), "final.norm": (D,)}
    for i, l in enumerate(cfg["layers"]):
        m, f, p = l["mixer"], l["mlp"], f"l{i}."
        H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        out.update({p + "norm1": (D,), p + "mix.q": (H * d, D), p + "mix.k": (G * d, D), p + "mix.v": (G * e, D), p + "mix.o": (D, H * e), p + "mix.q.norm": (d,),
                    p + "mix.k.norm": (d,)})
        if m["v_mix"]:
            out[p + "mix.vmix"] = ()
        if f is None:
            continue
        out[p + "norm2"] = (D,)
        if f["kind"] == "dense":
            parts = [("", f["ff"])]
        else:
            out[p + "mlp.router"] = (f["router"]["experts"], D)
            parts = [(f"e{j}.", f["expert"]["ff"]) for j in range(f["router"]["experts"])]
            if "shared" in f:
                parts.append(("shared.", f["shared"]["ff"]))
                out[p + "mlp.shared.sg"] = (1, D)
        for name, ff in parts:
            out.update({p + "mlp." + name + "gate": (ff, D), p + "mlp." + name + "up": (ff, D), p + "mlp." + name + "down": (D, ff)})
    return out


def random_tensors(cfg, seed=0):
    g, t = torch.Generator().manual_seed(seed), {}
    for name, shape in expected_tensors(cfg).items():
        x = torch.randn(shape, generator=g)
        if name.endswith(".vmix"):
            x = torch.tensor(0.3 + 0.1 * (int(name[1]) % 3))
        elif name.endswith("norm") or ".norm" in name:
            x = (1.6 if ".mix." in name else 1.0) + 0.3 * x     # sharp attention
        elif name == "embed":
            x = 0.5 * x
        else:
            x = x * (2.0 if "router" in name else 1.2) * shape[-1] ** -0.5
        t[name] = x.bfloat16().float()
    if any(chosen(l) for l in cfg["layers"]):
        settle_routers(cfg, t, g)
    return t


def chosen(l):
    """(experts, top) of a layer whose tokens leave some experts out."""
    r = (l["mlp"] or {}).get("router")
    return (r["experts"], r["top"]) if r is not None and r["top"] < r["experts"] else None


def settle_routers(cfg, t, g, own=8):
    """The last ``own`` dimensions decide: no norm weight there, large router weights there, and embedding rows drawn until the
    last chosen expert is well ahead of the next one in every layer."""
    for name in t:
        if ".norm1" in name or ".norm2" in name:
            t[name][-own:] = 0.0
        if name.endswith("router"):
            t[name][:, :-own] *= 0.0625
            t[name][:, -own:] = torch.randn(t[name].shape[0], own, generator=g).bfloat16().float()
    t["embed.norm"][-own:] = 1.0
    left = torch.arange(cfg["vocab"])
    for _ in range(2000):
        x = plain.rms_norm(t["embed"].double(), t["embed.norm"].double(), cfg["norm"]["eps"])
        gap = torch.full((cfg["vocab"],), 9.0).double()
        for i, l in enumerate(cfg["layers"]):
            if chosen(l):
                z = (x[:, -own:] @ t[f"l{i}.mlp.router"][:, -own:].double().t()).sort(-1, descending=True).values
                gap = torch.minimum(gap, z[:, chosen(l)[1] - 1] - z[:, chosen(l)[1]])
        left = torch.nonzero(gap < 0.4).flatten()
        if not len(left):
            return
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
    err = position_errors(got, want)
    limit = 1e-4 if place[1] == torch.float32 else 0.08
    assert float(err.max()) < limit, (name, what, float(err.max()), int(err.argmax()))


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
    assert {k: tuple(v.shape) for k, v in sd.items() if k != "lm_head.weight"} == expected_tensors(cfg)
    assert all(torch.equal(sd[k], t[k]) for k in t)
    assert arch.is_stack and arch.hidden_size == cfg["width"] and arch.to_hf_dict() == cfg and arch.num_parameters() >= sum(v.numel() for v in t.values())
    save_hf_weights(P, str(tmp_path))
    again = FlatParams(ModelConfig.from_pretrained(str(tmp_path)), dtype=torch.float32)
    load_hf_weights_into(again, str(tmp_path), strict=True)
    assert all(torch.equal(again.hf_state_dict()[k], t[k]) for k in t)


def test_missing_tensors_and_bad_configurations_are_errors(models):
    cfg, t, _ = models["mixed"]
    P = FlatParams(ModelConfig.from_hf_dict(cfg), dtype=torch.float32)
    for gone in ("l1.mlp.e3.up", "l2.mix.vmix", "l1.mlp.shared.sg", "embed.norm"):
        with pytest.raises(KeyError):
            P.load_hf_state_dict({k: v for k, v in t.items() if k != gone})
    for change in (lambda c: c["layers"][1].update(type="latent_attention"), lambda c: c["layers"][0]["mlp"].update(kind="other")):
        bad = json.loads(json.dumps(cfg))
        change(bad)
        with pytest.raises(NotImplementedError):
            ModelConfig.from_hf_dict(bad)
    for change in (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), lambda c: c["layers"][1]["mixer"].update(vdim=24)):
        bad = json.loads(json.dumps(cfg))
        change(bad)
        with pytest.raises(ValueError):
            ModelConfig.from_hf_dict(bad)
    with pytest.raises(NotImplementedError):
        build_decoder(P.cfg, P).forward_logprobs(PackedBatch.from_lengths(torch.tensor([1, 2]), [2]), torch.tensor([1, 2]), need_grad=True)


def test_flops_count_the_experts_a_token_uses(models):
    from verl_b200.utils.flops_counter import FlopsCounter

    count = lambda top: FlopsCounter(ModelConfig.from_hf_dict(config([layer(moe(8, top, 64))])))._dense_per_token()
    assert count(3) - count(1) == pytest.approx(2 * 3 * 64 * 72)


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
    """A cache with no room to spare: finished sequences leave full pages behind, the next ones must not see them."""
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


def test_far_keys_at_page_borders(place):
    """One layer in which some tokens match exactly one earlier token: the first ones of the sequence, those beside page borders,
    the one before. A key that is lost, or read from the wrong place, changes the logits by their whole size; so does a sink that
    is left out (tokens without a match have low scores only)."""
    n, T = 32, 200
    cfg = config([layer(None, heads=2, kv_heads=1, dim=n, vdim=n, rot=2, base=1e9, scale=1.0, cap=40.0)], width=2 * n, vocab=2 * T, mult=3.0, eps=1e-4)
    t = random_tensors(cfg, 9)
    content = torch.randn(T, n, generator=torch.Generator().manual_seed(3))
    content[:, :2] = 0                                      # nothing in the rotated pair: scores do not depend on the distance
    t["embed"].zero_()
    t["embed"][:T, :n], t["embed"][T:, n:] = content, content      # token p < T asks for token T + p
    eye, none = torch.eye(n), torch.zeros(n, n)
    t["l0.mix.q"], t["l0.mix.k"] = torch.cat([torch.cat([eye, none], 1)] * 2), torch.cat([none, eye], 1)
    t["l0.mix.v"], t["l0.mix.o"] = torch.cat([none, eye], 1), torch.cat([torch.cat([eye, none], 1), torch.cat([none, eye], 1)])
    t["l0.mix.q.norm"], t["l0.mix.k.norm"] = torch.full((n,), 1.1), torch.full((n,), 1.1)
    t = {k: v.bfloat16().float() for k, v in t.items()}
    ids, targets = [T + p for p in range(T)], {}
    for p in range(40, T, 3):
        far = [0, 1, 15, 16, 17, 31, 32, 63, 64, 65, p - 1, p - 16, p - 17][(p // 3) % 13]
        if far < p and ids[far] >= T:
            ids[p], targets[p] = ids[far] - T, far
    for p in (44, 80, 161):                                 # and a few questions without an answer
        ids[p] = 3
    assert len(set(targets.values())) > 12
    want = plain.forward(cfg, t, ids)
    for p, far in list(targets.items())[::7]:               # the inputs can tell: without the key the logits are others
        gone = list(ids)
        gone[far] = T + 199
        assert float((plain.forward(cfg, t, gone[: p + 1])[-1] - want[p]).abs().max()) > 0.5
    arch = ModelConfig.from_hf_dict(cfg)
    P = FlatParams(arch, dtype=place[1], device=place[0])
    P.load_hf_state_dict(t)
    for bs in (16, 64):
        eng = RolloutEngine(arch, P, max_num_seqs=2, max_model_len=256, block_size=bs, num_blocks=512 // bs)
        for cuts in ([T], [1], [50, 1], [16], [63, 65, 2]):
            close(feed_all(eng, {"a": ids}, cuts)["a"], want, place, "far", (bs, cuts))


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
    if place[1] == torch.float32:
        assert float(gap.max()) < 1e-3
    else:
        assert float(gap.max()) < 0.5, gap


@pytest.mark.parametrize("name", ["mixed", "odd", "wide", "plain"])
def test_greedy_generation_with_the_scheduler(models, name, place):
    """More requests than slots, unequal prompts and lengths, repeated prompts (prefilled once), slots, pages and cached prefixes
    used again."""
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
    assert eng.stats["prefix_cache_hit_tokens"] > 0
    assert len(eng.free_slots) == 3 and len(eng.free_blocks) + len(eng._idle_cached) == 40


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
