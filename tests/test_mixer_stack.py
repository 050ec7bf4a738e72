"""Mixer-stack models through the rollout engine: prompts, decoding, portions, batches, reused slots and pages, generation."""

import json
import os
import subprocess
import sys

import pytest
import torch

from oracles import mixer_stack_plain as plain
from stack_testing import PLACES, close, feed_all, tokens
from verl_b200.models import FlatParams, ModelConfig, PackedBatch, build_decoder
from verl_b200.utils.model import load_hf_weights_into, save_hf_weights
from verl_b200.workers.rollout.native.engine import RolloutEngine, SamplingParams

torch.set_num_threads(min(4, torch.get_num_threads()))
REPO = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.fixture(params=PLACES)
def place(request):
    return request.param


def attn(ff=None, heads=2, dim=16, rot_dim=8, vdim=24, q_rank=40, kv_rank=48, window=9, base=900.0, scaling="yarn", scale=0.3, rot_dims=None, **kw):
    rot = {"base": base, "dims": rot_dims or rot_dim}
    if scaling == "yarn":
        rot["scaling"] = {"factor": 3.0, "fast": 8.0, "original": 64, "slow": 1.0}
    return dict(type="latent_attention", mlp=None if ff is None else {"ff": ff, "kind": "dense"},
                mixer=dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, mask={"size": window}, rot=rot, scale=scale), **kw)


def mlstm(ff=None, heads=3, dim=16, vdim=24, gate_cap=7.0, **kw):
    return dict(type="mlstm", mlp=None if ff is None else {"ff": ff, "kind": "dense"}, mixer=dict(heads=heads, dim=dim, vdim=vdim, gate_cap=gate_cap), **kw)


def config(layers, width=56, vocab=96, scale=1.5, eps=1e-5):
    return {"architecture": "Zorelorn", "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


CONFIGS = {
    # every kind of layer, shared weights, with and without feed-forward
    "mixed": config([attn(72), mlstm(), attn(72, weights_of=0), mlstm(40, heads=2, dim=24, vdim=16), attn(None, heads=4, dim=8, rot_dim=16, window=17)]),
    # sizes that are no multiple of 8, one head, a window of one token
    "odd": config([mlstm(heads=1, dim=10, vdim=14), attn(22, heads=3, dim=10, rot_dim=6, vdim=14, q_rank=18, kv_rank=20, window=5, scaling=None), attn(30, window=1)],
                  width=42, vocab=61, scale=0.8),
    # recurrent layers share weights with a later owner; the window passes a page and a chunk
    "wide": config([mlstm(64, heads=2, dim=64, vdim=128, weights_of=2), attn(136, heads=6, dim=72, rot_dim=40, vdim=80, q_rank=88, kv_rank=136, window=65, scale=0.1),
                    mlstm(64, heads=2, dim=64, vdim=128)], width=128, vocab=200),
    # no window limit and partly rotated keys
    "full": config([attn(48, window=None, rot_dim=16, rot_dims=12), mlstm(48)]),
    "attention": config([attn(48, window=6), attn(48, window=40, heads=4)]),
}


def expected_tensors(cfg):
    """Checkpoint names and shapes, written from the format (not from the package)."""
    D, out = cfg["width"], {"embed": (cfg["vocab"], cfg["width"]), "head": (cfg["vocab"], cfg["width"])}

    def norm(name):
        out.update({name: (D,), name + ".b": (D,), name + ".alpha": ()})

    for i, l in enumerate(cfg["layers"]):
        if l.get("weights_of") is not None:
            continue
        m, p = l["mixer"], f"l{i}."
        H = m["heads"]
        norm(p + "norm1")
        if l["type"] == "mlstm":
            out.update({p + "mix.q": (H * m["dim"], D), p + "mix.k": (H * m["dim"], D), p + "mix.v": (H * m["vdim"], D), p + "mix.g": (H * m["vdim"], D),
                        p + "mix.o": (D, H * m["vdim"]), p + "mix.norm": (H * m["vdim"],), p + "mix.i": (H, D), p + "mix.i.b": (H,), p + "mix.f": (H, D), p + "mix.f.b": (H,)})
        else:
            out.update({p + "mix.dq": (m["q_rank"], D), p + "mix.dq.norm": (m["q_rank"],), p + "mix.uq": (H * (m["dim"] + m["rot_dim"]), m["q_rank"]),
                        p + "mix.dkv": (m["kv_rank"] + m["rot_dim"], D), p + "mix.dkv.norm": (m["kv_rank"],), p + "mix.uk": (H * m["dim"], m["kv_rank"]),
                        p + "mix.uv": (H * m["vdim"], m["kv_rank"]), p + "mix.sink": (H,), p + "mix.g": (H, D), p + "mix.o": (D, H * m["vdim"])})
        if l["mlp"] is not None:
            norm(p + "norm2")
            out.update({p + "mlp.up": (l["mlp"]["ff"], D), p + "mlp.down": (D, l["mlp"]["ff"])})
    norm("final.norm")
    return out


def random_tensors(cfg, seed=0):
    g, t = torch.Generator().manual_seed(seed), {}
    for name, shape in expected_tensors(cfg).items():
        x = torch.randn(shape, generator=g)
        if name.endswith(".alpha"):
            x = 0.4 + 0.2 * x.abs()
        elif name.endswith("mix.f.b"):
            x = 2.0 + x
        elif "norm" in name and not name.endswith(".b"):
            x = 1.0 + 0.3 * x
        elif len(shape) == 2 and name != "embed":
            x = x * (2.0 if ".uq" in name or ".uk" in name else 1.2) * shape[1] ** -0.5
        t[name] = x.bfloat16().float()
    return t


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


def want_logits(models, name, tokens):
    key = (name, tuple(tokens))
    if key not in _WANT:
        _WANT[key] = plain.forward(models[name][0], models[name][1], tokens)
    return _WANT[key]


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


def test_missing_tensors_and_unknown_layers_are_errors(models, tmp_path):
    cfg, t, _ = models["mixed"]
    P = FlatParams(ModelConfig.from_hf_dict(cfg), dtype=torch.float32)
    with pytest.raises(KeyError):
        P.load_hf_state_dict({k: v for k, v in t.items() if k != "l1.mix.f"})
    bad = json.loads(json.dumps(cfg))
    bad["layers"][1]["type"] = "convolution"
    with pytest.raises(NotImplementedError):
        ModelConfig.from_hf_dict(bad)
    model = build_decoder(P.cfg, P)
    with pytest.raises(NotImplementedError):
        model.forward_logprobs(PackedBatch.from_lengths(torch.tensor([1, 2]), [2]), torch.tensor([1, 2]), need_grad=True)


# ---------------------------------------------------------------------------------------------- logits
@pytest.mark.parametrize("name", list(CONFIGS))
def test_packed_prompts_without_cache(models, name, place):
    arch, P = load(models, name, place)
    seqs = [tokens(n, n, arch.vocab_size) for n in (1, 2, 30, 131)]
    model = build_decoder(arch, P)
    batch = PackedBatch.from_lengths(torch.tensor(sum(seqs, [])), [len(s) for s in seqs], device=place[0])
    want = torch.cat([want_logits(models, name, s) for s in seqs])
    close(model.forward_logits(batch), want, place)
    labels = torch.randint(0, arch.vocab_size, (want.shape[0],))
    lp, ent = model.forward_logprobs(batch, labels.to(place[0]), 1.0, need_grad=False)
    ref = torch.log_softmax(want, -1)
    tol = 1e-3 if place[1] == torch.float32 else 0.25
    assert float((lp.cpu() - ref.gather(-1, labels[:, None])[:, 0]).abs().max()) < tol
    assert float((ent.cpu() + (ref.exp() * ref).sum(-1)).abs().max()) < tol


@pytest.mark.parametrize("name", list(CONFIGS))
def test_token_by_token_equals_prompt(models, name, place):
    eng = engine(models, name, place)
    t = tokens(90, 3, eng.cfg.vocab_size)
    want = want_logits(models, name, t)
    for cuts in ([90], [1], [40, 1], [2, 1]):
        close(feed_all(eng, {"a": t}, cuts)["a"], want, place, cuts)


@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("cuts", [[2], [3, 2], [16], [17], [33, 1, 16], [64, 5]])
def test_portions(models, name, place, cuts):
    eng = engine(models, name, place)
    seqs = {"a": tokens(100, 5, eng.cfg.vocab_size), "b": tokens(71, 6, eng.cfg.vocab_size)}
    got = feed_all(eng, seqs, cuts)
    for k, t in seqs.items():
        close(got[k], want_logits(models, name, t), place, cuts)


@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
def test_unequal_batches_equal_each_alone(models, name, place):
    eng = engine(models, name, place)
    seqs = {str(n): tokens(n, 10 + n, eng.cfg.vocab_size) for n in (1, 2, 17, 64, 80)}
    for cuts in ([200], [30, 1]):
        together = feed_all(eng, seqs, cuts)
        for k, t in seqs.items():
            alone = feed_all(eng, {k: t}, cuts)[k]
            close(together[k], want_logits(models, name, t), place, (k, cuts))
            close(together[k], alone.double(), place if place[1] == torch.float32 else ("cuda", torch.bfloat16), (k, cuts))


@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_slots_and_pages_used_again(models, name, place):
    """A cache with no room to spare: finished sequences leave full pages and states behind, the next ones must not see them."""
    eng = engine(models, name, place, max_num_seqs=2, num_blocks=12, max_model_len=100)
    for round_ in range(4):
        seqs = {f"{round_}a": tokens(83 - 9 * round_, round_, eng.cfg.vocab_size), f"{round_}b": tokens(20 + 13 * round_, 50 + round_, eng.cfg.vocab_size)}
        got = feed_all(eng, seqs, [[200], [1], [20, 1], [7]][round_])
        for k, t in seqs.items():
            close(got[k], want_logits(models, name, t), place, k)
    assert len(eng.free_blocks) == 12 and len(eng.free_slots) == 2
    with pytest.raises(AssertionError):
        feed_all(eng, {"x": tokens(99, 1, eng.cfg.vocab_size), "y": tokens(98, 2, eng.cfg.vocab_size)}, [200])


@pytest.mark.parametrize("window", [1, 2, 15, 16, 17, 32, 48])
def test_every_window_edge(place, window):
    """One attention layer in which a query token matches exactly one key token: the last one inside its window, or the first one
    outside. A window that is off by one changes the output by its whole size."""
    T, n = 110, 32
    cfg = config([attn(None, heads=1, dim=n, vdim=n, q_rank=n, kv_rank=n, window=window, rot_dim=8, scaling=None, scale=0.5)], width=2 * n, vocab=2 * T)
    t = random_tensors(cfg, 9)
    t["embed"][:T, n:] = 0                                 # token p < T: a query with content p, no key
    t["embed"][T:, :n] = 0
    t["embed"][T:, n:] = t["embed"][:T, :n]                # token T + p: the key with content p
    eye, none = torch.eye(n), torch.zeros(n, n)
    t["l0.norm1"].fill_(1.0), t["l0.norm1.b"].zero_(), t["l0.mix.dq.norm"].fill_(1.0), t["l0.mix.dkv.norm"].fill_(1.0)
    t["l0.mix.dq"], t["l0.mix.dkv"] = torch.cat([eye, none], 1), torch.cat([torch.cat([none, eye], 1), torch.zeros(8, 2 * n)])
    t["l0.mix.uq"], t["l0.mix.uk"] = torch.cat([eye, torch.zeros(8, n)]), eye
    t["l0.mix.g"].zero_()
    ids = [T + p for p in range(T)]
    for p in range(2, T, 3):
        target = p - window + 1 if p % 2 else p - window   # inside / outside
        if 0 <= target < p and ids[target] >= T:
            ids[p] = target
    arch = ModelConfig.from_hf_dict(cfg)
    P = FlatParams(arch, dtype=place[1], device=place[0])
    P.load_hf_state_dict(t)
    eng = RolloutEngine(arch, P, max_num_seqs=2, max_model_len=256, block_size=16, num_blocks=40)
    want = plain.forward(cfg, t, ids)
    for off in (-1, 1):
        other = json.loads(json.dumps(cfg))
        other["layers"][0]["mixer"]["mask"]["size"] = window + off
        if window + off:
            assert float((plain.forward(other, t, ids) - want).abs().max()) > 0.3      # the inputs can tell the difference
    for cuts in ([T], [1], [50, 1], [16]):
        close(feed_all(eng, {"a": ids}, cuts)["a"], want, place, (window, cuts))


def test_long_decoding(models, place):
    eng = engine(models, "mixed", place)
    t = tokens(390, 21, eng.cfg.vocab_size)
    got = feed_all(eng, {"a": t, "b": t[:200]}, [5, 1])
    want = want_logits(models, "mixed", t)
    close(got["a"], want, place)
    close(got["b"], want[:200], place)


# ---------------------------------------------------------------------------------------------- generation
def check_greedy(models, name, prompt, generated, place):
    """Every generated token is the plain model's argmax for its prefix (bf16: within rounding of it)."""
    want = want_logits(models, name, list(prompt) + list(generated))[len(prompt) - 1 : -1]
    chosen = want.gather(-1, torch.tensor(generated)[:, None])[:, 0]
    slack = 1e-3 if place[1] == torch.float32 else 0.15
    assert float((want.max(-1).values - chosen).max()) < slack


@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
def test_greedy_generation_with_the_scheduler(models, name, place):
    """More requests than slots, unequal prompts and lengths, repeated prompts (prefilled once), slots and pages reused."""
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
    assert outs[1].token_ids == outs[5].token_ids == outs[6].token_ids[:12]
    assert len(eng.free_slots) == 3 and len(eng.free_blocks) + len(eng._idle_cached) == 40


def test_sampled_generation_and_log_probs(models, place):
    eng = engine(models, "mixed", place)
    prompt = tokens(21, 4, eng.cfg.vocab_size)
    outs = eng.generate([prompt] * 4, [SamplingParams(temperature=1.0, max_tokens=15, seed=s) for s in (1, 2, 3, 1)])
    assert outs[0].token_ids == outs[3].token_ids and outs[0].token_ids != outs[1].token_ids
    for o in outs:
        want = torch.log_softmax(want_logits(models, "mixed", prompt + o.token_ids)[len(prompt) - 1 : -1], -1)
        lp = want.gather(-1, torch.tensor(o.token_ids)[:, None])[:, 0]
        assert float((lp - torch.tensor(o.log_probs)).abs().max()) < (1e-3 if place[1] == torch.float32 else 0.25)


def test_prefill_decode_handoff_carries_the_state(models, place):
    pre, dec = engine(models, "mixed", place), engine(models, "mixed", place)
    prompts = [tokens(n, n, pre.cfg.vocab_size) for n in (9, 34)]
    sp = SamplingParams(temperature=0.0, max_tokens=14)
    hand = pre.prefill_only(prompts, sp)
    assert len(pre.free_slots) == 5 and not pre.running
    for i, h in enumerate(hand):
        dec.add_prefilled(h, sp, f"r{i}")
    got = {}
    while len(got) < 2:
        got.update({o.request_id: o.token_ids for o in dec.step()})
    for i, p in enumerate(prompts):
        check_greedy(models, "mixed", p, got[f"r{i}"], place)


def test_cache_release_and_abort(models, place):
    eng = engine(models, "mixed", place)
    prompt = tokens(12, 8, eng.cfg.vocab_size)
    first = eng.generate([prompt], SamplingParams(temperature=0.0, max_tokens=10))[0].token_ids
    eng.release_kv_cache()
    assert eng.kv is None and eng.cache.states is None
    eng.resume_kv_cache()
    eng.add_request(prompt, SamplingParams(temperature=0.0, max_tokens=200))
    eng.step()
    eng.abort()
    eng.step()
    assert eng.generate([prompt], SamplingParams(temperature=0.0, max_tokens=10))[0].token_ids == first


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

    cfg, _, path = models["mixed"]
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
    a, b = want_logits(models, "mixed", seqs["a"]), want_logits(models, "mixed", seqs["b"])
    close(read(0), a[[0, 19]], place)
    assert not (tmp_path / "1.f32").exists()
    close(read(2), torch.stack([a[21], b[10]]), place)
    close(read(10), a[[29]], place)
