"""Serving benchmark of a mixer-stack design beside the closest uniform decoder of equal size (same width, layers and parameters).

    python bench.py --design zorelorn            # all sizes: prefill and decode throughput of both models
    python bench.py --design zorelorn --kernels  # the kernels behind them, each against its roofline
    python bench.py --design tofinex [--kernels]
    python bench.py --design luzitar [--kernels]
    python bench.py --design fusazen [--kernels]

Random weights and tokens. Prefill runs packed prompts through the engine's prompt path into the cache, decode replays the
captured decode step over all slots; CUDA events around every timed region, after warm-up, on inputs larger than L2. One
JSON line per measurement.
"""

from __future__ import annotations

import gc
import json

import torch

from ....models import DecoderModel, FlatParams, ModelConfig
from ....ops import functional as F
from ....ops import mixers as X
from ....ops import native
from ....ops.bench_kernels import Timer, _peaks
from ....utils.profiler.clocks import ClockSampler
from .engine import RolloutEngine

SIZES = {  # name -> (width, heads, q_rank, window, ff, layers, prompts, prompt length, decode slots, decode context)
    "width2048": dict(width=2048, heads=16, q_rank=768, window=1024, ff=8192, layers=16, prompts=8, prompt_len=2048, slots=256, ctx=2048),
    "width4096": dict(width=4096, heads=32, q_rank=1536, window=4096, ff=16384, layers=8, prompts=4, prompt_len=4096, slots=128, ctx=4096),
}
VOCAB = 32768
# experts = 0: dense feed-forwards of size ff; else every layer has ``experts`` of size ff, ``top`` per token, and a shared one
TOFINEX_SIZES = {
    "dense2048": dict(width=2048, heads=16, kv_heads=4, ff=8192, experts=0, top=0, shared_ff=0, layers=12, prompts=8, prompt_len=2048, slots=256, ctx=2048),
    "moe2048": dict(width=2048, heads=16, kv_heads=4, ff=768, experts=64, top=6, shared_ff=1536, layers=8, prompts=8, prompt_len=2048, slots=256, ctx=2048),
    "moe4096": dict(width=4096, heads=32, kv_heads=8, ff=1536, experts=32, top=2, shared_ff=3072, layers=4, prompts=4, prompt_len=4096, slots=128, ctx=4096),
}
# layers in turn: lightning, windowed attention, latent attention, latent attention over the rows of the one before; experts everywhere
LUZITAR_SIZES = {
    "moe2048": dict(width=2048, heads=16, kv_heads=4, window=1024, keep=64, ff=768, experts=64, top=6, groups=8, group_keep=4, layers=8, prompts=8, prompt_len=2048, slots=256,
                    ctx=2048),
    "moe2048-long": dict(width=2048, heads=16, kv_heads=4, window=1024, keep=64, ff=768, experts=64, top=6, groups=8, group_keep=4, layers=8, prompts=1, prompt_len=16384, slots=32,
                         ctx=16384),
    "moe4096": dict(width=4096, heads=32, kv_heads=8, window=2048, keep=64, ff=1536, experts=32, top=2, groups=4, group_keep=2, layers=4, prompts=4, prompt_len=4096, slots=128,
                    ctx=4096),
}

# layers in turn: delta rule, differential attention, attention with norms over whole projections, differential attention over the rows of the one
# before; the decode steps run at the end of a chunk
FUSAZEN_SIZES = {
    "dense2048": dict(width=2048, heads=16, kv_heads=4, delta_dim=64, rank=64, chunk=1024, ff=8192, layers=12, prompts=8, prompt_len=2048, slots=256, ctx=2016),
    "dense2048-long": dict(width=2048, heads=16, kv_heads=4, delta_dim=64, rank=64, chunk=8192, ff=8192, layers=12, prompts=1, prompt_len=16384, slots=32, ctx=16352),
    "dense4096": dict(width=4096, heads=32, kv_heads=8, delta_dim=128, rank=128, chunk=2048, ff=16384, layers=8, prompts=4, prompt_len=4096, slots=128, ctx=4064),
}


def zorelorn_config(s: dict) -> ModelConfig:
    attn = dict(type="latent_attention", mlp={"kind": "dense", "ff": s["ff"]},
                mixer=dict(heads=s["heads"], dim=128, rot_dim=64, vdim=128, q_rank=s["q_rank"], kv_rank=512, mask={"size": s["window"]}, scale=192 ** -0.5,
                           rot=dict(base=500000.0, dims=64, scaling=dict(factor=8.0, original=8192, fast=32.0, slow=1.0))))
    mlstm = dict(type="mlstm", mlp=None, mixer=dict(heads=s["heads"] // 2, dim=128, vdim=256, gate_cap=15.0))
    return ModelConfig.from_hf_dict({"architecture": "Zorelorn", "embedding": {"scale": 1.0}, "norm": {"eps": 1e-6}, "vocab": VOCAB, "width": s["width"],
                                     "layers": [attn if i % 2 == 0 else mlstm for i in range(s["layers"])]})


def uniform_config(s: dict, params: int) -> ModelConfig:
    """Llama-type decoder of the same width and number of layers; its MLP is sized so that the parameters agree."""
    mk = lambda ff: ModelConfig(model_type="llama", vocab_size=VOCAB, hidden_size=s["width"], intermediate_size=ff, num_hidden_layers=s["layers"],
                                num_attention_heads=s["width"] // 128, num_key_value_heads=max(1, s["width"] // 512), head_dim=128, rope_theta=500000.0,
                                max_position_embeddings=8192)
    return mk(max(256, round((params - mk(0).num_parameters()) / (3 * s["width"] * s["layers"]) / 256) * 256))


def tofinex_config(s: dict) -> ModelConfig:
    mlp = {"kind": "dense", "ff": s["ff"]}
    if s["experts"]:
        mlp = {"kind": "moe", "expert": {"ff": s["ff"]}, "router": {"experts": s["experts"], "top": s["top"]}, "shared": {"ff": s["shared_ff"]}}
    mixer = dict(heads=s["heads"], kv_heads=s["kv_heads"], dim=128, vdim=128, scale=128 ** -0.5, softcap=30.0, v_mix=True, rot=dict(base=500000.0, dims=128))
    return ModelConfig.from_hf_dict({"architecture": "Tofinex", "logit_softcap": 20.0, "norm": {"eps": 1e-6}, "residual_mult": 0.5, "vocab": VOCAB, "width": s["width"],
                                     "layers": [{"type": "attention", "mixer": mixer, "mlp": mlp}] * s["layers"]})


def closest_to_tofinex(s: dict, params: int) -> ModelConfig:
    """Qwen-type decoder with the same attention sizes, query / key norms and feed-forwards (softmax router, shared expert)."""
    moe = s["experts"] > 0
    kw = dict(num_experts=s["experts"], num_experts_per_tok=s["top"], moe_intermediate_size=s["ff"], shared_expert_intermediate_size=s["shared_ff"]) if moe else {}
    return ModelConfig(model_type="qwen2_moe" if moe else "qwen3", vocab_size=VOCAB, hidden_size=s["width"], intermediate_size=s["ff"], num_hidden_layers=s["layers"],
                       num_attention_heads=s["heads"], num_key_value_heads=s["kv_heads"], head_dim=128, rope_theta=500000.0, max_position_embeddings=8192,
                       qk_norm=True, attention_bias=False, tie_word_embeddings=True, **kw)


def luzitar_config(s: dict) -> ModelConfig:
    H, layers = s["heads"], []
    mlp = {"kind": "moe", "expert": {"ff": s["ff"], "limit": 7.0},
           "router": {"experts": s["experts"], "top": s["top"], "groups": {"count": s["groups"], "keep": s["group_keep"]}}}
    latent = dict(heads=H, dim=128, rot_dim=64, vdim=128, kv_rank=512, scale=192 ** -0.5, rot=dict(base=500000.0, dims=64))
    for i in range(0, s["layers"], 4):
        layers += [("lightning", dict(heads=H, dim=128, vdim=128, decay=[1.0 - 2.0 ** (-2.0 - 6.0 * h / H) for h in range(H)])),
                   ("attention", dict(heads=H, kv_heads=s["kv_heads"], dim=128, vdim=128, conv=4, scale=128 ** 0.5, mask={"size": s["window"], "keep_first": s["keep"]},
                                      rot=dict(base=500000.0, dims=64, scaling=dict(factor=8.0, original=8192, fast=32.0, slow=1.0)))),
                   ("latent_attention", latent), ("latent_attention", {**latent, "kv_from": i + 2})]
    return ModelConfig.from_hf_dict({"architecture": "Luzitar", "logit_softcap": 20.0, "norm": {"eps": 1e-6}, "vocab": VOCAB, "width": s["width"],
                                     "layers": [{"type": t, "mixer": m, "mlp": mlp} for t, m in layers[: s["layers"]]]})


def closest_to_luzitar(s: dict, params: int) -> ModelConfig:
    """Qwen3-MoE-type decoder: full attention of the same head sizes in every layer, the same experts (softmax router)."""
    return ModelConfig(model_type="qwen3_moe", vocab_size=VOCAB, hidden_size=s["width"], intermediate_size=s["ff"], num_hidden_layers=s["layers"],
                       num_attention_heads=s["heads"], num_key_value_heads=s["kv_heads"], head_dim=128, rope_theta=500000.0, max_position_embeddings=1 << 15, qk_norm=True,
                       attention_bias=False, tie_word_embeddings=False, num_experts=s["experts"], num_experts_per_tok=s["top"], moe_intermediate_size=s["ff"])


def fusazen_config(s: dict) -> ModelConfig:
    H, G, layers = s["heads"], s["kv_heads"], []
    two = dict(heads=H, kv_heads=G, dim=64, vdim=128, diff=0.5, scale=64 ** -0.5, mask={"size": s["chunk"]}, rot=dict(base=500000.0, dims=64))
    for i in range(0, s["layers"], 4):
        layers += [("general_delta", dict(heads=s["width"] // s["delta_dim"], dim=s["delta_dim"], decay_rank=s["rank"])), ("attention", two),
                   ("attention_2", dict(heads=H, kv_heads=G, dim=128, vdim=128, scale=128 ** -0.5, mask={"size": s["chunk"]})), ("attention", {**two, "kv_from": i + 1})]
    return ModelConfig.from_hf_dict({"architecture": "Fusazen", "canon": {"taps": 4}, "embedding": {"scale": 1.0}, "norm": {"eps": 1e-6}, "vocab": VOCAB, "width": s["width"],
                                     "layers": [{"type": t, "mixer": m, "mlp": {"kind": "dense", "ff": s["ff"]}} for t, m in layers[: s["layers"]]]})


def closest_to_fusazen(s: dict, params: int) -> ModelConfig:
    """Qwen3-type decoder: full attention of the same head sizes in every layer; its MLP is sized so that the parameters agree."""
    mk = lambda ff: ModelConfig(model_type="qwen3", vocab_size=VOCAB, hidden_size=s["width"], intermediate_size=ff, num_hidden_layers=s["layers"], num_attention_heads=s["heads"],
                                num_key_value_heads=s["kv_heads"], head_dim=128, rope_theta=500000.0, max_position_embeddings=1 << 15, qk_norm=True, attention_bias=False,
                                tie_word_embeddings=False)
    return mk(max(256, round((params - mk(0).num_parameters()) / (3 * s["width"] * s["layers"]) / 256) * 256))


# design -> (sizes, its configuration, label and configuration of the closest existing model)
DESIGNS = {"zorelorn": (SIZES, zorelorn_config, "uniform decoder of equal size", uniform_config),
           "tofinex": (TOFINEX_SIZES, tofinex_config, "closest existing decoder", closest_to_tofinex),
           "luzitar": (LUZITAR_SIZES, luzitar_config, "closest existing decoder", closest_to_luzitar),
           "fusazen": (FUSAZEN_SIZES, fusazen_config, "closest existing decoder", closest_to_fusazen)}


def _events(fn, steps: int) -> float:
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    torch.cuda.synchronize()
    a.record()
    for _ in range(steps):
        fn()
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) / steps


def bench_model(cfg: ModelConfig, s: dict, steps: int, warmup: int) -> dict:
    dev = torch.device("cuda", torch.cuda.current_device())
    P = FlatParams(cfg, dtype=torch.bfloat16, device=dev)
    P.init_weights(seed=1, std=0.02)
    bs, S, n, L = 64, s["slots"], s["prompts"], s["prompt_len"]
    per = -(-(s["ctx"] + 64) // bs)
    eng = RolloutEngine(cfg, P, max_num_seqs=S, max_model_len=per * bs, block_size=bs, num_blocks=S * per, eos_token_id=-1)
    ids = torch.randint(0, VOCAB, (n * L,))
    table = torch.arange(S * per, dtype=torch.int32).view(S, per)

    def prefill():
        h, batch = eng._run_portions(ids, [0] * n, [L] * n, table[:n], list(range(n)))
        return eng._logits(h[batch.cu_seqlens[1:].long() - 1].contiguous())

    for _ in range(warmup):
        prefill()
    sampler = ClockSampler(dev.index or 0, period_s=0.02).start()
    ms_p = _events(prefill, steps)
    eng.block_table.copy_(table)
    for t, v in ((eng.tok, 5), (eng.pos, s["ctx"]), (eng.ctx, s["ctx"] + 1), (eng.gen, 1), (eng.max_new, 1 << 20)):
        t.fill_(v)
    eng.active.fill_(True)
    eng.ignore_eos.fill_(True)
    eng._ensure_out(64)
    eng._decode_steps(warmup)
    n0 = native.launch_count()
    ms_d = _events(lambda: eng._decode_steps(1), 16)
    launches = (native.launch_count() - n0) // 16
    clocks = sampler.stop()
    native.check_status()
    out = {"parameters": cfg.num_parameters(), "prefill_tokens_per_s": round(n * L / ms_p * 1e3), "prefill_ms": round(ms_p, 3),
           "decode_tokens_per_s": round(S / ms_d * 1e3), "decode_ms_per_step": round(ms_d, 3), "decode_kernels_per_step": launches, "clocks": clocks}
    del eng, P
    gc.collect()
    torch.cuda.empty_cache()
    return out


def run_models(design: str, steps: int, warmup: int, only=None) -> None:
    sizes, make, other, make_other = DESIGNS[design]
    for name, s in sizes.items():
        if only and name not in only:
            continue
        z = make(s)
        for label, cfg in ((design, z), (other, make_other(s, z.num_parameters()))):
            r = bench_model(cfg, s, steps, max(3, warmup))
            print(json.dumps({"bench": "serving", "size": name, "model": label, "intermediate_size": cfg.intermediate_size, **s, **r, "dtype": "bf16",
                              "data": "synthetic (random weights and tokens)"}), flush=True)


# --------------------------------------------------------------------------------------------- kernels
def _kernel_reporter(design: str, other: str, timer, only):
    pk = _peaks()

    def case(size, phase, kernel, fn, flops, nbytes, new):
        if only and kernel not in only:
            return
        ms = timer(fn)
        floor = max(flops / (pk["bf16_tflops"] * 1e9), nbytes / (pk["hbm_gbs"] * 1e6))
        print(json.dumps({"bench": "kernel", "size": size, "phase": phase, "kernel": kernel, "design": design if new else other, "us": round(ms * 1e3, 2),
                          "roofline_us": round(floor * 1e3, 2), "fraction_of_measured": round(floor / ms, 3), "bound": "flops" if flops / pk["bf16_tflops"] > nbytes / pk["hbm_gbs"] * 1e3 else "bytes",
                          "clocks": timer.clocks}), flush=True)

    return case


def run_kernels(iters: int = 20, only=None, sizes=None) -> None:
    dev = torch.device("cuda", torch.cuda.current_device())
    timer = Timer(dev, iters, 3)
    r = lambda *sh, sc=1.0, dt=torch.bfloat16: (torch.randn(*sh, device=dev) * sc).to(dt)
    case = _kernel_reporter("zorelorn", "uniform decoder", timer, only)

    for name, s in SIZES.items():
        if sizes and name not in sizes:
            continue
        W, H, qr, ff, w = s["width"], s["heads"], s["q_rank"], s["ff"], s["window"]
        Hm, d, e, kr, rot, dim, vd = H // 2, 128, 256, 512, 64, 128, 128
        for phase, T in (("prefill", s["prompts"] * s["prompt_len"]), ("decode", s["slots"])):
            h, x = r(T, W), torch.randn(T, W, device=dev)
            norm = (r(1), r(W), r(W))
            cut = qr + kr + rot
            w_in, w_up, w_down, w_o = r(cut + H, W, sc=0.02), r(ff, W, sc=0.02), r(W, ff, sc=0.02), r(W, H * vd, sc=0.02)
            act, att = r(T, ff), r(T, H * vd)
            mm = lambda m, n, k: (2.0 * m * n * k, 2.0 * (m * k + n * k + m * n))
            f, b = mm(T, cut + H, W)
            case(name, phase, "linear_split (latent input projections)", lambda: X.linear_split(h, w_in, cut), f, b, True)
            f, b = mm(T, ff, W)
            case(name, phase, "linear_act (up projection + gelu)", lambda: X.linear_act(h, w_up, "gelu_erf"), f, b, True)
            case(name, phase, "gemm (same product, no epilogue)", lambda: F.gemm(h, w_up), f, b, False)
            f, b = mm(T, W, ff)
            case(name, phase, "linear_residual (down projection + residual + norm)", lambda: X.linear_residual_(act, w_down, x, norm), f, b + 8.0 * T * W, True)
            case(name, phase, "gemm (same product, no epilogue, K deep)", lambda: F.gemm(act, w_down), f, b, False)
            f, b = mm(T, W, H * vd)
            case(name, phase, "linear_residual (output projection + residual + norm)", lambda: X.linear_residual_(att, w_o, x, norm), f, b + 8.0 * T * W, True)
            case(name, phase, "gemm (output projection)", lambda: F.gemm(att, w_o), f, b, False)
            y = r(T, W)
            case(name, phase, "rmsnorm with residual", lambda: F.rms_norm(h, norm[1], 1e-6, residual=y), 0, 8.0 * T * W, False)
            cos, sin = F.rope_table(8192, rot, 5e5, dev)
            pos = torch.arange(T, device=dev, dtype=torch.int32) % 4096
            p, qn, kn = r(T, cut), r(qr), r(kr)
            case(name, phase, "latent_prep (norms, rotation, rows)", lambda: X.latent_prep(p, qn, kn, 1e-6, pos, cos, sin, None, None, True), 0, 4.0 * T * cut, True)
            q = r(T, H, dim + rot)
            if phase == "prefill":
                case(name, phase, "rope_pairs (query rotation)", lambda: X.rope_pairs_(q, pos, cos, sin, dim), 0, 4.0 * T * H * rot, True)
                c = r(T, 128)
                cs2, sn2 = F.rope_table(8192, 128, 5e5, dev)
                qf = r(T, H, 128)
                case(name, phase, "rope (query rotation, uniform)", lambda: F.apply_rope_(qf, pos, cs2, sn2), 0, 4.0 * T * H * 128, False)
                n, L = s["prompts"], s["prompt_len"]
                cu = (torch.arange(n + 1, device=dev, dtype=torch.int32) * L)
                kv, rows, sink, gate = r(T, H * (dim + vd)), r(T, kr + rot), r(H), torch.randn(T, H, device=dev)
                ku, v = kv[:, : H * dim].view(T, H, dim), kv[:, H * dim :].view(T, H, vd)
                pairs = n * sum(min(i + 1, w) for i in range(L))
                case(name, phase, "latent_attention_prefill", lambda: X.latent_attention_prefill(q, ku, rows[:, kr:], v, cu, cu, w, 192 ** -0.5, sink, gate),
                     2.0 * pairs * H * (dim + rot + vd), 2.0 * T * (H * (dim + rot + dim + 2 * vd) + rot), True)
                nkv = max(1, W // 512)
                qq, kk, vv = r(T, W // 128, 128), r(T, nkv, 128), r(T, nkv, 128)
                case(name, phase, "attention_varlen (uniform, causal)", lambda: F.attention_varlen(qq, kk, vv, cu, L), 4.0 * n * L * (L + 1) / 2 * (W // 128) * 128,
                     2.0 * T * (2 * W + 2 * nkv * 128), False)
            else:
                S, ctx, bs = s["slots"], s["ctx"], 64
                per = -(-(ctx + 64) // bs)
                pages = r(S * per, bs, kr + rot, sc=0.5)
                table = torch.arange(S * per, device=dev, dtype=torch.int32).view(S, per)
                cl = torch.full((S,), ctx, device=dev, dtype=torch.int32)
                qa, sink, uk, uv, oc, gate = r(S, H, kr + rot), r(H), r(H, dim, kr), r(H, vd, kr), r(S, H, kr), torch.randn(S, H, device=dev)
                seen = min(ctx, w)
                case(name, phase, "latent_attention_decode", lambda: X.latent_attention_decode(qa, pages, table, cl, kr, w, 192 ** -0.5, sink),
                     2.0 * S * seen * H * (2 * kr + rot), 2.0 * S * seen * (kr + rot) + 2.0 * S * H * (2 * kr + rot), True)
                nkv = max(1, W // 512)
                kc, vc = r(S * per, bs, nkv, 128, sc=0.5), r(S * per, bs, nkv, 128, sc=0.5)
                qd = r(S, W // 128, 128)
                case(name, phase, "paged_decode_attention (uniform)", lambda: F.paged_decode_attention(qd, kc, vc, table, cl), 4.0 * S * ctx * W, 4.0 * S * ctx * nkv * 128, False)
                case(name, phase, "latent_absorb (query into latent space)", lambda: X.latent_absorb(q, uk, pos, cos, sin), 2.0 * S * H * dim * kr,
                     2.0 * (S * H * (dim + rot) + H * dim * kr + S * H * (kr + rot)), True)
                case(name, phase, "headwise_linear (values out of latent space + gate)", lambda: X.headwise_linear(oc, uv, False, gate), 2.0 * S * H * vd * kr,
                     2.0 * (S * H * kr + H * vd * kr + S * H * vd), True)
                del pages, kc, vc
            pm, gates, bias, nm = r(T, 2 * Hm * (d + e)), torch.randn(T, 2 * Hm, device=dev), r(Hm), r(Hm * e)
            io = 2.0 * T * (2 * Hm * (d + e) + Hm * e) + 8.0 * T * Hm
            if phase == "prefill":
                C = 64
                case(name, phase, "mlstm_prefill", lambda: X.mlstm_prefill(pm, gates, bias, bias, 15.0, nm, 1e-6, d, cu), 2.0 * T * Hm * (C / 2 * (d + e) + 2 * d * e), io, True)
            else:
                st = torch.zeros(T, Hm * (d * e + d + 1), device=dev)
                act_ = torch.ones(T, dtype=torch.bool, device=dev)
                case(name, phase, "mlstm_decode (step, norm, gate)", lambda: X.mlstm_decode(pm, gates, bias, bias, 15.0, nm, 1e-6, d, st, act_), 0, io + 8.0 * T * Hm * d * e, True)
            torch.cuda.empty_cache()
    native.check_status()


def run_tofinex_kernels(iters: int = 20, only=None, sizes=None) -> None:
    dev = torch.device("cuda", torch.cuda.current_device())
    timer = Timer(dev, iters, 3)
    r = lambda *sh, sc=1.0, dt=torch.bfloat16: (torch.randn(*sh, device=dev) * sc).to(dt)
    case = _kernel_reporter("tofinex", "closest decoder", timer, only)
    mm = lambda m, n, k: (2.0 * m * n * k, 2.0 * (m * k + n * k + m * n))
    for name, s in TOFINEX_SIZES.items():
        if sizes and name not in sizes:
            continue
        W, H, G, ff, E, top, sff, d = s["width"], s["heads"], s["kv_heads"], s["ff"], s["experts"], s["top"], s["shared_ff"], 128
        qkv, Q, scale, cap = (H + 2 * G) * d, H * d, d ** -0.5, 30.0
        cos, sin = F.rope_table(8192, d, 5e5, dev)
        nw, qn, kn, lam = r(W), r(d), r(d), r(1)
        for phase, T in (("prefill", s["prompts"] * s["prompt_len"]), ("decode", s["slots"])):
            h, x, att, res = r(T, W), torch.randn(T, W, device=dev), r(T, Q), r(T, W)
            w_in, w_o = r(qkv, W, sc=0.02), r(W, Q, sc=0.02)
            pos = torch.arange(T, device=dev, dtype=torch.int32) % 4096
            f, b = mm(T, qkv, W)
            case(name, phase, "linear_act (query, key and value projection)", lambda: X.linear_act(h, w_in), f, b, True)
            case(name, phase, "gemm (same product)", lambda: F.gemm(h, w_in), f, b, False)
            f, b = mm(T, W, Q)
            case(name, phase, "linear_partial (output projection)", lambda: X.linear_partial(att, w_o), f, b, True)
            case(name, phase, "gemm (output projection)", lambda: F.gemm(att, w_o), f, b, False)
            y = X.linear_partial(att, w_o)
            case(name, phase, "residual_rms (partial products, norm, residual, next input)", lambda: X.residual_rms_(x, y, nw, 1e-6, 0.5), 0,
                 y.numel() * y.element_size() + 10.0 * T * W, True)
            case(name, phase, "rmsnorm with residual", lambda: F.rms_norm(h, nw, 1e-6, residual=res), 0, 8.0 * T * W, False)
            p, first = r(T, qkv), r(T, G * d)
            case(name, phase, "qkv_prep (norms, rotation, value mix, rows)", lambda: X.qkv_prep(p, qn, kn, 1e-6, pos, cos, sin, H, G, d, first, lam, None, None, True), 0,
                 4.0 * T * qkv + 2.0 * T * G * d, True)
            q, k, v = r(T, H, d), r(T, G, d), r(T, G, d)
            case(name, phase, "rope (query rotation)", lambda: F.apply_rope_(q, pos, cos, sin), 0, 4.0 * T * Q, False)
            if phase == "prefill":
                n, L = s["prompts"], s["prompt_len"]
                cu = torch.arange(n + 1, device=dev, dtype=torch.int32) * L
                sink = torch.zeros(H, device=dev, dtype=torch.bfloat16)
                fl, by = 4.0 * n * L * (L + 1) / 2 * Q, 2.0 * T * (2 * Q + 2 * G * d)
                case(name, phase, "grouped_attention_prefill (capped scores, sink)", lambda: X.grouped_attention_prefill(q, k, v, cu, cu, 0, scale, cap, sink), fl, by, True)
                case(name, phase, "attention_varlen", lambda: F.attention_varlen(q, k, v, cu, L), fl, by, False)
            else:
                S, ctx, bs = s["slots"], s["ctx"], 64
                per = -(-(ctx + 64) // bs)
                pages, kc, vc = r(S * per, bs, 2 * G * d, sc=0.5), r(S * per, bs, G, d, sc=0.5), r(S * per, bs, G, d, sc=0.5)
                table = torch.arange(S * per, device=dev, dtype=torch.int32).view(S, per)
                cl = torch.full((S,), ctx, device=dev, dtype=torch.int32)
                sink = torch.zeros(H, device=dev, dtype=torch.bfloat16)
                fl, by = 4.0 * S * ctx * Q, 4.0 * S * ctx * G * d
                case(name, phase, "grouped_attention_decode (capped scores, sink)", lambda: X.grouped_attention_decode(q, pages, table, cl, G, d, 0, scale, cap, sink), fl, by, True)
                case(name, phase, "paged_decode_attention", lambda: F.paged_decode_attention(q, kc, vc, table, cl), fl, by, False)
                del pages, kc, vc
            if not E:
                w_gu, w_d, a = r(2 * ff, W, sc=0.02), r(W, ff, sc=0.02), r(T, ff)
                f, b = mm(T, 2 * ff, W)
                case(name, phase, "gated_up (gate, up, activation)", lambda: X.gated_up(h, w_gu), f, b - 2.0 * T * ff, True)
                case(name, phase, "gemm_swiglu", lambda: F.gemm_swiglu(h, w_gu)[0], f, b - 2.0 * T * ff, False)
                f, b = mm(T, W, ff)
                case(name, phase, "linear_partial (down projection)", lambda: X.linear_partial(a, w_d), f, b, True)
                case(name, phase, "gemm (down projection)", lambda: F.gemm(a, w_d), f, b, False)
                del w_gu, w_d, a
            else:
                w_m = r(2 * sff + -(-(E + 1) // 8) * 8, W, sc=0.02)
                w_u, w_dn = r(E * 2 * ff, W, sc=0.02), r(E * W, ff, sc=0.02)
                f, b = mm(T, w_m.shape[0], W)
                case(name, phase, "gated_up_split (shared expert, router, gate)", lambda: X.gated_up_split(h, w_m, 2 * sff), f, b - 2.0 * T * sff, True)
                w_gu, w_r = w_m[: 2 * sff].contiguous(), w_m[2 * sff :].contiguous()
                case(name, phase, "gemm_swiglu + router gemm", lambda: (F.gemm_swiglu(h, w_gu)[0], F.gemm(h, w_r)), f, b - 2.0 * T * sff, False)
                z = torch.randn(T, E + 8, device=dev)
                zb = z[:, :E].to(torch.bfloat16).contiguous()
                rows, used = T * top, min(E, T * top)
                by = 4.0 * T * E + 2.0 * T * W + 2.0 * rows * W
                case(name, phase, "expert_dispatch (route, place, copy)", lambda: X.expert_dispatch(h, z, E, top), 0, by, True)
                ops = native.ops()

                def route_other():
                    wts, idx, counts = ops.moe_route_topk(zb, top, False)
                    plan = DecoderModel._moe_plan(idx.long(), counts, T, top, E)
                    return plan, ops.moe_gather_rows(h, plan["src"], None), wts

                case(name, phase, "moe_route_topk + plan + gather_rows", route_other, 0, by, False)
                plan = X.expert_dispatch(h, z, E, top)
                act = X.expert_up(plan, w_u, ff)
                oplan, xp, wts = route_other()
                w3, d3 = w_u.view(E, 2 * ff, W), w_dn.view(E, W, ff)
                fl, by = 2.0 * rows * 2 * ff * W, 2.0 * (used * 2 * ff * W + rows * (W + ff))
                case(name, phase, "expert_up (gate, up, score, activation)", lambda: X.expert_up(plan, w_u, ff), fl, by, True)
                case(name, phase, "gemm_grouped_rows + swiglu", lambda: F.swiglu(ops.gemm_grouped_rows(xp, w3, False, oplan["tile_expert"], oplan["num_mtiles"])), fl, by, False)
                a2 = r(xp.shape[0], ff)
                fl, by = 2.0 * rows * ff * W, 2.0 * (used * ff * W + rows * (W + ff))
                case(name, phase, "expert_down", lambda: X.expert_down(act, w_dn, plan), fl, by, True)
                case(name, phase, "gemm_grouped_rows (down)", lambda: ops.gemm_grouped_rows(a2, d3, False, oplan["tile_expert"], oplan["num_mtiles"]), fl, by, False)
                out = X.expert_down(act, w_dn, plan)
                case(name, phase, "residual_rms (experts, gated shared part, norm, residual)", lambda: X.residual_rms_(x, h, nw, 1e-6, 0.5, None, (out, plan.slot), z[:, E]), 0,
                     2.0 * rows * W + 12.0 * T * W, True)
                yo = ops.gemm_grouped_rows(a2, d3, False, oplan["tile_expert"], oplan["num_mtiles"])
                case(name, phase, "moe_combine", lambda: ops.moe_combine(yo, oplan["slot"], wts), 0, 2.0 * rows * W + 2.0 * T * W, False)
                del w_m, w_u, w_dn, plan, act, xp, a2, out, yo
            ids, emb = torch.randint(0, VOCAB, (T,), device=dev), r(VOCAB, W)
            case(name, phase, "embed_rms", lambda: X.embed_rms(ids, emb, 1.0, nw, 1e-6), 0, 8.0 * T * W, True)
            case(name, phase, "embedding", lambda: F.embedding(ids, emb), 0, 4.0 * T * W, False)
            if phase == "decode":
                f, b = mm(T, VOCAB, W)
                case(name, phase, "linear_softcap (logits)", lambda: X.linear_softcap(h, emb, 20.0), f, b, True)
                case(name, phase, "gemm (logits)", lambda: F.gemm(h, emb), f, b, False)
            del emb
            torch.cuda.empty_cache()
    native.check_status()


def run_luzitar_kernels(iters: int = 20, only=None, sizes=None) -> None:
    dev = torch.device("cuda", torch.cuda.current_device())
    timer = Timer(dev, iters, 3)
    r = lambda *sh, sc=1.0, dt=torch.bfloat16: (torch.randn(*sh, device=dev) * sc).to(dt)
    case = _kernel_reporter("luzitar", "closest decoder", timer, only)
    mm = lambda m, n, k: (2.0 * m * n * k, 2.0 * (m * k + n * k + m * n))
    ops = native.ops()
    for name, s in LUZITAR_SIZES.items():
        if sizes and name not in sizes:
            continue
        W, H, G, E, top, ff, win, keep, d = s["width"], s["heads"], s["kv_heads"], s["experts"], s["top"], s["ff"], s["window"], s["keep"], 128
        Q, qkv, kr, rot, scale = H * d, (H + 2 * G) * d, 512, 64, 192 ** -0.5
        cos, sin = F.rope_table(1 << 15, d, 5e5, dev)
        cos2, sin2 = F.rope_table(1 << 15, rot, 5e5, dev)
        norm, post, nw = (r(1), r(W), r(W)), (r(1), r(W), r(W)), r(W)
        for phase, T in (("prefill", s["prompts"] * s["prompt_len"]), ("decode", s["slots"])):
            h, x, att = r(T, W), torch.randn(T, W, device=dev), r(T, Q)
            n, L, S, ctx, bs = s["prompts"], s["prompt_len"], s["slots"], s["ctx"], 64
            pos = torch.arange(T, device=dev, dtype=torch.int32) % L if phase == "prefill" else torch.full((T,), ctx, device=dev, dtype=torch.int32)
            cu = torch.arange(n + 1, device=dev, dtype=torch.int32) * L
            active = torch.ones(S, dtype=torch.bool, device=dev)
            table, cl = None, None
            if phase == "decode":
                per = -(-(ctx + 64) // bs)
                table = torch.arange(S * per, device=dev, dtype=torch.int32).view(S, per)
                cl = torch.full((S,), ctx, device=dev, dtype=torch.int32)
            # ---- attention of the closest model, the like kernel of every mixer
            q, k, v = r(T, H, d), r(T, G, d), r(T, G, d)
            if phase == "prefill":
                case(name, phase, "attention_varlen", lambda: F.attention_varlen(q, k, v, cu, L), 4.0 * n * L * (L + 1) / 2 * Q, 2.0 * T * (2 * Q + 2 * G * d), False)
            else:
                kc, vc = r(S * per, bs, G, d, sc=0.5), r(S * per, bs, G, d, sc=0.5)
                case(name, phase, "paged_decode_attention", lambda: F.paged_decode_attention(q, kc, vc, table, cl), 4.0 * S * ctx * Q, 4.0 * S * ctx * G * d, False)
                del kc, vc
            case(name, phase, "rope (query rotation)", lambda: F.apply_rope_(q, pos, cos, sin), 0, 4.0 * T * Q, False)
            case(name, phase, "rmsnorm with residual", lambda: F.rms_norm(h, nw, 1e-6, residual=att[:, :W].contiguous() if Q != W else att), 0, 8.0 * T * W, False)
            # ---- lightning
            w = r(4 * Q, W, sc=0.02)
            f, b = mm(T, 4 * Q, W)
            case(name, phase, "linear_silu (q, k, v with silu, g)", lambda: X.linear_silu(h, w, 3 * Q), f, b, True)
            case(name, phase, "gemm (q, k, v, g)", lambda: F.gemm(h, w), f, b, False)
            p, nm = r(T, 4 * Q, sc=0.5), r(Q)
            decay = torch.tensor([1.0 - 2.0 ** (-2.0 - 6.0 * i / H) for i in range(H)], device=dev)
            state = torch.zeros(max(n, S), H * d * d, device=dev)
            if phase == "prefill":
                slots, fresh = torch.arange(n, device=dev, dtype=torch.int32), torch.ones(n, device=dev, dtype=torch.int32)
                case(name, phase, "lightning_prefill", lambda: X.lightning_prefill(p, decay, d, d, cu, state, slots, fresh, True), 2.0 * T * H * (64 / 2 * 2 * d + 2 * d * d),
                     8.0 * T * Q + 4.0 * n * H * d * d, True)
            else:
                case(name, phase, "lightning_decode", lambda: X.lightning_decode(p, decay, d, d, state, active), 0, 8.0 * T * Q + 8.0 * T * H * d * d, True)
            case(name, phase, "gated_rms (norm of all heads, gate)", lambda: X.gated_rms(att, p[:, 3 * Q :], nm, 1e-6), 0, 6.0 * T * Q, True)
            del w, p, state
            # ---- windowed attention with convolved projections
            w, bias = r(qkv, W, sc=0.02), r(qkv)
            f, b = mm(T, qkv, W)
            case(name, phase, "linear_bias (q, k, v)", lambda: X.linear_bias(h, w, bias), f, b, True)
            case(name, phase, "gemm (q, k, v)", lambda: F.gemm(h, w), f, b, False)
            p, conv, state = r(T, qkv), r(qkv, 4, sc=0.5), torch.zeros(max(n, S), 3 * qkv, device=dev)
            if phase == "prefill":
                kw = dict(cu=cu, state=state, slots=slots, fresh=fresh, want_rows=True)
                by = 4.0 * T * qkv + 12.0 * n * qkv
            else:
                kw, by = dict(active=active, state=state, want_rows=True), 4.0 * T * qkv + 24.0 * T * qkv
            case(name, phase, "conv_qkv_prep (convolution, rotation, norms, rows)", lambda: X.conv_qkv_prep(p, conv, 1e-6, pos, cos2, sin2, H, G, d, d, True, **kw), 0, by, True)
            if phase == "prefill":
                pairs = n * sum(min(i + 1, win) + max(0, min(keep, i + 1 - win)) for i in range(L))
                case(name, phase, "grouped_attention_prefill (window, kept tokens)", lambda: X.grouped_attention_prefill(q, k, v, cu, cu, win, scale, 0.0, None, keep), 4.0 * pairs * Q,
                     2.0 * T * (2 * Q + 2 * G * d), True)
            else:
                pages, seen = r(S * per, bs, 2 * G * d, sc=0.5), min(ctx, win + keep)
                case(name, phase, "grouped_attention_decode (window, kept tokens)", lambda: X.grouped_attention_decode(q, pages, table, cl, G, d, win, scale, 0.0, None, keep),
                     4.0 * S * seen * Q, 4.0 * S * seen * G * d, True)
                del pages
                few = -(-seen // bs)
                kc, vc, ct = r(S * few, bs, G, d, sc=0.5), r(S * few, bs, G, d, sc=0.5), torch.arange(S * few, device=dev, dtype=torch.int32).view(S, few)
                case(name, phase, "paged_decode_attention (as many keys)", lambda: F.paged_decode_attention(q, kc, vc, ct, cl.clamp(max=seen)), 4.0 * S * seen * Q, 4.0 * S * seen * G * d,
                     False)
                del kc, vc, ct
            del w, p, state
            # ---- latent attention
            cut = H * (d + rot)
            w = r(cut + kr + rot, W, sc=0.02)
            f, b = mm(T, cut + kr + rot, W)
            case(name, phase, "linear_act (queries, latents)", lambda: X.linear_act(h, w), f, b, True)
            case(name, phase, "gemm (queries, latents)", lambda: F.gemm(h, w), f, b, False)
            p, kn = r(T, cut + kr + rot), r(kr)
            case(name, phase, "latent_prep (norm, rotation, rows)", lambda: X.latent_prep(p[:, cut:], None, kn, 1e-6, pos, cos2, sin2, None, None, True), 0, 4.0 * T * (kr + rot), True)
            ql = p[:, :cut].unflatten(1, (H, d + rot))
            if phase == "prefill":
                case(name, phase, "rope_pairs (query rotation)", lambda: X.rope_pairs_(ql, pos, cos2, sin2, d), 0, 4.0 * T * H * rot, True)
                rows, wkv = r(T, kr + rot), r(2 * Q, kr, sc=0.05)
                f, b = mm(T, 2 * Q, kr)
                case(name, phase, "linear_act (keys and values of the latents)", lambda: X.linear_act(rows[:, :kr], wkv), f, b, True)
                rc = rows[:, :kr].contiguous()
                case(name, phase, "gemm (keys and values of the latents)", lambda: F.gemm(rc, wkv), f, b, False)
                kv = r(T, 2 * Q)
                ku, vl = kv[:, :Q].view(T, H, d), kv[:, Q:].view(T, H, d)
                case(name, phase, "latent_attention_prefill", lambda: X.latent_attention_prefill(ql, ku, rows[:, kr:], vl, cu, cu, 0, scale), 2.0 * n * L * (L + 1) / 2 * H * (2 * d + rot),
                     2.0 * T * (H * (2 * d + rot + 2 * d) + rot), True)
                del rows, kv, ku, vl, wkv, rc
            else:
                pages, qa, uk, uv, oc = r(S * per, bs, kr + rot, sc=0.5), r(S, H, kr + rot), r(H, d, kr), r(H, d, kr), r(S, H, kr)
                case(name, phase, "latent_attention_decode", lambda: X.latent_attention_decode(qa, pages, table, cl, kr, 0, scale), 2.0 * S * ctx * H * (2 * kr + rot),
                     2.0 * S * ctx * (kr + rot) + 2.0 * S * H * (2 * kr + rot), True)
                case(name, phase, "latent_absorb (query into latent space)", lambda: X.latent_absorb(ql, uk, pos, cos2, sin2), 2.0 * S * H * d * kr,
                     2.0 * (S * H * (d + rot) + H * d * kr + S * H * (kr + rot)), True)
                case(name, phase, "headwise_linear (values out of latent space)", lambda: X.headwise_linear(oc, uv, False), 2.0 * S * H * d * kr,
                     2.0 * (S * H * kr + H * d * kr + S * H * d), True)
                del pages, qa, uk, uv, oc
            del w, p, ql
            # ---- output projection, experts
            w = r(W, Q, sc=0.02)
            f, b = mm(T, W, Q)
            case(name, phase, "linear_residual (output projection, both norms, residual)", lambda: X.linear_residual_(att, w, x, norm, post), f, b + 8.0 * T * W, True)
            case(name, phase, "gemm (output projection)", lambda: F.gemm(att, w), f, b, False)
            w, corr = r(E, W, sc=0.02), r(E)
            f, b = mm(T, E, W)
            case(name, phase, "linear_act (router, fp32)", lambda: X.linear_act(h, w, out_f32=True), f, b + 2.0 * T * E, True)
            case(name, phase, "gemm (router)", lambda: F.gemm(h, w), f, b, False)
            z = torch.randn(T, E, device=dev)
            zb, rows = z.to(torch.bfloat16), T * top
            used, by = min(E, rows), 4.0 * T * E + 2.0 * T * W + 2.0 * rows * W
            case(name, phase, "expert_dispatch (groups, route, place, copy)", lambda: X.expert_dispatch(h, z, E, top, True, corr, s["groups"], s["group_keep"]), 0, by, True)

            def route_other():
                wts, idx, counts = ops.moe_route_topk(zb, top, False)
                plan = DecoderModel._moe_plan(idx.long(), counts, T, top, E)
                return plan, ops.moe_gather_rows(h, plan["src"], None), wts

            case(name, phase, "moe_route_topk + plan + gather_rows", route_other, 0, by, False)
            w_u, w_d = r(E * 2 * ff, W, sc=0.02), r(E * W, ff, sc=0.02)
            plan = X.expert_dispatch(h, z, E, top, True, None, 1, 1)      # the same choices as the other router's
            oplan, xp, wts = route_other()
            w3, d3 = w_u.view(E, 2 * ff, W), w_d.view(E, W, ff)
            fl, by = 2.0 * rows * 2 * ff * W, 2.0 * (used * 2 * ff * W + rows * (W + ff))
            case(name, phase, "expert_up (gate, up, clipped activation, score)", lambda: X.expert_up(plan, w_u, ff, "clipped", 7.0), fl, by, True)
            case(name, phase, "gemm_grouped_rows + swiglu", lambda: F.swiglu(ops.gemm_grouped_rows(xp, w3, False, oplan["tile_expert"], oplan["num_mtiles"])), fl, by, False)
            act = X.expert_up(plan, w_u, ff, "clipped", 7.0)
            a2 = r(xp.shape[0], ff)
            fl, by = 2.0 * rows * ff * W, 2.0 * (used * ff * W + rows * (W + ff))
            case(name, phase, "expert_down", lambda: X.expert_down(act, w_d, plan), fl, by, True)
            case(name, phase, "gemm_grouped_rows (down)", lambda: ops.gemm_grouped_rows(a2, d3, False, oplan["tile_expert"], oplan["num_mtiles"]), fl, by, False)
            out = X.expert_down(act, w_d, plan)
            case(name, phase, "residual_dyt (experts, both norms, residual)", lambda: X.residual_dyt_(x, out, plan.slot, post, norm), 0, 2.0 * rows * W + 10.0 * T * W, True)
            yo = ops.gemm_grouped_rows(a2, d3, False, oplan["tile_expert"], oplan["num_mtiles"])
            case(name, phase, "moe_combine", lambda: ops.moe_combine(yo, oplan["slot"], wts), 0, 2.0 * rows * W + 2.0 * T * W, False)
            del w, w_u, w_d, plan, act, xp, a2, out, yo
            ids, emb = torch.randint(0, VOCAB, (T,), device=dev), r(VOCAB, W)
            case(name, phase, "embed_dyt2 (embedding, its norm, first norm)", lambda: X.embed_dyt2(ids, emb, post, norm), 0, 8.0 * T * W, True)
            case(name, phase, "embedding", lambda: F.embedding(ids, emb), 0, 4.0 * T * W, False)
            if phase == "decode":
                f, b = mm(T, VOCAB, W)
                case(name, phase, "linear_softcap (logits)", lambda: X.linear_softcap(h, emb, 20.0), f, b, True)
                case(name, phase, "gemm (logits)", lambda: F.gemm(h, emb), f, b, False)
            del emb, h, x, att, q, k, v
            torch.cuda.empty_cache()
    native.check_status()


def run_fusazen_kernels(iters: int = 20, only=None, sizes=None) -> None:
    """The like kernels are those of the closest decoder; those of the delta rule the lightning recurrence's."""
    dev = torch.device("cuda", torch.cuda.current_device())
    timer = Timer(dev, iters, 3)
    r = lambda *sh, sc=1.0, dt=torch.bfloat16: (torch.randn(*sh, device=dev) * sc).to(dt)
    case = _kernel_reporter("fusazen", "like kernel", timer, only)
    mm = lambda m, n, k: (2.0 * m * n * k, 2.0 * (m * k + n * k + m * n))
    for name, s in FUSAZEN_SIZES.items():
        if sizes and name not in sizes:
            continue
        W, H, G, dd, rank, chunk, ff = (s[k] for k in ("width", "heads", "kv_heads", "delta_dim", "rank", "chunk", "ff"))
        HD, d, e, taps = W // dd, 64, 128, 4
        Q, scale = H * e, d ** -0.5
        cos, sin = F.rope_table(1 << 15, 64, 5e5, dev)
        cos2, sin2 = F.rope_table(1 << 15, 128, 5e5, dev)
        nw, conv = r(W), r(W, taps, sc=0.4)
        for phase, T in (("prefill", s["prompts"] * s["prompt_len"]), ("decode", s["slots"])):
            pre = phase == "prefill"
            n, L, S, ctx, bs = s["prompts"], s["prompt_len"], s["slots"], s["ctx"], 64
            h, x, att = r(T, W), torch.randn(T, W, device=dev), r(T, Q)
            pos = torch.arange(T, device=dev, dtype=torch.int32) % L if pre else torch.full((T,), ctx, device=dev, dtype=torch.int32)
            cu = torch.arange(n + 1, device=dev, dtype=torch.int32) * L
            slots, fresh = torch.arange(n, device=dev, dtype=torch.int32), torch.ones(n, device=dev, dtype=torch.int32)
            active = torch.ones(S, dtype=torch.bool, device=dev)
            seen = ctx % chunk + 1                    # keys a step sees at position ctx
            per = -(-(ctx + 64) // bs)
            table = torch.arange(S * per, device=dev, dtype=torch.int32).view(S, per) if not pre else None
            cl = torch.full((S,), ctx + 1, device=dev, dtype=torch.int32)
            pairs = n * (sum(i % chunk + 1 for i in range(L)))
            # ---- stream
            ids, emb = torch.randint(0, VOCAB, (T,), device=dev), r(VOCAB, W)
            case(name, phase, "embed_rows", lambda: X.embed_rows(ids, emb, 1.0), 0, 6.0 * T * W, True)
            case(name, phase, "embedding", lambda: F.embedding(ids, emb), 0, 4.0 * T * W, False)
            state = torch.zeros(max(n, S), (taps - 1) * W, device=dev)
            if pre:
                case(name, phase, "rms_conv (norm, convolution)", lambda: X.rms_conv(x, nw, 1e-6, conv=conv, cu=cu, state=state, slots=slots, fresh=fresh), 0,
                     6.0 * T * W + 4.0 * n * (taps - 1) * W, True)
                case(name, phase, "rms_conv (norm)", lambda: X.rms_conv(x, nw, 1e-6), 0, 6.0 * T * W, True)
            else:
                y, bias = X.linear_partial(att, r(W, Q, sc=0.02)), r(W)
                planes = 4.0 * y.numel() if y.dim() == 3 else 2.0 * y.numel()
                case(name, phase, "rms_conv (partial products, norm, convolution)", lambda: X.rms_conv(x, nw, 1e-6, y, bias, conv, state=state, active=active), 0,
                     10.0 * T * W + planes + 8.0 * T * (taps - 1) * W, True)
                case(name, phase, "rms_conv (partial products, norm)", lambda: X.rms_conv(x, nw, 1e-6, y), 0, 10.0 * T * W + planes, True)
                del y
            res = r(T, W)
            case(name, phase, "rmsnorm with residual", lambda: F.rms_norm(h, nw, 1e-6, residual=res), 0, 8.0 * T * W, False)
            # ---- delta rule
            rows = 5 * W + rank
            w = r(rows, W, sc=0.02)
            f, b = mm(T, rows, W)
            case(name, phase, "linear_tanh (r, k, v, a, g, decay)", lambda: X.linear_tanh(h, w, 5 * W), f, b, True)
            case(name, phase, "gemm (r, k, v, a, g, decay)", lambda: F.gemm(h, w), f, b, False)
            p, w2 = r(T, rows), r(W, rank, sc=0.1)
            f, b = mm(T, W, rank)
            case(name, phase, "linear_act (decay, few columns)", lambda: X.linear_act(p[:, 5 * W :], w2), f, b, True)
            pc = p[:, 5 * W :].contiguous()
            case(name, phase, "gemm (decay, few columns)", lambda: F.gemm(pc, w2), f, b, False)
            zw, ab, w0, nm = r(T, W), r(W), r(W), r(W)
            mem = torch.zeros(max(n, S), W * dd, device=dev)
            decay = torch.tensor([1.0 - 2.0 ** (-2.0 - 6.0 * i / HD) for i in range(HD)], device=dev)
            if pre:
                case(name, phase, "delta_prefill", lambda: X.delta_prefill(p, zw, ab, w0, HD, cu, mem, slots, fresh), 10.0 * T * W * dd, 12.0 * T * W + 4.0 * n * W * dd, True)
                case(name, phase, "lightning_prefill", lambda: X.lightning_prefill(p, decay, dd, dd, cu, mem, slots, fresh, True), 4.0 * T * W * dd, 8.0 * T * W + 4.0 * n * W * dd, False)
                case(name, phase, "gated_rms (norm of every head, gate)", lambda: X.gated_rms(h, p[:, 4 * W : 5 * W], nm, 1e-6, HD), 0, 6.0 * T * W, True)
            else:
                case(name, phase, "delta_decode (with norm and gate)", lambda: X.delta_decode(p, zw, ab, w0, HD, nm, 1e-6, mem, active), 0, 14.0 * T * W + 8.0 * T * W * dd, True)
                case(name, phase, "lightning_decode", lambda: X.lightning_decode(p, decay, dd, dd, mem, active), 0, 8.0 * T * W + 8.0 * T * W * dd, False)
            del w, p, pc, zw, mem, w2
            # ---- differential attention
            vec = r(4 * d, sc=0.05)
            diff = (vec, 0.5, 1e-6)
            cols = 2 * H * d + G * (2 * d + e)
            w = r(cols, W, sc=0.02)
            f, b = mm(T, cols, W)
            case(name, phase, "linear_act (query and key maps, values)", lambda: X.linear_act(h, w), f, b, True)
            case(name, phase, "gemm (query and key maps, values)", lambda: F.gemm(h, w), f, b, False)
            p = r(T, cols)
            kw = dict(cu=cu) if pre else dict(active=active)
            case(name, phase, "conv_qkv_prep (rotation of the maps, rows)", lambda: X.conv_qkv_prep(p, None, 0.0, pos, cos, sin, 2 * H, 2 * G, d, e, True, want_rows=True, norm=False, v_heads=G,
                                                                                                     **kw), 0, 4.0 * T * cols, True)
            pq = r(T, 2 * H * d)
            case(name, phase, "conv_qkv_prep (rotation of the query maps alone)", lambda: X.conv_qkv_prep(pq, None, 0.0, pos, cos, sin, 2 * H, 0, d, e, True, norm=False, v_heads=0, **kw), 0,
                 8.0 * T * H * d, True)
            q = r(T, H, e)
            case(name, phase, "rope (query rotation)", lambda: F.apply_rope_(q, pos, cos2, sin2), 0, 4.0 * T * Q, False)
            k, v, q2, k2 = r(T, G, e), r(T, G, e), r(T, 2 * H, d), r(T, 2 * G, d)
            if pre:
                case(name, phase, "grouped_attention_prefill (differential)", lambda: X.grouped_attention_prefill(q2, k2, v, cu, cu, 0, scale, chunk=chunk, diff=diff),
                     4.0 * pairs * H * (d + e), 2.0 * T * (H * (2 * d + e) + G * (2 * d + e)), True)
                case(name, phase, "attention_varlen", lambda: F.attention_varlen(q, k, v, cu, L), 4.0 * n * L * (L + 1) / 2 * Q, 2.0 * T * (2 * Q + 2 * G * e), False)
            else:
                pages = r(S * per, bs, 2 * G * e, sc=0.5)
                case(name, phase, "grouped_attention_decode (differential)", lambda: X.grouped_attention_decode(q2, pages, table, cl, G, e, 0, scale, chunk=chunk, diff=diff),
                     4.0 * S * seen * H * (d + e), 2.0 * S * seen * G * (2 * d + e), True)
                few = -(-seen // bs)
                kc, vc, ct = r(S * few, bs, G, e, sc=0.5), r(S * few, bs, G, e, sc=0.5), torch.arange(S * few, device=dev, dtype=torch.int32).view(S, few)
                case(name, phase, "paged_decode_attention (as many keys)", lambda: F.paged_decode_attention(q, kc, vc, ct, cl.clamp(max=seen)), 4.0 * S * seen * Q, 4.0 * S * seen * G * e, False)
                del kc, vc, ct
            # ---- attention with norms over whole projections
            cols = (H + 2 * G) * e
            w, p, qn, kn, temp = r(cols, W, sc=0.02), r(T, cols), r(Q), r(G * e), r(H)
            f, b = mm(T, cols, W)
            case(name, phase, "linear_act (q, k, v)", lambda: X.linear_act(h, w), f, b, True)
            case(name, phase, "gemm (q, k, v)", lambda: F.gemm(h, w), f, b, False)
            case(name, phase, "whole_norm_prep (norms, rows)", lambda: X.whole_norm_prep(p, qn, kn, temp, 1e-6, H, G, e, want_rows=True), 0, 4.0 * T * cols, True)
            if pre:
                case(name, phase, "grouped_attention_prefill (chunks)", lambda: X.grouped_attention_prefill(q, k, v, cu, cu, 0, scale, chunk=chunk), 4.0 * pairs * Q, 2.0 * T * (2 * Q + 2 * G * e),
                     True)
            else:
                case(name, phase, "grouped_attention_decode (chunks)", lambda: X.grouped_attention_decode(q, pages, table, cl, G, e, 0, scale, chunk=chunk), 4.0 * S * seen * Q,
                     4.0 * S * seen * G * e, True)
                del pages
            del w, p, q, k, v, q2, k2, pq
            # ---- output projection, feed-forward
            wo, wu, wd, bu, bd, act = r(W, Q, sc=0.02), r(ff, W, sc=0.02), r(W, ff, sc=0.02), r(ff), r(W), r(T, ff)
            for label, a, w, bias in (("output projection", att, wo, None), ("down projection", act, wd, bd)):
                f, b = mm(T, W, a.shape[1])
                if pre:
                    case(name, phase, f"linear_residual ({label})", lambda: X.linear_residual_(a, w, x, bias=bias), f, b + 6.0 * T * W, True)
                else:
                    case(name, phase, f"linear_partial ({label})", lambda: X.linear_partial(a, w), f, b, True)
                case(name, phase, f"gemm ({label})", lambda: F.gemm(a, w), f, b, False)
            f, b = mm(T, ff, W)
            case(name, phase, "linear_bias (up projection, squared relu)", lambda: X.linear_bias(h, wu, bu, "relu2"), f, b, True)
            case(name, phase, "gemm (up projection)", lambda: F.gemm(h, wu), f, b, False)
            if not pre:
                f, b = mm(T, VOCAB, W)
                case(name, phase, "linear_act (logits)", lambda: X.linear_act(h, emb), f, b, True)
                case(name, phase, "gemm (logits)", lambda: F.gemm(h, emb), f, b, False)
            del wo, wu, wd, act, emb, h, x, att, res
            torch.cuda.empty_cache()
    native.check_status()


def main(args) -> None:
    native.load()
    if args.kernels:
        {"zorelorn": run_kernels, "tofinex": run_tofinex_kernels, "luzitar": run_luzitar_kernels, "fusazen": run_fusazen_kernels}[args.design]()
    else:
        run_models(args.design, args.steps if args.steps > 2 else 5, args.warmup)
