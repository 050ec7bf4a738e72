"""Replay of a token trace through the rollout engine: given tokens in, logits out, nothing sampled.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps.jsonl

``DIR`` holds ``config.json`` and the weights. Every line of standard input is a step: ``{"step": n, "entries": [{"id", "tokens",
"want"}], "end": [ids]}``; the entries are one batch of next tokens. Logits of the wanted places are written to
``OUT/<step>.f32`` (little-endian fp32, [wanted, vocab], in entry order), then ``done <step>`` is printed. Requests listed in
``end`` give their slot and pages back after the step. The steps run through the engine's own prompt and decode paths, cache
and kernels (``RolloutEngine.feed``). ``float32`` keeps weights, activations and cache in 32-bit without reduced-precision
products.
"""

from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np
import torch

__all__ = ["load_engine", "replay", "main"]


def load_engine(model_dir: str, dtype: torch.dtype, max_tokens: int, max_seqs: int = 64, block_size: int = 64, device=None):
    """Rollout engine over the weights of ``model_dir``, its cache sized for ``max_tokens`` live tokens."""
    from ....models import ModelConfig, make_flat_params
    from ....utils.model import load_hf_weights_into
    from .engine import RolloutEngine

    device = device if device is not None else (torch.device("cuda", 0) if torch.cuda.is_available() else torch.device("cpu"))
    cfg = ModelConfig.from_pretrained(model_dir)
    if cfg.is_generic:
        raise NotImplementedError(f"model_type={cfg.model_type!r} runs as a library module without the paged engine")
    if dtype != torch.bfloat16 and device.type == "cuda" and not cfg.is_stack:
        raise NotImplementedError(f"model_type={cfg.model_type!r} has no 32-bit GPU kernels")
    params = make_flat_params(cfg, dtype=dtype, device=device)
    load_hf_weights_into(params, model_dir, strict=True)
    max_tokens = max(int(max_tokens), block_size)
    blocks = -(-max_tokens // block_size) + max_seqs
    return RolloutEngine(cfg, params, max_num_seqs=max_seqs, max_model_len=max_tokens + 1, block_size=block_size, num_blocks=blocks,
                         use_cuda_graph=False)


def replay(engine, lines, out_dir: str, emit=lambda n: None) -> None:
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = [(str(e["id"]), e["tokens"], e.get("want") or []) for e in step["entries"]]
        for key, _, _ in entries:
            if key not in engine.sequences:
                engine.open_sequence(key)
        logits = engine.feed(entries) if entries else []
        rows = [l for l, (_, _, want) in zip(logits, entries) if len(want)]
        if rows:
            data = torch.cat(rows, 0).to("cpu", torch.float32).numpy().astype("<f4")
            tmp = os.path.join(out_dir, f".{step['step']}.part")
            data.tofile(tmp)
            os.replace(tmp, os.path.join(out_dir, f"{step['step']}.f32"))
        elif engine.is_cuda:
            torch.cuda.synchronize(engine.device)
        for key in step.get("end") or []:
            engine.close_sequence(str(key))
        emit(step["step"])


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a token trace through the rollout engine and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and the weights")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits, one <step>.f32 per step with wanted places")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    ap.add_argument("--device", default=None, help="cpu: the plain 32-bit or bf16 path of the CPU tests (default: the GPU when present)")
    a = ap.parse_args(argv)
    torch.backends.cuda.matmul.allow_tf32 = False
    torch.backends.cudnn.allow_tf32 = False
    try:
        engine = load_engine(a.model, getattr(torch, a.dtype), a.max_tokens, device=torch.device(a.device) if a.device else None)
    except NotImplementedError as e:
        print(f"trace_run: {e}", file=sys.stderr)
        return 3

    def emit(n):
        print(f"done {n}", flush=True)

    replay(engine, sys.stdin, a.out, emit)
    if engine.is_cuda:
        from ....ops import native

        native.check_status()
    return 0


if __name__ == "__main__":
    sys.exit(main())
