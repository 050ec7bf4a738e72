"""What the model tests of the mixer stacks share: places to run, token lists, comparison of logits, feeding an engine."""

import pytest
import torch

PLACES = [pytest.param(("cpu", torch.float32), id="cpu-fp32"),
          pytest.param(("cuda", torch.float32), id="cuda-fp32", marks=pytest.mark.gpu),
          pytest.param(("cuda", torch.bfloat16), id="cuda-bf16", marks=pytest.mark.gpu)]


def tokens(n, seed, vocab):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def position_errors(got, want):
    """Root-mean-square error over the vocabulary, relative to the logits' spread, of every position."""
    got, want = got.detach().cpu().double(), want.double()
    spread = (want - want.mean(-1, keepdim=True)).pow(2).mean().sqrt()
    d = got - want
    return (d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / spread


def close(got, want, place, what=""):
    err = position_errors(got, want)
    limit = 1e-4 if place[1] == torch.float32 else 0.06
    assert float(err.max()) < limit, (what, float(err.max()), int(err.argmax()))


def feed_all(eng, seqs, cuts, keep_open=False):
    """Feed the token lists in portions of the given sizes (last size repeats); logits of every position per sequence."""
    for k in seqs:
        eng.open_sequence(k)
    at, out = {k: 0 for k in seqs}, {k: [] for k in seqs}
    step = 0
    while any(at[k] < len(t) for k, t in seqs.items()):
        n = cuts[min(step, len(cuts) - 1)]
        entries = [(k, t[at[k] : at[k] + n], list(range(min(n, len(t) - at[k])))) for k, t in seqs.items() if at[k] < len(t)]
        for (k, part, _), l in zip(entries, eng.feed(entries)):
            out[k].append(l.cpu())
            at[k] += len(part)
        step += 1
    if not keep_open:
        for k in seqs:
            eng.close_sequence(k)
    return {k: torch.cat(v) for k, v in out.items()}
