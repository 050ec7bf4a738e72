"""Description of decoders whose layers differ: a list of token mixers and feed-forwards with their own sizes.

A *mixer stack* is a residual decoder in which every layer names its mixer (a kind of attention, a recurrent layer, ...), the
mixer's sizes, and its feed-forward or none; a layer may reuse another layer's weights. Norms sit in front of the sublayers or
on their outputs. The specs below are the typed form of such a configuration; ``DESIGNS`` maps the ``architecture`` of a
``config.json`` to the reader of its keys and is the place to register another design. Sizes and constants all come from the
configuration.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Callable, Optional, Union

__all__ = ["RotarySpec", "LatentAttentionSpec", "GroupedAttentionSpec", "MLstmSpec", "DenseMlpSpec", "GatedMlpSpec", "MoeSpec", "LayerSpec",
           "StackSpec", "DESIGNS", "is_stack_config", "parse_stack"]


@dataclass(frozen=True)
class RotarySpec:
    """Rotary positions: frequencies of ``dims`` dimensions at ``base``, ``pairing`` of the dimensions ("interleaved": 2i with
    2i + 1), and a context extension in the form ``ops.functional.rope_inv_freq`` reads."""

    dims: int
    base: float
    pairing: str = "interleaved"
    scaling: Optional[dict] = None

    def key(self) -> tuple:
        return (self.dims, self.base, tuple(sorted((self.scaling or {}).items())))


@dataclass(frozen=True)
class LatentAttentionSpec:
    """Attention whose keys and values are expanded from one cached latent row per token (``kv_rank`` normed dimensions and
    ``rot_dim`` rotated ones shared by all heads); queries go through a latent of ``q_rank``."""

    heads: int
    dim: int          # unrotated query / key size per head
    rot_dim: int      # rotated query / key size per head
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot: RotarySpec
    window: int = 0   # tokens a query sees, itself included; 0 = all
    kind: str = "latent_attention"

    @property
    def page_width(self) -> int:
        return self.kv_rank + self.rot_dim

    @property
    def state_size(self) -> int:
        return 0


@dataclass(frozen=True)
class GroupedAttentionSpec:
    """Grouped-query attention over cached keys and values: RMS norm per query / key head, rotation of the first ``rot.dims``
    dimensions, optional soft cap of the scores, an optional key of score 0 that has no value, and values mixed with those of
    the stack's first value-mixing layer."""

    heads: int
    kv_heads: int
    dim: int          # query / key size per head
    vdim: int
    scale: float
    rot: RotarySpec
    softcap: float = 0.0      # score = softcap * tanh(score / softcap); 0 = off
    zero_sink: bool = True    # one is added to the softmax denominator
    v_mix: bool = False
    window: int = 0
    kind: str = "attention"

    @property
    def page_width(self) -> int:
        return self.kv_heads * (self.dim + self.vdim)

    @property
    def state_size(self) -> int:
        return 0


@dataclass(frozen=True)
class MLstmSpec:
    """Matrix-memory recurrence with exponential gates: per head a state [dim, vdim], a normaliser [dim] and a running maximum."""

    heads: int
    dim: int
    vdim: int
    gate_cap: float
    kind: str = "mlstm"

    @property
    def page_width(self) -> int:
        return 0

    @property
    def state_size(self) -> int:
        return self.heads * (self.dim * self.vdim + self.dim + 1)


@dataclass(frozen=True)
class DenseMlpSpec:
    ff: int
    act: str = "gelu_erf"
    kind: str = "dense"


@dataclass(frozen=True)
class GatedMlpSpec:
    """``W_down (silu(W_gate h) * (W_up h))``."""

    ff: int
    kind: str = "gated"


@dataclass(frozen=True)
class MoeSpec:
    """Gated experts of which every token uses ``top``: sigmoid scores, the score of a chosen expert scales the expert's input
    (``renormalize``: scores divided by their sum first); a shared expert of ``shared_ff`` (0 = none) is added, multiplied by the
    sigmoid of its own gate."""

    experts: int
    top: int
    ff: int
    shared_ff: int = 0
    renormalize: bool = False
    kind: str = "moe"


@dataclass(frozen=True)
class LayerSpec:
    mixer: Union[LatentAttentionSpec, GroupedAttentionSpec, MLstmSpec]
    mlp: Union[DenseMlpSpec, GatedMlpSpec, MoeSpec, None]
    owner: int        # layer whose tensors this one uses (itself, or an earlier one with shared weights)


@dataclass(frozen=True)
class StackSpec:
    design: str
    embedding_scale: float
    norm: str         # "dynamic_tanh" | "rms"
    norm_eps: float   # eps of the RMS norms
    layers: tuple
    norm_on: str = "input"        # where a sublayer's norm sits: on its "input" or on its "output"
    residual_mult: float = 1.0    # factor on what a sublayer adds to the stream
    embedding_norm: bool = False  # the embedding passes the stack's norm
    tied_head: bool = False       # the output matrix is the embedding table
    logit_softcap: float = 0.0    # 0 = off

    @property
    def recurrent(self) -> bool:
        return any(l.mixer.state_size for l in self.layers)

    @property
    def value_source(self) -> int:
        """First value-mixing layer (-1: none): its values enter the mixes of the later ones."""
        return next((i for i, l in enumerate(self.layers) if getattr(l.mixer, "v_mix", False)), -1)


# --------------------------------------------------------------------------------------------- readers of config.json
def _rotary(d: dict) -> RotarySpec:
    scaling = None
    s = d.get("scaling")
    if s:
        import math

        scaling = {"rope_type": "yarn", "factor": float(s["factor"]), "original_max_position_embeddings": s["original"],
                   "beta_fast": float(s["fast"]), "beta_slow": float(s["slow"]), "attention_factor": 0.1 * math.log(float(s["factor"])) + 1.0}
    return RotarySpec(dims=int(d["dims"]), base=float(d["base"]), scaling=scaling)


def _latent_attention(m: dict) -> LatentAttentionSpec:
    mask = m.get("mask") or {}
    return LatentAttentionSpec(heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]), vdim=int(m["vdim"]), q_rank=int(m["q_rank"]),
                               kv_rank=int(m["kv_rank"]), scale=float(m["scale"]), rot=_rotary(m["rot"]), window=int(mask.get("size") or 0))


def _mlstm(m: dict) -> MLstmSpec:
    return MLstmSpec(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), gate_cap=float(m["gate_cap"]))


def _grouped_attention(m: dict) -> GroupedAttentionSpec:
    spec = GroupedAttentionSpec(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), scale=float(m["scale"]),
                                rot=_rotary(m["rot"]), softcap=float(m.get("softcap") or 0.0), v_mix=bool(m.get("v_mix", False)))
    if spec.heads % spec.kv_heads or spec.rot.dims % 2 or spec.rot.dims > spec.dim:
        raise ValueError(f"attention sizes: {spec}")
    return spec


MIXER_READERS: dict[str, Callable[[dict], Any]] = {"latent_attention": _latent_attention, "mlstm": _mlstm, "attention": _grouped_attention}


def _mlp(d: Optional[dict], gated: bool = False) -> Union[DenseMlpSpec, GatedMlpSpec, MoeSpec, None]:
    if d is None:
        return None
    if d.get("kind") == "dense":
        return GatedMlpSpec(ff=int(d["ff"])) if gated else DenseMlpSpec(ff=int(d["ff"]))
    if d.get("kind") == "moe" and gated:
        r = d["router"]
        return MoeSpec(experts=int(r["experts"]), top=int(r["top"]), ff=int(d["expert"]["ff"]), shared_ff=int((d.get("shared") or {}).get("ff", 0)))
    raise NotImplementedError(f"feed-forward kind {d.get('kind')!r}")


def _owner(layers: list, i: int) -> int:
    seen = set()
    while layers[i].get("weights_of") is not None:
        if i in seen:
            raise ValueError("layers share weights in a circle")
        seen.add(i)
        i = int(layers[i]["weights_of"])
    return i


def _layers(d: dict, mixers: tuple, gated: bool = False) -> tuple:
    layers = []
    for i, l in enumerate(d["layers"]):
        if l["type"] not in mixers:
            raise NotImplementedError(f"mixer type {l['type']!r}")
        layers.append(LayerSpec(mixer=MIXER_READERS[l["type"]](l["mixer"]), mlp=_mlp(l.get("mlp"), gated), owner=_owner(d["layers"], i)))
    return tuple(layers)


def parse_zorelorn(d: dict) -> StackSpec:
    return StackSpec(design="Zorelorn", embedding_scale=float(d["embedding"]["scale"]), norm="dynamic_tanh", norm_eps=float(d["norm"]["eps"]),
                     layers=_layers(d, ("latent_attention", "mlstm")))


def parse_tofinex(d: dict) -> StackSpec:
    spec = StackSpec(design="Tofinex", embedding_scale=1.0, norm="rms", norm_eps=float(d["norm"]["eps"]), layers=_layers(d, ("attention",), gated=True),
                     norm_on="output", residual_mult=float(d["residual_mult"]), embedding_norm=True, tied_head=True,
                     logit_softcap=float(d.get("logit_softcap") or 0.0))
    if len({(l.mixer.kv_heads, l.mixer.vdim) for l in spec.layers if l.mixer.v_mix}) > 1:
        raise ValueError("value-mixing layers need one number of value heads and one value size")
    return spec


DESIGNS: dict[str, Callable[[dict], StackSpec]] = {"Zorelorn": parse_zorelorn, "Tofinex": parse_tofinex}


def is_stack_config(d: dict) -> bool:
    return d.get("architecture") in DESIGNS


def parse_stack(d: dict) -> StackSpec:
    return DESIGNS[d["architecture"]](d)


# --------------------------------------------------------------------------------------------- parameter layout
def _up8(n: int) -> int:
    return (n + 7) // 8 * 8


def norm_tensors(spec: StackSpec, name: str, width: int) -> list:
    """``(name, shape, initialisation, weight decay)`` of one of the stack's norms."""
    if spec.norm == "rms":
        return [(name, (width,), "ones", False)]
    return [(name, (width,), "ones", False), (name + ".b", (width,), "zeros", False), (name + ".alpha", (1,), "fill:0.5", False)]


def model_tensors(spec: StackSpec, width: int, vocab: int) -> tuple:
    """Stored tensors in front of and behind the layers."""
    first = [("embed", (vocab, width), "normal", True)] + (norm_tensors(spec, "embed.norm", width) if spec.embedding_norm else [])
    last = norm_tensors(spec, "final.norm", width) + ([] if spec.tied_head else [("head", (vocab, width), "normal", True)])
    return first, last


def layer_tensors(spec: StackSpec, width: int, i: int) -> list:
    """Stored tensors of layer ``i`` (a weight owner): ``(name, shape, initialisation, weight decay)``. Projections of the same
    input are one matrix; its rows are padded to a multiple of 8."""
    l, p = spec.layers[i], f"l{i}."
    out = norm_tensors(spec, p + "norm1", width)
    m, f = l.mixer, l.mlp
    if m.kind == "latent_attention":
        out += [(p + "mix.in", (m.q_rank + m.kv_rank + m.rot_dim + _up8(m.heads), width), "normal", True),
                (p + "mix.dq.norm", (m.q_rank,), "ones", False), (p + "mix.dkv.norm", (m.kv_rank,), "ones", False),
                (p + "mix.uq", (m.heads * (m.dim + m.rot_dim), m.q_rank), "normal", True),
                (p + "mix.ukv", (m.heads * (m.dim + m.vdim), m.kv_rank), "normal", True),
                (p + "mix.sink", (m.heads,), "zeros", False), (p + "mix.o", (width, m.heads * m.vdim), "normal", True)]
    elif m.kind == "attention":
        out += [(p + "mix.in", (_up8((m.heads + m.kv_heads) * m.dim + m.kv_heads * m.vdim), width), "normal", True),
                (p + "mix.q.norm", (m.dim,), "ones", False), (p + "mix.k.norm", (m.dim,), "ones", False)]
        out += [(p + "mix.vmix", (1,), "fill:0.5", False)] if m.v_mix else []
        out += [(p + "mix.o", (width, m.heads * m.vdim), "normal", True)]
    else:
        out += [(p + "mix.in", (2 * m.heads * (m.dim + m.vdim) + _up8(2 * m.heads), width), "normal", True),
                (p + "mix.i.b", (m.heads,), "zeros", False), (p + "mix.f.b", (m.heads,), "fill:4.0", False),
                (p + "mix.norm", (m.heads * m.vdim,), "ones", False), (p + "mix.o", (width, m.heads * m.vdim), "normal", True)]
    if f is None:
        return out
    out += norm_tensors(spec, p + "norm2", width)
    if f.kind == "dense":
        out += [(p + "mlp.up", (f.ff, width), "normal", True), (p + "mlp.down", (width, f.ff), "normal", True)]
    elif f.kind == "gated":
        out += [(p + "mlp.in", (2 * f.ff, width), "normal", True), (p + "mlp.down", (width, f.ff), "normal", True)]
    else:
        # one matrix for everything that reads every token (shared expert, router, shared gate); the experts' are stacked
        out += [(p + "mlp.in", (2 * f.shared_ff + _up8(f.experts + (1 if f.shared_ff else 0)), width), "normal", True)]
        out += [(p + "mlp.shared.down", (width, f.shared_ff), "normal", True)] if f.shared_ff else []
        out += [(p + "mlp.experts.in", (f.experts * 2 * f.ff, width), "normal", True), (p + "mlp.experts.down", (f.experts * width, f.ff), "normal", True)]
    return out


def _consecutive(*parts) -> list:
    """(name, rows) pairs -> [(name, first row, rows)]"""
    out, at = [], 0
    for name, rows in parts:
        out.append((name, at, rows))
        at += rows
    return out


def fused_rows(spec: StackSpec, width: int, i: int) -> dict:
    """Fused tensor of layer ``i`` -> [(checkpoint name, first row, rows)]."""
    m, f, p = spec.layers[i].mixer, spec.layers[i].mlp, f"l{i}.mix."
    if m.kind == "latent_attention":
        out = {p + "in": _consecutive((p + "dq", m.q_rank), (p + "dkv", m.kv_rank + m.rot_dim), (p + "g", m.heads)),
               p + "ukv": _consecutive((p + "uk", m.heads * m.dim), (p + "uv", m.heads * m.vdim))}
    elif m.kind == "attention":
        out = {p + "in": _consecutive((p + "q", m.heads * m.dim), (p + "k", m.kv_heads * m.dim), (p + "v", m.kv_heads * m.vdim))}
    else:
        qk, v = m.heads * m.dim, m.heads * m.vdim
        out = {p + "in": _consecutive((p + "q", qk), (p + "k", qk), (p + "v", v), (p + "g", v), (p + "i", m.heads), (p + "f", m.heads))}
    p = f"l{i}.mlp."
    if f is not None and f.kind == "gated":
        out[p + "in"] = _consecutive((p + "gate", f.ff), (p + "up", f.ff))
    elif f is not None and f.kind == "moe":
        s = f.shared_ff
        shared = ((p + "shared.gate", s), (p + "shared.up", s)) if s else ()
        out[p + "in"] = _consecutive(*shared, (p + "router", f.experts), *([(p + "shared.sg", 1)] if s else []))
        out[p + "experts.in"] = _consecutive(*((f"{p}e{e}.{part}", f.ff) for e in range(f.experts) for part in ("gate", "up")))
        out[p + "experts.down"] = _consecutive(*((f"{p}e{e}.down", width) for e in range(f.experts)))
    return out


def checkpoint_parts(spec: StackSpec, width: int) -> dict:
    out: dict = {}
    for i, l in enumerate(spec.layers):
        if l.owner == i:
            out.update(fused_rows(spec, width, i))
    return out


def is_scalar(name: str) -> bool:
    """Stored with one element, a scalar in checkpoints."""
    return name.endswith((".alpha", ".vmix"))
