"""Description of decoders whose layers differ: a list of token mixers and feed-forwards with their own sizes.

A *mixer stack* is a pre-norm residual decoder in which every layer names its mixer (a kind of attention, a recurrent layer,
...), the mixer's sizes, and its feed-forward or none; a layer may reuse another layer's weights. The specs below are the
typed form of such a configuration; ``DESIGNS`` maps the ``architecture`` of a ``config.json`` to the reader of its keys and
is the place to register another design. Sizes and constants all come from the configuration.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Callable, Optional, Union

__all__ = ["RotarySpec", "LatentAttentionSpec", "MLstmSpec", "DenseMlpSpec", "LayerSpec", "StackSpec", "DESIGNS", "is_stack_config",
           "parse_stack"]


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
class LayerSpec:
    mixer: Union[LatentAttentionSpec, MLstmSpec]
    mlp: Optional[DenseMlpSpec]
    owner: int        # layer whose tensors this one uses (itself, or an earlier one with shared weights)


@dataclass(frozen=True)
class StackSpec:
    design: str
    embedding_scale: float
    norm: str         # "dynamic_tanh"
    norm_eps: float   # eps of the RMS norms inside the mixers
    layers: tuple

    @property
    def recurrent(self) -> bool:
        return any(l.mixer.state_size for l in self.layers)


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


MIXER_READERS: dict[str, Callable[[dict], Any]] = {"latent_attention": _latent_attention, "mlstm": _mlstm}


def _mlp(d: Optional[dict]) -> Optional[DenseMlpSpec]:
    if d is None:
        return None
    if d.get("kind") != "dense":
        raise NotImplementedError(f"feed-forward kind {d.get('kind')!r}")
    return DenseMlpSpec(ff=int(d["ff"]))


def _owner(layers: list, i: int) -> int:
    seen = set()
    while layers[i].get("weights_of") is not None:
        if i in seen:
            raise ValueError("layers share weights in a circle")
        seen.add(i)
        i = int(layers[i]["weights_of"])
    return i


def parse_zorelorn(d: dict) -> StackSpec:
    layers = []
    for i, l in enumerate(d["layers"]):
        if l["type"] not in MIXER_READERS:
            raise NotImplementedError(f"mixer type {l['type']!r}")
        layers.append(LayerSpec(mixer=MIXER_READERS[l["type"]](l["mixer"]), mlp=_mlp(l.get("mlp")), owner=_owner(d["layers"], i)))
    return StackSpec(design="Zorelorn", embedding_scale=float(d["embedding"]["scale"]), norm="dynamic_tanh", norm_eps=float(d["norm"]["eps"]),
                     layers=tuple(layers))


DESIGNS: dict[str, Callable[[dict], StackSpec]] = {"Zorelorn": parse_zorelorn}


def is_stack_config(d: dict) -> bool:
    return d.get("architecture") in DESIGNS


def parse_stack(d: dict) -> StackSpec:
    return DESIGNS[d["architecture"]](d)


# --------------------------------------------------------------------------------------------- parameter layout
def _up8(n: int) -> int:
    return (n + 7) // 8 * 8


def layer_tensors(spec: StackSpec, width: int, i: int) -> list:
    """Stored tensors of layer ``i`` (a weight owner): ``(name, shape, initialisation, weight decay)``. Projections of the same
    input are one matrix; its rows are padded to a multiple of 8."""
    l, p, out = spec.layers[i], f"l{i}.", []

    def norm(name):
        out.extend([(p + name, (width,), "ones", False), (p + name + ".b", (width,), "zeros", False), (p + name + ".alpha", (1,), "fill:0.5", False)])

    norm("norm1")
    m = l.mixer
    if m.kind == "latent_attention":
        out += [(p + "mix.in", (m.q_rank + m.kv_rank + m.rot_dim + _up8(m.heads), width), "normal", True),
                (p + "mix.dq.norm", (m.q_rank,), "ones", False), (p + "mix.dkv.norm", (m.kv_rank,), "ones", False),
                (p + "mix.uq", (m.heads * (m.dim + m.rot_dim), m.q_rank), "normal", True),
                (p + "mix.ukv", (m.heads * (m.dim + m.vdim), m.kv_rank), "normal", True),
                (p + "mix.sink", (m.heads,), "zeros", False), (p + "mix.o", (width, m.heads * m.vdim), "normal", True)]
    else:
        out += [(p + "mix.in", (2 * m.heads * (m.dim + m.vdim) + _up8(2 * m.heads), width), "normal", True),
                (p + "mix.i.b", (m.heads,), "zeros", False), (p + "mix.f.b", (m.heads,), "fill:4.0", False),
                (p + "mix.norm", (m.heads * m.vdim,), "ones", False), (p + "mix.o", (width, m.heads * m.vdim), "normal", True)]
    if l.mlp is not None:
        norm("norm2")
        out += [(p + "mlp.up", (l.mlp.ff, width), "normal", True), (p + "mlp.down", (width, l.mlp.ff), "normal", True)]
    return out


def fused_rows(spec: StackSpec, i: int) -> dict:
    """Fused tensor of layer ``i`` -> [(checkpoint name, first row, rows)]."""
    m, p = spec.layers[i].mixer, f"l{i}.mix."
    if m.kind == "latent_attention":
        a, b = m.q_rank, m.q_rank + m.kv_rank + m.rot_dim
        return {p + "in": [(p + "dq", 0, a), (p + "dkv", a, b - a), (p + "g", b, m.heads)],
                p + "ukv": [(p + "uk", 0, m.heads * m.dim), (p + "uv", m.heads * m.dim, m.heads * m.vdim)]}
    qk, v = m.heads * m.dim, m.heads * m.vdim
    g0 = 2 * (qk + v)
    return {p + "in": [(p + "q", 0, qk), (p + "k", qk, qk), (p + "v", 2 * qk, v), (p + "g", 2 * qk + v, v), (p + "i", g0, m.heads),
                       (p + "f", g0 + m.heads, m.heads)]}


def checkpoint_parts(spec: StackSpec) -> dict:
    out: dict = {}
    for i, l in enumerate(spec.layers):
        if l.owner == i:
            out.update(fused_rows(spec, i))
    return out
