"""Description of decoders whose layers differ: a list of token mixers and feed-forwards with their own sizes.

A *mixer stack* is a residual decoder in which every layer names its mixer (a kind of attention, a recurrent layer, ...), the
mixer's sizes, and its feed-forward or none; a layer may reuse another layer's weights or its cached latents. Norms sit in front
of the sublayers, on their outputs, or on both sides. The specs below are the typed form of such a configuration; ``DESIGNS`` maps the ``architecture`` of a
``config.json`` to the reader of its keys and is the place to register another design. Sizes and constants all come from the
configuration.
"""

from __future__ import annotations

from dataclasses import dataclass, replace
from typing import Any, Callable, Optional, Union

__all__ = ["RotarySpec", "LatentAttentionSpec", "GroupedAttentionSpec", "MLstmSpec", "LightningSpec", "DeltaSpec", "DenseMlpSpec", "GatedMlpSpec", "MoeSpec",
           "LayerSpec", "StackSpec", "DESIGNS", "is_stack_config", "sizes_from_tensors", "parse_stack"]


@dataclass(frozen=True)
class RotarySpec:
    """Rotary positions: frequencies of ``dims`` dimensions at ``base``, ``pairing`` of the dimensions ("interleaved": 2i with
    2i + 1; "halves": i with i + dims / 2), and a context extension in the form ``ops.functional.rope_inv_freq`` reads."""

    dims: int
    base: float
    pairing: str = "interleaved"
    scaling: Optional[dict] = None

    def key(self) -> tuple:
        return (self.dims, self.base, tuple(sorted((self.scaling or {}).items())))


@dataclass(frozen=True)
class LatentAttentionSpec:
    """Attention whose keys and values are expanded from one cached latent row per token (``kv_rank`` normed dimensions and
    ``rot_dim`` rotated ones shared by all heads). Queries go through a latent of ``q_rank`` (0: projected directly). A layer with
    ``kv_from`` reads the rows that layer ``kv_from`` cached and has none of its own."""

    heads: int
    dim: int          # unrotated query / key size per head
    rot_dim: int      # rotated query / key size per head
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot: RotarySpec
    window: int = 0   # tokens a query sees, itself included; 0 = all
    sink: bool = True         # one more score per head that has no value
    gate: bool = True         # output times the sigmoid of one gate per head
    kv_from: int = -1         # layer whose cached rows are used; -1: own rows
    keep_first: int = 0
    kind: str = "latent_attention"

    @property
    def span(self) -> tuple:
        return (self.window, self.keep_first, 0)

    @property
    def page_width(self) -> int:
        return self.kv_rank + self.rot_dim if self.kv_from < 0 else 0

    @property
    def state_size(self) -> int:
        return 0


@dataclass(frozen=True)
class GroupedAttentionSpec:
    """Grouped-query attention over cached keys and values: RMS norm per query / key head, rotation of the first ``rot.dims``
    dimensions, optional soft cap of the scores, an optional key of score 0 that has no value, and values mixed with those of
    the stack's first value-mixing layer. The norms carry weights and come before the rotation, or are plain and come after it
    (``norm_after_rot``), or span all heads (``norm_over`` "all"), or there are none. The projections may have biases and pass a
    causal convolution of ``conv`` taps over time per channel, whose last ``conv`` - 1 inputs are part of a sequence's state. With
    ``maps`` 2 (differential attention) every head has two query / key maps of ``dim`` over the same values; the head's output is the
    first map's minus lambda times the second's, normed, times 1 - ``diff``. A layer with ``kv_from`` reads the rows that layer cached."""

    heads: int
    kv_heads: int
    dim: int          # query / key size per head
    vdim: int
    scale: float
    rot: Optional[RotarySpec]
    softcap: float = 0.0      # score = softcap * tanh(score / softcap); 0 = off
    zero_sink: bool = True    # one is added to the softmax denominator
    v_mix: bool = False
    window: int = 0
    keep_first: int = 0       # first tokens of a sequence that every query sees besides its window
    norm_after_rot: bool = False
    bias: bool = False
    conv: int = 0             # taps; 0 = no convolution
    chunk: int = 0            # a query sees the keys of its own chunk of this many positions; 0 = all
    maps: int = 1             # 2: differential attention
    diff: float = 0.0
    norm_over: str = "head"   # what a query / key norm spans: "head" | "all" heads | "none"
    temp: bool = False        # scores times one number per head
    kv_from: int = -1         # layer whose cached rows are used; -1: own rows
    kind: str = "attention"

    @property
    def q_cols(self) -> int:
        return self.heads * self.maps * self.dim

    @property
    def k_cols(self) -> int:
        return self.kv_heads * self.maps * self.dim

    @property
    def row_width(self) -> int:
        """Cached row [keys | values]."""
        return self.k_cols + self.kv_heads * self.vdim

    @property
    def channels(self) -> int:
        """Projected columns."""
        return self.q_cols + (self.row_width if self.kv_from < 0 else 0)

    @property
    def page_width(self) -> int:
        return self.row_width if self.kv_from < 0 else 0

    @property
    def span(self) -> tuple:
        """What decides which cached rows a prompt portion reads."""
        return (self.window, self.keep_first, self.chunk)

    @property
    def state_size(self) -> int:
        return max(self.conv - 1, 0) * self.channels


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
class LightningSpec:
    """Linear recurrence with one fixed decay per head: S = decay S + k v^T, read with q; q, k and v pass a silu. The heads' outputs
    are normed together and gated."""

    heads: int
    dim: int
    vdim: int
    decay: tuple
    kind: str = "lightning"

    @property
    def page_width(self) -> int:
        return 0

    @property
    def state_size(self) -> int:
        return self.heads * self.dim * self.vdim


@dataclass(frozen=True)
class DeltaSpec:
    """Generalized delta rule on a matrix memory: per head S = diag(w) S - (a u) (u^T S) + k v^T, read with r; u is the unit key, the
    decay w and the removal rate a are numbers per head and key channel. The decay's pre-activation comes through ``rank`` channels
    with a tanh. Every head's output is normed, the heads are gated together."""

    heads: int
    dim: int
    rank: int
    kind: str = "general_delta"

    @property
    def vdim(self) -> int:
        return self.dim

    @property
    def width(self) -> int:
        return self.heads * self.dim

    @property
    def low(self) -> int:
        """First column of the decay's channels in the fused projection [r | k | v | a | g | decay]."""
        return _up8(5 * self.width)

    @property
    def page_width(self) -> int:
        return 0

    @property
    def state_size(self) -> int:
        return self.heads * self.dim * self.dim


@dataclass(frozen=True)
class DenseMlpSpec:
    ff: int
    act: str = "gelu_erf"     # "gelu_erf" | "relu2" (the square of relu)
    bias: bool = False
    kind: str = "dense"


@dataclass(frozen=True)
class GatedMlpSpec:
    """``W_down (silu(W_gate h) * (W_up h))``."""

    ff: int
    kind: str = "gated"


@dataclass(frozen=True)
class MoeSpec:
    """Gated experts of which every token uses ``top``: sigmoid scores, the score of a chosen expert scales the expert's input or
    output (``renormalize``: scores divided by their sum first); a shared expert of ``shared_ff`` (0 = none) is added, multiplied by
    the sigmoid of its own gate. Experts may be chosen by corrected scores (``correction``: one addend per expert) and from the
    ``keep`` best of ``groups`` groups of neighbours (a group's score: the sum of its two largest). ``act``: "silu", or "clipped":
    ``g sigmoid(1.702 g) (u + 1)`` with g <= ``limit`` and ``|u| <= limit``."""

    experts: int
    top: int
    ff: int
    shared_ff: int = 0
    renormalize: bool = False
    correction: bool = False
    groups: int = 1
    keep: int = 1
    act: str = "silu"         # "silu" scales the expert's input by the score, "clipped" its output
    limit: float = 0.0
    kind: str = "moe"


@dataclass(frozen=True)
class LayerSpec:
    mixer: Union[LatentAttentionSpec, GroupedAttentionSpec, MLstmSpec, LightningSpec, DeltaSpec]
    mlp: Union[DenseMlpSpec, GatedMlpSpec, MoeSpec, None]
    owner: int        # layer whose tensors this one uses (itself, or an earlier one with shared weights)


@dataclass(frozen=True)
class StackSpec:
    design: str
    embedding_scale: float
    norm: str         # "dynamic_tanh" | "rms"
    norm_eps: float   # eps of the RMS norms
    layers: tuple
    norm_on: str = "input"        # where a sublayer's norm sits: on its "input", on its "output", or on "both" sides
    residual_mult: float = 1.0    # factor on what a sublayer adds to the stream
    embedding_norm: bool = False  # the embedding passes the stack's norm
    tied_head: bool = False       # the output matrix is the embedding table
    logit_softcap: float = 0.0    # 0 = off
    input_conv: int = 0           # taps of the causal convolution that every mixer's input h passes, h + conv(h); the last taps - 1 h are state

    @property
    def recurrent(self) -> bool:
        return self.input_conv > 1 or any(l.mixer.state_size for l in self.layers)

    @property
    def value_source(self) -> int:
        """First value-mixing layer (-1: none): its values enter the mixes of the later ones."""
        return next((i for i, l in enumerate(self.layers) if getattr(l.mixer, "v_mix", False)), -1)


# --------------------------------------------------------------------------------------------- readers of config.json
def _rotary(d: dict, pairing: str = "interleaved") -> RotarySpec:
    scaling = None
    s = d.get("scaling")
    if s:
        import math

        scaling = {"rope_type": "yarn", "factor": float(s["factor"]), "original_max_position_embeddings": s["original"],
                   "beta_fast": float(s["fast"]), "beta_slow": float(s["slow"]), "attention_factor": 0.1 * math.log(float(s["factor"])) + 1.0}
    return RotarySpec(dims=int(d["dims"]), base=float(d["base"]), pairing=pairing, scaling=scaling)


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


def _shared_latent_attention(m: dict) -> LatentAttentionSpec:
    """Queries projected directly, no sink, no gate; the rows may be another layer's."""
    mask = m.get("mask") or {}
    return LatentAttentionSpec(heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]), vdim=int(m["vdim"]), q_rank=0, kv_rank=int(m["kv_rank"]),
                               scale=float(m["scale"]), rot=_rotary(m["rot"]), window=int(mask.get("size") or 0), keep_first=int(mask.get("keep_first") or 0),
                               sink=False, gate=False, kv_from=int(m["kv_from"]) if m.get("kv_from") is not None else -1)


def _convolved_attention(m: dict) -> GroupedAttentionSpec:
    """Biased, convolved projections; plain norms behind the rotation; a window that keeps the first tokens."""
    mask = m.get("mask") or {}
    spec = GroupedAttentionSpec(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), scale=float(m["scale"]),
                                rot=_rotary(m["rot"], "halves"), zero_sink=False, window=int(mask.get("size") or 0), keep_first=int(mask.get("keep_first") or 0),
                                norm_after_rot=True, bias=True, conv=int(m.get("conv") or 0))
    if spec.heads % spec.kv_heads or spec.rot.dims % 2 or spec.rot.dims > spec.dim or spec.conv < 0:
        raise ValueError(f"attention sizes: {spec}")
    return spec


def _lightning(m: dict) -> LightningSpec:
    spec = LightningSpec(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), decay=tuple(float(x) for x in m["decay"]))
    if len(spec.decay) != spec.heads:
        raise ValueError(f"one decay per head: {spec}")
    return spec


def _chunk(m: dict) -> int:
    return int((m.get("mask") or {}).get("size") or 0)


def _differential_attention(m: dict) -> GroupedAttentionSpec:
    """Two rotated query / key maps per head, no norms; keys and values may be another layer's."""
    return GroupedAttentionSpec(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), scale=float(m["scale"]),
                                rot=_rotary(m["rot"], "halves"), zero_sink=False, chunk=_chunk(m), maps=2, diff=float(m["diff"]), norm_over="none",
                                kv_from=int(m["kv_from"]) if m.get("kv_from") is not None else -1)


def _whole_norm_attention(m: dict) -> GroupedAttentionSpec:
    """Norms over the whole query and key projections, one temperature per head, no rotation."""
    return GroupedAttentionSpec(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), scale=float(m["scale"]), rot=None,
                                zero_sink=False, chunk=_chunk(m), norm_over="all", temp=True)


def _general_delta(m: dict) -> DeltaSpec:
    if "decay_rank" not in m:
        raise ValueError("a general_delta mixer needs decay_rank (read from the weights with sizes_from_tensors)")
    return DeltaSpec(heads=int(m["heads"]), dim=int(m["dim"]), rank=int(m["decay_rank"]))


MIXER_READERS: dict[str, Callable[[dict], Any]] = {"latent_attention": _latent_attention, "mlstm": _mlstm, "attention": _grouped_attention}


def _mlp(d: Optional[dict], gated: bool = False) -> Union[DenseMlpSpec, GatedMlpSpec, MoeSpec, None]:
    if d is None:
        return None
    if d.get("kind") == "dense":
        return GatedMlpSpec(ff=int(d["ff"])) if gated else DenseMlpSpec(ff=int(d["ff"]))
    if d.get("kind") == "moe" and gated:
        r = d["router"]
        if "limit" in d["expert"]:
            g = r.get("groups") or {}
            spec = MoeSpec(experts=int(r["experts"]), top=int(r["top"]), ff=int(d["expert"]["ff"]), renormalize=True, correction=True,
                           groups=int(g.get("count", 1)), keep=int(g.get("keep", g.get("count", 1))), act="clipped", limit=float(d["expert"]["limit"]))
            if spec.experts % spec.groups or not 1 <= spec.keep <= spec.groups or not 1 <= spec.top <= spec.keep * (spec.experts // spec.groups):
                raise ValueError(f"expert groups: {spec}")
            return spec
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
    """``mixers``: the design's mixer types, or a type -> reader mapping where they differ from ``MIXER_READERS``."""
    readers = mixers if isinstance(mixers, dict) else {t: MIXER_READERS[t] for t in mixers}
    layers = []
    for i, l in enumerate(d["layers"]):
        if l["type"] not in readers:
            raise NotImplementedError(f"mixer type {l['type']!r}")
        layers.append(LayerSpec(mixer=readers[l["type"]](l["mixer"]), mlp=_mlp(l.get("mlp"), gated), owner=_owner(d["layers"], i)))
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


def parse_luzitar(d: dict) -> StackSpec:
    readers = {"lightning": _lightning, "attention": _convolved_attention, "latent_attention": _shared_latent_attention}
    spec = StackSpec(design="Luzitar", embedding_scale=1.0, norm="dynamic_tanh", norm_eps=float(d["norm"]["eps"]), layers=_layers(d, readers, gated=True),
                     norm_on="both", embedding_norm=True, logit_softcap=float(d.get("logit_softcap") or 0.0))
    for i, l in enumerate(spec.layers):
        j = getattr(l.mixer, "kv_from", -1)
        if j < 0:
            continue
        m, src = l.mixer, spec.layers[j].mixer if j < i else None
        if src is None or src.kind != "latent_attention" or src.kv_from >= 0 or (src.kv_rank, src.rot_dim, src.rot) != (m.kv_rank, m.rot_dim, m.rot):
            raise ValueError(f"layer {i}: kv_from {j} must be an earlier latent layer with rows of its own, of the same sizes and rotation")
    return spec


def parse_fusazen(d: dict) -> StackSpec:
    readers = {"general_delta": _general_delta, "attention": _differential_attention, "attention_2": _whole_norm_attention}
    layers = tuple(replace(l, mlp=DenseMlpSpec(ff=l.mlp.ff, act="relu2", bias=True)) if l.mlp is not None else l for l in _layers(d, readers))
    spec = StackSpec(design="Fusazen", embedding_scale=float(d["embedding"]["scale"]), norm="rms", norm_eps=float(d["norm"]["eps"]), layers=layers,
                     input_conv=int(d["canon"]["taps"]))
    if spec.input_conv < 1:
        raise ValueError(f"taps of the input convolution: {spec.input_conv}")
    for i, l in enumerate(spec.layers):
        m = l.mixer
        if m.kind != "attention":
            continue
        if m.heads % m.kv_heads or m.chunk < 0 or (m.rot is not None and (m.rot.dims % 2 or m.rot.dims > m.dim)):
            raise ValueError(f"attention sizes: {m}")
        if m.kv_from >= 0:
            src = spec.layers[m.kv_from].mixer if m.kv_from < i else None
            same = lambda a: (a.kind, a.maps, a.kv_heads, a.dim, a.vdim, a.rot)
            if src is None or src.kind != "attention" or src.kv_from >= 0 or same(src) != same(m):
                raise ValueError(f"layer {i}: kv_from {m.kv_from} must be an earlier layer of the same kind with rows of its own, of the same sizes and rotation")
    return spec


DESIGNS: dict[str, Callable[[dict], StackSpec]] = {"Zorelorn": parse_zorelorn, "Tofinex": parse_tofinex, "Luzitar": parse_luzitar, "Fusazen": parse_fusazen}


def is_stack_config(d: dict) -> bool:
    return d.get("architecture") in DESIGNS


def sizes_from_tensors(d: dict, shape_of: Callable[[str], tuple]) -> dict:
    """The configuration with the sizes that only the weights tell; ``shape_of`` gives the shape of a stored tensor."""
    if d.get("architecture") != "Fusazen":
        return d
    layers = []
    for i, l in enumerate(d["layers"]):
        if l["type"] == "general_delta" and "decay_rank" not in l["mixer"]:
            l = {**l, "mixer": {**l["mixer"], "decay_rank": int(shape_of(f"l{i}.mix.w1")[0])}}
        layers.append(l)
    return {**d, "layers": layers}


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
    sides = lambda name: norm_tensors(spec, p + name, width) + (norm_tensors(spec, p + name + "b", width) if spec.norm_on == "both" else [])
    out = sides("norm1")
    out += [(p + "canon1", (width, spec.input_conv), "normal", False)] if spec.input_conv else []
    m, f = l.mixer, l.mlp
    if m.kind == "latent_attention":
        # queries (or their latent), key / value latent with the rotated key part, gates
        rows = m.kv_rank + m.rot_dim if m.kv_from < 0 else 0
        n = (m.q_rank or _up8(m.heads * (m.dim + m.rot_dim))) + rows
        out += [(p + "mix.in", (n + _up8(m.heads) if m.gate else _up8(n), width), "normal", True)]
        out += [(p + "mix.dq.norm", (m.q_rank,), "ones", False)] if m.q_rank else []
        out += [(p + "mix.dkv.norm", (m.kv_rank,), "ones", False)] if rows else []
        out += [(p + "mix.uq", (m.heads * (m.dim + m.rot_dim), m.q_rank), "normal", True)] if m.q_rank else []
        out += [(p + "mix.ukv", (m.heads * (m.dim + m.vdim), m.kv_rank), "normal", True)]
        out += [(p + "mix.sink", (m.heads,), "zeros", False)] if m.sink else []
        out += [(p + "mix.o", (width, m.heads * m.vdim), "normal", True)]
    elif m.kind == "attention":
        out += [(p + "mix.in", (_up8(m.channels), width), "normal", True)]
        out += [(p + "mix.in.b", (_up8(m.channels),), "zeros", False)] if m.bias else []
        out += [(p + "mix.in.conv", (m.channels, m.conv), "normal", False)] if m.conv else []
        if not m.norm_after_rot and m.norm_over != "none":
            out += [(p + "mix.q.norm", (m.dim if m.norm_over == "head" else m.q_cols,), "ones", False),
                    (p + "mix.k.norm", (m.dim if m.norm_over == "head" else m.k_cols,), "ones", False)]
        out += [(p + "mix.temp", (m.heads,), "ones", False)] if m.temp else []
        out += [(p + "mix.lambda", (4 * m.dim,), "zeros", False)] if m.maps == 2 else []
        out += [(p + "mix.vmix", (1,), "fill:0.5", False)] if m.v_mix else []
        out += [(p + "mix.o", (width, m.heads * m.vdim), "normal", True)]
    elif m.kind == "general_delta":
        n = m.width
        out += [(p + "mix.in", (m.low + _up8(m.rank), width), "normal", True), (p + "mix.a.b", (n,), "zeros", False), (p + "mix.w2", (n, m.rank), "normal", True),
                (p + "mix.w0", (n,), "zeros", False), (p + "mix.norm", (n,), "ones", False), (p + "mix.o", (width, n), "normal", True)]
    elif m.kind == "lightning":
        out += [(p + "mix.in", (_up8(2 * m.heads * (m.dim + m.vdim)), width), "normal", True), (p + "mix.norm", (m.heads * m.vdim,), "ones", False),
                (p + "mix.o", (width, m.heads * m.vdim), "normal", True)]
    else:
        out += [(p + "mix.in", (2 * m.heads * (m.dim + m.vdim) + _up8(2 * m.heads), width), "normal", True),
                (p + "mix.i.b", (m.heads,), "zeros", False), (p + "mix.f.b", (m.heads,), "fill:4.0", False),
                (p + "mix.norm", (m.heads * m.vdim,), "ones", False), (p + "mix.o", (width, m.heads * m.vdim), "normal", True)]
    if f is None:
        return out
    out += sides("norm2")
    if f.kind == "dense":
        out += [(p + "mlp.up", (f.ff, width), "normal", True), (p + "mlp.down", (width, f.ff), "normal", True)]
        out += [(p + "mlp.up.b", (f.ff,), "zeros", False), (p + "mlp.down.b", (width,), "zeros", False)] if f.bias else []
    elif f.kind == "gated":
        out += [(p + "mlp.in", (2 * f.ff, width), "normal", True), (p + "mlp.down", (width, f.ff), "normal", True)]
    else:
        # one matrix for everything that reads every token (shared expert, router, shared gate); the experts' are stacked
        out += [(p + "mlp.in", (2 * f.shared_ff + _up8(f.experts + (1 if f.shared_ff else 0)), width), "normal", True)]
        out += [(p + "mlp.correction", (f.experts,), "zeros", False)] if f.correction else []
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
        q = m.heads * (m.dim + m.rot_dim)
        rows = [("dq", 0, m.q_rank)] if m.q_rank else [("q", 0, q)]
        at = m.q_rank or _up8(q)
        if m.kv_from < 0:
            rows += [("dkv", at, m.kv_rank + m.rot_dim)]
            at += m.kv_rank + m.rot_dim
        rows += [("g", at, m.heads)] if m.gate else []
        out = {p + "in": [(p + name, r0, n) for name, r0, n in rows], p + "ukv": _consecutive((p + "uk", m.heads * m.dim), (p + "uv", m.heads * m.vdim))}
    elif m.kind == "attention":
        sizes = (("q", m.q_cols), *((("k", m.k_cols), ("v", m.kv_heads * m.vdim)) if m.kv_from < 0 else ()))
        out = {p + "in" + what: _consecutive(*((p + name + what, n) for name, n in sizes)) for what in ("", *([".b"] if m.bias else []), *([".conv"] if m.conv else []))}
        if m.maps == 2:
            out[p + "lambda"] = _consecutive(*((p + name, m.dim) for name in ("lq1", "lk1", "lq2", "lk2")))
    elif m.kind == "general_delta":
        out = {p + "in": _consecutive(*((p + name, m.width) for name in "rkvag")) + [(p + "w1", m.low, m.rank)]}
    elif m.kind == "lightning":
        qk, v = m.heads * m.dim, m.heads * m.vdim
        out = {p + "in": _consecutive((p + "q", qk), (p + "k", qk), (p + "v", v), (p + "g", v))}
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
