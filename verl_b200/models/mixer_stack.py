"""Decoder whose layers differ: attention and recurrent mixers, dense and mixture-of-experts feed-forwards on one fp32 residual
stream.

The model runs packed prompt portions (``forward_hidden``) and one-token steps over all slots (``decode_hidden``) against the
same cache object: a page pool for the rows of the attention layers and one fp32 state row per slot for the recurrent
layers (``workers/rollout/native/cache.py::StackCache``). Layers that share weights still have their own pages and state.

Step layout: every projection that reads a layer's input is one GEMM. Stacks with elementwise norms in front of the sublayers:
the GEMM that ends a sublayer adds to the residual stream and applies the next norm in its epilogue (with norms on both sides
also the one on the sublayer's output). Stacks with RMS norms on
the sublayers' outputs: one row kernel behind that GEMM adds up its partial products (and the experts' rows), norms them, adds
to the stream and writes the next sublayer's input. Stacks with RMS norms in front of the sublayers: the GEMM adds to the stream
(in decode steps the row kernel adds its partial products), one row kernel norms the stream and applies the input convolution. Feed-forward activations run in the epilogue of the up-projection. Latent
attention: prompts expand keys and values from the latents; decoding absorbs the key expansion into the query and applies the
value expansion to the attention output, so only latent rows are read; a layer may read another layer's rows. Grouped-query
attention caches normed, rotated keys and mixed or convolved values, the convolution's last inputs are state; experts run on
tokens grouped by expert without a host synchronisation.

Forward only: the stacks are served (rollout, log-probs), not trained.
"""

from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Callable, Optional

import torch

from ..ops import functional as F
from ..ops import mixers as X
from .config import ModelConfig
from .decoder import PackedBatch
from .weights import FlatParams

__all__ = ["MixerStackModel", "PortionCache"]


@dataclass
class PortionCache:
    """Where the tokens of a packed batch live: ``slot_map`` [T] page rows to append to, ``slots`` [B] state rows, ``starts`` [B]
    tokens of each sequence that are already in the cache, ``block_table`` [B, blocks]."""

    cache: object
    slot_map: torch.Tensor
    slots: torch.Tensor        # int32, device
    starts: list               # host
    block_table: torch.Tensor  # int32, device


class MixerStackModel:
    def __init__(self, cfg: ModelConfig, params: FlatParams, recompute: str = "none", max_positions: int = 0, **unused):
        self.cfg, self.params, self.spec = cfg, params, cfg.stack
        self.device = params.flat.device
        self.recompute = recompute
        # attributes the engines set on the hand-written decoder; none of them applies here
        self.tp = self.sp = self.ep = self.tsp = self.router_replay = self.offloader = self.vocab_parallel = self.fp8_weights = None
        self.kv_hook = self.prefix_kv = self.keep_layers_fn = None
        self.mlp_tile_tokens = 0
        self.stats_hook: Optional[Callable[[str, torch.Tensor], None]] = None  # called with (name, tensor) per layer output
        self._rope_len = 0
        self._rope: dict = {}
        self._ensure_rope(max_positions or 2048)
        self._zero_sinks: dict = {}
        self._row_readers = {l.mixer.kv_from for l in self.spec.layers if getattr(l.mixer, "kv_from", -1) >= 0}   # layers whose rows others use
        self._no_rotation = (torch.ones(1, 0, device=self.device), torch.zeros(1, 0, device=self.device))
        self._weights = [self._layer_weights(i) for i in range(len(self.spec.layers))]
        self._final_norm = self._norm("final.norm")
        self._embed_norm = self._norm("embed.norm") if self.spec.embedding_norm else None

    # ------------------------------------------------------------------------------------ weights and tables
    def _norm(self, name: str):
        P = self.params
        return P[name] if self.spec.norm == "rms" else (P[name + ".alpha"], P[name], P[name + ".b"])

    def _layer_weights(self, i: int) -> dict:
        layer = self.spec.layers[i]
        p = f"l{layer.owner}."
        W = {k[len(p):]: v for k, v in self.params.views.items() if k.startswith(p)}
        both = self.spec.norm_on == "both"
        out = {"norm1": self._norm(p + "norm1"), "norm1b": self._norm(p + "norm1b") if both else None,
               "canon1": W.get("canon1"), **{k[4:]: v for k, v in W.items() if k.startswith("mix.")}}
        m = layer.mixer
        if m.kind == "latent_attention":
            out["uk"] = out["ukv"][: m.heads * m.dim].view(m.heads, m.dim, m.kv_rank)
            out["uv"] = out["ukv"][m.heads * m.dim :].view(m.heads, m.vdim, m.kv_rank)
        elif m.kind == "lightning":
            out["decay"] = torch.tensor(m.decay, dtype=torch.float32, device=self.device)
        elif m.kind == "attention":
            if m.heads not in self._zero_sinks:
                self._zero_sinks[m.heads] = torch.zeros(m.heads, dtype=self.params.flat.dtype, device=self.device)
            out["sink"] = self._zero_sinks[m.heads] if m.zero_sink else None
        if layer.mlp is not None:
            out.update(norm2=self._norm(p + "norm2"), norm2b=self._norm(p + "norm2b") if both else None,
                       **{k: v for k, v in W.items() if k.startswith("mlp.")})
        return out

    def _ensure_rope(self, n: int) -> None:
        if n <= self._rope_len:
            return
        self._rope_len = int(2 ** math.ceil(math.log2(max(n, 16))))
        self._rope = {}
        for l in self.spec.layers:
            rot = getattr(l.mixer, "rot", None)
            if rot is not None and rot.key() not in self._rope:
                self._rope[rot.key()] = F.rope_table(self._rope_len, rot.dims, rot.base, self.device, rot.scaling)

    def activation_bytes_per_layer(self, num_tokens: int) -> int:
        return 0

    # ------------------------------------------------------------------------------------ mixers
    def _attention_in(self, W, m, h, pos, pages, slot_map, want_rows: bool):
        """Queries [T, heads, dim + rot_dim] (not rotated), the layer's own latent rows (None: it reads another layer's), gates."""
        cos, sin = self._rope[m.rot.key()]
        q_cols = m.heads * (m.dim + m.rot_dim)
        p, gate = X.linear_split(h, W["in"], m.q_rank + m.kv_rank + m.rot_dim) if m.gate else (X.linear_act(h, W["in"]), None)
        cq, rows = None, None
        if m.kv_from < 0:
            at = 0 if m.q_rank else -(-q_cols // 8) * 8
            cq, rows = X.latent_prep(p[:, at : at + m.q_rank + m.kv_rank + m.rot_dim], W["dq.norm"] if m.q_rank else None, W["dkv.norm"], self.spec.norm_eps,
                                     pos, cos, sin, pages, slot_map, want_rows)
        q = X.linear_act(cq, W["uq"]) if m.q_rank else p[:, :q_cols]
        return q.unflatten(1, (m.heads, m.dim + m.rot_dim)), rows, gate, cos, sin

    def _key_rows(self, src: int, m, rows, batch: PackedBatch, pages, pc: Optional[PortionCache], portion: Optional[dict], shared: dict):
        """(rows of the keys and values that layer ``src`` owns, their offsets per sequence); ``rows``: those of this pass when ``src`` is the
        running layer. ``shared``: rows that other layers of this pass may use."""
        key, cu_k = (src,), batch.cu_seqlens
        if portion is not None:      # earlier tokens of some sequence are in the cache: take the keys from the pages
            key = (src, m.span)
            lo, cu_k, total = portion[m.span]
        if key not in shared:
            rows = X.gather_pages(pages, pc.block_table, cu_k, lo, total) if portion is not None else rows
            if src not in self._row_readers:
                return rows, cu_k
            shared[key] = rows
        return shared[key], cu_k

    def _attention_prefill(self, i, W, m, h, batch: PackedBatch, pc: Optional[PortionCache], portion: Optional[dict], shared: dict):
        src = m.kv_from if m.kv_from >= 0 else i
        pages = pc.cache.pages(src) if pc is not None else None
        q, rows, gate, cos, sin = self._attention_in(W, m, h, batch.positions, pages, pc.slot_map if pc is not None else None, portion is None)
        X.rope_pairs_(q, batch.positions, cos, sin, m.dim)
        rows, cu_k = self._key_rows(src, m, rows, batch, pages, pc, portion, shared)
        kv = X.linear_act(rows[:, : m.kv_rank], W["ukv"])
        ku = kv[:, : m.heads * m.dim].view(-1, m.heads, m.dim)
        v = kv[:, m.heads * m.dim :].view(-1, m.heads, m.vdim)
        o = X.latent_attention_prefill(q, ku, rows[:, m.kv_rank :], v, batch.cu_seqlens, cu_k, m.window, m.scale, W.get("sink"), gate, m.keep_first)
        return o.view(h.shape[0], m.heads * m.vdim)

    def _attention_decode(self, i, W, m, h, pos, slot_map, ctx_len, block_table, cache):
        S, pages = h.shape[0], cache.pages(m.kv_from if m.kv_from >= 0 else i)
        q, _, gate, cos, sin = self._attention_in(W, m, h, pos, pages, slot_map, False)
        qa = X.latent_absorb(q, W["uk"], pos, cos, sin)
        oc = X.latent_attention_decode(qa, pages, block_table, ctx_len, m.kv_rank, m.window, m.scale, W.get("sink"), m.keep_first)
        return X.headwise_linear(oc, W["uv"], False, gate).view(S, m.heads * m.vdim)

    def _grouped_in(self, i, W, m, h, pos, pages, slot_map, want_rows: bool, first: dict, past: dict):
        """Queries and the row [keys | values] (none for a layer that reads another's); ``first`` carries the values of the stack's first
        value-mixing layer, ``past`` says where the inputs of a convolution go on from."""
        p = X.linear_bias(h, W["in"], W["in.b"]) if m.bias else X.linear_act(h, W["in"])
        if m.norm_over == "all":
            return X.whole_norm_prep(p, W["q.norm"], W["k.norm"], W["temp"], self.spec.norm_eps, m.heads, m.kv_heads, m.vdim, pages, slot_map, want_rows)
        cos, sin = self._rope[m.rot.key()] if m.rot is not None else self._no_rotation
        if m.norm_after_rot or m.norm_over == "none":
            own = m.kv_from < 0
            return X.conv_qkv_prep(p, W.get("in.conv"), self.spec.norm_eps, pos, cos, sin, m.heads * m.maps, m.kv_heads * m.maps if own else 0, m.dim, m.vdim,
                                   m.rot.pairing == "halves", **past, pages=pages if own else None, page_slots=slot_map, want_rows=want_rows and own,
                                   norm=m.norm_after_rot, v_heads=m.kv_heads if own else 0)
        v_first = None
        if m.v_mix:
            if i == self.spec.value_source:
                a = (m.heads + m.kv_heads) * m.dim
                first["values"] = p[:, a : a + m.kv_heads * m.vdim]
            else:
                v_first = first["values"]
        return X.qkv_prep(p, W["q.norm"], W["k.norm"], self.spec.norm_eps, pos, cos, sin, m.heads, m.kv_heads, m.vdim, v_first,
                          W["vmix"] if v_first is not None else None, pages, slot_map, want_rows)

    def _difference(self, W, m):
        return (W["lambda"], m.diff, self.spec.norm_eps) if m.maps == 2 else None

    def _grouped_prefill(self, i, W, m, h, batch: PackedBatch, pc: Optional[PortionCache], portion: Optional[dict], first: dict, fresh, shared: dict):
        src = m.kv_from if m.kv_from >= 0 else i
        pages = pc.cache.pages(src) if pc is not None else None
        past = {"cu": batch.cu_seqlens, "state": pc.cache.state(i), "slots": pc.slots, "fresh": fresh} if pc is not None and m.state_size else {"cu": batch.cu_seqlens}
        q, rows = self._grouped_in(i, W, m, h, batch.positions, pages, pc.slot_map if pc is not None else None, portion is None, first, past)
        rows, cu_k = self._key_rows(src, m, rows, batch, pages, pc, portion, shared)
        k, v = rows[:, : m.k_cols].unflatten(1, (m.kv_heads * m.maps, m.dim)), rows[:, m.k_cols :].unflatten(1, (m.kv_heads, m.vdim))
        return X.grouped_attention_prefill(q, k, v, batch.cu_seqlens, cu_k, m.window, m.scale, m.softcap, W["sink"], m.keep_first, m.chunk,
                                           self._difference(W, m)).flatten(1)

    def _grouped_decode(self, i, W, m, h, pos, slot_map, ctx_len, active, block_table, cache, first: dict):
        past = {"state": cache.state(i), "active": active} if m.state_size else {"active": active}
        pages = cache.pages(m.kv_from if m.kv_from >= 0 else i)
        q, _ = self._grouped_in(i, W, m, h, pos, pages, slot_map, False, first, past)
        return X.grouped_attention_decode(q, pages, block_table, ctx_len, m.kv_heads, m.vdim, m.window, m.scale, m.softcap, W["sink"],
                                          m.keep_first, m.chunk, self._difference(W, m)).flatten(1)

    def _delta_in(self, W, m, h):
        """The fused projection [r | k | v | a | g | ...] and the decay's pre-activation."""
        p = X.linear_tanh(h, W["in"], m.low)
        return p, X.linear_act(p[:, m.low : m.low + m.rank], W["w2"])

    def _lightning(self, W, m, h, recur: Callable) -> torch.Tensor:
        n = m.heads * (2 * m.dim + m.vdim)
        p = X.linear_silu(h, W["in"], n)
        return X.gated_rms(recur(p, W["decay"], m.dim, m.vdim), p[:, n : n + m.heads * m.vdim], W["norm"], self.spec.norm_eps)

    def _mlstm_in(self, W, m, h):
        return X.linear_split(h, W["in"], 2 * m.heads * (m.dim + m.vdim))

    # ------------------------------------------------------------------------------------ layer loop
    def _run(self, ids: torch.Tensor, mix: Callable, past: Callable) -> torch.Tensor:
        """Embedding, layers, final norm; ``mix(i, weights, mixer, h)`` is the layer's mixer up to its output projection, ``past(i)`` says where
        the convolution of a layer's input goes on from."""
        if self.spec.norm_on == "output":
            return self._run_output_norms(ids, mix)
        return self._run_input_norms(ids, mix) if self.spec.norm == "dynamic_tanh" else self._run_input_rms(ids, mix, past)

    def _layer_done(self, i: int, x: torch.Tensor) -> None:
        if self.stats_hook is not None:
            self.stats_hook(f"layers.{i}.residual", x)

    def _run_input_norms(self, ids: torch.Tensor, mix: Callable) -> torch.Tensor:
        """Dynamic Tanh in front of the sublayers, with ``norm_on`` "both" also on their outputs."""
        layers, Ws = self.spec.layers, self._weights
        if self._embed_norm is not None:
            x, h = X.embed_dyt2(ids, self.params["embed"], self._embed_norm, Ws[0]["norm1"])
        else:
            x, h = X.embed_dyt(ids, self.params["embed"], self.spec.embedding_scale, *Ws[0]["norm1"])
        for i, layer in enumerate(layers):
            W, f = Ws[i], layer.mlp
            nxt = Ws[i + 1]["norm1"] if i + 1 < len(layers) else self._final_norm
            o = mix(i, W, layer.mixer, h)
            h = X.linear_residual_(o, W["o"], x, nxt if f is None else W["norm2"], W["norm1b"])
            if f is not None and f.kind == "moe":
                plan = X.expert_dispatch(h, X.linear_act(h, W["mlp.in"], out_f32=True), f.experts, f.top, f.renormalize, W.get("mlp.correction"), f.groups, f.keep)
                rows = X.expert_down(X.expert_up(plan, W["mlp.experts.in"], f.ff, f.act, f.limit), W["mlp.experts.down"], plan)
                h = X.residual_dyt_(x, rows, plan.slot, W["norm2b"], nxt)
            elif f is not None:
                h = X.linear_residual_(X.linear_act(h, W["mlp.up"], f.act), W["mlp.down"], x, nxt, W["norm2b"])
            self._layer_done(i, x)
        return h

    def _run_input_rms(self, ids: torch.Tensor, mix: Callable, past: Callable) -> torch.Tensor:
        """RMS norms in front of the sublayers, with ``input_conv`` a convolution of the mixers' inputs."""
        layers, Ws, eps = self.spec.layers, self._weights, self.spec.norm_eps
        x = X.embed_rows(ids, self.params["embed"], self.spec.embedding_scale)
        y = bias = None        # what the row kernel still has to add to the stream
        steps = "active" in past(0)

        def add(a, w, b=None):
            if steps:
                return X.linear_partial(a, w), b
            X.linear_residual_(a, w, x, bias=b)
            return None, None

        for i, layer in enumerate(layers):
            W, f = Ws[i], layer.mlp
            h = X.rms_conv(x, W["norm1"], eps, y, bias, W["canon1"], **(past(i) if W["canon1"] is not None else {}))
            y, bias = add(mix(i, W, layer.mixer, h), W["o"])
            if f is not None:
                h = X.rms_conv(x, W["norm2"], eps, y, bias)
                up = X.linear_bias(h, W["mlp.up"], W["mlp.up.b"], f.act) if f.bias else X.linear_act(h, W["mlp.up"], f.act)
                y, bias = add(up, W["mlp.down"], W.get("mlp.down.b"))
            if self.stats_hook is not None:
                total = x if y is None else x + (y.float().sum(0) if y.dim() == 3 else y.float())
                self._layer_done(i, total if bias is None else total + bias.float())
        return X.rms_conv(x, self._final_norm, eps, y, bias)

    def _run_output_norms(self, ids: torch.Tensor, mix: Callable) -> torch.Tensor:
        spec, layers = self.spec, self.spec.layers
        eps, mult = spec.norm_eps, spec.residual_mult
        x, h = X.embed_rms(ids, self.params["embed"], spec.embedding_scale, self._embed_norm, eps)
        for i, layer in enumerate(layers):
            W, f = self._weights[i], layer.mlp
            nxt = self._final_norm if i + 1 == len(layers) else None   # the last sublayer's kernel applies the final norm
            h = X.residual_rms_(x, X.linear_partial(mix(i, W, layer.mixer, h), W["o"]), W["norm1"], eps, mult, nxt if f is None else None)
            if f is not None and f.kind == "moe":
                act, tail = X.gated_up_split(h, W["mlp.in"], 2 * f.shared_ff)     # tail: router logits, then the shared expert's gate
                plan = X.expert_dispatch(h, tail, f.experts, f.top, f.renormalize)
                rows = X.expert_down(X.expert_up(plan, W["mlp.experts.in"], f.ff), W["mlp.experts.down"], plan)
                y, gate = (X.linear_partial(act, W["mlp.shared.down"]), tail[:, f.experts]) if f.shared_ff else (None, None)
                h = X.residual_rms_(x, y, W["norm2"], eps, mult, nxt, (rows, plan.slot), gate)
            elif f is not None:
                h = X.residual_rms_(x, X.linear_partial(X.gated_up(h, W["mlp.in"]), W["mlp.down"]), W["norm2"], eps, mult, nxt)
            self._layer_done(i, x)
        return h

    @torch.no_grad()
    def forward_hidden(self, batch: PackedBatch, pc: Optional[PortionCache] = None) -> torch.Tensor:
        """Final-norm hidden states [T, width] of packed sequences; with ``pc`` the tokens enter the cache behind what each
        sequence already holds there."""
        assert batch.expand_index is None, "shared-prefix packing is for the attention-only decoders"
        starts = pc.starts if pc is not None else [0] * (batch.cu_seqlens.numel() - 1)
        lens = (batch.cu_seqlens_cpu[1:] - batch.cu_seqlens_cpu[:-1]).tolist()
        self._ensure_rope(max(s + n for s, n in zip(starts, lens)) + 1)
        portion = None
        if any(starts):
            portion = {}
            for w in {l.mixer.span for l in self.spec.layers if hasattr(l.mixer, "span")}:
                # rows a layer reads: from the window's or the chunk's start, or all where the first tokens stay visible
                window, keep, chunk = w
                lo = [s // chunk * chunk if chunk > 0 else max(0, s - window + 1) if window > 0 and keep == 0 else 0 for s in starts]
                cu = torch.zeros(len(lens) + 1, dtype=torch.int32)
                cu[1:] = torch.cumsum(torch.tensor([s + n - a for s, n, a in zip(starts, lens, lo)], dtype=torch.int32), 0)
                portion[w] = (torch.tensor(lo, dtype=torch.int32).to(self.device), cu.to(self.device), int(cu[-1]))
        fresh = torch.tensor([int(s == 0) for s in starts], dtype=torch.int32).to(self.device) if pc is not None and self.spec.recurrent else None
        first: dict = {}
        shared: dict = {}

        def mix(i, W, m, h):
            if m.kind == "latent_attention":
                return self._attention_prefill(i, W, m, h, batch, pc, portion, shared)
            if m.kind == "attention":
                return self._grouped_prefill(i, W, m, h, batch, pc, portion, first, fresh, shared)
            if m.kind == "general_delta":
                kept = (pc.cache.state(i), pc.slots, fresh) if pc is not None else (None, None, None)
                p, zw = self._delta_in(W, m, h)
                o = X.delta_prefill(p, zw, W["a.b"], W["w0"], m.heads, batch.cu_seqlens, *kept)
                return X.gated_rms(o, p[:, 4 * m.width : 5 * m.width], W["norm"], self.spec.norm_eps, m.heads)
            if m.kind == "lightning":
                kept = (pc.cache.state(i), pc.slots, fresh) if pc is not None else (None, None, None)
                return self._lightning(W, m, h, lambda *a: X.lightning_prefill(*a, batch.cu_seqlens, *kept, not any(starts)))
            p, gates = self._mlstm_in(W, m, h)
            return X.mlstm_prefill(p, gates, W["i.b"], W["f.b"], m.gate_cap, W["norm"], self.spec.norm_eps, m.dim, batch.cu_seqlens,
                                   pc.cache.state(i) if pc is not None else None, pc.slots if pc is not None else None, fresh, not any(starts))

        def past(i):
            kept = {"state": pc.cache.input_state(i), "slots": pc.slots, "fresh": fresh} if pc is not None and self.spec.input_conv > 1 else {}
            return {"cu": batch.cu_seqlens, **kept}

        return self._run(batch.input_ids, mix, past)

    @torch.no_grad()
    def decode_hidden(self, tok, pos, slot_map, ctx_len, active, block_table, cache) -> torch.Tensor:
        """One token for every slot (static shapes, capturable); inactive slots leave cache and state untouched."""
        first: dict = {}

        def mix(i, W, m, h):
            if m.kind == "latent_attention":
                return self._attention_decode(i, W, m, h, pos, slot_map, ctx_len, block_table, cache)
            if m.kind == "attention":
                return self._grouped_decode(i, W, m, h, pos, slot_map, ctx_len, active, block_table, cache, first)
            if m.kind == "general_delta":
                p, zw = self._delta_in(W, m, h)
                return X.delta_decode(p, zw, W["a.b"], W["w0"], m.heads, W["norm"], self.spec.norm_eps, cache.state(i), active)
            if m.kind == "lightning":
                return self._lightning(W, m, h, lambda *a: X.lightning_decode(*a, cache.state(i), active))
            p, gates = self._mlstm_in(W, m, h)
            return X.mlstm_decode(p, gates, W["i.b"], W["f.b"], m.gate_cap, W["norm"], self.spec.norm_eps, m.dim, cache.state(i), active)

        return self._run(tok, mix, lambda i: {"state": cache.input_state(i) if self.spec.input_conv > 1 else None, "active": active})

    # ------------------------------------------------------------------------------------ heads
    def logits(self, h: torch.Tensor) -> torch.Tensor:
        return X.linear_softcap(h, self.params.lm_head_weight, self.spec.logit_softcap)

    def forward_logits(self, batch: PackedBatch) -> torch.Tensor:
        return self.logits(self.forward_hidden(batch))

    def forward_logprobs(self, batch: PackedBatch, labels: torch.Tensor, temperature: float = 1.0, need_grad: Optional[bool] = None,
                         positions: Optional[torch.Tensor] = None, stage_input=None, position_labels: Optional[torch.Tensor] = None):
        """(log_probs, entropy) per packed position, or per entry of ``positions`` (forward only)."""
        need_grad = torch.is_grad_enabled() if need_grad is None else need_grad
        if need_grad:
            raise NotImplementedError(f"{self.spec.design}: this design is served and scored, not trained (no backward pass)")
        with torch.no_grad():
            h = self.forward_hidden(batch)
            if positions is not None:
                h = h.index_select(0, positions)
                labels = position_labels if position_labels is not None else labels.index_select(0, positions)
            cap, w = self.spec.logit_softcap, self.params.lm_head_weight
            # the fused head has no soft cap and serves bf16 sizes that are multiples of 8
            if cap > 0 or (h.is_cuda and (h.dtype != torch.bfloat16 or h.shape[1] % 8 or self.cfg.vocab_size % 8)):
                rows = max(256, (1 << 28) // self.cfg.vocab_size)
                parts = [self._row_logprobs(h[a : a + rows], w, labels[a : a + rows], cap, temperature) for a in range(0, h.shape[0], rows)]
                return torch.cat([p[0] for p in parts]), torch.cat([p[1] for p in parts])
            lp, ent, _ = F.lmhead_logprob_entropy(h, w, labels, temperature)
            return lp, ent

    @staticmethod
    def _row_logprobs(h, w, labels, cap: float, temperature: float):
        z = X.linear_act(h, w, out_f32=True)
        z = cap * torch.tanh(z / cap) if cap > 0 else z
        logp = torch.log_softmax(z / max(temperature, 1e-8), -1)
        return logp.gather(-1, labels.unsqueeze(-1)).squeeze(-1), -(logp.exp() * logp).sum(-1)
