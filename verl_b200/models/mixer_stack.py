"""Decoder whose layers differ: latent attention and matrix-memory recurrences on one fp32 residual stream.

The model runs packed prompt portions (``forward_hidden``) and one-token steps over all slots (``decode_hidden``) against the
same cache object: a page pool for the latent rows of the attention layers and one fp32 state row per slot for the recurrent
layers (``workers/rollout/native/cache.py::StackCache``). Layers that share weights still have their own pages and state.

Step layout: every projection that reads a layer's input is one GEMM; norms are elementwise, so the GEMM that ends a sublayer
adds to the residual stream and applies the next norm in its epilogue, and the feed-forward activation runs in the epilogue
of its up-projection. Prompts expand keys and values from the latents; decoding absorbs the key expansion into the query and
applies the value expansion to the attention output, so only latent rows are read.

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
        self._weights = [self._layer_weights(i) for i in range(len(self.spec.layers))]
        self._final_norm = self._norm("final.norm")

    # ------------------------------------------------------------------------------------ weights and tables
    def _norm(self, name: str) -> tuple:
        P = self.params
        return (P[name + ".alpha"], P[name], P[name + ".b"])

    def _layer_weights(self, i: int) -> dict:
        layer = self.spec.layers[i]
        p = f"l{layer.owner}."
        W = {k[len(p):]: v for k, v in self.params.views.items() if k.startswith(p)}
        out = {"norm1": self._norm(p + "norm1"), **{k[4:]: v for k, v in W.items() if k.startswith("mix.")}}
        m = layer.mixer
        if m.kind == "latent_attention":
            out["uk"] = out["ukv"][: m.heads * m.dim].view(m.heads, m.dim, m.kv_rank)
            out["uv"] = out["ukv"][m.heads * m.dim :].view(m.heads, m.vdim, m.kv_rank)
        if layer.mlp is not None:
            out.update(norm2=self._norm(p + "norm2"), up=W["mlp.up"], down=W["mlp.down"])
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
        cut = m.q_rank + m.kv_rank + m.rot_dim
        p, gate = X.linear_split(h, W["in"], cut)
        cos, sin = self._rope[m.rot.key()]
        cq, rows = X.latent_prep(p, W["dq.norm"], W["dkv.norm"], self.spec.norm_eps, pos, cos, sin, pages, slot_map, want_rows)
        q = X.linear_act(cq, W["uq"]).view(h.shape[0], m.heads, m.dim + m.rot_dim)
        return q, rows, gate, cos, sin

    def _attention_prefill(self, i, W, m, h, batch: PackedBatch, pc: Optional[PortionCache], portion: Optional[dict]):
        pages = pc.cache.pages(i) if pc is not None else None
        q, rows, gate, cos, sin = self._attention_in(W, m, h, batch.positions, pages, pc.slot_map if pc is not None else None, portion is None)
        X.rope_pairs_(q, batch.positions, cos, sin, m.dim)
        cu_k = batch.cu_seqlens
        if portion is not None:      # earlier tokens of some sequence are in the cache: take the keys from the pages
            lo, cu_k, total = portion[m.window]
            rows = X.gather_pages(pages, pc.block_table, cu_k, lo, total)
        kv = X.linear_act(rows[:, : m.kv_rank], W["ukv"])
        ku = kv[:, : m.heads * m.dim].view(-1, m.heads, m.dim)
        v = kv[:, m.heads * m.dim :].view(-1, m.heads, m.vdim)
        o = X.latent_attention_prefill(q, ku, rows[:, m.kv_rank :], v, batch.cu_seqlens, cu_k, m.window, m.scale, W["sink"], gate)
        return o.view(h.shape[0], m.heads * m.vdim)

    def _attention_decode(self, i, W, m, h, pos, slot_map, ctx_len, block_table, cache):
        S = h.shape[0]
        q, _, gate, cos, sin = self._attention_in(W, m, h, pos, cache.pages(i), slot_map, False)
        qa = X.latent_absorb(q, W["uk"], pos, cos, sin)
        oc = X.latent_attention_decode(qa, cache.pages(i), block_table, ctx_len, m.kv_rank, m.window, m.scale, W["sink"])
        return X.headwise_linear(oc, W["uv"], False, gate).view(S, m.heads * m.vdim)

    def _mlstm_in(self, W, m, h):
        return X.linear_split(h, W["in"], 2 * m.heads * (m.dim + m.vdim))

    # ------------------------------------------------------------------------------------ layer loop
    def _run(self, ids: torch.Tensor, mix: Callable) -> torch.Tensor:
        """Embedding, layers, final norm; ``mix(i, weights, mixer, h)`` is the layer's mixer up to its output projection."""
        layers, Ws = self.spec.layers, self._weights
        x, h = X.embed_dyt(ids, self.params["embed"], self.spec.embedding_scale, *Ws[0]["norm1"])
        for i, layer in enumerate(layers):
            W = Ws[i]
            nxt = Ws[i + 1]["norm1"] if i + 1 < len(layers) else self._final_norm
            o = mix(i, W, layer.mixer, h)
            if layer.mlp is None:
                h = X.linear_residual_(o, W["o"], x, nxt)
            else:
                h = X.linear_residual_(o, W["o"], x, W["norm2"])
                h = X.linear_residual_(X.linear_act(h, W["up"], layer.mlp.act), W["down"], x, nxt)
            if self.stats_hook is not None:
                self.stats_hook(f"layers.{i}.residual", x)
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
            for w in {l.mixer.window for l in self.spec.layers if l.mixer.kind == "latent_attention"}:
                lo = [max(0, s - w + 1) if w > 0 else 0 for s in starts]
                cu = torch.zeros(len(lens) + 1, dtype=torch.int32)
                cu[1:] = torch.cumsum(torch.tensor([s + n - a for s, n, a in zip(starts, lens, lo)], dtype=torch.int32), 0)
                portion[w] = (torch.tensor(lo, dtype=torch.int32).to(self.device), cu.to(self.device), int(cu[-1]))
        fresh = torch.tensor([int(s == 0) for s in starts], dtype=torch.int32).to(self.device) if pc is not None else None

        def mix(i, W, m, h):
            if m.kind == "latent_attention":
                return self._attention_prefill(i, W, m, h, batch, pc, portion)
            p, gates = self._mlstm_in(W, m, h)
            return X.mlstm_prefill(p, gates, W["i.b"], W["f.b"], m.gate_cap, W["norm"], self.spec.norm_eps, m.dim, batch.cu_seqlens,
                                   pc.cache.state(i) if pc is not None else None, pc.slots if pc is not None else None, fresh, not any(starts))

        return self._run(batch.input_ids, mix)

    @torch.no_grad()
    def decode_hidden(self, tok, pos, slot_map, ctx_len, active, block_table, cache) -> torch.Tensor:
        """One token for every slot (static shapes, capturable); inactive slots leave cache and state untouched."""

        def mix(i, W, m, h):
            if m.kind == "latent_attention":
                return self._attention_decode(i, W, m, h, pos, slot_map, ctx_len, block_table, cache)
            p, gates = self._mlstm_in(W, m, h)
            return X.mlstm_decode(p, gates, W["i.b"], W["f.b"], m.gate_cap, W["norm"], self.spec.norm_eps, m.dim, cache.state(i), active)

        return self._run(tok, mix)

    # ------------------------------------------------------------------------------------ heads
    def logits(self, h: torch.Tensor) -> torch.Tensor:
        return X.linear_act(h, self.params.lm_head_weight)

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
            if h.is_cuda and (h.dtype != torch.bfloat16 or h.shape[1] % 8 or self.cfg.vocab_size % 8):   # outside the fused head's sizes
                logp = torch.log_softmax(X.linear_act(h, self.params.lm_head_weight, out_f32=True) / max(temperature, 1e-8), -1)
                return logp.gather(-1, labels.unsqueeze(-1)).squeeze(-1), -(logp.exp() * logp).sum(-1)
            lp, ent, _ = F.lmhead_logprob_entropy(h, self.params.lm_head_weight, labels, temperature)
            return lp, ent
