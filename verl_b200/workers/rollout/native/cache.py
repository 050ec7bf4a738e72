"""What the rollout engine keeps per token and per sequence, behind one interface for its two kinds of models.

* :class:`DenseKVCache`: keys and values of a uniform decoder, one pool ``[layers, 2, blocks, block_size, kv_heads, head_dim]``.
* :class:`StackCache`: mixer stacks. Attention layers that cache a row per token share a page pool (a block holds the rows of
  all such layers for ``block_size`` tokens); recurrent layers and convolutions own parts of one fp32 state row per sequence slot.

A sequence is its block list plus its slot; ``copy_blocks`` / ``copy_slots`` duplicate them (samples of one prompt) and
``export`` / ``install`` move them between engines (prefill / decode disaggregation).
"""

from __future__ import annotations

from typing import Optional

import torch

__all__ = ["DenseKVCache", "StackCache", "make_cache"]


class DenseKVCache:
    has_state = False

    def __init__(self, cfg, dtype, device, block_size: int, num_slots: int, tp_size: int = 1):
        self.cfg, self.dtype, self.device, self.bs, self.tp = cfg, dtype, device, block_size, tp_size
        self.kv = None

    def bytes_per_block(self) -> int:
        c = self.cfg
        return c.num_hidden_layers * 2 * self.bs * (c.kv_size // self.tp) * torch.empty((), dtype=self.dtype).element_size()

    def allocate(self, blocks: int) -> None:
        c = self.cfg
        self.kv = torch.zeros(c.num_hidden_layers, 2, blocks, self.bs, c.num_key_value_heads // self.tp, c.head_dim, dtype=self.dtype,
                              device=self.device)

    def free(self) -> None:
        self.kv = None

    def copy_blocks(self, dst: torch.Tensor, src: torch.Tensor) -> None:
        self.kv[:, :, dst] = self.kv[:, :, src]

    def copy_slots(self, dst: torch.Tensor, src: torch.Tensor) -> None:
        pass

    def export(self, blocks: torch.Tensor, slot: int) -> dict:
        return {"kv": self.kv[:, :, blocks].clone()}

    def install(self, blocks: torch.Tensor, slot: int, data: dict) -> None:
        self.kv[:, :, blocks] = data["kv"].to(self.device, dtype=self.kv.dtype)


class StackCache:
    def __init__(self, cfg, dtype, device, block_size: int, num_slots: int, tp_size: int = 1):
        assert tp_size == 1, "mixer stacks are served on one GPU per replica"
        self.dtype, self.device, self.bs = dtype, device, block_size
        # element offsets of every layer inside a block (rows of the layer's tokens are contiguous) and inside a state row
        self._page_off, self._page_w, self._state_off, self._state_n = {}, {}, {}, {}
        past = max(cfg.stack.input_conv - 1, 0) * cfg.hidden_size
        off = st = 0
        for i, l in enumerate(cfg.stack.layers):
            w, n = l.mixer.page_width, l.mixer.state_size
            if w:
                self._page_off[i], self._page_w[i] = off, w
                off += -(-block_size * w // 8) * 8      # 16-byte aligned starts
            for key, n in ((i, n), ((i, "input"), past)):
                if n:
                    self._state_off[key], self._state_n[key] = st, n
                    st += -(-n // 4) * 4
        self.block_elems, self.state_elems = max(off, 8), st
        self.has_state = st > 0
        self.num_slots = num_slots
        self.kv = self.states = None

    def bytes_per_block(self) -> int:
        return self.block_elems * torch.empty((), dtype=self.dtype).element_size()

    def allocate(self, blocks: int) -> None:
        self.kv = torch.zeros(blocks, self.block_elems, dtype=self.dtype, device=self.device)
        self.states = torch.zeros(self.num_slots, self.state_elems, dtype=torch.float32, device=self.device) if self.has_state else None
        self._pages = {i: self.kv[:, o : o + self.bs * self._page_w[i]].view(blocks, self.bs, self._page_w[i]) for i, o in self._page_off.items()}

    def free(self) -> None:
        self.kv = self.states = None
        self._pages = {}

    def pages(self, layer: int) -> torch.Tensor:
        """[blocks, block_size, width] view of a layer's rows."""
        return self._pages[layer]

    def state(self, layer: int) -> torch.Tensor:
        """[slots, size] view of a recurrent layer's state."""
        return self._state_view(layer)

    def input_state(self, layer: int) -> Optional[torch.Tensor]:
        """[slots, (taps - 1) width] view of what the convolution of a layer's input keeps (None: it keeps nothing)."""
        return self._state_view((layer, "input")) if (layer, "input") in self._state_off else None

    def _state_view(self, key) -> torch.Tensor:
        o = self._state_off[key]
        return self.states[:, o : o + self._state_n[key]]

    def copy_blocks(self, dst: torch.Tensor, src: torch.Tensor) -> None:
        self.kv[dst] = self.kv[src]

    def copy_slots(self, dst: torch.Tensor, src: torch.Tensor) -> None:
        if self.has_state:
            self.states[dst] = self.states[src]

    def export(self, blocks: torch.Tensor, slot: int) -> dict:
        return {"kv": self.kv[blocks].clone(), "state": self.states[slot].clone() if self.has_state else None}

    def install(self, blocks: torch.Tensor, slot: int, data: dict) -> None:
        self.kv[blocks] = data["kv"].to(self.device, dtype=self.kv.dtype)
        if self.has_state:
            self.states[slot] = data["state"].to(self.device)


def make_cache(cfg, dtype, device, block_size: int, num_slots: int, tp_size: int = 1):
    return (StackCache if cfg.is_stack else DenseKVCache)(cfg, dtype, device, block_size, num_slots, tp_size)
