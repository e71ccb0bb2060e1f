"""Cache of models that mix latent-attention layers with recurrent layers, each layer with sizes of its own.

Latent layers share one page table: a token's row is [latent | rotated key part], one row for all heads, and a page of a
layer is ``page_size`` consecutive rows (row stride padded to 16 bytes so that a page is a TMA box).  Recurrent layers
keep a 32-bit [heads, dim, dim] state per sequence slot.  Pages of all layers live in one flat tensor (``values``), states
of all layers of a slot in one row of another.
"""
from __future__ import annotations

from typing import Optional

import torch

from ..models.config import ModelConfig
from ..ops.latent import LatentPages
from .hybrid import StateSlots
from .paged import KVSpec, PagedKVCache, PagePool


class LatentHybridCache(StateSlots, PagedKVCache):
    def __init__(self, cfg: ModelConfig, num_pages: int, device, max_seqs: int, latent_widths: dict, state_shapes: dict):
        """latent_widths: layer -> row width; state_shapes: layer -> (heads, dim)."""
        fmt = cfg.kv_format
        if fmt not in ("fp32", "bf16"):
            raise ValueError(f"latent pages are stored as bf16 or fp32, not {fmt!r}")
        self.device = torch.device(device)
        dt = torch.float32 if fmt == "fp32" else torch.bfloat16
        self.widths = dict(latent_widths)
        widest = max(self.widths.values(), default=0)
        self.spec = KVSpec(len(self.widths), 1, widest, cfg.page_size, fmt)
        self.pool = PagePool(num_pages, cfg.page_size)
        self.fp8 = self.nvfp4 = False
        self.scales: Optional[torch.Tensor] = None
        pad = 8                                             # elements: 16 bytes of bf16, 32 of fp32
        self._ld = {l: (w + pad - 1) // pad * pad for l, w in self.widths.items()}
        rows = num_pages * cfg.page_size
        self.values = torch.zeros(rows * sum(self._ld.values()), dtype=dt, device=self.device)
        self._layers, off = {}, 0
        for l, ld in self._ld.items():
            self._layers[l] = LatentPages(self.values[off:off + rows * ld].view(num_pages, cfg.page_size, ld), cfg.page_size)
            off += rows * ld
        offs, total = {}, 0
        for l, (h, d) in state_shapes.items():
            offs[l] = total
            total += (h * d * d + 3) // 4 * 4
        self.states = torch.zeros((max_seqs, max(total, 4)), dtype=torch.float32, device=self.device)
        self._states = {l: self.states[:, offs[l]:offs[l] + h * d * d].unflatten(1, (h, d, d)) for l, (h, d) in state_shapes.items()}
        self.init_slots(max_seqs, [(self.states, 0)])

    def layer(self, i: int) -> Optional[LatentPages]:
        return self._layers.get(i)

    def state(self, i: int) -> torch.Tensor:
        """[slots, heads, dim, dim] view of a recurrent layer (the slot stride is the whole state row)."""
        return self._states[i]

    def bytes_per_token(self) -> int:
        return sum(self._ld.values()) * self.values.element_size()

    def copy_page(self, src: int, dst: int) -> None:
        for kv in self._layers.values():
            kv.pages[dst].copy_(kv.pages[src])

    def export_pages(self, seq: int) -> dict:
        pages = torch.tensor(self.pool.pages(seq), dtype=torch.long, device=self.device)
        parts = [kv.pages[pages].reshape(-1).cpu() for kv in self._layers.values()]
        return {"values": torch.cat(parts) if parts else self.values.new_empty(0).cpu(), "length": self.pool.length(seq)}

    def import_pages(self, image: dict) -> int:
        seq = self.pool.new_seq()
        n = int(image["length"])
        try:
            self.pool.reserve(seq, n)
        except Exception:
            self.pool.free_seq(seq)
            raise
        pages = torch.tensor(self.pool.pages(seq), dtype=torch.long, device=self.device)
        off = 0
        for kv in self._layers.values():
            m = pages.numel() * kv.page_size * kv.pages.shape[2]
            kv.pages[pages] = image["values"][off:off + m].view(pages.numel(), kv.page_size, -1).to(self.device)
            off += m
        self.pool.commit(seq, n)
        return seq

    def export_token_major(self, seqs: list, max_tokens: int):
        raise ValueError("latent pages have no per-head keys and values to export")
