"""Cache of models whose layers differ in kind and size: pages of any width for some layers, a recurrent state for others
(or for the same ones).

All paged layers share one page table.  A layer has one or more planes; a plane's page is [heads, page_size, width], head
major, its row stride padded to 16 bytes so that a page is a TMA box.  Planes of all layers live in one flat tensor
(``values``).  A layer's state is a list of 32-bit arrays per sequence slot; the states of all layers of a slot are one row
of ``states``.
"""
from __future__ import annotations

import math
from typing import Optional

import torch

from ..models.config import ModelConfig
from .hybrid import StateSlots
from .paged import KVSpec, PagedKVCache, PagePool

PAD = 8                                             # elements: 16 bytes of bf16, 32 of fp32


class LayeredCache(StateSlots, PagedKVCache):
    def __init__(self, cfg: ModelConfig, num_pages: int, device, max_seqs: int, planes: dict, states: dict):
        """planes: layer -> [(heads, width)]; states: layer, or a key of a state that is no layer's -> [shape]."""
        fmt = cfg.kv_format
        if fmt not in ("fp32", "bf16"):
            raise ValueError(f"pages of this cache are stored as bf16 or fp32, not {fmt!r}")
        self.device = torch.device(device)
        dt = torch.float32 if fmt == "fp32" else torch.bfloat16
        dims = [p for ps in planes.values() for p in ps]
        self.spec = KVSpec(len(planes), max((h for h, _ in dims), default=1), max((w for _, w in dims), default=0), cfg.page_size, fmt)
        self.pool = PagePool(num_pages, cfg.page_size)
        self.fp8 = self.nvfp4 = False
        self.scales: Optional[torch.Tensor] = None
        rows = num_pages * cfg.page_size
        padded = [(l, h, (w + PAD - 1) // PAD * PAD) for l, ps in planes.items() for h, w in ps]
        self._row = sum(h * ld for _, h, ld in padded)
        self.values = torch.zeros(rows * self._row, dtype=dt, device=self.device)
        self._planes: dict = {l: [] for l in planes}
        off = 0
        for l, h, ld in padded:
            n = rows * h * ld
            self._planes[l].append(self.values[off:off + n].view(num_pages, h, cfg.page_size, ld))
            off += n
        self._layers = {l: self.wrap(ts) for l, ts in self._planes.items()}
        offs, total = {}, 0
        for l, shapes in states.items():
            offs[l] = []
            for s in shapes:
                offs[l].append((total, s))
                total += (math.prod(s) + 3) // 4 * 4
        self.states = torch.zeros((max_seqs, max(total, 4)), dtype=torch.float32, device=self.device)
        self._states = {l: [self.states[:, o:o + math.prod(s)].unflatten(1, tuple(s)) for o, s in parts] for l, parts in offs.items()}
        self.init_slots(max_seqs, [(self.states, 0)])

    def wrap(self, planes: list):
        """What ``layer`` returns for a layer with these planes ([num_pages, heads, page, row stride] each)."""
        return planes

    def layer(self, i: int):
        return self._layers.get(i)

    def state(self, i, part: int = 0) -> torch.Tensor:
        """[slots, *shape] view of one of a layer's state arrays (the slot stride is the whole state row)."""
        return self._states[i][part]

    def bytes_per_token(self) -> int:
        return self._row * self.values.element_size()

    def copy_page(self, src: int, dst: int) -> None:
        for ts in self._planes.values():
            for t in ts:
                t[dst].copy_(t[src])

    def export_pages(self, seq: int) -> dict:
        pages = torch.tensor(self.pool.pages(seq), dtype=torch.long, device=self.device)
        parts = [t[pages].reshape(-1).cpu() for ts in self._planes.values() for t in ts]
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
        for ts in self._planes.values():
            for t in ts:
                m = pages.numel() * t[0].numel()
                t[pages] = image["values"][off:off + m].view(pages.numel(), *t.shape[1:]).to(self.device)
                off += m
        self.pool.commit(seq, n)
        return seq

    def export_token_major(self, seqs: list, max_tokens: int):
        raise ValueError("layers of different widths have no common token-major view")


class KVLayeredCache(LayeredCache):
    """Layers with keys and values of their own widths: planes [(kv_heads, dim), (kv_heads, vdim)]."""

    def wrap(self, planes: list):
        from ..ops.kv_attention import KVPages
        k, v = planes
        return KVPages(k, v, k.shape[2])
