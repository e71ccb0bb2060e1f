"""KV pages for the full-attention layers plus O(1) recurrent state for the gated-delta-net layers.

A sequence owns one state slot for its lifetime: per GDN layer a rolling convolution window
[taps - 1, qkv width] (bf16) and a recurrent matrix [value heads, 128, 128] (fp32) - the reference's
`[3, 8192]` + `[32, 128, 128]` per layer (crates/sllm-core/src/linear_attention.rs).  The state always
describes the end of the sequence's computed tokens, so a prefix can be shared only at exactly that point and a
rewind needs a snapshot (`snapshot` / `restore`, used by speculative rollback and context rebuilds).
"""
from __future__ import annotations

from typing import Optional

import torch

from ..models.config import ModelConfig
from .paged import PagedKVCache


class StateSlots:
    """Per-sequence recurrent state in slots.  ``state_planes``: [(tensor, slot dimension)]; a slot is zeroed when a
    sequence takes it, so slots can be used again in any order."""

    def init_slots(self, max_seqs: int, planes: list) -> None:
        self.max_seqs = max_seqs
        self.state_planes = planes
        self._free = list(range(max_seqs - 1, -1, -1))
        self.slot_of: dict = {}

    def alloc_slot(self, seq_id: int) -> int:
        if not self._free:
            raise RuntimeError("no free recurrent-state slot")
        s = self._free.pop()
        self.slot_of[seq_id] = s
        for t, dim in self.state_planes:
            t.select(dim, s).zero_()
        return s

    def free_slot(self, seq_id: int) -> None:
        s = self.slot_of.pop(seq_id, None)
        if s is not None:
            self._free.append(s)

    def copy_slot(self, src_seq: int, dst_seq: int) -> None:
        a, b = self.slot_of[src_seq], self.slot_of[dst_seq]
        for t, dim in self.state_planes:
            t.select(dim, b).copy_(t.select(dim, a))

    def snapshot(self, seq_id: int):
        s = self.slot_of[seq_id]
        return tuple(t.select(dim, s).clone() for t, dim in self.state_planes)

    def restore(self, seq_id: int, snap) -> None:
        s = self.slot_of[seq_id]
        for (t, dim), v in zip(self.state_planes, snap):
            t.select(dim, s).copy_(v)

    def save_all(self):
        """Every slot's state (a graph capture runs the step once more than it counts)."""
        return tuple(t.clone() for t, _ in self.state_planes)

    def load_all(self, saved) -> None:
        for (t, _), v in zip(self.state_planes, saved):
            t.copy_(v)


class HybridCache(StateSlots, PagedKVCache):
    def __init__(self, cfg: ModelConfig, num_pages: int, device, max_seqs: int, kv_heads: Optional[int] = None,
                 tp_size: int = 1):
        """``tp_size``: the gated-delta-net heads (and with them the conv and recurrent state) are split over that
        many tensor-parallel ranks; this cache holds one rank's share."""
        self.full_layers = [i for i in range(cfg.n_layers) if (i + 1) % cfg.full_attention_interval == 0]
        self.gdn_layers = [i for i in range(cfg.n_layers) if i not in self.full_layers]
        import dataclasses
        kv_cfg = dataclasses.replace(cfg, n_layers=max(1, len(self.full_layers)))
        super().__init__(kv_cfg, num_pages, device, kv_heads)
        self._kv_index = {l: j for j, l in enumerate(self.full_layers)}
        self._gdn_index = {l: j for j, l in enumerate(self.gdn_layers)}
        hd = cfg.gdn_head_dim
        self.width = (2 * cfg.gdn_qk_heads + cfg.gdn_heads) // tp_size * hd
        n = max(1, len(self.gdn_layers))
        self.conv_state = torch.zeros((n, max_seqs, cfg.gdn_conv_kernel - 1, self.width), dtype=torch.bfloat16 if
                                      torch.device(device).type == "cuda" or cfg.weight_format != "fp32" else torch.float32,
                                      device=device)
        self.rec_state = torch.zeros((n, max_seqs, cfg.gdn_heads // tp_size, hd, hd), dtype=torch.float32, device=device)
        self.init_slots(max_seqs, [(self.conv_state, 1), (self.rec_state, 1)])

    def layer(self, i: int):
        j = self._kv_index.get(i)
        return None if j is None else self._layers[j]

    def gdn(self, i: int):
        j = self._gdn_index[i]
        return self.conv_state[j], self.rec_state[j]
