"""Resident weights from named source tensors, for families whose configuration lists their layers."""
from __future__ import annotations

from typing import Callable

import torch

from ..ops.core import LinearWeight


def pad8(n: int) -> int:
    return (n + 7) // 8 * 8


class SourceTensors:
    """Checked access to source tensors.  ``get(name)`` returns one (any float type, any device), ``shapes`` says what is
    expected; matrices come in the model's type, vectors in fp32."""

    def __init__(self, cfg, get: Callable, shapes: dict, device):
        self.get, self.shapes, self.device = get, shapes, torch.device(device)
        self.dtype = torch.float32 if cfg.weight_format == "fp32" else torch.bfloat16

    def fetch(self, name: str) -> torch.Tensor:
        t, want = self.get(name), self.shapes[name]
        if want == () and t.numel() == 1:
            return t.reshape(())
        if tuple(t.shape) != want:
            raise ValueError(f"{name}: shape {tuple(t.shape)}, expected {want}")
        return t

    def raw(self, name: str) -> torch.Tensor:
        return self.fetch(name).to(device=self.device, dtype=self.dtype)

    def mat(self, *names) -> LinearWeight:
        return LinearWeight("dense", torch.cat([self.raw(n) for n in names], dim=0).contiguous())

    def f32(self, name: str) -> torch.Tensor:
        return self.fetch(name).to(device=self.device, dtype=torch.float32).contiguous()

    def vec(self, *names) -> torch.Tensor:
        return torch.cat([self.f32(n).reshape(-1) for n in names]).contiguous()

    def taps(self, *names) -> torch.Tensor:
        """Filters [channels, taps] of the named tensors, as [taps, all channels]."""
        return torch.cat([self.f32(n) for n in names]).t().contiguous()

    def second_factor(self, name: str) -> LinearWeight:
        """Second factor [n, rank] of a low-rank product, its rank padded with zeros to a multiple of 8."""
        w = self.raw(name)
        out = w.new_zeros((w.shape[0], pad8(w.shape[1])))
        out[:, :w.shape[1]] = w
        return LinearWeight("dense", out)

    def packed(self, prefix: str, parts: list):
        """One matrix of many: (LinearWeight, [(name, first row, rows)]).  parts: lists of names whose rows follow each other;
        every list starts at a multiple of 8 rows."""
        rows, blocks, at = [], [], 0
        for names in parts:
            for n in names:
                w = self.raw(prefix + n)
                rows.append((n, at, w.shape[0]))
                blocks.append(w)
                at += w.shape[0]
            if at % 8:
                blocks.append(blocks[-1].new_zeros((8 - at % 8, blocks[-1].shape[1])))
                at = pad8(at)
        return LinearWeight("dense", torch.cat(blocks).contiguous()), rows
