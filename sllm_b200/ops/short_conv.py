"""Short causal convolution with its inputs in a ring per state slot (PyTorch form; the CUDA kernels that consume the
convolution's result compute it themselves: csrc/kv_attention.cu, csrc/rglru.cu, csrc/linear_state.cu).

ring [slots, taps, channels], fp32: row (position mod taps) holds the conv input of that position, for the last ``taps``
positions of the slot's sequence.  A decoded token reads the rows of the taps - 1 positions before it and writes its own."""
from __future__ import annotations

import torch


def causal_conv(u: torch.Tensor, w: torch.Tensor, ring: torch.Tensor, row_off: torch.Tensor, slots: torch.Tensor,
                positions: torch.Tensor) -> torch.Tensor:
    """u [T, C] fp32 conv inputs of a flat batch, w [taps, C] (last row: the current token) -> [T, C]; the ring is updated."""
    taps = w.shape[0]
    y = torch.empty_like(u)
    offs = row_off.tolist()
    for s, slot in enumerate(slots.tolist()):
        r0, r1 = offs[s], offs[s + 1]
        if r0 == r1:
            continue
        p0 = int(positions[r0])
        past = [ring[slot, (p0 - b) % taps] if p0 - b >= 0 else torch.zeros_like(u[0]) for b in range(taps - 1, 0, -1)]
        x = torch.cat([torch.stack(past), u[r0:r1]]) if past else u[r0:r1]
        n = r1 - r0
        y[r0:r1] = sum(w[t] * x[t:t + n] for t in range(taps))
        for r in range(max(r0, r1 - taps), r1):
            ring[slot, (p0 + r - r0) % taps] = u[r]
    return y
