"""Generalised delta rule with a decay and a removal rate per key channel (kernels in csrc/delta_rule.cu; the PyTorch
branch restates them for CPU tensors).  State slots [dim keys, dim values] per head, fp32, updated in place."""
from __future__ import annotations

import ctypes as C
import math
from dataclasses import dataclass
from typing import Optional

import torch

from . import _lib

P, I, F, L = C.c_void_p, C.c_int, C.c_float, C.c_longlong


class DeltaArgs(C.Structure):
    _fields_ = [(n, P) for n in ("proj", "decay", "w2", "w0", "a_bias", "norm_w", "state", "row_off", "slots", "scratch", "out")] + \
        [("slot_stride", L), ("scratch_floats", L)] + \
        [(n, I) for n in ("ldp", "off_r", "off_k", "off_v", "off_a", "off_g", "off_w1", "rank", "ld_decay", "ld_w2", "heads", "dim",
                          "tokens", "sequences", "fp32", "decode")] + [("eps_u", F), ("eps", F)]


_SIGS = {
    "sllm_general_delta": (I, [P, P]),
    "sllm_tanh_rows": (I, [P, P, I, I, I, I, I, P]),
    "sllm_delta_abi": (I, [P, I]),
}
UNIT_EPS = 1e-6              # of the unit key u = k / sqrt(sum k^2 + UNIT_EPS)


def _k():
    for n, s in _SIGS.items():
        _lib.EXTRA_KERNEL_SIGNATURES.setdefault(n, s)
    return _lib.kernels()


@dataclass
class DeltaSpec:
    """Sizes of one layer and the columns of its packed input projection r | k | v | a | g | low-rank decay input."""
    heads: int
    dim: int
    rank: int

    @property
    def size(self) -> int:
        return self.heads * self.dim

    @property
    def columns(self) -> dict:
        n = self.size
        return {"r": 0, "k": n, "v": 2 * n, "a": 3 * n, "g": 4 * n, "w1": 5 * n}


def _pad(dim: int) -> int:
    p = 16
    while p < dim:
        p *= 2
    return p


def tanh_rows(x: torch.Tensor, n_pad: int) -> torch.Tensor:
    """tanh of [T, n] (row stride allowed), zero-padded to n_pad columns."""
    t, n = x.shape
    if _lib.on_cpu(x):
        y = torch.zeros((t, n_pad), dtype=x.dtype)
        y[:, :n] = torch.tanh(x.float()).to(x.dtype)
        return y
    from .core import _p, _stream
    y = torch.empty((t, n_pad), dtype=x.dtype, device=x.device)
    rc = _k().sllm_tanh_rows(_p(x), _p(y), t, x.stride(0), n, n_pad, int(x.dtype == torch.float32), _stream())
    _lib.check(rc, "tanh_rows")
    return y


def general_delta(proj: torch.Tensor, spec: DeltaSpec, w2, w0: torch.Tensor, a_bias: torch.Tensor, norm_w: torch.Tensor,
                  eps: float, state: torch.Tensor, row_off: torch.Tensor, slots: torch.Tensor, one_row_each: bool) -> torch.Tensor:
    """proj [T, *] packed projections, w2 LinearWeight [heads * dim, rank padded to 8]; state [slots, heads, dim, dim].
    ``one_row_each``: the batch holds exactly one row per sequence (a decode step).  Returns [T, heads * dim]."""
    t, H, D = proj.shape[0], spec.heads, spec.dim
    col = spec.columns
    if _lib.on_cpu(proj):
        f = lambda name: proj[:, col[name]:col[name] + H * D].float().view(t, H, D)
        r, k, v = f("r"), f("k"), f("v")
        low = torch.tanh(proj[:, col["w1"]:col["w1"] + spec.rank].float())
        w = torch.exp(-math.exp(-0.5) * torch.sigmoid(low @ w2.w[:, :spec.rank].float().t() + w0)).view(t, H, D)
        a = torch.sigmoid(f("a") + a_bias.view(H, D))
        u = k / torch.sqrt((k * k).sum(-1, keepdim=True) + UNIT_EPS)
        o = torch.empty((t, H, D))
        offs = row_off.tolist()
        for s, slot in enumerate(slots.tolist()):
            S = state[slot].clone()
            for i in range(offs[s], offs[s + 1]):
                old = torch.einsum("hk,hkv->hv", u[i], S)
                S = w[i].unsqueeze(-1) * S - (a[i] * u[i]).unsqueeze(-1) * old.unsqueeze(1) + k[i].unsqueeze(-1) * v[i].unsqueeze(1)
                o[i] = torch.einsum("hkv,hk->hv", S, r[i])
            state[slot] = S
        y = o / torch.sqrt((o * o).mean(-1, keepdim=True) + eps)
        return (y.view(t, H * D) * norm_w * torch.sigmoid(f("g").view(t, H * D))).to(proj.dtype)
    from .core import _p, _stream, linear
    out = torch.empty((t, H * D), dtype=proj.dtype, device=proj.device)
    decay: Optional[torch.Tensor] = None
    scratch: Optional[torch.Tensor] = None
    if not one_row_each:
        decay = linear(tanh_rows(proj[:, col["w1"]:col["w1"] + spec.rank], w2.in_features), w2)
        scratch = torch.empty(H * t * (5 * _pad(D) + (D + 3) // 4 * 4 + 4) + t * H * D, dtype=torch.float32, device=proj.device)
    v = lambda x: None if x is None else x.data_ptr()
    args = DeltaArgs(v(proj), v(decay), v(w2.w), v(w0), v(a_bias), v(norm_w), v(state), v(row_off), v(slots), v(scratch), v(out),
                     state.stride(0), 0 if scratch is None else scratch.numel(), proj.stride(0), col["r"], col["k"], col["v"],
                     col["a"], col["g"], col["w1"], spec.rank, 0 if decay is None else decay.stride(0), w2.w.stride(0), H, D, t,
                     slots.numel(), int(proj.dtype == torch.float32), int(one_row_each), UNIT_EPS, eps)
    _lib.check(_k().sllm_general_delta(C.byref(args), _stream()), "general_delta")
    return out
