"""Gated linear recurrence of a Griffin-style block: short convolution, block-diagonal gates, per-channel fp32 state, GELU
output gate (kernels in csrc/rglru.cu; the PyTorch branch restates them for CPU tensors)."""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import Optional

import torch
import torch.nn.functional as F_

from . import _lib
from .short_conv import causal_conv

P, I, L = C.c_void_p, C.c_int, C.c_longlong
DECAY_SCALE = 8.0              # log a = -DECAY_SCALE * r * softplus(lambda)
TILE, CHANNELS, MAX_BLOCK, MAX_TAPS = 64, 128, 256, 4      # of the tensor-core form


class RglruArgs(C.Structure):
    _fields_ = [(n, P) for n in ("proj", "bias_y", "bias_x", "conv_w", "conv_b", "bias_r", "bias_i", "decay", "gate_r", "gate_i",
                                 "gate_tiles", "state", "ring", "row_off", "slots", "positions", "seq_index", "tiles", "h", "prod",
                                 "out", "status")] + \
        [("state_stride", L), ("ring_stride", L)] + \
        [(n, I) for n in ("ldp", "off_y", "off_x", "width", "blocks", "bs", "taps", "tokens", "sequences", "n_tiles", "fp32", "decode")]


_SIGS = {"sllm_rglru": (I, [P, P]), "sllm_rglru_simt": (I, [P, P]), "sllm_rglru_abi": (I, [P, I])}


def _k():
    for n, s in _SIGS.items():
        _lib.EXTRA_KERNEL_SIGNATURES.setdefault(n, s)
    return _lib.kernels()


@dataclass
class RglruSpec:
    """Sizes of one layer; its packed input projection is y | x."""
    width: int
    blocks: int
    taps: int

    @property
    def block(self) -> int:
        return self.width // self.blocks


@dataclass
class RglruWeights:
    """Vectors are fp32; gates [blocks, out, in] in the model's type, ``tiles`` their packed form for the tensor-core kernel."""
    bias_y: torch.Tensor
    bias_x: torch.Tensor
    conv_w: torch.Tensor       # [taps, width], last row: the current token
    conv_b: torch.Tensor
    gate_r: torch.Tensor
    gate_i: torch.Tensor
    bias_r: torch.Tensor       # [width]
    bias_i: torch.Tensor
    lam: torch.Tensor
    decay: torch.Tensor        # -DECAY_SCALE softplus(lam)
    tiles: Optional[torch.Tensor] = None

    @staticmethod
    def make(spec: RglruSpec, **kw) -> "RglruWeights":
        kw["decay"] = -DECAY_SCALE * F_.softplus(kw["lam"].double()).float()
        w = RglruWeights(**kw)
        if w.gate_r.is_cuda and tensor_core(spec, w.gate_r.dtype):
            w.tiles = pack_gates(spec, w.gate_r, w.gate_i)
        return w


def tensor_core(spec: RglruSpec, dtype) -> bool:
    """Whether the tensor-core form takes this layer."""
    return dtype == torch.bfloat16 and spec.block % 8 == 0 and spec.block <= MAX_BLOCK and spec.taps <= MAX_TAPS


def pack_gates(spec: RglruSpec, gate_r: torch.Tensor, gate_i: torch.Tensor) -> torch.Tensor:
    """[blocks, channel tiles, 2, 128, block padded to 64], zero padded."""
    b = spec.block
    ct, kp = (b + CHANNELS - 1) // CHANNELS, (b + 63) // 64 * 64
    out = gate_r.new_zeros((spec.blocks, 2, ct * CHANNELS, kp))
    out[:, 0, :b, :b], out[:, 1, :b, :b] = gate_r, gate_i
    return out.view(spec.blocks, 2, ct, CHANNELS, kp).transpose(1, 2).contiguous()


def plan_tiles(row_off: list, device) -> torch.Tensor:
    """int32 [tiles, 4]: first row, rows, sequence, tile number within the sequence | last << 24."""
    out = []
    for s in range(len(row_off) - 1):
        r0, r1 = row_off[s], row_off[s + 1]
        n = (r1 - r0 + TILE - 1) // TILE
        out += [(r0 + TILE * c, min(TILE, r1 - r0 - TILE * c), s, c | (int(c == n - 1) << 24)) for c in range(n)]
    return torch.tensor(out, dtype=torch.int32, device=device)


def terms(u: torch.Tensor, spec: RglruSpec, w: RglruWeights) -> tuple:
    """(a, b) of S <- a S + b for conv outputs u [T, width], fp32."""
    t = u.shape[0]
    x = u.view(t, spec.blocks, spec.block)
    r = torch.sigmoid(torch.einsum("tbi,boi->tbo", x, w.gate_r.float()).reshape(t, -1) + w.bias_r)
    i = torch.sigmoid(torch.einsum("tbi,boi->tbo", x, w.gate_i.float()).reshape(t, -1) + w.bias_i)
    la = w.decay * r
    return torch.exp(la), torch.sqrt(-torch.expm1(2 * la)) * i * u


def rglru(proj: torch.Tensor, spec: RglruSpec, w: RglruWeights, state: torch.Tensor, ring: torch.Tensor, b,
          impl: Optional[str] = None) -> torch.Tensor:
    """proj [T, >= 2 width] = y | x projections of a ForwardBatch's rows (biases not yet added); state [slots, width] and ring
    [slots, taps, width] are fp32 views with a common slot stride.  Returns S gelu(y), [T, width].  ``impl`` "cuda_core"
    forces the any-size kernels."""
    t, W = proj.shape[0], spec.width
    if _lib.on_cpu(proj):
        u = causal_conv(proj[:, W:2 * W].float() + w.bias_x, w.conv_w, ring, b.row_off, b.slots, b.positions) + w.conv_b
        a, x = terms(u, spec, w)
        y = F_.gelu(proj[:, :W].float() + w.bias_y, approximate="tanh")
        out = torch.empty((t, W), dtype=torch.float32)
        offs = b.row_off.tolist()
        for s, slot in enumerate(b.slots.tolist()):
            S = state[slot].clone()
            for r in range(offs[s], offs[s + 1]):
                S = a[r] * S + x[r]
                out[r] = S
            state[slot] = S
        return (out * y).to(proj.dtype)
    from .core import _p, _stream, workspace
    decode = b.row_off_host is None and t == b.slots.numel()
    fast = w.tiles is not None and impl != "cuda_core" and (decode or b.row_off_host is not None)
    out = torch.empty((t, W), dtype=proj.dtype, device=proj.device)
    h = prod = tiles = None
    if not (fast and decode):
        h, prod = (torch.empty((t, W), dtype=torch.float32, device=proj.device) for _ in range(2))
    if fast and not decode:
        tiles = b.plans.get("rglru")
        if tiles is None:
            tiles = b.plans["rglru"] = plan_tiles(b.row_off_host, proj.device)
    v = lambda x: None if x is None else x.data_ptr()
    args = RglruArgs(v(proj), v(w.bias_y), v(w.bias_x), v(w.conv_w), v(w.conv_b), v(w.bias_r), v(w.bias_i), v(w.decay), v(w.gate_r),
                     v(w.gate_i), v(w.tiles), v(state), v(ring), v(b.row_off), v(b.slots), v(b.positions), v(b.seq_index), v(tiles),
                     v(h), v(prod), v(out), v(workspace(proj.device).status), state.stride(0), ring.stride(0), proj.stride(0), 0, W, W,
                     spec.blocks, spec.block, spec.taps, t, b.slots.numel(), 0 if tiles is None else tiles.shape[0],
                     int(proj.dtype == torch.float32), int(decode))
    if _lib.audit_enabled():
        _lib.record_dispatch("rglru", "rglru_tile_kernel" if fast else "rglru_terms_kernel", rows=t, width=W, blocks=spec.blocks,
                             decode=decode)
    fn = _k().sllm_rglru if fast else _k().sllm_rglru_simt
    _lib.check(fn(C.byref(args), _stream()), "rglru")
    return out
