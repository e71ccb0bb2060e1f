"""Linear attention with a matrix-valued fp32 state per head: gated linear attention, retention, and a delta rule with a decay
per key channel or per head (kernels in csrc/linear_state.cu; the PyTorch branch restates them for CPU tensors)."""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import Optional

import torch
import torch.nn.functional as F_

from . import _lib
from .short_conv import causal_conv

P, I, F, L = C.c_void_p, C.c_int, C.c_float, C.c_longlong
GATED, FIXED, DELTA, HEAD_DELTA = 0, 1, 2, 3
UNIT_EPS = 1e-6              # of the delta forms' unit vectors x / sqrt(sum x^2 + UNIT_EPS)


class LinearStateArgs(C.Structure):
    _fields_ = [(n, P) for n in ("proj", "decay", "gate", "w_a", "w_g", "bias", "rate", "conv_w", "ring", "norm_w", "state", "row_off", "slots",
                                 "positions", "seq_index", "scratch", "out")] + \
        [(n, L) for n in ("ring_stride", "slot_stride", "scratch_floats")] + \
        [(n, I) for n in ("form", "ldp", "off_q", "off_k", "off_v", "off_g", "off_a", "off_b", "ld_decay", "ld_gate", "ld_wa", "ld_wg", "rank_a",
                          "rank_g", "taps", "heads", "kv_heads", "dim", "vdim", "tokens", "sequences", "fp32", "decode")] + \
        [(n, F) for n in ("inv_tau", "q_scale", "k_scale", "unit_eps", "eps")]


_SIGS = {
    "sllm_linear_state": (I, [P, P]),
    "sllm_linear_state_abi": (I, [P, I]),
    "sllm_linear_state_floats": (L, [I, I, I, I, I]),
}


def _k():
    for n, s in _SIGS.items():
        _lib.EXTRA_KERNEL_SIGNATURES.setdefault(n, s)
    return _lib.kernels()


@dataclass
class StateSpec:
    """Sizes and constants of one layer.  ``form``: GATED (decay sigmoid(z)^(1 / tau) per key channel, z low-rank), FIXED (one
    decay per head), DELTA (delta rule with a decay exp(-rate softplus(z)) per key channel, short convolutions with SiLU on q,
    k and v, unit query and key) or HEAD_DELTA (the same with one decay per head, z a column of the projection plus a bias, and
    an output gate as in the first two).  ``columns``: where the parts of the packed input projection start: q, k, v, g, a
    (low-rank decay input, in the head form z), b (write strengths); in the delta forms q, k and v are consecutive, and in the
    channel form g is the gate's low-rank input."""
    form: int
    heads: int
    kv_heads: int            # query / key heads (value heads are a multiple)
    dim: int
    vdim: int
    columns: dict
    q_scale: float = 1.0
    k_scale: float = 1.0
    tau: float = 1.0
    taps: int = 1
    rank_a: int = 0
    rank_g: int = 0

    @property
    def delta(self) -> bool:
        return self.form in (DELTA, HEAD_DELTA)

    @property
    def channels(self) -> int:
        """Columns that the short convolution covers."""
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim

    @property
    def out_cols(self) -> int:
        return self.heads * self.vdim


@dataclass
class StateWeights:
    """Vectors are fp32; the low-rank second factors [*, rank padded to 8] are in the model's type."""
    w_a: Optional[object] = None                # LinearWeight [heads * dim, rank_a padded]
    w_g: Optional[object] = None                # LinearWeight [heads * vdim, rank_g padded]
    bias: Optional[torch.Tensor] = None         # [heads * dim], of z (HEAD_DELTA: [heads])
    rate: Optional[torch.Tensor] = None         # [heads]: the decay itself (FIXED), exp(A_log) (the delta forms)
    conv_w: Optional[torch.Tensor] = None       # [taps, channels], last row: the current token
    norm: Optional[torch.Tensor] = None         # [vdim]


def _recur(q, k, v, g, beta, state, b) -> torch.Tensor:
    """q, k, g [T, H, D], v [T, H, V], beta [T, H] or None (no removal); state updated in place."""
    o = torch.empty_like(v)
    offs = b.row_off.tolist()
    for s, slot in enumerate(b.slots.tolist()):
        S = state[slot].clone()
        for r in range(offs[s], offs[s + 1]):
            S = g[r].unsqueeze(-1) * S
            u = v[r] if beta is None else beta[r].unsqueeze(-1) * (v[r] - torch.einsum("hkv,hk->hv", S, k[r]))
            S = S + k[r].unsqueeze(-1) * u.unsqueeze(1)
            o[r] = torch.einsum("hkv,hk->hv", S, q[r])
        state[slot] = S
    return o


def _cpu(proj, spec: StateSpec, w: StateWeights, eps, state, ring, b) -> torch.Tensor:
    t, H, G, D, V, col = proj.shape[0], spec.heads, spec.kv_heads, spec.dim, spec.vdim, spec.columns
    f = lambda name, n: proj[:, col[name]:col[name] + n].float()
    low = lambda name, r, m: f(name, r) @ m.w[:, :r].float().t()
    if spec.delta:
        x = F_.silu(causal_conv(f("q", spec.channels), w.conv_w, ring, b.row_off, b.slots, b.positions))
        q, k, v = x.split([G * D, G * D, H * V], dim=1)
    else:
        q, k, v = f("q", G * D), f("k", G * D), f("v", H * V)
    q, k, v = q.reshape(t, G, D), k.reshape(t, G, D), v.reshape(t, H, V)
    beta = None
    if spec.delta:
        q, k = (y / torch.sqrt((y * y).sum(-1, keepdim=True) + UNIT_EPS) for y in (q, k))
        beta = torch.sigmoid(f("b", H))
    q, k = ((y * s).repeat_interleave(H // G, dim=1) for y, s in ((q, spec.q_scale), (k, spec.k_scale)))
    if spec.form == FIXED:
        g = w.rate.view(1, H, 1).expand(t, H, D)
    elif spec.form == HEAD_DELTA:
        g = torch.exp(-w.rate * F_.softplus(f("a", H) + w.bias)).unsqueeze(-1).expand(t, H, D)
    else:
        z = (low("a", spec.rank_a, w.w_a) + w.bias).view(t, H, D)
        g = torch.exp(-F_.softplus(-z) / spec.tau) if spec.form == GATED else torch.exp(-w.rate.view(1, H, 1) * F_.softplus(z))
    o = _recur(q, k, v, g, beta, state, b)
    o = o / torch.sqrt((o * o).mean(-1, keepdim=True) + eps)
    if w.norm is not None:
        o = o * w.norm
    gate = torch.sigmoid(low("g", spec.rank_g, w.w_g)) if spec.form == DELTA else F_.silu(f("g", H * V))
    return (o.reshape(t, H * V) * gate).to(proj.dtype)


def linear_state(proj: torch.Tensor, spec: StateSpec, w: StateWeights, eps: float, state: torch.Tensor, ring: Optional[torch.Tensor],
                 b) -> torch.Tensor:
    """proj [T, *] packed projections of a ForwardBatch's rows; state [slots, heads, dim, vdim] and ring [slots, taps, channels]
    (delta forms) are fp32 views with a common slot stride, updated in place.  Returns [T, heads * vdim], normed and gated."""
    t, H, D, V, col = proj.shape[0], spec.heads, spec.dim, spec.vdim, spec.columns
    if _lib.on_cpu(proj):
        return _cpu(proj, spec, w, eps, state, ring, b)
    from .core import _stream, linear
    decode = b.row_off_host is None and t == b.slots.numel()
    out = torch.empty((t, spec.out_cols), dtype=proj.dtype, device=proj.device)
    decay = gate = scratch = None
    if not decode:
        if spec.form in (GATED, DELTA):
            decay = linear(proj[:, col["a"]:col["a"] + w.w_a.in_features], w.w_a, out_fp32=True)
        if spec.form == DELTA:
            gate = linear(proj[:, col["g"]:col["g"] + w.w_g.in_features], w.w_g)
        scratch = torch.empty(int(_k().sllm_linear_state_floats(spec.form, H, D, V, t)), dtype=torch.float32, device=proj.device)
    v = lambda x: None if x is None else x.data_ptr()
    lw = lambda x: None if x is None else x.w.data_ptr()
    ld = lambda x: 0 if x is None else x.w.stride(0)
    st = lambda x: 0 if x is None else x.stride(0)
    args = LinearStateArgs(v(proj), v(decay), v(gate), lw(w.w_a), lw(w.w_g), v(w.bias), v(w.rate), v(w.conv_w), v(ring), v(w.norm), v(state),
                           v(b.row_off), v(b.slots), v(b.positions), v(b.seq_index), v(scratch), v(out), st(ring), state.stride(0),
                           0 if scratch is None else scratch.numel(), spec.form, proj.stride(0), col["q"], col["k"], col["v"], col["g"],
                           col.get("a", 0), col.get("b", 0), st(decay), st(gate), ld(w.w_a), ld(w.w_g), spec.rank_a, spec.rank_g, spec.taps, H,
                           spec.kv_heads, D, V, t, b.slots.numel(), int(proj.dtype == torch.float32), int(decode), 1.0 / spec.tau, spec.q_scale,
                           spec.k_scale, UNIT_EPS, eps)
    if _lib.audit_enabled():
        _lib.record_dispatch("linear_state", "linear_decode_kernel" if decode else "state_scan_kernel", rows=t, heads=H, dim=D, vdim=V,
                             form=spec.form)
    _lib.check(_k().sllm_linear_state(C.byref(args), _stream()), "linear_state")
    return out
