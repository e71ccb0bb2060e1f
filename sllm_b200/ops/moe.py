"""Mixture-of-experts ops: routing, permutation, grouped expert GEMMs, combine - CUDA kernels with CPU oracles.

The CPU path is the oracle of the same contract (reference: reference_sparse_moe_route,
crates/sllm-core/src/moe.rs:229: top-k by logit, ties to the lower index, softmax over the selected logits).
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import Optional

import torch

from . import _lib
from .w4 import W4Weight, linear_w4

P, I, L, F = C.c_void_p, C.c_int, C.c_longlong, C.c_float
_SIGS = {
    "sllm_moe_route": (I, [P, I, I, P, I, P, P, P]),
    "sllm_moe_router": (I, [P, I, P, I, I, P, I, P, P, P]),
    "sllm_moe_route_abi": (I, [P, I]),
    "sllm_moe_grouped": (I, [P, P, P, I, I, I, I, P, F, F, F, P, I, I, I, I, I, P, P]),
    "sllm_moe_grouped_simt": (I, [P, I, P, P, P, I, I, I, I, P, F, F, F, P, I, I, I, I, P]),
    "sllm_moe_permute": (I, [P, P, I, I, I, I, P, P, P, P, P, P]),
    "sllm_moe_gather": (I, [P, I, P, P, I, P, I, I, P]),
    "sllm_moe_combine": (I, [P, P, I, P, P, I, I, P]),
    "sllm_moe_shared_add": (I, [P, P, P, I, P, I, I, P]),
    "sllm_moe_owner_plan": (I, [P, P, P, I, I, L, L, P, I, I, I, I, P, P, P]),
    "sllm_moe_owner_combine": (I, [P, P, P, I, I, L, L, I, P, P, I, I, I, I, P, P, P, P]),
    "sllm_moe_combine_allreduce": (I, [P, P, I, I, P, P, I, P, P, I, I, I, L, I, P, P, P]),
}


def _k():
    for n, s in _SIGS.items():
        _lib.EXTRA_KERNEL_SIGNATURES.setdefault(n, s)
    return _lib.kernels()


class RouteArgs(C.Structure):
    _fields_ = [("correction", P)] + [(n, I) for n in ("experts", "top_k", "mode", "groups", "keep", "group_top")] + [("scale", F)]


@dataclass
class SigmoidScores:
    """Experts are chosen by sigmoid(logit) + correction; their weights are scale * sigmoid(logit), not renormalised."""
    correction: Optional[torch.Tensor] = None      # fp32 [E]
    scale: float = 1.0


def _route_args(e: int, top_k: int, softmax_all: bool, groups: int, keep: int, group_top: int, sigmoid: Optional[SigmoidScores]):
    c = None if sigmoid is None or sigmoid.correction is None else sigmoid.correction.data_ptr()
    return C.byref(RouteArgs(c, e, top_k, 2 if sigmoid is not None else int(softmax_all), groups, keep, group_top,
                             1.0 if sigmoid is None else sigmoid.scale))


def route(logits: torch.Tensor, top_k: int, softmax_all: bool = False, groups: int = 1, keep: int = 1, group_top: int = 1,
          sigmoid: Optional[SigmoidScores] = None):
    """[T, E] (bf16 or fp32) -> (idx int32 [T, k], weights fp32 [T, k]).  ``groups`` > 1: neighbouring experts form equal
    groups, a group's score is the sum of its ``group_top`` (1 or 2) largest, and only experts of the ``keep`` best groups are
    selected.  ``sigmoid`` replaces the softmax."""
    t, e = logits.shape
    if _lib.on_cpu(logits):
        lf = torch.nan_to_num(logits.float(), nan=float("-inf"))
        if sigmoid is not None:
            score = torch.sigmoid(lf)
            lf = score if sigmoid.correction is None else score + sigmoid.correction
        pick = lf
        if groups > 1 and keep < groups:
            top = lf.view(t, groups, e // groups).topk(min(group_top, e // groups), -1).values.sum(-1)
            best = torch.sort(-top, dim=1, stable=True).indices[:, :keep]
            shut = torch.ones((t, groups), dtype=torch.bool).scatter(1, best, False)
            pick = lf.masked_fill(shut.repeat_interleave(e // groups, dim=1), float("-inf"))
        # stable ordering: larger logit first, ties to the lower index
        order = torch.sort(-pick, dim=1, stable=True).indices[:, :top_k]
        sel = torch.gather(lf, 1, order)
        if sigmoid is not None:
            w = score.gather(1, order) * sigmoid.scale
        elif softmax_all:
            w = torch.softmax(lf, dim=1).gather(1, order)
        else:
            w = torch.softmax(sel, dim=1)
        return order.to(torch.int32), w.float()
    from .core import _p, _stream
    idx = torch.empty((t, top_k), dtype=torch.int32, device=logits.device)
    w = torch.empty((t, top_k), dtype=torch.float32, device=logits.device)
    rc = _k().sllm_moe_route(_p(logits), logits.stride(0), t, _route_args(e, top_k, softmax_all, groups, keep, group_top, sigmoid),
                             int(logits.dtype == torch.float32), _p(idx), _p(w), _stream())
    _lib.check(rc, "moe_route")
    return idx, w


ROUTER_FUSED_ROWS = 64         # up to this many tokens the product and the selection are one launch


def router(x: torch.Tensor, w, top_k: int, softmax_all: bool = False, groups: int = 1, keep: int = 1, group_top: int = 1,
           sigmoid: Optional[SigmoidScores] = None):
    """Routing from fp32 router logits: x [T, d], w LinearWeight [E, d] of the type of x.  Returns (idx, weights) as `route`."""
    from . import core
    t, e = x.shape[0], w.out_features
    if _lib.on_cpu(x) or (t > ROUTER_FUSED_ROWS and x.dtype == torch.bfloat16 and w.in_features % 8 == 0):
        return route(core.linear(x, w, out_fp32=True), top_k, softmax_all, groups, keep, group_top, sigmoid)
    idx = torch.empty((t, top_k), dtype=torch.int32, device=x.device)
    wt = torch.empty((t, top_k), dtype=torch.float32, device=x.device)
    rc = _k().sllm_moe_router(core._p(x), x.stride(0), core._p(w.w), t, w.in_features,
                              _route_args(e, top_k, softmax_all, groups, keep, group_top, sigmoid), int(x.dtype == torch.float32),
                              core._p(idx), core._p(wt), core._stream())
    _lib.check(rc, "moe_router")
    return idx, wt


PERMUTE_CHUNK = 1024           # assignments of one CTA of the chunked permutation


def permute(idx: torch.Tensor, w: torch.Tensor, e_lo: int, e_hi: int):
    """Groups assignments by local expert.  Returns (tok_off [n_local + 1], perm_src [T*k], perm_dst [T, k],
    perm_w [T*k]); rows beyond tok_off[-1] are unused."""
    t, k = idx.shape
    n_local = e_hi - e_lo
    dev = idx.device
    tok_off = torch.zeros(n_local + 1, dtype=torch.int32, device=dev)
    perm_src = torch.zeros(t * k, dtype=torch.int32, device=dev)
    perm_dst = torch.full((t, k), -1, dtype=torch.int32, device=dev)
    perm_w = torch.zeros(t * k, dtype=torch.float32, device=dev)
    if _lib.on_cpu(idx):
        flat = idx.reshape(-1).tolist()
        wf = w.reshape(-1).tolist()
        cur = 0
        for e in range(e_lo, e_hi):
            tok_off[e - e_lo] = cur
            for a, ex in enumerate(flat):
                if ex == e:
                    perm_src[cur] = a // k
                    perm_w[cur] = wf[a]
                    perm_dst[a // k, a % k] = cur
                    cur += 1
        tok_off[n_local] = cur
        return tok_off, perm_src, perm_dst, perm_w
    from .core import _p, _stream
    chunks = (t * k + PERMUTE_CHUNK - 1) // PERMUTE_CHUNK
    counts = torch.empty(chunks * n_local, dtype=torch.int32, device=dev) if chunks > 1 else None
    rc = _k().sllm_moe_permute(_p(idx), _p(w), t, k, e_lo, e_hi, _p(tok_off), _p(perm_src), _p(perm_dst), _p(perm_w), _p(counts), _stream())
    _lib.check(rc, "moe_permute")
    return tok_off, perm_src, perm_dst, perm_w


def gather(x: torch.Tensor, perm_src: torch.Tensor, tok_off: torch.Tensor) -> torch.Tensor:
    rows = perm_src.numel()
    if _lib.on_cpu(x):
        return x[perm_src.long()]
    from .core import _p, _stream
    xp = torch.empty((rows, x.shape[1]), dtype=torch.bfloat16, device=x.device)
    rc = _k().sllm_moe_gather(_p(x), x.stride(0), _p(perm_src), _p(tok_off), tok_off.numel() - 1, _p(xp), x.shape[1], rows,
                              _stream())
    _lib.check(rc, "moe_gather")
    return xp


def combine(yp: torch.Tensor, perm_dst: torch.Tensor, residual: Optional[torch.Tensor]) -> torch.Tensor:
    t, k = perm_dst.shape
    d = yp.shape[1]
    if _lib.on_cpu(yp):
        out = torch.zeros((t, d), dtype=torch.float32)
        for j in range(k):
            p = perm_dst[:, j].long()
            m = p >= 0
            out[m] += yp.float()[p[m]]
        if residual is not None:
            out = out + residual.float()
        return out if yp.dtype == torch.float32 else out.to(torch.bfloat16)
    from .core import _p, _stream
    y = torch.empty((t, d), dtype=torch.bfloat16, device=yp.device)
    rc = _k().sllm_moe_combine(_p(yp), _p(perm_dst), k, _p(residual), _p(y), t, d, _stream())
    _lib.check(rc, "moe_combine")
    return y


def shared_add(a: torch.Tensor, b: torch.Tensor, gate: torch.Tensor) -> torch.Tensor:
    """a + sigmoid(gate) * b with one gate logit per row: a, b [T, d]; gate [T] (any stride, e.g. a column of the
    router logits)."""
    if _lib.on_cpu(a):
        out = a.float() + torch.sigmoid(gate.float()).unsqueeze(1) * b.float()
        return out if a.dtype == torch.float32 else out.to(torch.bfloat16)
    from .core import _p, _stream
    y = torch.empty_like(a)
    rc = _k().sllm_moe_shared_add(_p(a), _p(b), _p(gate), gate.stride(0), _p(y), a.shape[0], a.shape[1], _stream())
    _lib.check(rc, "moe_shared_add")
    return y


def expert_mlp(x: torch.Tensor, tok_off: torch.Tensor, perm_src: torch.Tensor, perm_w: torch.Tensor, gate_up: W4Weight,
               down: W4Weight, act: str, row_ptr: Optional[torch.Tensor] = None) -> Optional[torch.Tensor]:
    """The gated MLP of the local experts over the routed rows (grouped by expert: `tok_off`), routing weights applied:
    y_perm [T*k, d], or None when `row_ptr` scatters the rows (see `linear_w4`).

    W4A16 (default): gather rows -> grouped gate_up GEMM -> SiLU*up -> grouped down GEMM, bf16 activations.
    W4A4 (`ops.w4.set_w4a4`): the quantiser reads the routed rows in place (no gather), both GEMMs run on the
    block-scaled 4-bit tensor-core kernel, and SiLU*up is computed inside the quantiser of the down projection
    (reference: the fused expert kernels, native/hip/src/moe_expert_kernel.hip.cpp:88,176)."""
    from . import core
    from . import w4 as W
    t = x.shape[0]
    # 4-bit activations serve the decode regime; with more than 32 routed rows per expert on average (a prompt) the
    # rows are compute bound and keep bf16 activations on the W4A16 kernel, whose token tiles are 128 wide
    if W.w4a4_enabled() and x.dtype == torch.bfloat16 and perm_src.numel() <= W.W4A4_MAX_DENSE_ROWS * gate_up.groups:
        rows = perm_src.numel()
        n_rows = tok_off[-1:] if x.is_cuda else None
        if not x.is_cuda:
            rows = int(tok_off[-1])
        q = W.act_quant_fp4(x, gate_up.fmt, src_row=perm_src, tokens=rows, n_rows=n_rows)
        gu = W.linear_w4a4(None, gate_up, tok_off=tok_off, max_group_tokens=t, quantized=q)
        q2 = W.act_quant_fp4(gu, down.fmt, n_rows=n_rows, gated=act)
        y = W.linear_w4a4(None, down, tok_off=tok_off, tok_scale=perm_w[:rows], max_group_tokens=t, quantized=q2,
                          row_ptr=row_ptr)
        if y is not None and y.shape[0] < perm_src.numel():
            y = torch.cat([y, y.new_zeros((perm_src.numel() - y.shape[0], y.shape[1]))])
        return y
    xp = gather(x, perm_src, tok_off)
    a = core.gated_act(linear_w4(xp, gate_up, tok_off=tok_off, max_group_tokens=t), act)
    return linear_w4(a, down, tok_off=tok_off, tok_scale=perm_w, max_group_tokens=t, row_ptr=row_ptr)


def experts_forward(x: torch.Tensor, idx: torch.Tensor, w: torch.Tensor, gate_up: W4Weight, down: W4Weight, act: str,
                    e_lo: int, e_hi: int):
    """Runs the local experts [e_lo, e_hi) on the tokens routed to them.  Returns (y_perm [T*k, d] with the routing
    weights applied, perm_dst [T, k])."""
    tok_off, perm_src, perm_dst, perm_w = permute(idx, w, e_lo, e_hi)
    return expert_mlp(x, tok_off, perm_src, perm_w, gate_up, down, act), perm_dst


# ------------------------------------------------------------------------------------------ experts with dense weights
@dataclass
class GatedAct:
    """g sigmoid(alpha g) (u + shift) with g = min(gate, limit), u = clamp(up, -limit, limit).  alpha 1, shift 0 and an
    infinite limit give SiLU(gate) * up."""
    limit: float = float("inf")
    alpha: float = 1.0
    shift: float = 0.0


GATE_BLOCK = 64                # gate rows, then the up rows of the same features, in blocks of this many


@dataclass
class ExpertBank:
    """bf16 / fp32 experts of one layer.  gate_up [E, 2 * padded, d]: blocks of 64 gate rows and the 64 up rows of the same
    features; down [E, d, padded]; ``ff`` real features, the rest is zero."""
    gate_up: torch.Tensor
    down: torch.Tensor
    ff: int
    act: GatedAct

    @property
    def experts(self) -> int:
        return self.gate_up.shape[0]

    @property
    def padded(self) -> int:
        return self.down.shape[2]

    @staticmethod
    def pack(gates: list, ups: list, downs: list, act: GatedAct) -> "ExpertBank":
        """Per-expert [ff, d], [ff, d] and [d, ff] matrices."""
        ff, d = gates[0].shape
        n = (ff + GATE_BLOCK - 1) // GATE_BLOCK * GATE_BLOCK
        gate_up = gates[0].new_zeros((len(gates), n // GATE_BLOCK, 2, GATE_BLOCK, d))
        down = gates[0].new_zeros((len(gates), d, n))
        for e, (g, u, w) in enumerate(zip(gates, ups, downs)):
            for part, m in enumerate((g, u)):
                rows = m.new_zeros((n, d))
                rows[:ff] = m
                gate_up[e, :, part] = rows.view(-1, GATE_BLOCK, d)
            down[e, :, :ff] = w
        return ExpertBank(gate_up.view(len(gates), 2 * n, d), down, ff, act)

    def matrices(self, e: int) -> tuple:
        """(gate, up, down) of expert ``e``: the inverse of `pack`."""
        d = self.gate_up.shape[2]
        g = self.gate_up[e].view(-1, 2, GATE_BLOCK, d)
        return (g[:, 0].reshape(-1, d)[:self.ff], g[:, 1].reshape(-1, d)[:self.ff], self.down[e, :, :self.ff])


def _grouped(x, src, w, tok_off, mode, row_w, act, features, rows, tile_rows, bn):
    from .core import _p, _stream, workspace
    e, n, k = w.shape
    y = torch.empty((rows, features), dtype=x.dtype, device=x.device)
    if tile_rows:
        rc = _k().sllm_moe_grouped(_p(x), _p(w), _p(tok_off), e, n, k, mode, _p(row_w), act.limit, act.alpha, act.shift, _p(y), features,
                                   features, rows, tile_rows, bn, _p(workspace(x.device).status), _stream())
    else:
        rc = _k().sllm_moe_grouped_simt(_p(x), x.stride(0), _p(src), _p(w), _p(tok_off), e, n, k, mode, _p(row_w), act.limit, act.alpha,
                                        act.shift, _p(y), features, features, rows, int(x.dtype == torch.float32), _stream())
    _lib.check(rc, "moe_grouped")
    return y


def bank_forward(x: torch.Tensor, idx: torch.Tensor, w: torch.Tensor, bank: ExpertBank):
    """The experts' outputs with routing weights applied: (y_perm [T * k, d], perm_dst [T, k]); row perm_dst[t, j] belongs to
    the j-th expert of token t (`combine` or `add_group_norm(terms=)` sum them)."""
    tok_off, perm_src, perm_dst, perm_w = permute(idx, w, 0, bank.experts)
    d, act = x.shape[1], bank.act
    if _lib.on_cpu(x):
        y = torch.zeros((perm_src.numel(), d), dtype=x.dtype)
        offs = tok_off.tolist()
        for e in range(bank.experts):
            lo, hi = offs[e], offs[e + 1]
            if lo == hi:
                continue
            gate, up, down = (m.float() for m in bank.matrices(e))
            h = x[perm_src[lo:hi].long()].float()
            g, u = torch.clamp(h @ gate.t(), max=act.limit), torch.clamp(h @ up.t(), min=-act.limit, max=act.limit)
            a = (g * torch.sigmoid(act.alpha * g) * (u + act.shift)).to(x.dtype).float()
            y[lo:hi] = ((a @ down.t()) * perm_w[lo:hi, None]).to(x.dtype)
        return y, perm_dst
    rows = perm_src.numel()
    if x.dtype == torch.float32 or d % 8:
        a = _grouped(x, perm_src, bank.gate_up, tok_off, 0, None, act, bank.padded, rows, 0, 0)
        return _grouped(a, None, bank.down, tok_off, 1, perm_w, act, d, rows, 0, 0), perm_dst
    tile_rows, bn = (32, 128) if rows <= 24 * bank.experts else (128, 256)
    if _lib.audit_enabled():
        _lib.record_dispatch("moe_experts", "grouped_gemm_kernel", rows=rows, experts=bank.experts, d=d, ff=bank.ff, tile_rows=tile_rows,
                             bn=bn)
    a = _grouped(gather(x, perm_src, tok_off), None, bank.gate_up, tok_off, 0, None, act, bank.padded, rows, tile_rows, bn)
    return _grouped(a, None, bank.down, tok_off, 1, perm_w, act, d, rows, tile_rows, bn), perm_dst
