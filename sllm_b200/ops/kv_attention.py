"""Attention with keys and values of different widths: biases or short convolutions on q, k and v, rotation in neighbouring or
half-split pairs with scaled frequencies, query / key norms (per head or over all heads) and value norms, values mixed with
another layer's, a sink in the softmax, a window with kept first positions or chunks of positions, slopes or learned biases over
the distance, and an output gate per channel or head, each optional (kernels in csrc/kv_attention.cu; PyTorch restatements here for CPU tensors).

A layer runs  prepare  (everything between the projection and the scores, page write) -> attention.  Decoded tokens and short
portions read the pages row by row; long portions gather them once and run on the tensor cores (csrc/latent_prefill.cu).  A
layer that takes its keys and values from another one prepares queries only and is handed that layer's pages."""
from __future__ import annotations

import ctypes as C
import math
from dataclasses import dataclass
from typing import Optional

import torch

from . import _lib
from .latent import plan_portions, rotate
from .short_conv import causal_conv

P, I, F, L = C.c_void_p, C.c_int, C.c_float, C.c_longlong


class KvPrepareArgs(C.Structure):
    _fields_ = [(n, P) for n in ("proj", "conv_w", "bias", "q_norm", "k_norm", "ring", "inv_freq", "row_off", "slots", "positions", "seq_index", "block_table", "q",
                                 "k_pages", "v_pages", "v_other")] + [("ring_stride", L)] + \
        [(n, I) for n in ("ldp", "max_blocks", "heads", "kv_heads", "dim", "vdim", "q_pad", "ld_k", "ld_v", "rot_dims", "taps",
                          "page_size", "tokens", "sequences", "norm", "decode", "fp32", "interleaved", "ld_other", "v_norm")] + \
        [("v_mix", F), ("eps", F)]


_SIGS = {
    "sllm_kv_prepare": (I, [P, P]),
    "sllm_kv_abi": (I, [P, I]),
    "sllm_paged_attention_any": (I, [P, I, P, P, I, I, P, I, P, P] + [I] * 9 + [F, P, P, P, I, I, P, L, I, P, I, P, L, P, I, P]),
    "sllm_kv_gather": (I, [P, P, I, P, I, P, I, I, P, I, I, I, P]),
    "sllm_kv_attention": (I, [P, P, P, P, L, P, P, I, P, P, I, I, I, I, I, I, I, I, I, I, I, I, P, P, I, I, I, F, P, I, P]),
    "sllm_kv_prefill": (I, [P, I, P, I, P, I, I, I, I, I, I, I, I, P, P, I, I, F, P, P, L, I, P, P, P]),
}


def _k():
    for n, s in _SIGS.items():
        _lib.EXTRA_KERNEL_SIGNATURES.setdefault(n, s)
    return _lib.kernels()


def rope_frequencies(base: float, dims: int, scaling: Optional[dict] = None) -> torch.Tensor:
    """fp64 [dims / 2].  ``scaling`` {factor, low, high, original} stretches long wavelengths: pairs that turn more than `high`
    times within `original` positions stay, those that turn less than `low` times are slowed down by `factor`, and between
    the two the rates are blended."""
    f = float(base) ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims)
    if not scaling:
        return f
    turns = float(scaling["original"]) * f / (2 * math.pi)
    low, high, slow = float(scaling["low"]), float(scaling["high"]), f / float(scaling["factor"])
    s = (turns - low) / (high - low) if high != low else torch.zeros_like(f)
    return torch.where(turns > high, f, torch.where(turns < low, slow, (1 - s) * slow + s * f))


@dataclass
class KVSpec:
    """Sizes and constants of one layer; its packed input projection is q | k | v | g (q | g without keys of its own).  A row sees
    all earlier positions, the last ``window`` and the first ``keep_first`` ones, or those of its own ``chunk``."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_base: float
    rot_dims: int
    taps: int = 1
    rot_scaling: Optional[dict] = None
    qk_norm: bool = True
    window: int = 0
    own_kv: bool = True
    keep_first: int = 0
    chunk: int = 0
    interleaved: bool = True         # rotary pairs (2i, 2i + 1); else (i, i + rot_dims / 2)
    norm_all: bool = False           # the query / key norm goes over all heads at once; else over each
    v_norm: bool = False             # each head's value is divided by its root mean square
    gate_heads: bool = False         # the output gate has one logit per head; else one per channel

    @property
    def q_cols(self) -> int:
        return self.heads * self.dim

    @property
    def channels(self) -> int:
        """Columns that the short convolution covers."""
        return self.q_cols + (self.kv_heads * (self.dim + self.vdim) if self.own_kv else 0)

    @property
    def out_cols(self) -> int:
        return self.heads * self.vdim

    @property
    def q_pad(self) -> int:
        return (self.dim + 63) // 64 * 64

    def sees(self, i: int, j: torch.Tensor) -> torch.Tensor:
        """Which of the positions ``j`` <= i position i sees."""
        if self.chunk:
            return j // self.chunk == i // self.chunk
        return (i - j < self.window) | (j < self.keep_first) if self.window else torch.ones_like(j, dtype=torch.bool)

    def inv_freq(self, device) -> torch.Tensor:
        return rope_frequencies(self.rot_base, self.rot_dims, self.rot_scaling).float().to(device)


def distance_slopes(heads: int, device) -> torch.Tensor:
    """fp32 [heads]: 2^(-8 (h + 1) / heads), the geometric slopes of linear distance biases."""
    return torch.exp2(-8.0 * torch.arange(1, heads + 1, dtype=torch.float64) / heads).float().to(device)


DIST_FRONT, DIST_BACK = 256, 256            # of attention_common.cuh


def distance_buckets(rows: int, far: float, limit: int) -> list:
    """Row of a table of learned distance biases for the distances 0, 1, ...: a row each below half the table, logarithmic steps
    from there to distance ``far``, the last row from there on.  The list ends with the last row's first distance, or after
    ``limit`` entries."""
    near, out = rows // 2, []
    for n in range(limit):
        b = n
        if n >= near:
            steps = math.log(n / near) / math.log(far / near) * (rows - near) if near > 0 and far > near else rows
            b = min(rows - 1, near + math.floor(steps))
        out.append(b)
        if b == rows - 1:
            break
    return out


@dataclass
class DistanceBias:
    """What joins a score by its distance.  table fp32 [heads, DIST_FRONT + n + DIST_BACK]: the entries of distances 0 .. n - 1
    behind DIST_FRONT unused ones; the last holds for all distances beyond and is repeated."""
    table: torch.Tensor
    n: int

    @staticmethod
    def make(rel: torch.Tensor, far: float, limit: int) -> "DistanceBias":
        """``rel`` [rows, heads], read by ``distance_buckets``."""
        b = distance_buckets(rel.shape[0], far, limit)
        rows = torch.tensor([b[0]] * DIST_FRONT + b + [b[-1]] * DIST_BACK, device=rel.device)
        return DistanceBias(rel.float()[rows].t().contiguous(), len(b))

    def at(self, distance: torch.Tensor) -> torch.Tensor:
        """[heads, *distance.shape]"""
        return self.table[:, DIST_FRONT + distance.clamp(max=self.n - 1)]


@dataclass
class KVPages:
    """One layer's pages: k [num_pages, kv_heads, page, >= dim], v [num_pages, kv_heads, page, >= vdim]."""
    k: torch.Tensor
    v: torch.Tensor
    page_size: int

    # what ops.paged_attention reads of a layer
    k_scale = v_scale = None
    fp8 = nvfp4 = False
    k_static = v_static = 0.0
    mode = 0


def prepare(proj: torch.Tensor, spec: KVSpec, conv_w: Optional[torch.Tensor], inv_freq: Optional[torch.Tensor], eps: float,
            kv: Optional[KVPages], ring: Optional[torch.Tensor], b, bias: Optional[torch.Tensor] = None,
            q_norm: Optional[torch.Tensor] = None, k_norm: Optional[torch.Tensor] = None, mix: Optional[tuple] = None) -> torch.Tensor:
    """proj [T, >= channels]; conv_w [taps, channels] and ring [slots, taps, channels], or neither; bias fp32 [channels]; q_norm,
    k_norm fp32 [dim] weights of the norms (``norm_all``: [heads * dim], [kv_heads * dim]); ``mix``: (values [T, kv_heads * vdim],
    their share lambda), v <- (1 - lambda) v + lambda values; ``kv`` the layer's own pages (None: the layer has no keys of its own).  Returns q
    [T, heads, q_pad], zero past ``dim``."""
    t, H, G, D, V = proj.shape[0], spec.heads, spec.kv_heads, spec.dim, spec.vdim
    if _lib.on_cpu(proj):
        x = proj[:, :spec.channels].float()
        if bias is not None:
            x = x + bias
        if conv_w is not None:
            x = causal_conv(x, conv_w, ring, b.row_off, b.slots, b.positions)

        def turned(y, w):
            if spec.qk_norm:
                y = y / torch.sqrt((y * y).mean((1, 2) if spec.norm_all else -1, keepdim=True) + eps)
                y = y if w is None else y * (w.view(y.shape[1:]) if spec.norm_all else w)
            return rotate(y, b.positions, inv_freq, spec.rot_dims, spec.interleaved) if spec.rot_dims else y
        q = torch.zeros((t, H, spec.q_pad), dtype=proj.dtype)
        q[..., :D] = turned(x[:, :spec.q_cols].reshape(t, H, D), q_norm).to(proj.dtype)
        if kv is not None:
            k = turned(x[:, spec.q_cols:spec.q_cols + G * D].reshape(t, G, D), k_norm)
            v = x[:, spec.q_cols + G * D:].reshape(t, G, V)
            if spec.v_norm:
                v = v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)
            if mix is not None:
                v = (1 - mix[1]) * v + mix[1] * mix[0].float().reshape(t, G, V)
            pos = b.positions.long()
            blk = b.block_table[b.seq_index.long(), pos // kv.page_size].long()
            kv.k[blk, :, pos % kv.page_size, :D] = k.to(kv.k.dtype)
            kv.v[blk, :, pos % kv.page_size, :V] = v.to(kv.v.dtype)
        return q
    from .core import _stream
    q = torch.empty((t, H, spec.q_pad), dtype=proj.dtype, device=proj.device)
    p = lambda x: None if x is None else x.data_ptr()
    decode = b.row_off_host is None and t == b.slots.numel()
    own = kv is not None
    other, share = mix if mix is not None else (None, 0.0)
    args = KvPrepareArgs(p(proj), p(conv_w), p(bias), p(q_norm), p(k_norm), p(ring), p(inv_freq), p(b.row_off), p(b.slots), p(b.positions), p(b.seq_index),
                         p(b.block_table), p(q), p(kv.k) if own else None, p(kv.v) if own else None, p(other), 0 if ring is None else ring.stride(0), proj.stride(0),
                         b.block_table.stride(0), H, G if own else 0, D, V, spec.q_pad, kv.k.shape[3] if own else 0,
                         kv.v.shape[3] if own else 0, spec.rot_dims, spec.taps, kv.page_size if own else 1, t, b.slots.numel(),
                         (2 if spec.norm_all else 1) if spec.qk_norm else 0, int(decode), int(proj.dtype == torch.float32),
                         int(spec.interleaved), 0 if other is None else other.stride(0), int(spec.v_norm), share, eps)
    _lib.check(_k().sllm_kv_prepare(C.byref(args), _stream()), "kv_prepare")
    return q


def paged_rows(q: torch.Tensor, gate: Optional[torch.Tensor], spec: KVSpec, kv: KVPages, sinks: Optional[torch.Tensor], block_table,
               seq_index, kv_lens, max_kv: int = 0, out: Optional[torch.Tensor] = None, impl: Optional[str] = None,
               slopes: Optional[torch.Tensor] = None, dist: Optional[DistanceBias] = None) -> torch.Tensor:
    """Rows q [R, heads, q_pad] over their sequences' pages -> [R, heads * vdim].  ``impl`` "cuda_core_any" forces the any-size
    kernel."""
    from . import core
    r, H, G, D, V = q.shape[0], spec.heads, spec.kv_heads, spec.dim, spec.vdim
    if _lib.on_cpu(q):
        res = torch.empty((r, H, V))
        for i in range(r):
            n = int(kv_lens[i])
            blks = block_table[int(seq_index[i]), :(n + kv.page_size - 1) // kv.page_size].long()
            j = torch.arange(n)
            j = j[spec.sees(n - 1, j)]
            k = kv.k[blks].transpose(1, 2).reshape(-1, G, kv.k.shape[3])[j, :, :D].float().repeat_interleave(H // G, dim=1)
            v = kv.v[blks].transpose(1, 2).reshape(-1, G, kv.v.shape[3])[j, :, :V].float().repeat_interleave(H // G, dim=1)
            s = torch.einsum("hd,jhd->hj", q[i, :, :D].float(), k) * spec.scale
            if slopes is not None:
                s = s - slopes[:, None] * (n - 1 - j).float()
            if dist is not None:
                s = s + dist.at(n - 1 - j)
            if sinks is not None:
                s = torch.cat([s, sinks[:, None]], dim=1)
            p = torch.softmax(s, dim=-1)[:, :j.numel()]
            res[i] = torch.einsum("hj,jhv->hv", p, v)
        if gate is not None:
            res = res * torch.sigmoid(gate.float()).reshape(r, H, -1)
        res = res.reshape(r, H * V)
        res = res.to(q.dtype)
        if out is not None:
            out.copy_(res)
        return res
    g = H // G
    if q.dtype == torch.bfloat16 and D == V and D in (64, 128, 256) and g in (1, 2, 4, 8) and impl != "cuda_core_any":
        return core.paged_attention(q.view(r, H * D), kv, block_table, seq_index, kv_lens, H, G, D, window=spec.window,
                                    sm_scale=spec.scale, max_kv=max_kv, sinks=sinks, gate=gate, out=out, gate_heads=spec.gate_heads,
                                    keep_first=spec.keep_first, chunk=spec.chunk, slopes=slopes, dist=dist)
    out = torch.empty((r, H * V), dtype=q.dtype, device=q.device) if out is None else out
    if q.dtype == torch.bfloat16 and max(D, V) <= 256 and kv.k.shape[3] % 8 == 0 and kv.v.shape[3] % 8 == 0 and impl != "cuda_core_any":
        ws = core.workspace(q.device)
        mk = max_kv if max_kv > 0 else block_table.shape[1] * kv.page_size
        mk = min(mk, spec.window + spec.keep_first) if spec.window else min(mk, spec.chunk) if spec.chunk else mk
        splits = core._attn_splits(r, H // math.gcd(H // G, 8), mk)
        if _lib.audit_enabled():
            _lib.record_dispatch("paged_attention", "paged_attention_kernel", rows=r, hq=H, hkv=G, hd=D, window=spec.window, splits=splits)
        rc = _k().sllm_paged_attention_any(core._p(q), spec.q_pad, core._p(kv.k), core._p(kv.v), kv.k.shape[3], kv.v.shape[3],
                                           core._p(block_table), block_table.stride(0), core._p(seq_index), core._p(kv_lens), r, H, G, D, V,
                                           kv.page_size, spec.window, spec.keep_first, spec.chunk, spec.scale, core._p(sinks),
                                           core._p(slopes), *core.dist_args(dist), core._p(gate), gate.stride(0) if gate is not None else 0,
                                           int(spec.gate_heads), core._p(out), splits, core._p(ws.ws), ws.ws.numel(), core._p(ws.counters),
                                           ws.counters.numel(), core._stream())
        _lib.check(rc, "paged_attention_any")
        return out
    rc = _k().sllm_kv_attention(core._p(q), core._p(kv.k), core._p(kv.v), core._p(gate), gate.stride(0) if gate is not None else 0,
                                core._p(sinks), core._p(block_table), block_table.stride(0), core._p(seq_index), core._p(kv_lens), r, H,
                                G, D, V, spec.q_pad, kv.k.shape[3], kv.v.shape[3], kv.page_size, spec.window, spec.keep_first, spec.chunk,
                                core._p(slopes), *core.dist_args(dist), int(spec.gate_heads), spec.scale, core._p(out),
                                int(q.dtype == torch.float32), core._stream())
    _lib.check(rc, "kv_attention")
    return out


def gatherable(spec: KVSpec, dtype, gate: Optional[torch.Tensor]) -> bool:
    """Whether long portions of this layer run on the tensor cores."""
    return (dtype == torch.bfloat16 and spec.dim % 8 == 0 and spec.vdim % 8 == 0 and spec.dim <= 192 and spec.vdim <= 128
            and (gate is None or spec.gate_heads or (gate.stride(0) % 8 == 0 and gate.data_ptr() % 16 == 0)))


def attend_gathered(q, gate, spec: KVSpec, kv: KVPages, sinks, b, pt, out, slopes=None, dist=None) -> None:
    """Rows [pt.lo, pt.hi) of a batch (q, gate and out are those rows)."""
    from .core import _p, _stream, dist_args, workspace
    key = ("gathered", pt.lo)
    held = b.plans.get(key)
    if spec.own_kv or held is None or held[0] is not kv:      # a layer that borrows its keys finds them gathered already
        rows = torch.empty((pt.context, spec.kv_heads * (spec.dim + spec.vdim)), dtype=q.dtype, device=q.device)
        rc = _k().sllm_kv_gather(_p(kv.k), _p(kv.v), kv.page_size, _p(b.block_table), b.block_table.stride(0), _p(pt.spans),
                                 pt.spans.shape[0], pt.longest, _p(rows), spec.kv_heads, spec.dim, spec.vdim, _stream())
        _lib.check(rc, "kv_gather")
        held = b.plans[key] = (kv, rows)
    if _lib.audit_enabled():
        _lib.record_dispatch("kv_attention", "latent_prefill_kernel", rows=q.shape[0], heads=spec.heads, context=pt.context,
                             window=spec.window, grid=[pt.tiles.shape[0], spec.heads])
    rc = _k().sllm_kv_prefill(_p(q), q.shape[0], _p(held[1]), pt.context, _p(pt.tiles), pt.tiles.shape[0], spec.heads, spec.kv_heads,
                              spec.dim, spec.vdim, spec.window, spec.keep_first, spec.chunk, _p(slopes), *dist_args(dist), spec.scale, _p(sinks), _p(gate),
                              gate.stride(0) if gate is not None else 0, int(spec.gate_heads), _p(out), _p(workspace(q.device).status), _stream())
    _lib.check(rc, "kv_prefill")


def attention(q: torch.Tensor, gate: Optional[torch.Tensor], spec: KVSpec, kv: KVPages, sinks: Optional[torch.Tensor], b,
              slopes: Optional[torch.Tensor] = None, dist: Optional[DistanceBias] = None) -> torch.Tensor:
    """Attention of a ForwardBatch's rows over ``kv`` (already appended to) -> [T, heads * vdim], gated."""
    t = q.shape[0]

    def rows(lo, hi, out=None):
        return paged_rows(q[lo:hi], None if gate is None else gate[lo:hi], spec, kv, sinks, b.block_table, b.seq_index[lo:hi],
                          b.kv_lens[lo:hi], b.max_kv, out, slopes=slopes, dist=dist)

    if b.row_off_host is None or not q.is_cuda or _lib.fake_active() or not gatherable(spec, q.dtype, gate):
        return rows(0, t)
    key = ("portions", spec.window, spec.keep_first, spec.chunk)
    portions = b.plans.get(key)
    if portions is None:
        portions = b.plans[key] = plan_portions(b.row_off_host, b.starts_host, spec.window, q.device, spec.keep_first, spec.chunk)
    if len(portions) == 1 and portions[0].spans is None:
        return rows(0, t)
    out = torch.empty((t, spec.out_cols), dtype=q.dtype, device=q.device)
    for pt in portions:
        if pt.spans is None:
            rows(pt.lo, pt.hi, out[pt.lo:pt.hi])
        else:
            attend_gathered(q[pt.lo:pt.hi], None if gate is None else gate[pt.lo:pt.hi], spec, kv, sinks, b, pt, out[pt.lo:pt.hi],
                            slopes, dist)
    return out
