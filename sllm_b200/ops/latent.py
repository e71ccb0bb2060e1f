"""Latent attention ops: one cached row [latent | rotated key part] per token serves every head (kernels in
csrc/latent_attention.cu; PyTorch restatements here for CPU tensors).

A layer runs  append  (norms of the query / key latents, rotation of the shared key part, page write) ->
absorb  (q_h W_uk[h] and the query's rotated part: queries of the width of a cache row) -> attend  (softmax over the
visible rows, result in latent space) -> values  (W_uv[h] and the output gate).  Long prompt portions take the expanded
form instead (csrc/latent_prefill.cu): keys and values of every head are materialised once for the whole portion.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import Optional

import torch

from . import _lib

P, I, F, L = C.c_void_p, C.c_int, C.c_float, C.c_longlong
_SIGS = {
    "sllm_latent_append": (I, [P, I, I, I, I, I, I, P, P, F, P, P, I, I, I, P, P, P, P, I, I, I, I, P]),
    "sllm_head_matmul": (I, [P, L, I, P, P, L, I, I, I, I, I, P, L, I, P, P, I, I, I, P]),
    "sllm_latent_decode_workspace_floats": (L, [I, I, I, I]),
    "sllm_latent_decode": (I, [P, P, L, I, I, I, P, P, P, I, I, I, I, I, F, P, I, P, L, P, P]),
    "sllm_latent_gather": (I, [P, I, I, P, I, P, I, I, P, P, I, I, I, P]),
    "sllm_latent_pack_q": (I, [P, L, P, I, I, I, I, I, I, P, P, I, I, P]),
    "sllm_latent_prefill": (I, [P, I, P, P, I, P, I, I, I, I, I, I, F, P, L, P, P, P]),
    "sllm_latent_attention": (I, [P, P, I, I, I, P, P, P, I, I, I, I, I, F, P, I, P]),
}


def _k():
    for n, s in _SIGS.items():
        _lib.EXTRA_KERNEL_SIGNATURES.setdefault(n, s)
    return _lib.kernels()


@dataclass
class LatentSpec:
    """Sizes and constants of one latent-attention layer."""
    heads: int
    dim: int                  # unrotated query / key channels per head
    rot_dim: int              # rotated channels per head (the key's are shared by all heads)
    vdim: int
    kv_rank: int
    scale: float
    rot_base: float
    rot_dims: int             # channels of rot_dim that turn
    interleaved: bool         # rotary pairs (2i, 2i + 1); else (i, i + rot_dims / 2)
    q_rank: int = 0           # 0: queries come straight from the layer input
    window: int = 0           # 0: every earlier position is visible
    gated: bool = False       # one sigmoid output gate per head

    @property
    def width(self) -> int:
        return self.kv_rank + self.rot_dim

    def inv_freq(self, device) -> torch.Tensor:
        i = torch.arange(self.rot_dims // 2, dtype=torch.float64)
        return (float(self.rot_base) ** (-2.0 * i / self.rot_dims)).float().to(device)


@dataclass
class LatentPages:
    """One layer's pages: [num_pages, page, ld], columns [0, kv_rank) the latent, then the rotated key part."""
    pages: torch.Tensor
    page_size: int


def rotate(x: torch.Tensor, positions: torch.Tensor, inv_freq: torch.Tensor, dims: int, interleaved: bool) -> torch.Tensor:
    """x [T, ..., R] in fp32: the first ``dims`` channels turned by positions * inv_freq."""
    ang = positions.float().view(-1, *([1] * (x.dim() - 1))) * inv_freq
    c, s = ang.cos(), ang.sin()
    out = x.clone()
    if interleaved:
        u, v = x[..., 0:dims:2], x[..., 1:dims:2]
        out[..., 0:dims:2], out[..., 1:dims:2] = u * c - v * s, v * c + u * s
    else:
        u, v = x[..., :dims // 2], x[..., dims // 2:dims]
        out[..., :dims // 2], out[..., dims // 2:dims] = u * c - v * s, v * c + u * s
    return out


def append(proj: torch.Tensor, off_q: int, off_kv: int, spec: LatentSpec, q_norm: Optional[torch.Tensor], kv_norm: torch.Tensor,
           eps: float, inv_freq: torch.Tensor, kv: LatentPages, positions, seq_index, block_table) -> Optional[torch.Tensor]:
    """proj [T, *]: columns off_q.. hold the query latent (with ``q_rank``), off_kv.. [key latent | rotated part].  Writes
    each token's cache row; returns the normed query latent [T, q_rank] or None."""
    t = proj.shape[0]
    if _lib.on_cpu(proj):
        def rms(x, w):
            x = x.float()
            return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w
        x = proj[:, off_kv:off_kv + spec.width]
        c = rms(x[:, :spec.kv_rank], kv_norm)
        kr = rotate(x[:, spec.kv_rank:].float(), positions, inv_freq, spec.rot_dims, spec.interleaved)
        pos = positions.long()
        blk = block_table[seq_index.long(), pos // kv.page_size].long()
        kv.pages[blk, pos % kv.page_size, :spec.width] = torch.cat([c, kr], dim=1).to(kv.pages.dtype)
        return rms(proj[:, off_q:off_q + spec.q_rank], q_norm).to(proj.dtype) if spec.q_rank else None
    from .core import _p, _stream
    cq = torch.empty((t, spec.q_rank), dtype=proj.dtype, device=proj.device) if spec.q_rank else None
    rc = _k().sllm_latent_append(_p(proj), proj.stride(0), off_q, off_kv, spec.q_rank, spec.kv_rank, spec.rot_dim, _p(q_norm),
                                 _p(kv_norm), eps, _p(cq), _p(kv.pages), kv.pages.shape[2], kv.page_size, block_table.stride(0),
                                 _p(positions), _p(seq_index), _p(block_table), _p(inv_freq), spec.rot_dims, int(spec.interleaved),
                                 t, int(proj.dtype == torch.float32), _stream())
    _lib.check(rc, "latent_append")
    return cq


def absorb(q: torch.Tensor, spec: LatentSpec, uk: torch.Tensor, inv_freq: torch.Tensor, positions: torch.Tensor) -> torch.Tensor:
    """q [T, heads * (dim + rot_dim)] (row stride allowed), uk [heads, dim, kv_rank] -> [T, heads, kv_rank + rot_dim]."""
    t, h, hd = q.shape[0], spec.heads, spec.dim + spec.rot_dim
    if _lib.on_cpu(q):
        x = q.reshape(t, h, hd).float()
        a = torch.einsum("thd,hdc->thc", x[..., :spec.dim], uk.float())
        r = rotate(x[..., spec.dim:], positions, inv_freq, spec.rot_dims, spec.interleaved)
        return torch.cat([a, r], dim=-1).to(q.dtype)
    from .core import _p, _stream
    out = torch.empty((t, h, spec.width), dtype=q.dtype, device=q.device)
    rc = _k().sllm_head_matmul(_p(q), q.stride(0), hd, _p(uk), _p(out), h * spec.width, spec.width, t, h, spec.dim, spec.kv_rank,
                               None, 0, spec.rot_dim, _p(positions), _p(inv_freq), spec.rot_dims, int(spec.interleaved),
                               int(q.dtype == torch.float32), _stream())
    _lib.check(rc, "latent_absorb")
    return out


def _tensor_core_rows(qa: torch.Tensor, spec: LatentSpec, kv: LatentPages) -> bool:
    """Whether the page-streaming kernel (csrc/latent_decode.cu) takes this layer."""
    return (qa.dtype == torch.bfloat16 and spec.width <= 576 and spec.kv_rank <= 512 and spec.kv_rank % 8 == 0
            and spec.width % 2 == 0 and kv.page_size in (8, 16, 32))


def _splits(rows: int, groups: int, keys: int) -> int:
    """KV splits of the page-streaming kernel: one CTA per SM, so the number of waves times the tiles of a split (and a
    tile's worth of start-up and merging) is what a launch costs."""
    tiles = max(1, (keys + 63) // 64)
    best, cost = 1, None
    for s in range(1, min(32, tiles) + 1):
        waves = (rows * groups * s + 147) // 148
        c = waves * ((tiles + s - 1) // s + 1.5 + (0.5 if s > 1 else 0.0))
        if cost is None or c < cost - 1e-9:
            best, cost = s, c
    return best


def attend(qa: torch.Tensor, spec: LatentSpec, kv: LatentPages, block_table, seq_index, kv_lens, max_kv: int = 0,
           impl: Optional[str] = None) -> torch.Tensor:
    """Absorbed queries [R, heads, width] over their sequences' pages -> [R, heads, kv_rank].  ``max_kv``: host-side bound
    on kv_lens (split heuristics); ``impl`` "cuda_core" forces the any-size kernel."""
    r = qa.shape[0]
    if _lib.on_cpu(qa):
        out = torch.empty((r, spec.heads, spec.kv_rank), dtype=torch.float32)
        for i in range(r):
            n = int(kv_lens[i])
            blks = block_table[int(seq_index[i]), :(n + kv.page_size - 1) // kv.page_size].long()
            lo = max(0, n - spec.window) if spec.window else 0
            rows = kv.pages[blks].flatten(0, 1)[lo:n, :spec.width].float()
            p = torch.softmax(qa[i].float() @ rows.t() * spec.scale, dim=-1)
            out[i] = p @ rows[:, :spec.kv_rank]
        return out.to(qa.dtype)
    from .core import _p, _stream, workspace
    out = torch.empty((r, spec.heads, spec.kv_rank), dtype=qa.dtype, device=qa.device)
    if impl != "cuda_core" and _tensor_core_rows(qa, spec, kv):
        wsp = workspace(qa.device)
        groups = (spec.heads + 31) // 32
        keys = max_kv if max_kv > 0 else block_table.shape[1] * kv.page_size
        if spec.window:
            keys = min(keys, spec.window + kv.page_size)
        splits = _splits(r, groups, keys)
        while splits > 1 and r * groups * splits * 32 * (spec.kv_rank + 2) > wsp.ws.numel():
            splits -= 1
        if _lib.audit_enabled():
            _lib.record_dispatch("latent_attention", "latent_decode_kernel", rows=r, heads=spec.heads, width=spec.width,
                                 window=spec.window, splits=splits, grid=[r, groups, splits])
        rc = _k().sllm_latent_decode(_p(qa), _p(kv.pages), kv.pages.shape[0] * kv.page_size, kv.pages.shape[2], kv.page_size,
                                     block_table.stride(0), _p(block_table), _p(seq_index), _p(kv_lens), r, spec.heads, spec.kv_rank,
                                     spec.width, spec.window, spec.scale, _p(out), splits, _p(wsp.ws), wsp.ws.numel(),
                                     _p(wsp.status), _stream())
        _lib.check(rc, "latent_decode")
        return out
    rc = _k().sllm_latent_attention(_p(qa), _p(kv.pages), kv.pages.shape[2], kv.page_size, block_table.stride(0), _p(block_table),
                                    _p(seq_index), _p(kv_lens), r, spec.heads, spec.kv_rank, spec.width, spec.window, spec.scale,
                                    _p(out), int(qa.dtype == torch.float32), _stream())
    _lib.check(rc, "latent_attention")
    return out


def values(o: torch.Tensor, spec: LatentSpec, uvt: torch.Tensor, gate: Optional[torch.Tensor],
           out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """o [T, heads, kv_rank], uvt [heads, kv_rank, vdim], gate [T, heads] logits or None -> [T, heads * vdim] (``out``)."""
    t, h = o.shape[0], spec.heads
    if _lib.on_cpu(o):
        y = torch.einsum("thc,hcv->thv", o.float(), uvt.float())
        if gate is not None:
            y = y * torch.sigmoid(gate.float()).unsqueeze(-1)
        return y.reshape(t, h * spec.vdim).to(o.dtype)
    from .core import _p, _stream
    if out is None:
        out = torch.empty((t, h * spec.vdim), dtype=o.dtype, device=o.device)
    rc = _k().sllm_head_matmul(_p(o), h * spec.kv_rank, spec.kv_rank, _p(uvt), _p(out), h * spec.vdim, spec.vdim, t, h, spec.kv_rank,
                               spec.vdim, _p(gate), gate.stride(0) if gate is not None else 0, 0, None, None, 0, 0,
                               int(o.dtype == torch.float32), _stream())
    _lib.check(rc, "latent_values")
    return out


# ------------------------------------------------------------------------------------------ expanded form (prompts)
EXPAND_MIN_ROWS = 64           # a sequence with at least this many rows in the batch takes the expanded form
EXPAND_MAX_CONTEXT = 1 << 16   # context rows expanded at a time (one sequence may exceed it)
TILE = 128


def expandable(spec: LatentSpec, dtype) -> bool:
    """Whether csrc/latent_prefill.cu takes this layer's sizes."""
    nq = (spec.dim + 63) // 64 + (spec.rot_dim + 63) // 64
    return (dtype == torch.bfloat16 and spec.dim % 8 == 0 and spec.vdim % 8 == 0 and spec.kv_rank % 8 == 0 and nq <= 3
            and spec.vdim <= 128)


@dataclass
class Portion:
    """Consecutive rows of a batch that take one form; ``spans`` / ``tiles`` are set for the expanded one."""
    lo: int
    hi: int
    spans: Optional[torch.Tensor] = None     # int32 [sequences, 4]: table row, first position, context rows, gathered row
    tiles: Optional[torch.Tensor] = None     # int32 [tiles, 8], rows relative to ``lo``
    context: int = 0
    longest: int = 0


def plan_portions(row_off: list, starts: list, window: int, device, keep_first: int = 0, chunk: int = 0) -> list:
    """Splits a flat batch into runs of sequences with few rows (absorbed form) and with many (expanded form).  The context of
    a portion starts where its first row's window, or chunk of positions, does; ``keep_first`` positions that a window does not
    reach are gathered ahead of it."""
    out: list = []
    run: list = []

    def flush():
        nonlocal run
        if not run:
            return
        lo, spans, tiles, rows = row_off[run[0]], [], [], 0
        for s in run:
            n, st = row_off[s + 1] - row_off[s], starts[s]
            k_lo = max(0, st - window + 1) if window else st // chunk * chunk if chunk else 0
            if k_lo <= keep_first and not chunk:
                k_lo = 0
            start = rows
            if keep_first and k_lo:
                spans.append((s, 0, keep_first, rows))
                rows += keep_first
            ctx = st + n - k_lo
            spans.append((s, k_lo, ctx, rows))
            for q0 in range(0, n, TILE):
                tiles.append((row_off[s] - lo + q0, min(TILE, n - q0), st + q0, rows, k_lo, start, 0, 0))
            rows += ctx
        tiles.sort(key=lambda t: -(t[2] - t[4]))         # most keys first
        out.append(Portion(lo, row_off[run[-1] + 1], torch.tensor(spans, dtype=torch.int32, device=device),
                           torch.tensor(tiles, dtype=torch.int32, device=device), rows, max(x[2] for x in spans)))
        run = []

    ctx_run = 0
    for s in range(len(row_off) - 1):
        n = row_off[s + 1] - row_off[s]
        if n >= EXPAND_MIN_ROWS:
            ctx = starts[s] + n
            if run and ctx_run + ctx > EXPAND_MAX_CONTEXT:
                flush()
            ctx_run = ctx if not run else ctx_run + ctx
            run.append(s)
            continue
        flush()
        if n == 0:
            continue
        if out and out[-1].spans is None and out[-1].hi == row_off[s]:
            out[-1].hi = row_off[s + 1]
        else:
            out.append(Portion(row_off[s], row_off[s + 1]))
    flush()
    return out


def attend_expanded(q: torch.Tensor, spec: LatentSpec, expand, inv_freq, kv: LatentPages, block_table, positions, gate, pt: Portion,
                    out: torch.Tensor) -> None:
    """Rows [pt.lo, pt.hi) of a batch: q [rows, heads * (dim + rot_dim)], ``expand`` LinearWeight [heads * (dim + vdim),
    kv_rank] (all heads' W_uk, then all heads' W_uv); writes out [rows, heads * vdim]."""
    from .core import _p, _stream, linear, workspace
    t, h = q.shape[0], spec.heads
    dp, rp = (spec.dim + 63) // 64 * 64, (spec.rot_dim + 63) // 64 * 64
    dev = q.device
    c = torch.empty((pt.context, spec.kv_rank), dtype=q.dtype, device=dev)
    r = torch.empty((pt.context, max(rp, 64)), dtype=q.dtype, device=dev)
    k = _k()
    rc = k.sllm_latent_gather(_p(kv.pages), kv.pages.shape[2], kv.page_size, _p(block_table), block_table.stride(0), _p(pt.spans),
                              pt.spans.shape[0], pt.longest, _p(c), _p(r), spec.kv_rank, spec.rot_dim, r.shape[1], _stream())
    _lib.check(rc, "latent_gather")
    exp = linear(c, expand)
    qp = torch.empty((t, h, dp + rp), dtype=q.dtype, device=dev)
    rc = k.sllm_latent_pack_q(_p(q), q.stride(0), _p(qp), t, h, spec.dim, spec.rot_dim, dp, rp, _p(positions), _p(inv_freq),
                              spec.rot_dims, int(spec.interleaved), _stream())
    _lib.check(rc, "latent_pack_q")
    if _lib.audit_enabled():
        _lib.record_dispatch("latent_attention", "latent_prefill_kernel", rows=t, heads=h, context=pt.context, window=spec.window,
                             grid=[pt.tiles.shape[0], h])
    rc = k.sllm_latent_prefill(_p(qp), t, _p(exp), _p(r), pt.context, _p(pt.tiles), pt.tiles.shape[0], h, spec.dim, spec.rot_dim,
                               spec.vdim, spec.window, spec.scale, _p(gate), gate.stride(0) if gate is not None else 0, _p(out),
                               _p(workspace(dev).status), _stream())
    _lib.check(rc, "latent_prefill")


def attention(q: torch.Tensor, gate: Optional[torch.Tensor], spec: LatentSpec, uk, uvt, expand, inv_freq, kv: LatentPages, b):
    """Attention of a ForwardBatch's rows (already appended to the pages) -> [T, heads * vdim], gated."""
    def absorbed(lo, hi, out=None):
        pos = b.positions[lo:hi]
        qa = absorb(q[lo:hi], spec, uk, inv_freq, pos)
        o = attend(qa, spec, kv, b.block_table, b.seq_index[lo:hi], b.kv_lens[lo:hi], b.max_kv)
        return values(o, spec, uvt, None if gate is None else gate[lo:hi], out)

    t = q.shape[0]
    if b.row_off_host is None or not q.is_cuda or _lib.fake_active() or not expandable(spec, q.dtype):
        return absorbed(0, t)
    key = ("latent", spec.window)
    portions = b.plans.get(key)
    if portions is None:
        portions = b.plans[key] = plan_portions(b.row_off_host, b.starts_host, spec.window, q.device)
    if len(portions) == 1 and portions[0].spans is None:
        return absorbed(0, t)
    out = torch.empty((t, spec.heads * spec.vdim), dtype=q.dtype, device=q.device)
    for pt in portions:
        if pt.spans is None:
            absorbed(pt.lo, pt.hi, out[pt.lo:pt.hi])
        else:
            attend_expanded(q[pt.lo:pt.hi], spec, expand, inv_freq, kv, b.block_table, b.positions[pt.lo:pt.hi],
                            None if gate is None else gate[pt.lo:pt.hi], pt, out[pt.lo:pt.hi])
    return out
