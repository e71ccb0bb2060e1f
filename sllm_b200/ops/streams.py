"""A residual of several parallel streams (hyper-connections), fp32 [T, streams, d] (kernel in csrc/hyper_streams.cu; the PyTorch
branches restate it for CPU tensors).

start_streams (embedding, optionally with an embedding of the token pair) -> per sublayer join_streams -> read_streams of the rows
that need logits.  Each returns the RMS norm of a weighted sum of the streams, the input of what comes next."""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import Optional

import torch

from . import _lib

P, I, F, L = C.c_void_p, C.c_int, C.c_float, C.c_longlong
MAX_STREAMS = 16
MAX_TOKEN = 1 << 24          # ids below are exact in the fp32 slot that carries a sequence's last token


class StreamArgs(C.Structure):
    _fields_ = [(n, P) for n in ("table", "pair", "ids", "positions", "seq_index", "row_off", "slots", "last", "y", "y2", "mix", "out", "x",
                                 "row_idx", "read", "w", "z")] + \
        [(n, L) for n in ("last_stride", "mul_prev", "mul_cur")] + \
        [(n, I) for n in ("vocab", "buckets", "ldy", "ldy2", "w_step", "rows", "d", "streams", "fp32")] + \
        [(n, F) for n in ("table_scale", "coef", "coef2", "eps")]


_SIGS = {"sllm_streams": (I, [P, P]), "sllm_streams_abi": (I, [P, I])}


def _k():
    for n, s in _SIGS.items():
        _lib.EXTRA_KERNEL_SIGNATURES.setdefault(n, s)
    return _lib.kernels()


@dataclass
class PairEmbedding:
    """Embedding of (previous token, token): row (prev mul_prev + cur mul_cur) mod buckets of ``table`` [buckets + 1, d], for a
    sequence's first token the last row."""
    table: torch.Tensor
    mul_prev: int
    mul_cur: int

    @property
    def buckets(self) -> int:
        return self.table.shape[0] - 1


@dataclass
class Connection:
    """How a sublayer meets the streams (fp32): it reads sum_s read[s] x_s and its output y gives
    x_t <- sum_s mix[s, t] x_s + out[t] y."""
    read: torch.Tensor        # [streams]
    mix: torch.Tensor         # [streams, streams]
    out: torch.Tensor         # [streams]


def _norm(u: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return u / torch.sqrt((u * u).mean(-1, keepdim=True) + eps) * w


def _sum(x: torch.Tensor, read: Optional[torch.Tensor]) -> torch.Tensor:
    return x.sum(1) if read is None else torch.einsum("s,tsd->td", read, x)


def _launch(x, rows, dtype, z, *, read=None, w=None, eps=0.0, **kw) -> None:
    v = lambda t: None if t is None else t.data_ptr()
    a = StreamArgs(x=v(x), read=v(read), w=v(w), z=v(z), w_step=int(w is not None and w.numel() > 1), rows=rows, d=x.shape[2],
                   streams=x.shape[1], fp32=int(dtype == torch.float32), eps=eps, **{k: v(t) if isinstance(t, torch.Tensor) else t
                                                                                    for k, t in kw.items()})
    from .core import _stream
    _lib.check(_k().sllm_streams(C.byref(a), _stream()), "streams")


def start_streams(table: torch.Tensor, b, scale: float, pair: Optional[PairEmbedding], last: Optional[torch.Tensor], streams: int,
                  read: Optional[torch.Tensor], w: torch.Tensor, eps: float):
    """(x [T, streams, d] with every stream ``scale`` table[id] plus the pair's row, the norm of its weighted sum in the table's
    type).  ``last`` fp32 [slots, 1]: the last token of each slot's sequence, read and updated with ``pair``; ``w`` [d] or one
    number."""
    t, d = b.tokens.numel(), table.shape[1]
    if _lib.on_cpu(table):
        e = table[b.tokens.long()].float() * scale
        if pair is not None:
            rows, offs, ids = [], b.row_off.tolist(), b.tokens.tolist()
            for s, slot in enumerate(b.slots.tolist()):
                for r in range(offs[s], offs[s + 1]):
                    prev = ids[r - 1] if r > offs[s] else int(last[slot, 0]) if int(b.positions[r]) > 0 else None
                    rows.append(pair.buckets if prev is None else (prev * pair.mul_prev + ids[r] * pair.mul_cur) % pair.buckets)
                if offs[s + 1] > offs[s]:
                    last[slot, 0] = float(ids[offs[s + 1] - 1])
            e = e + pair.table[torch.tensor(rows)].float()
        x = e.unsqueeze(1).repeat(1, streams, 1)
        return x, _norm(_sum(x, read), w, eps).to(table.dtype)
    x = torch.empty((t, streams, d), dtype=torch.float32, device=table.device)
    z = torch.empty((t, d), dtype=table.dtype, device=table.device)
    kw = dict(table=table, ids=b.tokens, vocab=table.shape[0], table_scale=scale)
    if pair is not None:
        kw.update(pair=pair.table, positions=b.positions, seq_index=b.seq_index, row_off=b.row_off, slots=b.slots, last=last,
                  last_stride=last.stride(0), buckets=pair.buckets, mul_prev=pair.mul_prev, mul_cur=pair.mul_cur)
    _launch(x, t, table.dtype, z, read=read, w=w, eps=eps, **kw)
    return x, z


def join_streams(x: torch.Tensor, y: torch.Tensor, c: Connection, read: Optional[torch.Tensor], w: Optional[torch.Tensor], eps: float,
                 coef: float = 1.0, second: Optional[tuple] = None) -> Optional[torch.Tensor]:
    """Streams after a sublayer, in place: its output is coef y, with ``second`` (y2, coef2) coef y + coef2 y2.  Returns the norm of
    the next weighted sum ``read`` in the type of ``y``, or None without ``w``."""
    if _lib.on_cpu(x):
        v = y.float() * coef
        if second is not None:
            v = v + second[0].float() * second[1]
        x.copy_(torch.einsum("st,rsd->rtd", c.mix, x) + c.out.view(1, -1, 1) * v.unsqueeze(1))
        return None if w is None else _norm(_sum(x, read), w, eps).to(y.dtype)
    z = None if w is None else torch.empty((x.shape[0], x.shape[2]), dtype=y.dtype, device=x.device)
    y2, c2 = second or (None, 0.0)
    _launch(x, x.shape[0], y.dtype, z, read=read, w=w, eps=eps, y=y, ldy=y.stride(0), mix=c.mix, out=c.out, coef=coef, y2=y2,
            ldy2=0 if y2 is None else y2.stride(0), coef2=c2)
    return z


def read_streams(x: torch.Tensor, w: torch.Tensor, eps: float, dtype, rows: Optional[torch.Tensor] = None,
                 read: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Norm of the weighted sum ``read`` (None: the sum) of the streams, of all rows or those listed (int64), in ``dtype``."""
    if _lib.on_cpu(x):
        return _norm(_sum(x if rows is None else x.index_select(0, rows), read), w, eps).to(dtype)
    n = x.shape[0] if rows is None else rows.numel()
    z = torch.empty((n, x.shape[2]), dtype=dtype, device=x.device)
    if n > 0:
        _launch(x, n, dtype, z, read=read, w=w, eps=eps, row_idx=rows)
    return z
