"""Zokuvik beside the framework's closest model - the gated-delta-net hybrid - at equal size (`bench.py --compare zokuvik`).

Sizes are those of a served model's layers with random weights: 8 layers (6 recurrent, 2 attention), equal width, head
count, recurrent state and feed-forward parameters, bf16.  Reported per size: prompt and decode throughput of both models
through their engines, and every kernel of the new design with its roofline fraction beside the kernel that does the like
work in the other model.  Kernel times are steady-state times inside a captured graph over rotating buffers that together
exceed the L2.
"""
from __future__ import annotations

import dataclasses
import json

import torch

from .. import ops
from ..engine.batch import make_prefill_batch
from ..engine.engine import build_engine
from ..models.config import qwen35_hybrid_shape
from ..models.zokuvik import zokuvik_shape
from ..ops import delta as D
from ..ops import gdn as G
from ..ops import latent as A
from ..ops import prefill as PF
from ..ops.core import KVLayer, LinearWeight, _p, _stream, workspace
from .kernel_bench import peaks, timed_graph

SIZES = {"2k": dict(width=2048, heads=16, ffn=6144), "4k": dict(width=4096, heads=32, ffn=12288)}
LAYERS = 8


def configs(size: str, ctx: int):
    """(zokuvik, hybrid): the hybrid's gated feed-forward has three matrices, the other two, so the inner sizes differ by 3/2."""
    s = SIZES[size]
    z = zokuvik_shape(LAYERS, s["width"], s["heads"], s["ffn"] * 3 // 2)
    q = qwen35_hybrid_shape(LAYERS)
    q = dataclasses.replace(q, d_model=s["width"], n_heads=s["heads"], n_kv_heads=s["heads"] // 4, head_dim=128, rotary_dim=64,
                            ffn=s["ffn"], gdn_heads=s["heads"], gdn_qk_heads=s["heads"])
    z.max_context = q.max_context = ctx
    return z, q


# ------------------------------------------------------------------------------------------ whole models
def model_rates(cfg, batch: int, prompt: int, steps: int, warmup: int) -> dict:
    eng = build_engine(cfg, "cuda", seed=0, max_batch=batch)
    g = torch.Generator().manual_seed(1)
    prompts = torch.randint(0, cfg.vocab, (batch, prompt), generator=g).tolist()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    grp = min(4, batch)
    times = []
    for _ in range(6):                                # the first three are warm-up
        seqs = [eng.new_sequence(p) for p in prompts[:grp]]
        torch.cuda.synchronize()
        e0.record()
        eng.prefill(seqs)
        e1.record()
        torch.cuda.synchronize()
        times.append(e0.elapsed_time(e1))
        for s in seqs:
            eng.free_sequence(s)
    pre = sorted(times[3:])[1]
    seqs = [eng.new_sequence(p) for p in prompts]
    for i in range(0, batch, 4):
        for s, t in zip(seqs[i:i + 4], eng.prefill(seqs[i:i + 4])):
            s.tokens.append(t)
    for _ in range(warmup):
        for s, t in zip(seqs, eng.decode(seqs)):
            s.tokens.append(t)
    torch.cuda.synchronize()
    e0.record()
    for _ in range(steps):
        for s, t in zip(seqs, eng.decode(seqs)):
            s.tokens.append(t)
    e1.record()
    torch.cuda.synchronize()
    ms = e0.elapsed_time(e1) / steps
    out = {"prefill_tok_s": round(grp * prompt / pre * 1e3), "prefill_ms": round(pre, 3), "prefill_seqs": grp,
           "decode_tok_s": round(batch / ms * 1e3), "decode_ms_per_step": round(ms, 4),
           "decode_launches": int(eng._graph_launches[(batch, True)])}
    for s in seqs:
        eng.free_sequence(s)
    out["device_status"] = ops.device_status(torch.device("cuda"))
    eng.release()
    del eng
    torch.cuda.empty_cache()
    return out


# ------------------------------------------------------------------------------------------ kernels
class _Table:
    """Rows {kernel, us, bound, frac, like, like_us, like_frac, distance}; distance = like_frac / frac: how many times
    further from its roofline the kernel is than the like one."""

    def __init__(self):
        self.bw, self.tf, self.label = peaks()
        self.rows: list = []

    def add(self, name, us, like, like_us, *, nbytes=None, flops=None, like_bytes=None, like_flops=None):
        f = (nbytes / self.bw if nbytes else flops / self.tf) / (us * 1e-6)
        lf = (like_bytes / self.bw if like_bytes else like_flops / self.tf) / (like_us * 1e-6)
        self.rows.append({"kernel": name, "us": round(us, 1), "bound": "bytes" if nbytes else "flops", "frac": round(f, 3),
                          "like": like, "like_us": round(like_us, 1), "like_frac": round(lf, 3), "distance": round(lf / f, 2)})


def _bf(*shape):
    return torch.randn(*shape, device="cuda").to(torch.bfloat16)


def _us(fns) -> float:
    return timed_graph(fns) * 1e6


RANK, ROT, DIM, VDIM, QRANK, PAGE, COPIES = 512, 64, 128, 128, 1024, 16, 6


def _spec(heads: int, **kw) -> A.LatentSpec:
    return A.LatentSpec(heads, DIM, ROT, VDIM, RANK, (DIM + ROT) ** -0.5, 1e6, ROT, True, **kw)


def attention_decode(tab: _Table, heads: int, batch: int, ctx: int) -> None:
    hkv, hd, spec = heads // 4, 128, _spec(heads)
    W, nb = spec.width, ctx // PAGE
    table = torch.randperm(nb * batch).view(batch, nb).int().cuda()
    si, kl = torch.arange(batch, device="cuda").int(), torch.full((batch,), ctx, device="cuda").int()
    pos, f = kl - 1, spec.inv_freq("cuda")
    qa, q, gate = _bf(batch, heads, W), _bf(batch, heads * hd), _bf(batch, heads)
    lat = [A.LatentPages(_bf(nb * batch, PAGE, W), PAGE) for _ in range(COPIES)]
    kv = [KVLayer(_bf(nb * batch, hkv, PAGE, hd), _bf(nb * batch, hkv, PAGE, hd), None, None, False, PAGE) for _ in range(COPIES)]
    tab.add(f"latent_decode (batch {batch}, {ctx} keys)", _us([lambda k=k: A.attend(qa, spec, k, table, si, kl, ctx) for k in lat]),
            "paged_attention", _us([lambda k=k: ops.paged_attention(q, k, table, si, kl, heads, hkv, hd, max_kv=ctx) for k in kv]),
            nbytes=batch * ctx * W * 2, like_bytes=2 * batch * ctx * hkv * hd * 2)
    # the page appends of a step
    proj, n1, n2 = _bf(batch, QRANK + W + heads), torch.ones(QRANK, device="cuda"), torch.ones(RANK, device="cuda")
    qkv, sq = _bf(batch, (heads + 2 * hkv) * hd), _spec(heads, q_rank=QRANK)
    tab.add("latent_append (decode)", _us([lambda k=k: A.append(proj, 0, QRANK, sq, n1, n2, 1e-6, f, k, pos, si, table) for k in lat]),
            "rope_kv_append", _us([lambda k=k: ops.rope_kv_append(qkv, pos, si, table, k, heads, hkv, hd, 1e6, 64) for k in kv]),
            nbytes=batch * (2 * QRANK + 2 * W) * 2, like_bytes=batch * (2 * heads + 4 * hkv) * hd * 2)
    # per-head products beside a dense product that reads as much
    many = 3 * COPIES
    uk, uv = [_bf(heads, DIM, RANK) for _ in range(many)], [_bf(heads, RANK, VDIM) for _ in range(many)]
    wl = [LinearWeight("dense", _bf(heads * DIM, RANK)) for _ in range(many)]
    qx, ol, xr = _bf(batch, heads * (DIM + ROT)), _bf(batch, heads, RANK), _bf(batch, RANK)
    lin = _us([lambda w=w: ops.linear(xr, w) for w in wl])
    lin_bytes = heads * DIM * RANK * 2 + batch * (RANK + heads * DIM) * 2
    tab.add("head_matmul (absorb)", _us([lambda u=u: A.absorb(qx, spec, u, f, pos) for u in uk]), "gemm_tcgen05, equal weights", lin,
            nbytes=heads * DIM * RANK * 2 + batch * heads * (DIM + ROT + W) * 2, like_bytes=lin_bytes)
    tab.add("head_matmul (values)", _us([lambda u=u: A.values(ol, spec, u, gate) for u in uv]), "gemm_tcgen05, equal weights", lin,
            nbytes=heads * VDIM * RANK * 2 + batch * heads * (RANK + VDIM) * 2, like_bytes=lin_bytes)


def attention_prompt(tab: _Table, heads: int, seqs: int, n: int) -> None:
    hkv, hd, spec = heads // 4, 128, _spec(heads)
    W, T, nb = spec.width, seqs * n, n // PAGE
    table = torch.randperm(nb * seqs).view(seqs, nb).int().cuda()
    b = make_prefill_batch([[0] * n] * seqs, table, "cuda")
    kv = KVLayer(_bf(nb * seqs, hkv, PAGE, hd), _bf(nb * seqs, hkv, PAGE, hd), None, None, False, PAGE)
    lat = A.LatentPages(_bf(nb * seqs, PAGE, W), PAGE)
    q, qkv = _bf(T, heads * hd), _bf(T, (heads + 2 * hkv) * hd)
    qx, gate, out = _bf(T, heads * (DIM + ROT)), _bf(T, heads), _bf(T, heads * VDIM)
    ex, f = LinearWeight("dense", _bf(heads * (DIM + VDIM), RANK)), spec.inv_freq("cuda")
    pt = A.plan_portions(b.row_off_host, b.starts_host, 0, "cuda")[0]
    k, c, r, qp = A._k(), _bf(T, RANK), _bf(T, 64), _bf(T, heads, DIM + 64)
    e, status = ops.linear(c, ex), workspace(q.device).status
    paged = _us([lambda: ops.paged_attention(q, kv, table, b.seq_index, b.kv_lens, heads, hkv, hd, max_kv=n)] * 2)
    dense = _us([lambda: PF.prefill_attention(qkv, b, heads, hkv, hd)] * 3)
    attn = _us([lambda: k.sllm_latent_prefill(_p(qp), T, _p(e), _p(r), T, _p(pt.tiles), pt.tiles.shape[0], heads, DIM, ROT, VDIM, 0,
                                              spec.scale, _p(gate), gate.stride(0), _p(out), _p(status), _stream())] * 3)
    pairs = seqs * n * (n + 1) / 2 * heads
    for like, us in (("paged_attention (the hybrid's prompts)", paged), ("prefill_attention (dense models)", dense)):
        tab.add(f"latent_prefill ({seqs} x {n})", attn, like, us, flops=pairs * 2 * (DIM + ROT + VDIM), like_flops=pairs * 4 * hd)
    append = _us([lambda: ops.rope_kv_append(qkv, b.positions, b.seq_index, table, kv, heads, hkv, hd, 1e6, 64)] * 3)
    ab = T * (2 * heads + 4 * hkv) * hd * 2
    tab.add("latent_gather", _us([lambda: k.sllm_latent_gather(_p(lat.pages), W, PAGE, _p(table), table.stride(0), _p(pt.spans), seqs, n,
                                                               _p(c), _p(r), RANK, ROT, 64, _stream())] * 3),
            "rope_kv_append", append, nbytes=T * 2 * W * 2, like_bytes=ab)
    tab.add("latent_pack_q", _us([lambda: k.sllm_latent_pack_q(_p(qx), qx.stride(0), _p(qp), T, heads, DIM, ROT, DIM, 64, _p(b.positions),
                                                               _p(f), ROT, 1, _stream())] * 3),
            "rope_kv_append", append, nbytes=T * 2 * heads * (DIM + ROT) * 2, like_bytes=ab)
    proj, n1, n2 = _bf(T, QRANK + W + heads), torch.ones(QRANK, device="cuda"), torch.ones(RANK, device="cuda")
    sq = _spec(heads, q_rank=QRANK)
    tab.add("latent_append (prompt)", _us([lambda: A.append(proj, 0, QRANK, sq, n1, n2, 1e-6, f, lat, b.positions, b.seq_index, table)] * 3),
            "rope_kv_append", append, nbytes=T * (2 * QRANK + 2 * W) * 2, like_bytes=ab)
    whole = _us([lambda: A.attend_expanded(qx, spec, ex, f, lat, table, b.positions, gate, pt, out)] * 3)
    tab.rows.append({"kernel": f"attention of a prompt, all launches ({seqs} x {n})", "us": round(whole, 1),
                     "of which expansion GEMM": round(_us([lambda: ops.linear(c, ex)] * 3), 1), "of which attention": round(attn, 1)})


def recurrence(tab: _Table, heads: int, batch: int, seqs: int, n: int) -> None:
    ds, T = D.DeltaSpec(heads, 128, 64), seqs * n
    nz = ds.size
    w2, v0, one = LinearWeight("dense", _bf(nz, 64)), torch.zeros(nz, device="cuda"), torch.ones(nz, device="cuda")
    proj, qkv, z, ba = _bf(T, 5 * nz + 64), _bf(T, 3 * nz), _bf(T, nz), _bf(T, 2 * heads)
    a_log, dtb, nw = torch.zeros(heads, device="cuda"), _bf(heads), torch.ones(128, device="cuda")

    def new(rows, st, off, slots, one_each):
        return D.general_delta(proj[:rows], ds, w2, v0, v0, one, 1e-6, st, off, slots, one_each)

    def old(rows, st, off, slots):
        return G.recurrent(qkv[:rows], z[:rows], ba[:rows, :heads], ba[:rows, heads:], a_log, dtb, nw, st, off, slots, heads, heads)

    st = torch.zeros(seqs, heads, 128, 128, device="cuda")
    off, slots = torch.arange(0, T + 1, n, device="cuda").int(), torch.arange(seqs, device="cuda").int()
    sb = 2 * seqs * heads * 128 * 128 * 4
    tab.add(f"general_delta, prompt ({seqs} x {n})", _us([lambda: new(T, st, off, slots, False)] * 2), "gated delta net, prompt form",
            _us([lambda: old(T, st, off, slots)] * 2), nbytes=T * 6 * nz * 2 + sb, like_bytes=T * 5 * nz * 2 + sb)
    off, slots = torch.arange(batch + 1, device="cuda").int(), torch.arange(batch, device="cuda").int()
    sts = [torch.zeros(batch, heads, 128, 128, device="cuda") for _ in range(COPIES)]
    sb = 2 * batch * heads * 128 * 128 * 4
    tab.add(f"general_delta, decode (batch {batch})", _us([lambda x=x: new(batch, x, off, slots, True) for x in sts]),
            "gated delta net, decode", _us([lambda x=x: old(batch, x, off, slots) for x in sts]),
            nbytes=sb + batch * 6 * nz * 2 + nz * 128, like_bytes=sb + batch * 5 * nz * 2)


def norms(tab: _Table, d: int, rows: dict) -> None:
    for name, m in rows.items():
        x, y, xb = torch.randn(m, d, device="cuda"), _bf(m, d), _bf(m, d)
        w, wb = torch.ones(d, device="cuda"), _bf(d)
        tab.add(f"group_norm (x += norm(y), z = norm(x)), {name}", _us([lambda: ops.add_group_norm(x, y, w, w, 1e-6, 1)] * 3), "rmsnorm",
                _us([lambda: ops.rmsnorm(xb, wb, 1e-6)] * 3), nbytes=m * d * (2 + 4 + 4 + 2), like_bytes=m * d * 4)


def kernel_rows(size: str, batch: int, ctx: int) -> list:
    s, tab = SIZES[size], _Table()
    attention_decode(tab, s["heads"], batch, ctx)
    torch.cuda.empty_cache()
    attention_prompt(tab, s["heads"], 4, 2048)
    torch.cuda.empty_cache()
    recurrence(tab, s["heads"], batch, 4, 2048)
    torch.cuda.empty_cache()
    norms(tab, s["width"], {"prompt": 4 * 2048, "decode": batch})
    return tab.rows


def main(args) -> int:
    out = {"metric": "zokuvik_beside_hybrid", "data": "synthetic: seeded random prompts and weights", "layers": LAYERS,
           "prompt": args.prompt, "steps": args.steps, "roofline": peaks()[2], "sizes": {}}
    for size in SIZES:
        z, q = configs(size, ((args.prompt + args.warmup + args.steps + 64 + 255) // 256) * 256)
        models = {name: {f"batch{b}": model_rates(cfg, b, args.prompt, args.steps, args.warmup) for b in (args.batch, 1)}
                  for name, cfg in (("zokuvik", z), ("hybrid", q))}
        out["sizes"][size] = {"shape": SIZES[size], "models": models, "kernels": kernel_rows(size, args.batch, args.prompt)}
        torch.cuda.empty_cache()
    print(json.dumps(out))
    return 0
