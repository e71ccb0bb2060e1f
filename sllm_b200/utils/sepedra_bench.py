"""Sepedra beside the framework's closest model - the gated-delta-net hybrid with routed experts - at equal size
(`bench.py --compare sepedra`).

Sizes are those of a served model's layers with random weights: 8 layers (6 recurrent, 2 attention), equal width, head
count, experts and experts per token.  Sepedra's experts are bf16, the hybrid's MXFP4 (the only form its experts have).
Reported as in family_bench: throughput of both models through their engines, and every kernel of the new design with its
roofline fraction beside the kernel that does the like work in the other model.
"""
from __future__ import annotations

import dataclasses
import json

import torch

from .. import ops
from ..engine.batch import ForwardBatch, make_prefill_batch
from ..models.config import qwen35_hybrid_shape
from ..models.sepedra import sepedra_shape
from ..ops import gdn as G
from ..ops import kv_attention as A
from ..ops import moe as M
from ..ops import prefill as PF
from ..ops import rglru as R
from ..ops.core import KVLayer, LinearWeight, _p, _stream, workspace
from ..ops.w4 import W4Weight, linear_w4
from .family_bench import COPIES, LAYERS, PAGE, _bf, _Table, _us, model_rates
from .kernel_bench import peaks

SIZES = {"2k": dict(width=2048, heads=16, experts=64, top=8, ff=1024), "4k": dict(width=4096, heads=32, experts=64, top=8, ff=1536)}
HD = 128


def configs(size: str, ctx: int):
    """(sepedra, hybrid)."""
    s = SIZES[size]
    z = sepedra_shape(LAYERS, s["width"], s["heads"], s["experts"], s["top"], s["ff"])
    q = dataclasses.replace(qwen35_hybrid_shape(LAYERS), d_model=s["width"], n_heads=s["heads"], n_kv_heads=s["heads"] // 4, head_dim=HD,
                            rotary_dim=64, gdn_heads=s["heads"], gdn_qk_heads=s["heads"], n_experts=s["experts"], top_k=s["top"],
                            expert_ffn=s["ff"])
    z.max_context = q.max_context = ctx
    return z, q


# ------------------------------------------------------------------------------------------ kernels
def _decode_batch(batch: int, ctx: int, table=None) -> ForwardBatch:
    pos = torch.full((batch,), ctx - 1, dtype=torch.int32, device="cuda")
    ar = torch.arange(batch + 1, dtype=torch.int32, device="cuda")
    return ForwardBatch(pos, pos, ar[:batch], pos + 1, table, None, ctx, row_off=ar, slots=ar[:batch])


def _attn_spec(heads: int) -> A.KVSpec:
    return A.KVSpec(heads, heads // 4, HD, HD, HD ** -0.5, 5e5, HD, 4, {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192})


def attention(tab: _Table, heads: int, batch: int, ctx: int, seqs: int, n: int) -> None:
    spec, hkv = _attn_spec(heads), heads // 4
    f, sinks = spec.inv_freq("cuda"), torch.zeros(heads, device="cuda")
    nb = ctx // PAGE
    table = torch.randperm(nb * batch).view(batch, nb).int().cuda()
    b = _decode_batch(batch, ctx, table)
    kv = [KVLayer(_bf(nb * batch, hkv, PAGE, HD), _bf(nb * batch, hkv, PAGE, HD), None, None, False, PAGE) for _ in range(COPIES)]
    own = [A.KVPages(k.k, k.v, PAGE) for k in kv]
    q, gate = _bf(batch, heads, HD), _bf(batch, heads * HD)
    kvb = 2 * batch * ctx * hkv * HD * 2
    tab.add(f"paged_attention with sink and gate (batch {batch}, {ctx} keys)",
            _us([lambda k=k: A.paged_rows(q, gate, spec, k, sinks, table, b.seq_index, b.kv_lens, ctx) for k in own]), "paged_attention",
            _us([lambda k=k: ops.paged_attention(q.view(batch, -1), k, table, b.seq_index, b.kv_lens, heads, hkv, HD, max_kv=ctx) for k in kv]),
            nbytes=kvb, like_bytes=kvb)
    cw, ring = torch.randn(4, spec.channels, device="cuda"), torch.zeros(batch, 4, spec.channels, device="cuda")
    proj, qkv = _bf(batch, spec.channels + spec.out_cols), _bf(batch, (heads + 2 * hkv) * HD)
    new, old = 2 * spec.channels * 2 + 4 * spec.channels * 4, (2 * heads + 4 * hkv) * HD * 2
    tab.add("kv_prepare (decode)", _us([lambda k=k: A.prepare(proj, spec, cw, f, 1e-6, k, ring, b) for k in own]), "rope_kv_append",
            _us([lambda k=k: ops.rope_kv_append(qkv, b.positions, b.seq_index, table, k, heads, hkv, HD, 1e6, HD) for k in kv]),
            nbytes=batch * new, like_bytes=batch * old)
    T, nb = seqs * n, n // PAGE
    table = torch.randperm(nb * seqs).view(seqs, nb).int().cuda()
    b = make_prefill_batch([[0] * n] * seqs, table, "cuda")
    b.slots = torch.arange(seqs, device="cuda").int()
    kl = KVLayer(_bf(nb * seqs, hkv, PAGE, HD), _bf(nb * seqs, hkv, PAGE, HD), None, None, False, PAGE)
    pages = A.KVPages(kl.k, kl.v, PAGE)
    proj, qkv, q = _bf(T, spec.channels + spec.out_cols), _bf(T, (heads + 2 * hkv) * HD), _bf(T, heads, HD)
    gate, out = proj[:, spec.channels:], _bf(T, heads * HD)
    append = _us([lambda: ops.rope_kv_append(qkv, b.positions, b.seq_index, table, kl, heads, hkv, HD, 1e6, HD)] * 3)
    tab.add("kv_prepare + conv_ring (prompt)", _us([lambda: A.prepare(proj, spec, cw, f, 1e-6, pages, ring, b)] * 3), "rope_kv_append", append,
            nbytes=T * 2 * spec.channels * 2, like_bytes=T * old)
    pt, k = A.plan_portions(b.row_off_host, b.starts_host, 0, "cuda")[0], A._k()
    rows, status = _bf(T, hkv * 2 * HD), workspace(q.device).status
    tab.add("kv_gather", _us([lambda: k.sllm_kv_gather(_p(pages.k), _p(pages.v), PAGE, _p(table), table.stride(0), _p(pt.spans), seqs, n,
                                                       _p(rows), hkv, HD, HD, _stream())] * 3),
            "rope_kv_append", append, nbytes=T * 2 * hkv * 2 * HD * 2, like_bytes=T * old)
    attn = _us([lambda: k.sllm_kv_prefill(_p(q), T, _p(rows), T, _p(pt.tiles), pt.tiles.shape[0], heads, hkv, HD, HD, 0, 0, 0, None, None, 0, 0, spec.scale,
                                          _p(sinks), _p(gate), gate.stride(0), 0, _p(out), _p(status), _stream())] * 3)
    paged = _us([lambda: ops.paged_attention(q.view(T, -1), kl, table, b.seq_index, b.kv_lens, heads, hkv, HD, max_kv=n)] * 2)
    dense = _us([lambda: PF.prefill_attention(qkv, b, heads, hkv, HD)] * 3)
    fl = seqs * n * (n + 1) / 2 * heads * 4 * HD
    for like, us in (("paged_attention (the hybrid's prompts)", paged), ("prefill_attention (dense models)", dense)):
        tab.add(f"kv_prefill ({seqs} x {n})", attn, like, us, flops=fl, like_flops=fl)


def recurrence(tab: _Table, width: int, batch: int, seqs: int, n: int) -> None:
    heads, T = width // HD, seqs * n
    spec = R.RglruSpec(width, width // 256, 4)
    v = lambda: torch.randn(width, device="cuda")
    many = 3 * COPIES
    ws = [R.RglruWeights.make(spec, bias_y=v(), bias_x=v(), conv_w=torch.randn(4, width, device="cuda"), conv_b=v(), bias_r=v(), bias_i=v(),
                              gate_r=_bf(spec.blocks, 256, 256), gate_i=_bf(spec.blocks, 256, 256), lam=v() - 4) for _ in range(many)]
    proj, qkv, z, ba = _bf(T, 2 * width), _bf(T, 3 * width), _bf(T, width), _bf(T, 2 * heads)
    cw, a_log, dtb, nw = _bf(3 * width, 4), torch.zeros(heads, device="cuda"), _bf(heads), torch.ones(HD, device="cuda")

    def old(rows, cs, st, b):
        x = G.conv_silu(qkv[:rows], cw, cs, b.row_off, b.slots)
        return G.recurrent(x, z[:rows], ba[:rows, :heads], ba[:rows, heads:], a_log, dtb, nw, st, b.row_off, b.slots, heads, heads)

    b = make_prefill_batch([[0] * n] * seqs, torch.zeros((seqs, 1), dtype=torch.int32, device="cuda"), "cuda")
    b.slots = torch.arange(seqs, device="cuda").int()
    S, ring = torch.zeros(seqs, width, device="cuda"), torch.zeros(seqs, 4, width, device="cuda")
    st, cs = torch.zeros(seqs, heads, HD, HD, device="cuda"), torch.zeros(seqs, 3, 3 * width, device="cuda", dtype=torch.bfloat16)
    sb = 2 * seqs * heads * HD * HD * 4
    tab.add(f"rglru, prompt ({seqs} x {n}), two launches", _us([lambda w=w: R.rglru(proj, spec, w, S, ring, b) for w in ws[:3]]),
            "gated delta net, conv + prompt form", _us([lambda: old(T, cs, st, b)] * 2), nbytes=T * 3 * width * 2 + 2 * width * 256 * 2,
            like_bytes=T * 5 * width * 2 + sb)
    b = _decode_batch(batch, 512)
    S, ring = torch.zeros(batch, width, device="cuda"), torch.zeros(batch, 4, width, device="cuda")
    sts = [torch.zeros(batch, heads, HD, HD, device="cuda") for _ in range(COPIES)]
    cs = torch.zeros(batch, 3, 3 * width, device="cuda", dtype=torch.bfloat16)
    sb = 2 * batch * heads * HD * HD * 4
    mine = _us([lambda w=w: R.rglru(proj[:batch], spec, w, S, ring, b) for w in ws])
    nbytes = 2 * width * 256 * 2 + batch * width * (3 * 2 + 2 * 4 + 4 * 4)
    tab.add(f"rglru, decode (batch {batch})", mine, "gated delta net, conv + decode form", _us([lambda x=x: old(batch, cs, x, b) for x in sts]),
            nbytes=nbytes, like_bytes=sb + batch * 5 * width * 2)
    wl = [LinearWeight("dense", _bf(2 * width, 256)) for _ in range(many)]
    xr = _bf(batch, 256)
    tab.add(f"rglru, decode (batch {batch})", mine, "gemm_tcgen05 with as many weights", _us([lambda w=w: ops.linear(xr, w) for w in wl]),
            nbytes=nbytes, like_bytes=2 * width * 256 * 2 + batch * (256 + 2 * width) * 2)


def experts(tab: _Table, d: int, E: int, top: int, ff: int, rows: dict) -> None:
    act = M.GatedAct(7.0, 1.702, 1.0)
    gu, dn = _bf(E, 2 * ff, d).mul_(d ** -0.5), _bf(E, d, ff).mul_(ff ** -0.5)
    g4, d4 = (W4Weight.quantize_device("mxfp4", w.float()) for w in (gu, dn))
    wr = LinearWeight("dense", _bf(E, d))
    bank = M.ExpertBank(gu, dn, ff, act)
    for name, t in rows.items():
        x = _bf(t, d)
        idx, wt = M.router(x, wr, top, True, 8, 4)
        off, src, dst, pw = M.permute(idx, wt, 0, E)
        P = t * top
        xp, a = M.gather(x, src, off), _bf(P, ff)
        tile_rows, bn = (32, 128) if P <= 24 * E else (128, 256)
        used = int((off[1:] > off[:-1]).sum())
        for part, w, w4, xin, n, k, mode in (("gate, up, activation", gu, g4, xp, 2 * ff, d, 0), ("down", dn, d4, a, d, ff, 1)):
            mine = _us([lambda: M._grouped(xin, None, w, off, mode, pw, act, n // 2 if mode == 0 else n, P, tile_rows, bn)] * 3)
            if mode == 0:
                like = _us([lambda: ops.gated_act(linear_w4(xin, w4, tok_off=off, max_group_tokens=t), "silu")] * 3)
            else:
                like = _us([lambda: linear_w4(xin, w4, tok_off=off, tok_scale=pw, max_group_tokens=t)] * 3)
            out = n // 2 if mode == 0 else n
            label, other = f"grouped_gemm, {part}, {name} ({P} rows, {used} experts)", "W4A16 grouped GEMM" + (" + gated_act" if mode == 0 else "")
            if P <= 24 * E:
                tab.add(label, mine, other, like, nbytes=used * n * k * 2 + P * (k + out) * 2, like_bytes=used * n * k * 17 / 32 + P * (k + out) * 2)
            else:
                tab.add(label, mine, other, like, flops=2.0 * P * n * k, like_flops=2.0 * P * n * k)
        lg = ops.linear(x, wr)
        tab.add(f"router, {name}", _us([lambda: M.router(x, wr, top, True, 8, 4)] * 3), "gemm_tcgen05 + moe_route",
                _us([lambda: M.route(ops.linear(x, wr), top)] * 3), nbytes=t * d * 2 + E * d * 2, like_bytes=t * d * 2 + E * d * 2)
        del lg
        y, res, w1, wb, xb = _bf(P, d), torch.randn(t, d, device="cuda"), torch.ones(d, device="cuda"), _bf(d), _bf(t, d)
        tab.add(f"group_norm over a token's experts, {name}", _us([lambda: ops.add_group_norm(res, y, w1, None, 1e-6, terms=dst, raw=True)] * 3),
                "moe_combine + rmsnorm", _us([lambda: ops.rmsnorm(M.combine(y, dst, xb), wb, 1e-6)] * 3),
                nbytes=t * d * (top * 2 + 4 + 4 + 2), like_bytes=t * d * (top * 2 + 2 + 2 + 2 + 2))
        y = _bf(t, d)
        tab.add(f"group_norm (x += norm(y), z = x), {name}", _us([lambda: ops.add_group_norm(res, y, w1, None, 1e-6, raw=True)] * 3), "rmsnorm",
                _us([lambda: ops.rmsnorm(xb, wb, 1e-6)] * 3), nbytes=t * d * (2 + 4 + 4 + 2), like_bytes=t * d * 4)


def head(tab: _Table, d: int, vocab: int, batch: int) -> None:
    ws, x = [LinearWeight("dense", _bf(vocab, d)) for _ in range(2)], _bf(batch, d)
    nbytes = vocab * d * 2 + batch * (vocab + d) * 2
    tab.add("output product with soft cap (decode)", _us([lambda w=w: ops.linear(x, w, act="softcap", act_arg=30.0) for w in ws]), "gemm_tcgen05",
            _us([lambda w=w: ops.linear(x, w) for w in ws]), nbytes=nbytes, like_bytes=nbytes)


def kernel_rows(size: str, batch: int, ctx: int) -> list:
    s, tab = SIZES[size], _Table()
    for part in (lambda: attention(tab, s["heads"], batch, ctx, 4, 2048), lambda: recurrence(tab, s["width"], batch, 4, 2048),
                 lambda: experts(tab, s["width"], s["experts"], s["top"], s["ff"], {"prompt": 4 * 2048, "decode": batch}),
                 lambda: head(tab, s["width"], 151936, batch)):
        part()
        torch.cuda.empty_cache()
    return tab.rows


def main(args) -> int:
    out = {"metric": "sepedra_beside_hybrid", "data": "synthetic: seeded random prompts and weights", "layers": LAYERS,
           "prompt": args.prompt, "steps": args.steps, "roofline": peaks()[2], "sizes": {}}
    for size in SIZES:
        z, q = configs(size, ((args.prompt + args.warmup + args.steps + 64 + 255) // 256) * 256)
        models = {name: {f"batch{b}": model_rates(cfg, b, args.prompt, args.steps, args.warmup) for b in (args.batch, 1)}
                  for name, cfg in (("sepedra", z), ("hybrid", q))}
        out["sizes"][size] = {"shape": SIZES[size], "models": models, "kernels": kernel_rows(size, args.batch, args.prompt)}
        torch.cuda.empty_cache()
    print(json.dumps(out))
    return 0
