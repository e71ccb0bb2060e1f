"""Kegorax beside the framework's closest model - the gated-delta-net hybrid with routed experts - at equal size
(`bench.py --compare kegorax`).

Sizes are those of a served model's layers with random weights: 8 layers (6 delta-rule ones, one of each parallel kind against
the hybrid's 6 recurrent and 2 attention layers), equal width, head count, experts and experts per token.  Half of Kegorax's
feed-forwards are dense; its experts are bf16, the hybrid's MXFP4 (the only form its experts have).  Reported as in
family_bench: throughput of both models through their engines, and every kernel of the new design with its roofline fraction
beside the kernel that does the like work in the other model.
"""
from __future__ import annotations

import json

import torch

from .. import ops
from ..engine.batch import make_prefill_batch
from ..models.kegorax import kegorax_shape
from ..ops import gdn as G
from ..ops import kv_attention as A
from ..ops import linear_state as S
from ..ops import moe as M
from ..ops import prefill as PF
from ..ops.core import KVLayer, LinearWeight, _p, _stream, workspace
from . import sepedra_bench
from .family_bench import COPIES, LAYERS, PAGE, _bf, _Table, _us, model_rates
from .kernel_bench import peaks
from .sepedra_bench import SIZES, _decode_batch

HD, RANK = 128, 64
FF = 3                         # dense feed-forward: this many widths


def configs(size: str, ctx: int):
    """(kegorax, hybrid)."""
    s = SIZES[size]
    z = kegorax_shape(LAYERS, s["width"], s["heads"], FF * s["width"], s["experts"], s["top"], s["ff"])
    z.max_context = ctx
    return z, sepedra_bench.configs(size, ctx)[1]


# ------------------------------------------------------------------------------------------ kernels
def _specs(heads: int) -> dict:
    kw = dict(heads=heads, kv_heads=heads // 4, dim=HD, vdim=HD, scale=HD ** -0.5, interleaved=False, gate_heads=True)
    return {"chunks": A.KVSpec(rot_base=5e5, rot_dims=64, chunk=2048, qk_norm=False, **kw),
            "window": A.KVSpec(rot_base=1.0, rot_dims=0, window=1024, keep_first=4, **kw)}


def attention(tab: _Table, heads: int, batch: int, ctx: int, seqs: int, n: int) -> None:
    hkv = heads // 4
    sinks, slopes, norm = torch.zeros(heads, device="cuda"), A.distance_slopes(heads, "cuda"), torch.ones(HD, device="cuda")
    nb = ctx // PAGE
    table = torch.randperm(nb * batch).view(batch, nb).int().cuda()
    b = _decode_batch(batch, ctx, table)
    kv = [KVLayer(_bf(nb * batch, hkv, PAGE, HD), _bf(nb * batch, hkv, PAGE, HD), None, None, False, PAGE) for _ in range(COPIES)]
    own = [A.KVPages(k.k, k.v, PAGE) for k in kv]
    q = _bf(batch, heads, HD)
    cols = (heads + 2 * hkv) * HD
    bias = torch.zeros(cols, device="cuda")
    proj, qkv = _bf(batch, cols + 64), _bf(batch, cols)
    gate, old = proj[:, cols:cols + heads], (2 * heads + 4 * hkv) * HD * 2
    append = _us([lambda k=k: ops.rope_kv_append(qkv, b.positions, b.seq_index, table, k, heads, hkv, HD, 1e6, 64) for k in kv])
    for name, spec in _specs(heads).items():
        extra = dict(bias=bias, q_norm=norm, k_norm=norm) if spec.window else {}
        f, sl, g = spec.inv_freq("cuda"), slopes if spec.window else None, None if spec.window else gate
        keys = min(ctx, spec.window + spec.keep_first) if spec.window else ctx
        like = _us([lambda k=k: ops.paged_attention(q.view(batch, -1), k, table, b.seq_index, b.kv_lens, heads, hkv, HD, window=spec.window,
                                                    max_kv=ctx) for k in kv])
        kvb = 2 * batch * hkv * HD * 2
        tab.add(f"paged_attention, {name} (batch {batch}, {keys} keys)",
                _us([lambda k=k: A.paged_rows(q, g, spec, k, sinks, table, b.seq_index, b.kv_lens, ctx, slopes=sl) for k in own]),
                "paged_attention", like, nbytes=kvb * keys, like_bytes=kvb * (min(ctx, spec.window) if spec.window else ctx))
        tab.add(f"kv_prepare, {name} (decode)", _us([lambda k=k: A.prepare(proj, spec, None, f, 1e-6, k, None, b, **extra) for k in own]),
                "rope_kv_append", append, nbytes=batch * 2 * cols * 2, like_bytes=batch * old)
    T, nb = seqs * n, n // PAGE
    table = torch.randperm(nb * seqs).view(seqs, nb).int().cuda()
    b = make_prefill_batch([[0] * n] * seqs, table, "cuda")
    b.slots = torch.arange(seqs, device="cuda").int()
    kl = KVLayer(_bf(nb * seqs, hkv, PAGE, HD), _bf(nb * seqs, hkv, PAGE, HD), None, None, False, PAGE)
    pages = A.KVPages(kl.k, kl.v, PAGE)
    proj, qkv, q, out, rows = _bf(T, cols + 64), _bf(T, cols), _bf(T, heads, HD), _bf(T, heads * HD), _bf(T, hkv * 2 * HD)
    gate, status, k = proj[:, cols:cols + heads], workspace(q.device).status, A._k()
    append = _us([lambda: ops.rope_kv_append(qkv, b.positions, b.seq_index, table, kl, heads, hkv, HD, 1e6, 64)] * 3)
    dense = _us([lambda: PF.prefill_attention(qkv, b, heads, hkv, HD)] * 3)
    full = seqs * n * (n + 1) / 2 * heads * 4 * HD
    for name, spec in _specs(heads).items():
        extra = dict(bias=bias, q_norm=norm, k_norm=norm) if spec.window else {}
        f, sl, g = spec.inv_freq("cuda"), slopes if spec.window else None, None if spec.window else gate
        tab.add(f"kv_prepare, {name} (prompt)", _us([lambda: A.prepare(proj, spec, None, f, 1e-6, pages, None, b, **extra)] * 3), "rope_kv_append",
                append, nbytes=T * 2 * cols * 2, like_bytes=T * old)
        pt = A.plan_portions(b.row_off_host, b.starts_host, spec.window, "cuda", spec.keep_first, spec.chunk)[0]
        run = lambda: k.sllm_kv_prefill(_p(q), T, _p(rows), T, _p(pt.tiles), pt.tiles.shape[0], heads, hkv, HD, HD, spec.window, spec.keep_first,
                                        spec.chunk, _p(sl), None, 0, 0, spec.scale, _p(sinks), _p(g), g.stride(0) if g is not None else 0, 1, _p(out),
                                        _p(status), _stream())
        paged = _us([lambda: ops.paged_attention(q.view(T, -1), kl, table, b.seq_index, b.kv_lens, heads, hkv, HD, window=spec.window, max_kv=n)] * 2)
        w = spec.window
        pairs = seqs * (w * (w + 1) / 2 + (n - w) * (w + spec.keep_first)) if w else seqs * n * (n + 1) / 2
        us, fl = _us([run] * 3), pairs * heads * 4 * HD
        for like, t, lf in (("paged_attention (the hybrid's prompts)", paged, fl), ("prefill_attention (dense models)", dense, full)):
            tab.add(f"kv_prefill, {name} ({seqs} x {n})", us, like, t, flops=fl, like_flops=lf)


def recurrences(tab: _Table, heads: int, batch: int, seqs: int, n: int) -> None:
    T, nz = seqs * n, heads * HD
    lw = lambda: LinearWeight("dense", _bf(nz, RANK).mul_(RANK ** -0.5))
    zero, one, rate = torch.zeros(nz, device="cuda"), torch.ones(HD, device="cuda"), torch.full((heads,), 0.9, device="cuda")
    wide = {"q": 0, "k": nz, "v": 2 * nz}
    kw = dict(heads=heads, kv_heads=heads, dim=HD, vdim=HD)
    forms = {
        "gated linear": (S.StateSpec(S.GATED, columns=dict(wide, g=3 * nz, a=4 * nz), q_scale=HD ** -0.5, tau=16.0, rank_a=RANK, **kw),
                         S.StateWeights(w_a=lw(), bias=zero, norm=one)),
        "retention": (S.StateSpec(S.FIXED, columns=dict(wide, g=3 * nz), k_scale=HD ** -0.5, **kw), S.StateWeights(rate=rate)),
        "channel delta": (S.StateSpec(S.DELTA, columns=dict(wide, b=3 * nz, a=3 * nz + 64, g=3 * nz + 64 + RANK), q_scale=HD ** -0.5, taps=4,
                                      rank_a=RANK, rank_g=RANK, **kw),
                          S.StateWeights(w_a=lw(), w_g=lw(), bias=zero, rate=rate, conv_w=torch.randn(4, 3 * nz, device="cuda"), norm=one))}
    proj, qkv, z, ba = _bf(T, 4 * nz + RANK), _bf(T, 3 * nz), _bf(T, nz), _bf(T, 2 * heads)
    cw, a_log, dtb = _bf(3 * nz, 4), torch.zeros(heads, device="cuda"), _bf(heads)

    def old(rows, cs, st, b, conv):
        x = G.conv_silu(qkv[:rows], cw, cs, b.row_off, b.slots) if conv else qkv[:rows]
        return G.recurrent(x, z[:rows], ba[:rows, :heads], ba[:rows, heads:], a_log, dtb, one, st, b.row_off, b.slots, heads, heads)

    b = make_prefill_batch([[0] * n] * seqs, torch.zeros((seqs, 1), dtype=torch.int32, device="cuda"), "cuda")
    b.slots = torch.arange(seqs, device="cuda").int()
    st, cs = torch.zeros(seqs, heads, HD, HD, device="cuda"), torch.zeros(seqs, 3, 3 * nz, device="cuda", dtype=torch.bfloat16)
    ring = torch.zeros(batch, 4, 3 * nz, device="cuda")
    sb = 2 * seqs * heads * HD * HD * 4
    like = {c: _us([lambda: old(T, cs, st, b, c)] * 2) for c in (False, True)}
    for name, (spec, w) in forms.items():
        d = spec.form == S.DELTA
        tab.add(f"{name}, prompt ({seqs} x {n}), all launches", _us([lambda: S.linear_state(proj, spec, w, 1e-6, st, ring if d else None, b)] * 2),
                "gated delta net" + (", conv + prompt form" if d else ", prompt form"), like[d], nbytes=T * 5 * nz * 2 + sb,
                like_bytes=T * 5 * nz * 2 + sb)
    b = _decode_batch(batch, 512)
    sts = [torch.zeros(batch, heads, HD, HD, device="cuda") for _ in range(COPIES)]
    cs = torch.zeros(batch, 3, 3 * nz, device="cuda", dtype=torch.bfloat16)
    sb = 2 * batch * heads * HD * HD * 4
    like = {c: _us([lambda x=x: old(batch, cs, x, b, c) for x in sts]) for c in (False, True)}
    for name, (spec, w) in forms.items():
        d = spec.form == S.DELTA
        tab.add(f"{name}, decode (batch {batch})",
                _us([lambda x=x: S.linear_state(proj[:batch], spec, w, 1e-6, x, ring if d else None, b) for x in sts]),
                "gated delta net" + (", conv + decode form" if d else ", decode form"), like[d],
                nbytes=sb + batch * 5 * nz * 2, like_bytes=sb + batch * 5 * nz * 2)


def norms_and_feed_forward(tab: _Table, d: int, E: int, top: int, ff: int, rows: dict) -> None:
    act = M.GatedAct()
    gu, dn = _bf(E, 2 * ff, d).mul_(d ** -0.5), _bf(E, d, ff).mul_(ff ** -0.5)
    wr, sc = LinearWeight("dense", _bf(E, d)), M.SigmoidScores(torch.zeros(E, device="cuda"), 2.5)
    bank = M.ExpertBank(gu, dn, ff, act)
    table, w, wb = _bf(1000, d), torch.ones(d, device="cuda"), _bf(d)
    for name, t in rows.items():
        x = _bf(t, d)
        route = lambda: M.router(x, wr, top, groups=8, keep=4, group_top=2, sigmoid=sc)
        tab.add(f"router (corrected sigmoid, groups), {name}", _us([route] * 3), "gemm_tcgen05 + moe_route",
                _us([lambda: M.route(ops.linear(x, wr), top)] * 3), nbytes=t * d * 2 + E * d * 2, like_bytes=t * d * 2 + E * d * 2)
        idx, wt = route()
        dst = M.bank_forward(x, idx, wt, bank)[1]
        yp, res, y, y2 = _bf(t * top, d), torch.randn(t, d, device="cuda"), _bf(t, d), _bf(t, d)
        ids = torch.randint(0, 1000, (t,), device="cuda").int()
        rms = _us([lambda: ops.rmsnorm(x, wb, 1e-6)] * 3)
        tab.add(f"group_norm over a token's experts, {name}", _us([lambda: ops.add_group_norm(res, yp, None, w, 1e-6, terms=dst)] * 3),
                "moe_combine + rmsnorm", _us([lambda: ops.rmsnorm(M.combine(yp, dst, x), wb, 1e-6)] * 3),
                nbytes=t * d * (top * 2 + 4 + 4 + 2), like_bytes=t * d * (top * 2 + 2 + 2 + 2 + 2))
        tab.add(f"group_norm (x += y, z = norm(x)), {name}", _us([lambda: ops.add_group_norm(res, y, None, w, 1e-6)] * 3), "rmsnorm", rms,
                nbytes=t * d * (2 + 4 + 4 + 2), like_bytes=t * d * 4)
        tab.add(f"group_norm (x += norm(y) + norm(y2), z = norm(x)), {name}",
                _us([lambda: ops.add_group_norm(res, y, w, w, 1e-6, coef=0.5, second=(y2, w, 0.5))] * 3), "rmsnorm", rms,
                nbytes=t * d * (2 + 2 + 4 + 4 + 2), like_bytes=t * d * 4)
        tab.add(f"group_norm (x += y + embedding + step, z = norm(x)), {name}",
                _us([lambda: ops.add_group_norm(res, y, None, w, 1e-6, again=ops.Again(table, ids, 2.0, w))] * 3), "rmsnorm", rms,
                nbytes=t * d * (2 + 2 + 4 + 4 + 2), like_bytes=t * d * 4)


def kernel_rows(size: str, batch: int, ctx: int) -> list:
    s, tab = SIZES[size], _Table()
    rows = {"prompt": 4 * 2048, "decode": batch}
    for part in (lambda: attention(tab, s["heads"], batch, ctx, 4, 2048), lambda: recurrences(tab, s["heads"], batch, 4, 2048),
                 lambda: norms_and_feed_forward(tab, s["width"], s["experts"], s["top"], s["ff"], rows)):
        part()
        torch.cuda.empty_cache()
    return tab.rows


def main(args) -> int:
    out = {"metric": "kegorax_beside_hybrid", "data": "synthetic: seeded random prompts and weights", "layers": LAYERS,
           "prompt": args.prompt, "steps": args.steps, "roofline": peaks()[2], "sizes": {}}
    for size in SIZES:
        z, q = configs(size, ((args.prompt + args.warmup + args.steps + 64 + 255) // 256) * 256)
        models = {name: {f"batch{b}": model_rates(cfg, b, args.prompt, args.steps, args.warmup) for b in (args.batch, 1)}
                  for name, cfg in (("kegorax", z), ("hybrid", q))}
        out["sizes"][size] = {"shape": SIZES[size], "models": models, "kernels": kernel_rows(size, args.batch, args.prompt)}
        torch.cuda.empty_cache()
    print(json.dumps(out))
    return 0
