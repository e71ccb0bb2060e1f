"""Fekolorn beside the framework's closest model - the gated-delta-net hybrid - at equal size (`bench.py --compare fekolorn`).

Sizes are those of a served model's layers with random weights: 8 layers (6 with attention and a delta rule side by side, 2 with
windowed attention, against the hybrid's 6 recurrent and 2 attention layers), equal width, head count, recurrent state and
feed-forward parameters, bf16.  Reported as in family_bench: throughput of both models through their engines, and every kernel of
the new design with its roofline fraction beside the kernel that does the like work in the other model.
"""
from __future__ import annotations

import json

import torch

from .. import ops
from ..engine.batch import make_prefill_batch
from ..models.fekolorn import fekolorn_shape
from ..ops import gdn as G
from ..ops import kv_attention as A
from ..ops import linear_state as S
from ..ops import prefill as PF
from ..ops import streams as R
from ..ops.core import KVLayer, _p, _stream, workspace
from . import family_bench
from .family_bench import COPIES, LAYERS, PAGE, SIZES, _bf, _Table, _us, model_rates
from .kernel_bench import peaks
from .sepedra_bench import _decode_batch

HD, STREAMS, WINDOW, BIAS_MAX = 128, 2, 1024, 512


def configs(size: str, ctx: int):
    """(fekolorn, hybrid): the hybrid's gated feed-forward has three matrices, the other two, so the inner sizes differ by 3/2."""
    s = SIZES[size]
    z = fekolorn_shape(LAYERS, s["width"], s["heads"], s["ffn"] * 3 // 2, STREAMS)
    z.max_context = ctx
    return z, family_bench.configs(size, ctx)[1]


# ------------------------------------------------------------------------------------------ kernels
def attention(tab: _Table, heads: int, batch: int, ctx: int, seqs: int, n: int) -> None:
    hkv = heads // 4
    kw = dict(heads=heads, kv_heads=hkv, dim=HD, vdim=HD, scale=HD ** -0.5, interleaved=False)
    specs = {"full": A.KVSpec(rot_base=5e5, rot_dims=64, qk_norm=False, v_norm=True, **kw),
             "window": A.KVSpec(rot_base=1.0, rot_dims=0, window=WINDOW, norm_all=True, **kw)}
    sinks = torch.zeros(heads, device="cuda")
    dist = A.DistanceBias.make(torch.randn(32, heads, device="cuda"), BIAS_MAX, WINDOW)
    norms = dict(q_norm=torch.ones(heads * HD, device="cuda"), k_norm=torch.ones(hkv * HD, device="cuda"))
    cols, old = (heads + 2 * hkv) * HD, (2 * heads + 4 * hkv) * HD * 2

    def extras(name, proj):
        if name == "full":
            return None, dict()
        return dist, dict(norms, mix=(proj[:, cols - hkv * HD:cols], 0.3))

    nb = ctx // PAGE
    table = torch.randperm(nb * batch).view(batch, nb).int().cuda()
    b = _decode_batch(batch, ctx, table)
    kv = [KVLayer(_bf(nb * batch, hkv, PAGE, HD), _bf(nb * batch, hkv, PAGE, HD), None, None, False, PAGE) for _ in range(COPIES)]
    own = [A.KVPages(k.k, k.v, PAGE) for k in kv]
    q, proj, qkv = _bf(batch, heads, HD), _bf(batch, cols), _bf(batch, cols)
    append = _us([lambda k=k: ops.rope_kv_append(qkv, b.positions, b.seq_index, table, k, heads, hkv, HD, 1e6, 64) for k in kv])
    for name, spec in specs.items():
        d, extra = extras(name, proj)
        f, keys = spec.inv_freq("cuda"), min(ctx, spec.window) if spec.window else ctx
        like = _us([lambda k=k: ops.paged_attention(q.view(batch, -1), k, table, b.seq_index, b.kv_lens, heads, hkv, HD, window=spec.window,
                                                    max_kv=ctx) for k in kv])
        kvb = 2 * batch * hkv * HD * 2 * keys
        tab.add(f"paged_attention, {name} (batch {batch}, {keys} keys)",
                _us([lambda k=k: A.paged_rows(q, None, spec, k, sinks, table, b.seq_index, b.kv_lens, ctx, dist=d) for k in own]),
                "paged_attention", like, nbytes=kvb, like_bytes=kvb)
        tab.add(f"kv_prepare, {name} (decode)", _us([lambda k=k: A.prepare(proj, spec, None, f, 1e-6, k, None, b, **extra) for k in own]),
                "rope_kv_append", append, nbytes=batch * 2 * cols * 2, like_bytes=batch * old)
    dim, vdim = 96, 64                                # heads that the kernel for any sizes takes
    spec = A.KVSpec(heads=heads, kv_heads=hkv, dim=dim, vdim=vdim, scale=dim ** -0.5, rot_base=5e5, rot_dims=64)
    own = [A.KVPages(_bf(nb * batch, hkv, PAGE, dim), _bf(nb * batch, hkv, PAGE, vdim), PAGE) for _ in range(COPIES)]
    like = _us([lambda k=k: ops.paged_attention(q.view(batch, -1), k, table, b.seq_index, b.kv_lens, heads, hkv, HD, max_kv=ctx) for k in kv])
    tab.add(f"paged_attention, keys of {dim}, values of {vdim} (batch {batch}, {ctx} keys)",
            _us([lambda k=k: A.paged_rows(q, None, spec, k, sinks, table, b.seq_index, b.kv_lens, ctx) for k in own]), "paged_attention", like,
            nbytes=batch * hkv * ctx * (dim + vdim) * 2, like_bytes=2 * batch * hkv * HD * 2 * ctx)
    T, nb = seqs * n, n // PAGE
    table = torch.randperm(nb * seqs).view(seqs, nb).int().cuda()
    b = make_prefill_batch([[0] * n] * seqs, table, "cuda")
    b.slots = torch.arange(seqs, device="cuda").int()
    kl = KVLayer(_bf(nb * seqs, hkv, PAGE, HD), _bf(nb * seqs, hkv, PAGE, HD), None, None, False, PAGE)
    pages = A.KVPages(kl.k, kl.v, PAGE)
    proj, qkv, q, out, rows = _bf(T, cols), _bf(T, cols), _bf(T, heads, HD), _bf(T, heads * HD), _bf(T, hkv * 2 * HD)
    status, k = workspace(q.device).status, A._k()
    append = _us([lambda: ops.rope_kv_append(qkv, b.positions, b.seq_index, table, kl, heads, hkv, HD, 1e6, 64)] * 3)
    dense = _us([lambda: PF.prefill_attention(qkv, b, heads, hkv, HD)] * 3)
    full = seqs * n * (n + 1) / 2 * heads * 4 * HD
    pt = A.plan_portions(b.row_off_host, b.starts_host, 0, "cuda")[0]
    tab.add("kv_gather", _us([lambda: k.sllm_kv_gather(_p(pages.k), _p(pages.v), PAGE, _p(table), table.stride(0), _p(pt.spans), seqs, n,
                                                       _p(rows), hkv, HD, HD, _stream())] * 3),
            "rope_kv_append", append, nbytes=T * 4 * hkv * HD * 2, like_bytes=T * old)
    for name, spec in specs.items():
        d, extra = extras(name, proj)
        f = spec.inv_freq("cuda")
        tab.add(f"kv_prepare, {name} (prompt)", _us([lambda: A.prepare(proj, spec, None, f, 1e-6, pages, None, b, **extra)] * 3), "rope_kv_append",
                append, nbytes=T * 2 * cols * 2, like_bytes=T * old)
        pt = A.plan_portions(b.row_off_host, b.starts_host, spec.window, "cuda")[0]
        args = ops.core.dist_args(d)
        run = lambda: k.sllm_kv_prefill(_p(q), T, _p(rows), T, _p(pt.tiles), pt.tiles.shape[0], heads, hkv, HD, HD, spec.window, 0, 0, None, *args,
                                        spec.scale, _p(sinks), None, 0, 0, _p(out), _p(status), _stream())
        paged = _us([lambda: ops.paged_attention(q.view(T, -1), kl, table, b.seq_index, b.kv_lens, heads, hkv, HD, window=spec.window, max_kv=n)] * 2)
        w = spec.window
        us, fl = _us([run] * 3), (seqs * (w * (w + 1) / 2 + (n - w) * w) if w else seqs * n * (n + 1) / 2) * heads * 4 * HD
        for like, t, lf in (("paged_attention (the hybrid's prompts)", paged, fl), ("prefill_attention (dense models)", dense, full)):
            tab.add(f"kv_prefill, {name} ({seqs} x {n})", us, like, t, flops=fl, like_flops=lf)


def recurrence(tab: _Table, heads: int, batch: int, seqs: int, n: int) -> None:
    T, nz = seqs * n, heads * HD
    one = torch.ones(HD, device="cuda")
    spec = S.StateSpec(S.HEAD_DELTA, heads, heads, HD, HD, {"q": 0, "k": nz, "v": 2 * nz, "g": 3 * nz, "a": 4 * nz, "b": 4 * nz + heads},
                       q_scale=HD ** -0.5, taps=4)
    w = S.StateWeights(bias=torch.zeros(heads, device="cuda"), rate=torch.full((heads,), 0.9, device="cuda"),
                       conv_w=torch.randn(4, 3 * nz, device="cuda"), norm=one)
    proj, qkv, z, ba = _bf(T, 4 * nz + 2 * heads), _bf(T, 3 * nz), _bf(T, nz), _bf(T, 2 * heads)
    cw, a_log, dtb = _bf(3 * nz, 4), torch.zeros(heads, device="cuda"), _bf(heads)

    def old(rows, cs, st, b):
        x = G.conv_silu(qkv[:rows], cw, cs, b.row_off, b.slots)
        return G.recurrent(x, z[:rows], ba[:rows, :heads], ba[:rows, heads:], a_log, dtb, one, st, b.row_off, b.slots, heads, heads)

    b = make_prefill_batch([[0] * n] * seqs, torch.zeros((seqs, 1), dtype=torch.int32, device="cuda"), "cuda")
    b.slots = torch.arange(seqs, device="cuda").int()
    st, cs = torch.zeros(seqs, heads, HD, HD, device="cuda"), torch.zeros(seqs, 3, 3 * nz, device="cuda", dtype=torch.bfloat16)
    ring = torch.zeros(batch, 4, 3 * nz, device="cuda")
    nbytes = T * 5 * nz * 2 + 2 * seqs * heads * HD * HD * 4
    tab.add(f"head delta, prompt ({seqs} x {n}), all launches", _us([lambda: S.linear_state(proj, spec, w, 1e-6, st, ring, b)] * 2),
            "gated delta net, conv + prompt form", _us([lambda: old(T, cs, st, b)] * 2), nbytes=nbytes, like_bytes=nbytes)
    b = _decode_batch(batch, 512)
    sts = [torch.zeros(batch, heads, HD, HD, device="cuda") for _ in range(COPIES)]
    cs = torch.zeros(batch, 3, 3 * nz, device="cuda", dtype=torch.bfloat16)
    nbytes = 2 * batch * heads * HD * HD * 4 + batch * 5 * nz * 2
    tab.add(f"head delta, decode (batch {batch})", _us([lambda x=x: S.linear_state(proj[:batch], spec, w, 1e-6, x, ring, b) for x in sts]),
            "gated delta net, conv + decode form", _us([lambda x=x: old(batch, cs, x, b) for x in sts]), nbytes=nbytes, like_bytes=nbytes)


def streams_and_feed_forward(tab: _Table, d: int, ff: int, rows: dict) -> None:
    """``ff``: the hybrid's inner size; the new design's is 3/2 of it."""
    one, wb, n = torch.ones(1, device="cuda"), _bf(d), STREAMS
    c = R.Connection(torch.full((n,), 1.0 / n, device="cuda"), torch.eye(n, device="cuda"), torch.ones(n, device="cuda"))
    table, pair = _bf(20000, d), R.PairEmbedding(_bf(20001, d), 31, 17)
    coef, wide = torch.tensor([0.6, 0.3, 0.3, 0.0], device="cuda"), ff * 3 // 2
    for name, t in rows.items():
        x, xb, y, y2 = torch.randn(t, n, d, device="cuda"), _bf(t, d), _bf(t, d), _bf(t, d)
        rms = _us([lambda: ops.rmsnorm(xb, wb, 1e-6)] * 3)
        tab.add(f"streams (join y, z = norm of the next sum), {name}", _us([lambda: R.join_streams(x, y, c, c.read, one, 1e-6)] * 3), "rmsnorm", rms,
                nbytes=t * d * (8 * n + 2 + 2), like_bytes=t * d * 4)
        tab.add(f"streams (join two outputs), {name}",
                _us([lambda: R.join_streams(x, y, c, c.read, one, 1e-6, 0.7, (y2, 0.7))] * 3), "rmsnorm", rms,
                nbytes=t * d * (8 * n + 4 + 2), like_bytes=t * d * 4)
        b = _decode_batch(t, 64)
        b.tokens = torch.randint(0, 20000, (t,), device="cuda").int()
        last = torch.zeros(t, 1, device="cuda")
        tab.add(f"streams (start, pair embedding), {name}",
                _us([lambda: R.start_streams(table, b, 2.0, pair, last, n, c.read, one, 1e-6)] * 3), "embedding",
                _us([lambda: ops.embedding(table, b.tokens)] * 3), nbytes=t * d * (4 + 4 * n + 2), like_bytes=t * d * 4)
        tab.add(f"streams (z = norm of the sum), {name}", _us([lambda: R.read_streams(x, one, 1e-6, torch.bfloat16)] * 3), "rmsnorm", rms,
                nbytes=t * d * (4 * n + 2), like_bytes=t * d * 4)
        u, gu = _bf(t, wide), _bf(t, 2 * ff)
        tab.add(f"poly_norm, {name}", _us([lambda: ops.poly_norm(u, coef, 1e-6)] * 3), "gated_act", _us([lambda: ops.gated_act(gu)] * 3),
                nbytes=t * wide * 4, like_bytes=t * ff * 6)


def kernel_rows(size: str, batch: int, ctx: int) -> list:
    s, tab = SIZES[size], _Table()
    rows = {"prompt": 4 * 2048, "decode": batch}
    for part in (lambda: attention(tab, s["heads"], batch, ctx, 4, 2048), lambda: recurrence(tab, s["heads"], batch, 4, 2048),
                 lambda: streams_and_feed_forward(tab, s["width"], s["ffn"], rows)):
        part()
        torch.cuda.empty_cache()
    return tab.rows


def main(args) -> int:
    out = {"metric": "fekolorn_beside_hybrid", "data": "synthetic: seeded random prompts and weights", "layers": LAYERS,
           "prompt": args.prompt, "steps": args.steps, "roofline": peaks()[2], "sizes": {}}
    for size in SIZES:
        z, q = configs(size, ((args.prompt + args.warmup + args.steps + 64 + 255) // 256) * 256)
        models = {name: {f"batch{b}": model_rates(cfg, b, args.prompt, args.steps, args.warmup) for b in (args.batch, 1)}
                  for name, cfg in (("fekolorn", z), ("hybrid", q))}
        out["sizes"][size] = {"shape": SIZES[size], "models": models, "kernels": kernel_rows(size, args.batch, args.prompt)}
        torch.cuda.empty_cache()
    print(json.dumps(out))
    return 0
