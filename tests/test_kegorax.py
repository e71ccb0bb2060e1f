"""Kegorax against its plain restatement (tests/kegorax_oracle.py): every mechanism, whole prompts, portions, decoding, mixed
batches, pages and slots used again, the scheduler, files and the command line - on the CPU oracle path of the ops and, where a
GPU is present, on the CUDA kernels in fp32 and bf16."""
import json
import os

import pytest
import torch

import kegorax_cases as K
import kegorax_oracle as O
from sllm_b200 import ops
from sllm_b200.cache.paged import OutOfPages
from sllm_b200.engine.batch import ForwardBatch, make_prefill_batch
from sllm_b200.ops import kv_attention as A
from sllm_b200.ops import linear_state as S
from sllm_b200.ops import moe as M
from sllm_b200.ops.core import LinearWeight

RUNS = [("cpu", "fp32"), pytest.param("cuda", "fp32", marks=pytest.mark.gpu), pytest.param("cuda", "bf16", marks=pytest.mark.gpu)]
DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]


@pytest.fixture(scope="module", autouse=True)
def _one_thread():
    """The sizes are tiny: a thread pool per operation costs more than the operations."""
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


@pytest.fixture(scope="module")
def cases(tmp_path_factory):
    made = {}

    def get(name, seed=0):
        if (name, seed) not in made:
            made[name, seed] = K.Case(tmp_path_factory.mktemp("kg"), name, seed)
        return made[name, seed]
    return get


# ------------------------------------------------------------------------------------------ mechanisms
def test_order_of_runs_and_their_additions():
    from sllm_b200.models.kegorax import layer_runs
    for n, loop in ((4, (1, 3, 3)), (3, (0, 3, 2)), (5, (2, 5, 1)), (2, (0, 1, 4)), (3, None)):
        cfg = {"layers": [0] * n}
        if loop:
            cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
        want = O.order(cfg)
        got = layer_runs(n, cfg.get("loop"))
        assert [i for i, _ in got] == [i for i, _ in want]
        assert [t for _, t in got] == [t if t is not None and i == loop[0] else None for i, t in want]


def test_masks_and_slopes_as_stated():
    j = torch.arange(60)
    for i in (0, 1, 9, 10, 11, 39, 59):
        c = A.KVSpec(1, 1, 4, 4, 1.0, 1.0, 0, chunk=10)
        w = A.KVSpec(1, 1, 4, 4, 1.0, 1.0, 0, window=7, keep_first=3)
        k = j[:i + 1]
        assert c.sees(i, k).tolist() == [O.sees_chunk(i, int(x), 10) for x in k]
        assert w.sees(i, k).tolist() == [O.sees_window(i, int(x), 7, 3) for x in k]
    for n in (1, 3, 8, 12):
        assert torch.allclose(A.distance_slopes(n, "cpu").double(), torch.tensor([O.slope(h, n) for h in range(n)]).double(), rtol=1e-6)


@pytest.mark.parametrize("window,keep,chunk", [(70, 0, 0), (70, 9, 0), (70, 200, 0), (0, 0, 96), (0, 0, 500), (130, 64, 0)])
def test_portions_gather_what_their_rows_see(window, keep, chunk):
    """Gathered positions of a portion: everything that any of its rows sees, kept positions first."""
    row_off, starts = [0, 100, 103, 403], [0, 40, 290]
    port = [p for p in A.plan_portions(row_off, starts, window, "cpu", keep, chunk) if p.spans is not None]
    spec = A.KVSpec(1, 1, 4, 4, 1.0, 1.0, 0, window=window, keep_first=keep, chunk=chunk)
    seen_seqs = set()
    for p in port:
        at = {}
        for s, lo, n, row in p.spans.tolist():
            for x in range(n):
                assert at.setdefault((s, row + x), lo + x) == lo + x
        assert sorted(r for _, r in at) == list(range(p.context))
        for q_row, rows, q0, ctx, lo, start, _, _ in p.tiles.tolist():
            s = next(i for i in range(3) if row_off[i] <= p.lo + q_row < row_off[i + 1])
            seen_seqs.add(s)
            assert q0 == starts[s] + p.lo + q_row - row_off[s] and at[s, ctx] == lo
            held = {pos for (ss, _), pos in at.items() if ss == s}
            for i in (q0, q0 + rows - 1):
                j = torch.arange(i + 1)
                assert set(j[spec.sees(i, j)].tolist()) <= held
            if keep and lo > keep:
                assert all(at[s, start + x] == x for x in range(keep))
            elif keep:
                assert start == ctx and lo == 0
    assert seen_seqs == {0, 2}


def _state_case(form, H, G, D, V, taps, ra, rg, seed=0):
    """(spec, weights in fp32, columns of a packed projection)."""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, generator=g)
    pad = lambda n: (n + 7) // 8 * 8
    widths = [("q", G * D), ("k", G * D), ("v", H * V), ("g", rg if form == S.DELTA else H * V), ("a", ra), ("b", H)]
    col, at = {}, 0
    for n, w in widths:
        col[n] = at
        at += w
        if form != S.DELTA or n not in ("q", "k"):
            at = pad(at)
    mat = lambda n, r: LinearWeight("dense", torch.cat([0.5 * rnd(n, r), torch.zeros(n, pad(r) - r)], 1))
    w = S.StateWeights()
    kw = {}
    if form == S.FIXED:
        w.rate = 1 - torch.rand(H, generator=g) * 0.2
        kw = dict(k_scale=D ** -0.5)
    else:
        w.w_a, w.bias, w.norm = mat(H * D, ra), rnd(H * D) + (1 if form == S.GATED else -2), 1 + 0.3 * rnd(V)
        kw = dict(q_scale=D ** -0.5, tau=4.0 if form == S.GATED else 1.0, rank_a=ra)
    if form == S.DELTA:
        w.w_g, w.rate, w.conv_w = mat(H * V, rg), torch.exp(0.7 * rnd(H)), 0.7 * rnd(taps, 2 * G * D + H * V)
        kw.update(rank_g=rg, taps=taps)
    return S.StateSpec(form, H, G, D, V, col, **kw), w, at


def _state_want(proj, spec, w, eps):
    """fp64 outputs of one sequence from its start."""
    p, t, H, G, D, V, col = proj.double(), proj.shape[0], spec.heads, spec.kv_heads, spec.dim, spec.vdim, spec.columns
    f = lambda n, m: p[:, col[n]:col[n] + m]
    dec = lambda lw: lw.w.double()
    q, k, v = f("q", G * D), f("k", G * D), f("v", H * V)
    if spec.form == S.DELTA:
        c = w.conv_w.double().T
        q, k, v = (O.silu(O.causal_conv(x, cw)) for x, cw in zip((q, k, v), c.split([G * D, G * D, H * V])))
    q, k, v = q.reshape(t, G, D), k.reshape(t, G, D), v.reshape(t, H, V)
    if spec.form == S.DELTA:
        q, k = O.unit(q), O.unit(k)
    q, k = (spec.q_scale * q).repeat_interleave(H // G, 1), (spec.k_scale * k).repeat_interleave(H // G, 1)
    if spec.form == S.FIXED:
        o = O.linear_states(q, k, v, w.rate.double()[None, :, None].expand(t, H, D))
    else:
        z = (f("a", spec.rank_a) @ dec(w.w_a)[:, :spec.rank_a].T + w.bias.double()).view(t, H, D)
        if spec.form == S.GATED:
            o = O.linear_states(q, k, v, torch.sigmoid(z) ** (1 / spec.tau))
        else:
            o = O.delta_states(q, k, v, torch.exp(-w.rate.double()[None, :, None] * torch.log1p(torch.exp(z))), torch.sigmoid(f("b", H)))
    o = O.rms(o, eps) * (1 if w.norm is None else w.norm.double())
    gate = torch.sigmoid(f("g", spec.rank_g) @ dec(w.w_g)[:, :spec.rank_g].T) if spec.form == S.DELTA else O.silu(f("g", H * V))
    return o.reshape(t, -1) * gate


def _to(w, device, dtype):
    out = S.StateWeights(**vars(w))
    for n, x in vars(w).items():
        if isinstance(x, LinearWeight):
            setattr(out, n, LinearWeight("dense", x.w.to(device, dtype)))
        elif x is not None:
            setattr(out, n, x.to(device))
    return out


STATE_SIZES = [(2, 2, 12, 20, 3, 5, 9), (3, 1, 16, 16, 1, 8, 8), (4, 2, 64, 128, 4, 16, 24), (6, 3, 10, 7, 5, 3, 11), (2, 1, 200, 33, 2, 40, 8),
               (1, 1, 128, 264, 4, 64, 64), (2, 2, 300, 24, 4, 8, 16)]


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("form", [S.GATED, S.FIXED, S.DELTA])
@pytest.mark.parametrize("H,G,D,V,taps,ra,rg", STATE_SIZES)
def test_recurrences_over_portions_and_steps(device, dtype, form, H, G, D, V, taps, ra, rg):
    """Unequal portions of several sequences in slots out of order, then single tokens, each going on where it was."""
    G = G if form == S.DELTA else H
    dt = torch.float32 if dtype == "fp32" else torch.bfloat16
    spec, w32, width = _state_case(form, H, G, D, V, taps, ra, rg)
    w = _to(w32, device, dt)
    if dtype == "bf16":
        w32 = _to(w, "cpu", torch.float32)
    lens, steps = [[1, 17, 2], [9, 2, 1], [20, 1, 3]], 4
    total = [sum(x) + steps for x in lens]
    g = torch.Generator().manual_seed(5)
    proj = [torch.randn(n, width, generator=g).to(dt) for n in total]
    slots = [4, 0, 2]
    state = torch.full((5, H, D, V), 7.0, device=device)
    ring = torch.full((5, taps, spec.channels), 99.0, device=device) if form == S.DELTA else None
    state[slots] = 0
    out, at = [[], [], []], [0, 0, 0]
    table = torch.zeros((3, 1), dtype=torch.int32, device=device)
    for k in range(3 + steps):
        n = [x[k] for x in lens] if k < 3 else [1] * 3
        if k < 3:
            b = make_prefill_batch([[0] * m for m in n], table, device, at)
        else:
            pos = torch.tensor(at, dtype=torch.int32, device=device)
            ar = torch.arange(4, dtype=torch.int32, device=device)
            b = ForwardBatch(pos, pos, ar[:3], pos + 1, table, row_off=ar)
        b.slots = torch.tensor(slots, dtype=torch.int32, device=device)
        y = S.linear_state(torch.cat([proj[i][at[i]:at[i] + n[i]] for i in range(3)]).to(device), spec, w, 1e-5, state, ring, b)
        for i, part in enumerate(y.float().cpu().split(n)):
            out[i].append(part)
            at[i] += n[i]
    for i in range(3):
        want, got = _state_want(proj[i], spec, w32, 1e-5), torch.cat(out[i]).double()
        tol = 3e-5 if dtype == "fp32" else 2e-2
        assert (got - want).pow(2).mean().sqrt() < tol * want.pow(2).mean().sqrt(), i
        assert (got - want).abs().max() < 6 * tol * want.abs().max(), i
    assert (state[[1, 3]] == 7).all() and (ring is None or (ring[[1, 3]] == 99).all())


def _attn_inputs(device, dt, spec, ends, seed=0):
    g = torch.Generator().manual_seed(seed)
    up = lambda n: (n + 7) // 8 * 8
    nb = (max(ends) + 15) // 16
    n = nb * len(ends) + 2
    kv = A.KVPages(*(torch.randn(n, spec.kv_heads, 16, up(x), generator=g).to(device, dt) for x in (spec.dim, spec.vdim)), 16)
    table = torch.randperm(n, generator=g)[:nb * len(ends)].view(len(ends), nb).int().to(device)
    proj = [torch.randn(e, up(spec.channels) + up(spec.heads), generator=g).to(dt) for e in ends]
    return kv, table, proj


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,rot,size,keep", [
    (4, 2, 64, 64, 32, 40, None), (6, 3, 20, 24, 20, 33, None), (3, 1, 72, 40, 8, 150, None), (5, 5, 7, 9, 2, 16, None), (2, 1, 256, 256, 0, 50, None),
    (4, 2, 64, 64, 0, 24, 5), (8, 1, 128, 128, 0, 70, 20), (6, 2, 20, 24, 0, 33, 0), (3, 1, 72, 40, 0, 140, 150), (2, 2, 10, 14, 0, 1, 1),
    (5, 1, 64, 64, 0, 64, 129)])
def test_attention_over_portions_and_steps(device, dtype, heads, kv_heads, dim, vdim, rot, size, keep):
    """Chunked (keep None) and windowed attention with all that belongs to them, from projections to gated outputs."""
    dt = torch.float32 if dtype == "fp32" else torch.bfloat16
    chunked = keep is None
    spec = A.KVSpec(heads, kv_heads, dim, vdim, 1.5 * dim ** -0.5, 3e3, rot, qk_norm=not chunked, chunk=size if chunked else 0,
                    window=0 if chunked else size, keep_first=keep or 0, interleaved=False, gate_heads=True)
    lens = [[90, 2, 130], [1, 3, 40], [65, 64, 1]] if device == "cuda" else [[30, 2, 20], [1, 3, 20], [17, 16, 1]]
    ends = [sum(x) + 3 for x in lens]
    kv, table, proj = _attn_inputs(device, dt, spec, ends)
    g = torch.Generator().manual_seed(9)
    rnd = lambda n, m=0.0: (m + 0.4 * torch.randn(n, generator=g)).to(device)
    bias, qn, kn = (None, None, None) if chunked else (rnd(spec.channels), rnd(dim, 1.0), rnd(dim, 1.0))
    sinks = 3 * rnd(heads) if chunked else torch.zeros(heads, device=device)
    slopes = None if chunked else A.distance_slopes(heads, device)
    gcol = (spec.channels + 7) // 8 * 8
    f = spec.inv_freq(device)
    out, at = [[], [], []], [0, 0, 0]
    for k in range(6):
        n = [x[k] for x in lens] if k < 3 else [1] * 3
        if k < 3:
            b = make_prefill_batch([[0] * m for m in n], table, device, at)
        else:
            pos = torch.tensor(at, dtype=torch.int32, device=device)
            ar = torch.arange(4, dtype=torch.int32, device=device)
            b = ForwardBatch(pos, pos, ar[:3], pos + 1, table, row_off=ar)
        b.slots = torch.arange(3, dtype=torch.int32, device=device)
        x = torch.cat([proj[i][at[i]:at[i] + n[i]] for i in range(3)]).to(device)
        q = A.prepare(x, spec, None, f, 1e-5, kv, None, b, bias=bias, q_norm=qn, k_norm=kn)
        gate = x[:, gcol:gcol + heads] if chunked else None
        y = A.attention(q, gate, spec, kv, sinks, b, slopes)
        if device == "cuda":                                # the any-size kernel over the same pages
            z = A.paged_rows(q, gate, spec, kv, sinks, table, b.seq_index, b.kv_lens, b.max_kv, impl="cuda_core_any", slopes=slopes)
            assert (y.float() - z.float()).abs().max() < (2e-5 if dtype == "fp32" else 4e-2) * z.float().abs().max()
        for i, part in enumerate(y.float().cpu().split(n)):
            out[i].append(part)
            at[i] += n[i]
    c64 = lambda v: v.double().cpu()
    for i, e in enumerate(ends):
        p = proj[i].double()
        x = p[:, :spec.channels] + (0 if bias is None else c64(bias))
        q, k, v = (y.reshape(e, -1, m) for y, m in zip(x.split([heads * dim, kv_heads * dim, kv_heads * vdim], 1), (dim, dim, vdim)))
        if chunked:
            q, k = (O.rotate(y, {"base": 3e3, "dims": rot}) for y in (q, k))
            seen = O.visible(e, lambda a, b: O.sees_chunk(a, b, size))
        else:
            q, k = O.rms(q, 1e-5) * c64(qn), O.rms(k, 1e-5) * c64(kn)
            seen = O.visible(e, lambda a, b: O.sees_window(a, b, size, keep))
        want = O.attend(q, k, v, spec.scale, seen, c64(sinks), None if chunked else [O.slope(h, heads) for h in range(heads)])
        if chunked:
            want = want * torch.sigmoid(p[:, gcol:gcol + heads])[:, :, None]
        d = torch.cat(out[i]).double() - want.reshape(e, -1)
        assert d.abs().max() < (3e-5 if dtype == "fp32" else 5e-2) * want.abs().max(), i
        assert d.pow(2).mean().sqrt() < (1e-5 if dtype == "fp32" else 1e-2) * want.pow(2).mean().sqrt(), i


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("E,top,count,keep", [(15, 4, 5, 3), (8, 1, 8, 1), (64, 8, 8, 4), (5, 5, 1, 1), (200, 20, 10, 3), (6, 2, 2, 2), (256, 6, 64, 2)])
def test_corrected_sigmoid_routing(device, E, top, count, keep):
    """Choice by score + correction (negative ones too) from the groups with the best pair, weights by the score alone."""
    g = torch.Generator().manual_seed(E)
    z, c = torch.randn(40, E, generator=g) * 2, torch.randn(E, generator=g) * 0.5 - 0.6
    sc = M.SigmoidScores(c.to(device), 2.5)
    idx, w = M.route(z.to(device), top, groups=count, keep=keep, group_top=2, sigmoid=sc)
    plain = M.route(z.to(device), top, groups=count, keep=keep, group_top=2, sigmoid=M.SigmoidScores(None, 2.5))[0]
    single = M.route(z.to(device), top, groups=count, keep=keep, group_top=1, sigmoid=sc)[0]
    for t in range(40):
        want = O.route(z[t].double(), c.double(), {"top": top, "scale": 2.5, "groups": {"count": count, "keep": keep}})
        assert idx[t].tolist() == [e for e, _ in want]
        assert torch.allclose(w[t].double().cpu(), torch.stack([s for _, s in want]), rtol=1e-5)
    assert (torch.sigmoid(z) + c < 0).any()
    if top < E:
        assert (idx != plain).any()                          # the correction decides for some token
    if 1 < keep < count and count < E:
        assert (idx != single).any()                         # so does the second of a group's pair
    x, wr = torch.randn(9, 24, generator=g), torch.randn(E, 24, generator=g)
    i2, w2 = M.router(x.to(device), LinearWeight("dense", wr.to(device)), top, groups=count, keep=keep, group_top=2, sigmoid=sc)
    i1, w1 = M.route(x @ wr.T, top, groups=count, keep=keep, group_top=2, sigmoid=M.SigmoidScores(c, 2.5))
    assert torch.equal(i1, i2.cpu()) and torch.allclose(w1, w2.cpu(), rtol=1e-4)


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("d", [56, 61, 1024])
def test_what_joins_the_residual(device, dtype, d):
    dt = torch.float32 if dtype == "fp32" else torch.bfloat16
    g = torch.Generator().manual_seed(d)
    rnd = lambda *s: torch.randn(*s, generator=g).to(device)
    table, ids, step = rnd(30, d).to(dt), torch.tensor([3, 29, 0], dtype=torch.int32, device=device), rnd(d)
    w1, w2, wo = rnd(d), rnd(d), rnd(d)
    c = lambda t: t.double().cpu()
    close = lambda got, want, tol=3e-5: (c(got) - want).abs().max() < tol * want.abs().max()
    zt = 3e-5 if dtype == "fp32" else 5e-3
    x, z = ops.embed_group_norm(table, ids, wo, 1e-5, scale=2.5, step=step)
    want = 2.5 * c(table)[ids.long().cpu()] + c(step)
    assert close(x, want) and close(z, O.rms(want, 1e-5) * c(wo), zt)
    y, y2 = rnd(3, d).to(dt), rnd(3, d).to(dt)
    for post, post2, again in ((w1, w2, None), (None, None, ops.Again(table, ids, 2.5, step)), (w1, None, ops.Again(step=step))):
        z = ops.add_group_norm(x, y, post, wo, 1e-5, coef=0.7, second=(y2, post2, -0.3), again=again)
        n = lambda v, p: c(v) if p is None else O.rms(c(v), 1e-5) * c(p)
        want = want + 0.7 * n(y, post) - 0.3 * n(y2, post2)
        if again is not None:
            want = want + c(step) + (2.5 * c(table)[ids.long().cpu()] if again.table is not None else 0)
        assert close(x, want) and close(z, O.rms(want, 1e-5) * c(wo), zt)
    assert ops.add_group_norm(x, y, None, None, 1e-5) is None and close(x, want + c(y))


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("ff,ld", [(40, 80), (36, 72), (24, 56)])
def test_gated_gelu(device, dtype, ff, ld):
    x = torch.randn(5, ld, generator=torch.Generator().manual_seed(ff)).to(device, torch.float32 if dtype == "fp32" else torch.bfloat16)
    x = x[:, :2 * ff]
    want = O.gelu_tanh(x[:, :ff].double().cpu()) * x[:, ff:].double().cpu()
    got = ops.gated_act(x, "gelu_tanh").double().cpu()
    assert (got - want).abs().max() < (1e-5 if dtype == "fp32" else 2e-2) * want.abs().max()


@pytest.mark.gpu
@pytest.mark.parametrize("m,n,k,off,ld", [(1, 40, 24, 8, 80), (70, 136, 64, 64, 200), (300, 72, 8, 16, 32), (129, 1000, 72, 0, 80)])
def test_products_over_columns_of_a_wider_matrix(m, n, k, off, ld):
    x, w = torch.randn(m, ld, device="cuda").bfloat16(), torch.randn(n, k, device="cuda").bfloat16()
    want = x[:, off:off + k].double() @ w.double().T
    for kw in ({}, {"out_fp32": True}):
        y = ops.linear(x[:, off:off + k], LinearWeight("dense", w), **kw).double()
        assert (y - want).abs().max() < (1e-4 if kw else 1e-2) * want.abs().max()
    assert ops.device_status(torch.device("cuda")) == 0


# ------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("name", list(K.CASES))
def test_prompt_portions_and_decoding_agree_with_the_oracle(cases, name, device, dtype):
    c = cases(name)
    n = 150 if device == "cuda" else 45
    toks = c.prompt(n, 1)
    want = c.oracle(toks)
    eng = c.engine(device, dtype)
    whole = K.run_cut(eng, toks, [n])
    assert K.agrees(whole, want, dtype)
    for cuts in ([2], [1], [3, 5, 2], [16], [17, 1, 64, 2], [n - 9, 1]):
        assert K.agrees(K.run_cut(eng, toks, cuts), want, dtype), cuts
    assert eng.cache.pool.stats()["free"] == eng.cache.pool.stats()["pages"] and len(eng.cache._free) == 4
    if device == "cuda":
        assert ops.device_status(torch.device("cuda")) == 0


@pytest.mark.parametrize("device", DEVICES)
def test_routes_follow_the_residual(tmp_path, device):
    """Routers that read every channel of what the layers before them wrote (the other models' routes hang on the token)."""
    cfg = K.CASES["mixed"]
    c = K.Case(tmp_path, "free", cfg=cfg, weights=K.random_weights(cfg, 11, clear_routes=False))
    toks = c.prompt(50, 2)
    eng = c.engine(device, "fp32")
    for cuts in ([50], [7, 1]):
        assert K.agrees(K.run_cut(eng, toks, cuts), c.oracle(toks), "fp32")


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_batches_of_unequal_requests_equal_each_alone(cases, name, device, dtype):
    """Portions of some requests beside single tokens of others, requests that pause, and pages and slots that are taken
    again by later requests, in a pool that just fits the live ones."""
    c = cases(name, 3)
    lens = {"a": 45, "b": 3, "c": 61, "d": 30, "e": 52, "f": 17}
    if device == "cuda":
        lens.update(c=161)
    toks = {k: c.prompt(n, 7 + i) for i, (k, n) in enumerate(lens.items())}
    want = {k: c.oracle(t) for k, t in toks.items()}
    eng = c.engine(device, dtype, max_tokens=240 if device == "cpu" else 352)     # live: at most a, c, d, e
    c0 = 33 if device == "cpu" else 133
    schedule = [{"a": 20, "b": 2, "c": 2}, {"a": 1, "b": 1, "c": c0}, {"c": 5, "d": 16}, {"a": 1, "d": 1, "c": 1}, {"a": 7, "d": 2},
                {"a": 1, "c": 1, "d": 1, "e": 40}, {"a": 1, "c": 1, "d": 1, "e": 1}, {"e": 1, "c": 2}, {"a": 14, "c": 16, "d": 9},
                {"e": 10, "f": 2}, {"f": 15}]
    live, at = {}, {k: 0 for k in lens}
    for step in schedule:
        seqs, wanted = [], []
        for k, n in step.items():
            s = live.setdefault(k, None) or eng.new_sequence([])
            live[k] = s
            s.tokens.extend(toks[k][at[k]:at[k] + n])
            seqs.append(s)
            wanted.append(list(range(n)))
        out = eng.step(seqs, wanted)
        r = 0
        for k, n in step.items():
            assert K.agrees(out[r:r + n], want[k][at[k]:at[k] + n], dtype), (step, k)
            r, at[k] = r + n, at[k] + n
            if at[k] == lens[k]:
                eng.free_sequence(live.pop(k))
    assert eng.cache.pool.stats()["high_water"] <= (15 if device == "cpu" else 22)


def test_pool_and_slots_are_bounded(cases):
    eng = cases("mixed").engine("cpu", "fp32", max_tokens=64, max_seqs=2)
    a, b = eng.new_sequence([]), eng.new_sequence([])
    with pytest.raises(RuntimeError):
        eng.new_sequence([])
    a.tokens.extend([1] * 48)
    eng.step([a], [[]])
    b.tokens.extend([2] * 17)
    with pytest.raises(OutOfPages):
        eng.step([b], [[16]])


# (key, query) pairs just inside and just outside of every edge, small sizes and sizes that reach the tensor-core kernel
EDGES = {
    ("chunk", 24): [(0, 23), (0, 24), (23, 24), (24, 47), (24, 48), (16, 17), (15, 16), (30, 31)],
    ("window", 21, 5): [(30, 50), (29, 50), (4, 50), (5, 50), (0, 25), (0, 20), (4, 24), (5, 26), (5, 25), (15, 16), (31, 32)],
    ("chunk", 150): [(0, 149), (149, 150), (150, 299), (150, 300), (16, 140), (128, 149)],
    ("window", 140, 5): [(61, 200), (60, 200), (4, 200), (5, 200), (0, 300), (5, 144), (5, 145), (160, 299)],
    ("window", 70, 130): [(129, 290), (130, 290), (221, 290), (220, 290), (0, 290), (127, 290), (128, 290)],
}


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("dim", [16, 64])
@pytest.mark.parametrize("mask", list(EDGES), ids=str)
def test_one_far_key_decides(tmp_path, device, dtype, dim, mask):
    """A token that only one query looks for, at every edge: the logits show whether position i sees position j, in prompts,
    portions and decoding."""
    if device == "cpu" and (mask[1] > 30 or dim > 16):
        pytest.skip("long prompts run on the GPU")
    att, lin = (2, 1, dim, dim), (1, 8, 8)
    if mask[0] == "chunk":
        layer = K.parallel(None, att=att, chunk=mask[1], lin=lin, rot=4, base=1e6, scale=24.0 / dim)
    else:
        layer = K.parallel_2(None, att=att, window=mask[1], keep=mask[2], ret=lin, decay=[0.9], scale=40.0 / dim)
    cfg = K.config([layer], width=64, vocab=40)
    w = K.random_weights(cfg, 5)
    w["l0.mix.right.o"].zero_()                              # the state would carry the token past the edges
    w["embed"][:, :K.CODE] *= 0.2
    h = O.rms(w["embed"].double() * 3, 1e-5) * w["l0.norm1"].double()
    q, k = ((h @ w[f"l0.mix.left.{x}"].double().T).view(40, -1, dim)[:, -1] for x in ("q", "k"))     # the head of the smaller slope
    if mask[0] == "window":
        q, k = (O.rms(y + w[f"l0.mix.left.{x}.b"].double().view(-1, dim)[-1], 1e-5) * w[f"l0.mix.left.{x}.norm"].double()
                for x, y in (("q", q), ("k", k)))
    sc = q @ k.T
    qi, kj = divmod(int(sc.argmax()), 40)
    filler = int(sc[qi].argmin())
    c = K.Case(tmp_path, f"far{device}{dtype}{dim}", cfg=cfg, weights=w)
    eng = c.engine(device, dtype)
    rule = (lambda i, j: O.sees_chunk(i, j, mask[1])) if mask[0] == "chunk" else (lambda i, j: O.sees_window(i, j, *mask[1:]))
    shown = set()
    for j, i in EDGES[mask]:
        toks = [filler] * (i + 1)
        toks[j], toks[-1] = kj, qi
        base = list(toks)
        base[j] = filler
        with_key, without = c.oracle(toks)[-1], c.oracle(base)[-1]
        moved = float((with_key - without).pow(2).mean().sqrt() / without.pow(2).mean().sqrt())
        assert moved > 0.1 if rule(i, j) else moved < 1e-9, (j, i, moved)
        shown.add(rule(i, j))
        for cuts in ([i + 1], [i, 1], [i - 1, 2], [2] if i < 60 else [i - 70, 71]):
            got = K.run_cut(eng, toks, cuts)[-1:]
            assert K.error(got, with_key[None]) < (0.05 if dtype == "bf16" else 1e-3), (j, i, cuts)
    assert shown == {True, False}


@pytest.mark.parametrize("device,dtype", RUNS)
def test_planted_mistakes_show(tmp_path, monkeypatch, device, dtype):
    """With one thing wrong in the oracle, positions that hang on it come out different by far more than the tolerance."""
    cfg = K.config([K.parallel(None, att=(4, 2, 64, 64), chunk=30, lin=(2, 16, 16), rot=64, scale=0.3),
                    K.parallel_2(None, att=(4, 2, 64, 64), window=20, keep=4, ret=(2, 16, 16), decay=[0.9, 0.99], scale=0.3)],
                   width=64, vocab=50, loop=(0, 2, 2))
    c = K.Case(tmp_path, f"planted{device}{dtype}", 2, cfg=cfg)
    toks = c.prompt(70, 3)
    want = c.oracle(toks)
    plant = {"no sink": ("softmax_sink", lambda s, k: torch.softmax(s, -1), slice(0, 3)),
             "chunk cut": ("sees_chunk", lambda i, j, n: j <= i and (i + 1) // n == (j + 1) // n, slice(28, 34)),
             "window one off": ("sees_window", lambda i, j, n, f: j <= i and (i - j <= n or j < f), slice(24, 70)),
             "kept one off": ("sees_window", lambda i, j, n, f: j <= i and (i - j < n or j < f + 1), slice(26, 70)),
             "no slope": ("slope", lambda h, n: 0.0, slice(10, 70)),
             "state lost": ("linear_states", lambda q, k, v, d: (k * q).sum(-1, keepdim=True) * v, slice(2, 70))}
    tol = 2e-2 if dtype == "bf16" else 1e-4
    for name, (fn, wrong, rows) in plant.items():
        monkeypatch.setattr(O, fn, wrong)
        bad = O.forward(toks, cfg, c.w64)
        monkeypatch.undo()
        assert K.error(bad[rows], want[rows]) > (1.5 if dtype == "bf16" else 100) * tol, name
    for cuts in ([70], [1], [29, 2]):
        assert K.error(K.run_cut(c.engine(device, dtype), toks, cuts), want) < tol


@pytest.mark.parametrize("device,dtype", RUNS)
def test_long_decoding_keeps_the_state(cases, device, dtype):
    c = cases("odd" if dtype == "fp32" else "grouped", 2)
    n = 300 if device == "cuda" else 90
    toks = c.prompt(n, 4)
    assert K.agrees(K.run_cut(c.engine(device, dtype), toks, [5, 1]), c.oracle(toks), dtype)


# ------------------------------------------------------------------------------------------ serving
def _greedy(c, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(c.oracle(toks)[-1].argmax()))
    return toks[len(prompt):]


@pytest.mark.parametrize("device", DEVICES)
def test_greedy_generation_through_the_engine_and_the_scheduler(cases, device):
    from sllm_b200.engine.scheduler import EngineLoop, GenRequest
    import threading
    c = cases("mixed", 1)
    prompts = [c.prompt(n, 20 + n) for n in (1, 9, 34)]
    want = [_greedy(c, p, 5) for p in prompts]
    eng = c.engine(device, "fp32")
    assert eng.generate(prompts, 5) == want
    loop = EngineLoop(eng, max_batch=3, prefill_chunk_tokens=7)
    out, done = [[] for _ in prompts], [threading.Event() for _ in prompts]
    try:
        for i, p in enumerate(prompts):
            loop.submit(GenRequest(prompt=p, max_new_tokens=5, on_token=lambda t, s, i=i: out[i].append(t),
                                   on_done=lambda r, i=i: done[i].set()))
        assert all(d.wait(120) for d in done)
    finally:
        loop.shutdown(5)
    assert out == want


def test_fork_copies_pages_and_state(cases):
    c = cases("mixed")
    toks = c.prompt(40, 9)
    eng = c.engine("cpu", "fp32")
    a = eng.new_sequence([])
    a.tokens.extend(toks[:21])
    eng.step([a], [[]])
    b = eng.fork_sequence(a, toks)
    assert b.num_computed == 21
    assert K.agrees(eng.step([b], [[18]]), c.oracle(toks)[-1:], "fp32")
    a.tokens.append(toks[21])
    assert K.agrees(eng.step([a], [[0]]), c.oracle(toks[:22])[-1:], "fp32")


def test_every_pass_has_its_own_pages_and_states(cases):
    eng = cases("mixed").engine("cpu", "fp32")
    assert len(eng.model.runs) == 8 and len(eng.model.w.layers) == 4
    assert [next(i for i, l in enumerate(eng.model.w.layers) if l is r.layer) for r in eng.model.runs] == [0, 1, 2, 1, 2, 1, 2, 3]
    tokens = 4 * (2 * (24 + 24) + 3 * 2 * (24 + 16) + (16 + 16))          # fp32 rows, widths padded to 8
    assert eng.cache.bytes_per_token() == tokens
    ptrs = {eng.cache.state(j).data_ptr() for j in range(8)}
    assert len(ptrs) == 8 and len({eng.cache.layer(j).k.data_ptr() for j in (0, 1, 3, 5, 7)}) == 5 and eng.cache.layer(2) is None


@pytest.mark.parametrize("device", DEVICES)
def test_trace_session_writes_logits(cases, tmp_path, device):
    from sllm_b200.cli.trace import TraceSession
    import numpy as np
    c = cases("mixed")
    toks = c.prompt(12, 3)
    want = c.oracle(toks)
    t = TraceSession(c.engine(device, "fp32", max_tokens=64), str(tmp_path))
    t.run({"step": 0, "entries": [{"id": "x", "tokens": toks[:7], "want": [0, 6]}, {"id": "y", "tokens": toks[:2], "want": []}], "end": ["y"]})
    t.run({"step": 1, "entries": [{"id": "x", "tokens": toks[7:11], "want": []}], "end": []})
    t.run({"step": 2, "entries": [{"id": "x", "tokens": toks[11:], "want": [0]}], "end": ["x"]})
    got = [torch.from_numpy(np.fromfile(os.path.join(tmp_path, f"{i}.f32"), dtype="<f4").reshape(-1, c.cfg["vocab"])) for i in (0, 2)]
    assert not os.path.exists(os.path.join(tmp_path, "1.f32")) and got[0].shape[0] == 2
    assert K.agrees(got[0], want[[0, 6]], "fp32") and K.agrees(got[1], want[11:], "fp32")


# ------------------------------------------------------------------------------------------ files, registry, command line
def test_config_is_read_and_refused(cases, tmp_path):
    from sllm_b200.models import registry
    from sllm_b200.models.config import NAMED
    c = cases("mixed")
    cfg = registry.read_folder_config(c.path, "fp32")
    assert (cfg.family, cfg.n_layers, cfg.vocab, cfg.embedding_scale, cfg.layer_loop) == ("kegorax", 4, 211, 3.0, {"start": 1, "stop": 3, "times": 3})
    assert NAMED["kegorax"]().family == "kegorax"
    L = c.cfg["layers"]

    def bad(i, part=None, **mixer):
        m = dict(L[i]["mixer"])
        if part is None:
            m.update(mixer)
        else:
            m[part] = dict(m[part], **mixer)
        return {"layers": L[:i] + [dict(L[i], mixer=m)] + L[i + 1:]}

    for change in ({"architecture": "Other"}, {"layers": [{"type": "x", "mixer": {}, "mlp": None}]}, bad(0, "left", kv_heads=4),
                   bad(0, "left", mask={"size": 0, "keep_first": 1}), bad(0, "right", decay=[0.9]), bad(1, "left", rot={"base": 10.0, "dims": 26}),
                   bad(1, "right", tau=0), bad(2, kv_heads=3), bad(2, conv=0), {"loop": {"start": 1, "stop": 5, "times": 2}},
                   {"loop": {"start": 2, "stop": 2, "times": 2}}, {"loop": {"start": 1, "stop": 3, "times": 0}},
                   {"layers": [K.delta(K.moe(experts=6, top=3, ff=8, count=3, keep=1), heads=1, kv_heads=1, dim=4, vdim=4, conv=1)]},
                   {"layers": [K.delta({"kind": "other"}, heads=1, kv_heads=1, dim=4, vdim=4, conv=1)]}):
        p = K.write_folder(tmp_path / "bad", dict(c.cfg, **change), {})
        with pytest.raises(registry.ModelFolderError):
            registry.read_folder_config(p)
    w = dict(c.w)
    del w["l1.mix.left.sink"]
    with pytest.raises(registry.ModelFolderError):
        registry.load_folder_weights(K.write_folder(tmp_path / "short", c.cfg, w), cfg, "cpu")
    w = dict(c.w, **{"l0.mlp.down": c.w["l0.mlp.down"].T.contiguous()})
    with pytest.raises(registry.ModelFolderError):
        registry.load_folder_weights(K.write_folder(tmp_path / "turned", c.cfg, w), cfg, "cpu")


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_packed_weights_unpack_to_the_source(cases, name):
    from sllm_b200.models import kegorax, registry
    c = cases(name)
    cfg = registry.read_folder_config(c.path, "fp32")
    got = dict(kegorax.named_tensors(cfg, registry.load_folder_weights(c.path, cfg, "cpu")))
    assert set(got) == set(c.w) and all(got[n].shape == c.w[n].shape and torch.equal(got[n].float(), c.w[n]) for n in got)


def test_convert_and_generate_on_the_command_line(cases, tmp_path, capsys):
    from sllm_b200.cli import convert
    from sllm_b200.cli import main as cli
    from sllm_b200.formats import model_lock as ML
    c = cases("mixed")
    lock, gguf, dlock = tmp_path / "lock.json", str(tmp_path / "m.gguf"), str(tmp_path / "m.lock")
    lock.write_text(json.dumps(ML.make_model_lock(c.path, "local/kegorax", "0" * 40, ["kegorax"], {"family": "kegorax"}, {"kind": "none"})))
    args = ["--lock", str(lock), "--cache", c.path, "--output", gguf, "--derived-lock", dlock, "--weight-format", "fp32"]
    assert convert.main(["--kind", "sepedra", *args]) != 0      # another family's folder
    assert convert.main(["--kind", "kegorax", *args]) == 0
    capsys.readouterr()
    prompt = c.prompt(9, 5)
    assert cli.main(["decode", "--gguf", gguf, "--derived-lock", dlock, "--cpu", "--max-new-tokens", "4",
                     "--input-token-ids", ",".join(map(str, prompt))]) == 0
    rec = json.loads(capsys.readouterr().out.strip().splitlines()[-1])
    assert rec["output_tokens"] == _greedy(c, prompt, 4)


def test_random_shape_round_trips_through_gguf(tmp_path, capsys):
    from sllm_b200.cli import convert
    from sllm_b200.formats import gguf as G
    from sllm_b200.models import kegorax, loader, registry
    gguf, dlock = str(tmp_path / "t.gguf"), str(tmp_path / "t.lock")
    for extra, layers in (([], 3), (["--layers", "1"], 1)):
        assert convert.main(["--kind", "random-llama", "--artifact", "tiny-kegorax", "--output", gguf, "--derived-lock", dlock, *extra]) == 0
        cfg, w, family = loader.load_model_gguf(G.verify_gguf(gguf, G.read_derived_lock(dlock)), "cpu")
        assert family == "kegorax" and cfg.weight_format == "bf16" and len(w.layers) == layers
        if not torch.cuda.is_available():
            ref = dict(kegorax.named_tensors(cfg, registry.init_random_weights(cfg, "cpu", 0)))
            assert all(torch.equal(t, ref[n]) for n, t in kegorax.named_tensors(cfg, w))


def test_argument_blocks_match_the_library():
    import ctypes as C
    from sllm_b200.ops import _lib, core
    if not _lib.kernels_available():
        pytest.skip("kernel library not built")
    for fn, cls, last in ((S._k().sllm_linear_state_abi, S.LinearStateArgs, "eps"), (A._k().sllm_kv_abi, A.KvPrepareArgs, "eps"),
                          (M._k().sllm_moe_route_abi, M.RouteArgs, "scale"), (S._k().sllm_group_norm_abi, core.GroupNormArgs, "eps")):
        out = (C.c_int * 2)()
        assert fn(out, 2) == 2
        assert list(out) == [C.sizeof(cls), getattr(cls, last).offset]
