"""Fekolorn against its plain restatement (tests/fekolorn_oracle.py): every mechanism, whole prompts, portions, decoding, mixed
batches, pages and slots used again, the scheduler, files and the command line - on the CPU oracle path of the ops and, where a
GPU is present, on the CUDA kernels in fp32 and bf16."""
import json
import os

import pytest
import torch

import fekolorn_cases as K
import fekolorn_oracle as O
from sllm_b200 import ops
from sllm_b200.cache.paged import OutOfPages
from sllm_b200.engine.batch import ForwardBatch, make_prefill_batch
from sllm_b200.ops import kv_attention as A
from sllm_b200.ops import linear_state as S
from sllm_b200.ops import streams as R

RUNS = [("cpu", "fp32"), pytest.param("cuda", "fp32", marks=pytest.mark.gpu), pytest.param("cuda", "bf16", marks=pytest.mark.gpu)]
DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]


def _type(dtype):
    return torch.float32 if dtype == "fp32" else torch.bfloat16


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
            made[name, seed] = K.Case(tmp_path_factory.mktemp("fk"), name, seed)
        return made[name, seed]
    return get


def _steps(lens, steps, device):
    """Batches over three sequences: unequal portions, then ``steps`` single tokens of each; yields (batch, rows, starts)."""
    at = [0, 0, 0]
    for k in range(len(lens[0]) + steps):
        n = [x[k] for x in lens] if k < len(lens[0]) else [1] * 3
        if k < len(lens[0]):
            b = make_prefill_batch([[0] * m for m in n], None, device, at)
        else:
            pos = torch.tensor(at, dtype=torch.int32, device=device)
            ar = torch.arange(4, dtype=torch.int32, device=device)
            b = ForwardBatch(pos, pos, ar[:3], pos + 1, None, row_off=ar)
        yield b, n, list(at)
        at = [a + m for a, m in zip(at, n)]


# ------------------------------------------------------------------------------------------ mechanisms
@pytest.mark.parametrize("rows,far", [(32, 90), (6, 5), (16, 30), (10, 300), (2, 7), (1, 4), (12, 6), (12, 3), (7, 20), (64, 4000)])
def test_distance_buckets_as_stated(rows, far):
    got = A.distance_buckets(rows, far, 5000)
    near = rows // 2
    want = [O.bucket(n, rows, far) if near > 0 and far > near or n < near else rows - 1 for n in range(5000)]
    assert got == want[:len(got)] and got[-1] == rows - 1 and set(want[len(got) - 1:]) == {rows - 1}
    assert A.distance_buckets(rows, far, 3) == got[:3]
    rel = torch.randn(rows, 3)
    d = A.DistanceBias.make(rel, far, 5000)
    n = torch.arange(5000)
    assert torch.equal(d.at(n), rel[torch.tensor(want)].T)
    assert d.table.shape == (3, A.DIST_FRONT + len(got) + A.DIST_BACK)
    assert (d.table[:, A.DIST_FRONT + len(got) - 1:] == rel[-1][:, None]).all()


def _state_case(H, G, D, V, taps, seed=0):
    """(spec, weights in fp32, columns of a packed projection)."""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, generator=g)
    col, at = {}, 0
    for n, w in (("q", G * D), ("k", G * D), ("v", H * V), ("g", H * V), ("a", H), ("b", H)):
        col[n], at = at, at + w
        if n not in ("q", "k"):
            at = (at + 7) // 8 * 8
    w = S.StateWeights(bias=rnd(H) - 2, rate=torch.exp(0.7 * rnd(H)), conv_w=0.7 * rnd(taps, 2 * G * D + H * V), norm=1 + 0.3 * rnd(V))
    return S.StateSpec(S.HEAD_DELTA, H, G, D, V, col, q_scale=D ** -0.5, taps=taps), w, at


def _state_want(proj, spec, w, eps):
    """fp64 outputs of one sequence from its start."""
    p, t, H, G, D, V = proj.double(), proj.shape[0], spec.heads, spec.kv_heads, spec.dim, spec.vdim
    f = lambda n, m: p[:, spec.columns[n]:spec.columns[n] + m]
    c = w.conv_w.double().T.split([G * D, G * D, H * V])
    q, k, v = (O.silu(O.causal_conv(f(n, x.shape[0]), x)) for n, x in zip(("q", "k", "v"), c))
    q, k = ((O.unit(x.view(t, G, D))).repeat_interleave(H // G, 1) for x in (q, k))
    decay = torch.exp(-w.rate.double() * O.softplus(f("a", H) + w.bias.double()))
    o = O.delta_states(q * spec.q_scale, k, v.view(t, H, V), decay, torch.sigmoid(f("b", H)))
    return (O.rms(o, eps) * w.norm.double()).reshape(t, -1) * O.silu(f("g", H * V))


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("H,G,D,V,taps", [(2, 2, 12, 20, 3), (3, 1, 16, 16, 1), (4, 2, 64, 128, 4), (6, 3, 10, 7, 5), (2, 1, 200, 33, 2),
                                          (1, 1, 128, 264, 4), (2, 2, 300, 24, 4), (8, 8, 32, 64, 2)])
def test_recurrence_over_portions_and_steps(device, dtype, H, G, D, V, taps):
    """Unequal portions of several sequences in slots out of order, then single tokens, each going on where it was."""
    spec, w32, width = _state_case(H, G, D, V, taps)
    w = S.StateWeights(**{n: x if x is None else x.to(device) for n, x in vars(w32).items()})
    lens, steps, slots = [[1, 17, 2], [9, 2, 1], [20, 1, 3]], 4, [4, 0, 2]
    g = torch.Generator().manual_seed(5)
    proj = [torch.randn(sum(x) + steps, width, generator=g).to(_type(dtype)) for x in lens]
    state = torch.full((5, H, D, V), 7.0, device=device)
    ring = torch.full((5, taps, spec.channels), 99.0, device=device)
    state[slots] = 0
    out = [[], [], []]
    for b, n, at in _steps(lens, steps, device):
        b.slots = torch.tensor(slots, dtype=torch.int32, device=device)
        y = S.linear_state(torch.cat([proj[i][at[i]:at[i] + n[i]] for i in range(3)]).to(device), spec, w, 1e-5, state, ring, b)
        for i, part in enumerate(y.float().cpu().split(n)):
            out[i].append(part)
    for i in range(3):
        want, got = _state_want(proj[i], spec, w32, 1e-5), torch.cat(out[i]).double()
        tol = 3e-5 if dtype == "fp32" else 2e-2
        assert (got - want).pow(2).mean().sqrt() < tol * want.pow(2).mean().sqrt(), i
        assert (got - want).abs().max() < 6 * tol * want.abs().max(), i
    assert (state[[1, 3]] == 7).all() and (ring[[1, 3]] == 99).all()


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,rot,window,rows,far", [
    (4, 2, 64, 64, 32, 0, 0, 0), (6, 3, 20, 24, 20, 0, 0, 0), (3, 1, 72, 40, 8, 0, 0, 0), (5, 5, 7, 9, 2, 0, 0, 0), (2, 1, 256, 256, 0, 0, 0, 0),
    (12, 2, 96, 64, 48, 0, 0, 0),
    (4, 2, 64, 64, 0, 24, 16, 20), (8, 1, 128, 128, 0, 70, 32, 60), (6, 2, 20, 24, 0, 33, 8, 100), (3, 1, 72, 40, 0, 140, 10, 130),
    (2, 2, 10, 14, 0, 1, 6, 8), (5, 1, 64, 64, 0, 64, 12, 3), (6, 6, 192, 128, 0, 0, 64, 5000), (3, 3, 40, 16, 0, 129, 2, 9)])
def test_attention_over_portions_and_steps(device, dtype, heads, kv_heads, dim, vdim, rot, window, rows, far):
    """From projections to outputs: rotation and normed values (no bias rows), or norms over all heads, distance biases and values
    mixed with others."""
    dt, rich = _type(dtype), rows > 0
    spec = A.KVSpec(heads, kv_heads, dim, vdim, 1.5 * dim ** -0.5, 3e3, rot, qk_norm=rich, norm_all=rich, v_norm=not rich, window=window,
                    interleaved=False)
    lens = [[90, 2, 130], [1, 3, 40], [65, 64, 1]] if device == "cuda" else [[30, 2, 20], [1, 3, 20], [17, 16, 1]]
    ends = [sum(x) + 3 for x in lens]
    up = lambda n: (n + 7) // 8 * 8
    g = torch.Generator().manual_seed(dim)
    nb = (max(ends) + 15) // 16
    table = torch.randperm(3 * nb + 2, generator=g)[:3 * nb].view(3, nb).int().to(device)
    kv = A.KVPages(*(torch.zeros(3 * nb + 2, kv_heads, 16, up(x)).to(device, dt) for x in (dim, vdim)), 16)
    for t, x in ((kv.k, dim), (kv.v, vdim)):
        t[..., :x] = 50.0                                    # what a page held before; the padding behind a row is zero
    nv = kv_heads * vdim
    proj = [torch.randn(e, up(spec.channels) + up(nv), generator=g).to(dt) for e in ends]
    rnd = lambda *s, m=0.0: (m + 0.4 * torch.randn(*s, generator=g)).to(device)
    qn, kn = (rnd(heads * dim, m=1.0), rnd(kv_heads * dim, m=1.0)) if rich else (None, None)
    sinks, rel = 3 * rnd(heads), 3 * rnd(max(rows, 1), heads)
    dist = A.DistanceBias.make(rel, far, window or far + 9) if rich else None
    f, c0, lam = spec.inv_freq(device), up(spec.channels), 0.3
    out = [[], [], []]
    for b, n, at in _steps(lens, 3, device):
        b.block_table, b.slots = table, torch.arange(3, dtype=torch.int32, device=device)
        x = torch.cat([proj[i][at[i]:at[i] + n[i]] for i in range(3)]).to(device)
        q = A.prepare(x, spec, None, f, 1e-5, kv, None, b, q_norm=qn, k_norm=kn, mix=(x[:, c0:c0 + nv], lam) if rich else None)
        y = A.attention(q, None, spec, kv, sinks, b, dist=dist)
        if device == "cuda":                                 # the page-walking kernels over the same pages
            z = A.paged_rows(q, None, spec, kv, sinks, table, b.seq_index, b.kv_lens, b.max_kv, impl="cuda_core_any", dist=dist)
            z2 = A.paged_rows(q, None, spec, kv, sinks, table, b.seq_index, b.kv_lens, b.max_kv, dist=dist)
            for got in (y, z2):
                assert (got.float() - z.float()).abs().max() < (2e-5 if dtype == "fp32" else 4e-2) * z.float().abs().max()
        for i, part in enumerate(y.float().cpu().split(n)):
            out[i].append(part)
    c64 = lambda v: v.double().cpu()
    for i, e in enumerate(ends):
        p = proj[i].double()
        q, k, v = p[:, :spec.channels].split([heads * dim, kv_heads * dim, nv], 1)
        if rich:
            q, k = O.rms(q, 1e-5) * c64(qn), O.rms(k, 1e-5) * c64(kn)
            v = O.mixed_values(v, p[:, c0:c0 + nv], lam)
        q, k, v = (y.reshape(e, -1, m) for y, m in zip((q, k, v), (dim, dim, vdim)))
        if not rich:
            q, k, v = O.rotate(q, {"base": 3e3, "dims": rot}), O.rotate(k, {"base": 3e3, "dims": rot}), O.rms(v, 1e-5)
        seen = O.visible(e, lambda a, b: j_ok(a, b, window))
        bias = None
        if rich:
            full = torch.tensor([x for x in A.distance_buckets(rows, far, 6000)])
            gap = (torch.arange(e)[:, None] - torch.arange(e)[None, :]).clamp(min=0, max=len(full) - 1)
            bias = c64(rel)[full[gap]].permute(2, 0, 1)
        d = torch.cat(out[i]).double()
        want = O.attend(q, k, v, spec.scale, seen, c64(sinks), bias).reshape(e, -1)
        assert (d - want).abs().max() < (3e-5 if dtype == "fp32" else 5e-2) * want.abs().max(), i
        assert (d - want).pow(2).mean().sqrt() < (1e-5 if dtype == "fp32" else 1e-2) * want.pow(2).mean().sqrt(), i
    if device == "cuda":
        assert ops.device_status(torch.device("cuda")) == 0


def j_ok(i, j, window):
    return O.sees_window(i, j, window) if window else j <= i


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("n,ld", [(1, 1), (24, 56), (37, 37), (1000, 1000), (2056, 2064), (8192, 8192), (12296, 12296), (20000, 20000)])
def test_normed_polynomial(device, dtype, n, ld):
    g = torch.Generator().manual_seed(n)
    x = (torch.randn(4, ld, generator=g) * torch.tensor([1.0, 30.0, 0.02, 0.0])[:, None]).to(_type(dtype))[:, :n]
    coef = torch.tensor([0.7, -0.4, 0.3, 0.1])
    want = O.poly_norm(x.double(), coef.double(), 1e-5)
    got = ops.poly_norm(x.to(device), coef.to(device), 1e-5).double().cpu()
    assert ((got - want).abs() < (2e-5 if dtype == "fp32" else 8e-3) * want.abs().amax(1, keepdim=True)).all()


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("n,d", [(1, 56), (2, 61), (3, 1024), (4, 40), (5, 72), (9, 1031), (16, 64)])
def test_streams_are_read_and_written(device, dtype, n, d):
    dt, t = _type(dtype), 5
    g = torch.Generator().manual_seed(d)
    rnd = lambda *s: torch.randn(*s, generator=g).to(device)
    close = lambda got, want, tol=3e-5: (got.double().cpu() - want).abs().max() < tol * want.abs().max()
    zt, c = 3e-5 if dtype == "fp32" else 5e-3, lambda v: v.double().cpu()
    x, y, y2 = rnd(t, n, d), rnd(t, d).to(dt), rnd(t, d + 8).to(dt)[:, :d]
    conn, read, one, wide = R.Connection(rnd(n), rnd(n, n), rnd(n)), rnd(n), rnd(1), rnd(d)
    for w, second in ((one, None), (wide, (y2, -0.3)), (None, (y2, 0.5))):
        old = [c(x)[:, s] for s in range(n)]
        out = 0.7 * c(y) + (0 if second is None else second[1] * c(y2))
        want = O.write(old, out, c(conn.mix), c(conn.out))
        z = R.join_streams(x, y, conn, read, w, 1e-5, 0.7, second)
        assert close(x, torch.stack(want, 1))
        if w is None:
            assert z is None
        else:
            assert close(z, O.rms(O.read(want, c(read)), 1e-5) * c(w), zt)
    rows = torch.tensor([4, 0, 0], device=device)
    got = R.read_streams(x, one, 1e-5, dt, rows)
    assert close(got, (O.rms(c(x).sum(1), 1e-5) * c(one))[rows.cpu()], zt) and R.read_streams(x, one, 1e-5, dt, rows[:0]).shape == (0, d)
    assert close(R.read_streams(x, wide, 1e-5, dt, read=read), O.rms(O.read([c(x)[:, s] for s in range(n)], c(read)), 1e-5) * c(wide), zt)


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("n,d,buckets", [(2, 56, 101), (1, 61, 7), (3, 24, 1)])
def test_pairs_of_tokens_across_portions(device, dtype, n, d, buckets):
    """The token before a portion comes from the sequence's slot; a sequence's first token has a row of its own, also in a slot
    that another sequence has left."""
    dt, vocab, slots = _type(dtype), 5000, [4, 0, 2]
    g = torch.Generator().manual_seed(d)
    rnd = lambda *s: torch.randn(*s, generator=g).to(device)
    table, pair = rnd(vocab, d).to(dt), R.PairEmbedding(rnd(buckets + 1, d).to(dt), 2 ** 40 + 7, 1009)
    spec = {"buckets": buckets, "mul_prev": 2 ** 40 + 7, "mul_cur": 1009}
    cfg, w = {"embedding": {"scale": 2.5, "bigram": spec}}, {"embed": table.double().cpu(), "bigram": pair.table.double().cpu()}
    lens = [[1, 7, 2], [4, 2, 1], [3, 1, 30]]
    toks = [torch.randint(0, vocab, (sum(x) + 3,), generator=g).tolist() for x in lens]
    last, read, one = torch.full((5, 1), 17.0, device=device), rnd(n), rnd(1)
    for b, m, at in _steps(lens, 3, device):
        b.slots = torch.tensor(slots, dtype=torch.int32, device=device)
        b.tokens = torch.tensor([t for i in range(3) for t in toks[i][at[i]:at[i] + m[i]]], dtype=torch.int32, device=device)
        x, z = R.start_streams(table, b, 2.5, pair, last, n, read, one, 1e-5)
        want = torch.cat([O.embedding(toks[i][:at[i] + m[i]], cfg, w)[at[i]:] for i in range(3)])
        assert all((x[:, s].double().cpu() - want).abs().max() < 1e-5 * want.abs().max() for s in range(n))
        wz = O.rms(want * read.double().cpu().sum(), 1e-5) * one.double().cpu()
        assert (z.double().cpu() - wz).abs().max() < (3e-5 if dtype == "fp32" else 5e-3) * wz.abs().max()
    assert last[[4, 0, 2], 0].tolist() == [t[-1] for t in toks] and (last[[1, 3]] == 17).all()
    x, _ = R.start_streams(table, b, 1.0, None, None, n, None, one, 1e-5)
    assert torch.equal(x[:, 0], table[b.tokens.long()].float())


# ------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("name", list(K.CASES))
def test_prompt_portions_and_decoding_agree_with_the_oracle(cases, name, device, dtype):
    c = cases(name)
    n = 150 if device == "cuda" else 45
    toks = c.prompt(n, 1)
    want = c.oracle(toks)
    eng = c.engine(device, dtype)
    for cuts in ([n], [2], [1], [3, 5, 2], [16], [17, 1, 64, 2], [n - 9, 1]):
        assert K.agrees(K.run_cut(eng, toks, cuts), want, dtype), cuts
    assert eng.cache.pool.stats()["free"] == eng.cache.pool.stats()["pages"] and len(eng.cache._free) == 4
    if device == "cuda":
        assert ops.device_status(torch.device("cuda")) == 0


def test_residual_after_every_layer(cases, monkeypatch):
    """The sum of the streams behind each layer."""
    from sllm_b200.models import fekolorn as F
    c = cases("mixed")
    toks = c.prompt(20, 6)
    eng = c.engine("cpu", "fp32")
    seen, join = [], R.join_streams

    def spy(x, *a, **k):
        z = join(x, *a, **k)
        seen.append(x.sum(1).double())
        return z
    monkeypatch.setattr(F.R, "join_streams", spy)
    K.run_cut(eng, toks, [20])
    want = []
    O.forward(toks, c.cfg, c.w64, want)
    ends, k = [], -1
    for e in c.cfg["layers"]:
        k += 1 if e["mlp"] is None else 2
        ends.append(k)
    assert len(seen) == k + 1
    for i, j in enumerate(ends):
        assert (seen[j] - want[i]).abs().max() < 1e-5 * want[i].abs().max(), i


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


# window (0: every earlier position) -> (key, query) pairs at page borders, and just inside and outside of every edge
EDGES = {
    21: [(30, 50), (29, 50), (0, 20), (0, 21), (15, 16), (16, 17), (31, 32), (16, 36), (16, 37)],
    1: [(5, 5), (4, 5), (15, 16), (16, 16)],
    0: [(0, 50), (15, 16), (16, 31), (47, 50), (0, 1)],
    140: [(61, 200), (60, 200), (0, 139), (0, 140), (160, 299), (159, 299), (128, 129)],
    -1: [(0, 400), (127, 128), (128, 383), (16, 399), (255, 256)],
}


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("dims", [(16, 16), (64, 64), (48, 24)], ids=str)
@pytest.mark.parametrize("window", list(EDGES))
def test_one_far_key_decides(tmp_path, device, dtype, dims, window):
    """A token that only one query looks for, at every edge: the logits show whether position i sees position j, in prompts,
    portions and decoding."""
    if device == "cpu" and (window not in (21, 1, 0) or dims != (16, 16)):
        pytest.skip("long prompts run on the GPU")
    att = (2, 1, *dims)
    if window > 0:
        layer = K.attention(None, att=att, window=window, far=40, scale=60.0 / dims[0])
    else:
        layer = K.parallel(None, att=att, delta=(1, 1, 8, 8), conv=2, rot=4, base=1e6, scale=24.0 / dims[0], scales=(1.0, 0.5))
    cfg = K.config([layer], width=64, vocab=40, streams=2)
    w = K.random_weights(cfg, 5)
    w["bigram"].zero_()                                      # a pair would show the neighbour
    p = "l0.mix." if window > 0 else "l0.mix.left."
    if window > 0:
        w[p + "rel"] *= 0.3
    else:
        w["l0.mix.right.o"].zero_()                          # so would the state
    h = O.rms(w["embed"].double() * 3 * w["l0.hc1.in"].double().sum(), 1e-5) * w["l0.norm1"].double()
    q, k = (h @ w[p + x].double().T for x in ("q", "k"))
    if window > 0:
        q, k = (O.rms(y, 1e-5) * w[f"{p}{x}.norm"].double() for x, y in (("q", q), ("k", k)))
    sc = q[:, :dims[0]] @ k.T
    qi, kj = divmod(int(sc.argmax()), 40)
    filler = int(sc[qi].argmin())
    c = K.Case(tmp_path, f"far{window}{device}{dtype}{dims[0]}", cfg=cfg, weights=w)
    eng = c.engine(device, dtype)
    rule = lambda i, j: j_ok(i, j, max(window, 0))
    shown = set()
    for j, i in EDGES[window]:
        toks = [filler] * (i + 1)
        toks[j] = kj
        base = list(toks)
        base[j] = filler
        if j != i:
            toks[-1] = base[-1] = qi
        with_key, without = c.oracle(toks)[-1], c.oracle(base)[-1]
        moved = float((with_key - without).pow(2).mean().sqrt() / without.pow(2).mean().sqrt())
        assert moved > 0.1 if rule(i, j) else moved < 1e-9, (j, i, moved)
        shown.add(rule(i, j))
        for cuts in ([i + 1], [i, 1], [i - 1, 2], [2] if i < 60 else [i - 70, 71]):
            if min(cuts) < 1:
                continue
            got = K.run_cut(eng, toks, cuts)[-1:]
            assert K.error(got, with_key[None]) < (0.05 if dtype == "bf16" else 1e-3), (j, i, cuts)
    assert shown == ({True, False} if window > 0 else {True})


@pytest.mark.parametrize("device,dtype", RUNS)
def test_planted_mistakes_show(tmp_path, monkeypatch, device, dtype):
    """With one thing wrong in the oracle, positions that hang on it come out different by far more than the tolerance."""
    cfg = K.config([K.attention(None, att=(4, 2, 64, 32), window=20, far=14, scale=0.3),
                    K.parallel(K.dense(48), att=(4, 2, 64, 64), delta=(4, 2, 16, 16), conv=3, rot=64, scale=0.3),
                    K.attention(K.dense(48), att=(4, 2, 64, 32), window=31, far=50, scale=0.3)], width=64, vocab=50, streams=3)
    c = K.Case(tmp_path, f"planted{device}{dtype}", 2, cfg=cfg)
    toks = c.prompt(70, 3)
    want = c.oracle(toks)
    right = {n: getattr(O, n) for n in ("bucket", "write", "delta_states", "causal_conv")}
    plant = {"no sink": ("softmax_sink", lambda s, k: torch.softmax(s, -1), slice(0, 3)),
             "window one off": ("sees_window", lambda i, j, n: 0 <= i - j <= n, slice(24, 70)),
             "bias one off": ("bucket", lambda n, r, far: right["bucket"](n + 1, r, far), slice(0, 70)),
             "bias never far": ("bucket", lambda n, r, far: min(n, r // 2 - 1), slice(24, 70)),
             "own values": ("mixed_values", lambda v, first, lam: v, slice(0, 70)),
             "first token": ("bigram_row", lambda p, t, s: ((p or 0) * s["mul_prev"] + t * s["mul_cur"]) % s["buckets"], slice(0, 1)),
             "previous token": ("bigram_row", lambda p, t, s: s["buckets"] if p is None else (p * s["mul_cur"] + t * s["mul_prev"]) % s["buckets"],
                                slice(1, 70)),
             "mix turned": ("write", lambda x, y, m, o: right["write"](x, y, m.T, o), slice(0, 70)),
             "state lost": ("delta_states", lambda q, k, v, d, b: right["delta_states"](q, k, v, 0 * d, b), slice(2, 70)),
             "no decay": ("head_decay", lambda h, w, p: torch.ones_like(h @ w[p + "a"].T), slice(3, 70)),
             "conv lost": ("causal_conv", lambda u, w: u * w[:, -1], slice(1, 70))}
    tol = 3e-2 if dtype == "bf16" else 1e-4
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


def test_cache_holds_what_each_layer_needs(cases):
    eng = cases("mixed").engine("cpu", "fp32")
    assert eng.cache.bytes_per_token() == 4 * (2 * (24 + 16) + 2 * (24 + 24) + 2 * (16 + 24) + (16 + 16) + (16 + 8))   # widths padded to 8
    assert eng.cache.state(0).shape == (4, 4, 12, 20) and eng.cache.state(0, 1).shape == (4, 3, 2 * 24 + 80)
    assert eng.cache.state("last_token").shape == (4, 1)
    with pytest.raises(KeyError):
        eng.cache.state(1)


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
    assert (cfg.family, cfg.n_layers, cfg.vocab, cfg.embedding_scale, cfg.streams) == ("fekolorn", 5, 211, 3.0, 3)
    assert cfg.bigram == {"buckets": 53, "mul_prev": 31, "mul_cur": 7}
    assert NAMED["fekolorn"]().family == "fekolorn"
    L = c.cfg["layers"]

    def bad(i, part=None, **mixer):
        m = dict(L[i]["mixer"])
        if part is None:
            m.update(mixer)
        else:
            m[part] = dict(m[part], **mixer)
        return {"layers": L[:i] + [dict(L[i], mixer=m)] + L[i + 1:]}

    for change in ({"architecture": "Other"}, {"layers": [{"type": "x", "mixer": {}, "mlp": None}]}, {"layers": []}, {"streams": 0}, {"streams": 17},
                   bad(0, "left", kv_heads=3), bad(0, "left", rot={"base": 10.0, "dims": 26}), bad(0, "right", kv_heads=3), bad(0, "right", conv=0),
                   bad(1, mask={"size": 0}), bad(1, bias_max=0), bad(1, vdim=25), {"vocab": 2 ** 24 + 1},
                   {"embedding": {"scale": 1.0, "bigram": {"buckets": 0, "mul_prev": 1, "mul_cur": 1}}},
                   {"layers": [dict(L[0], mlp={"kind": "other"})]}):
        p = K.write_folder(tmp_path / "bad", dict(c.cfg, **change), {})
        with pytest.raises(registry.ModelFolderError):
            registry.read_folder_config(p)
    w = dict(c.w)
    del w["l1.mix.sink"]
    with pytest.raises(registry.ModelFolderError):
        registry.load_folder_weights(K.write_folder(tmp_path / "short", c.cfg, w), cfg, "cpu")
    for name, t in (("l0.mlp.down", c.w["l0.mlp.down"].T.contiguous()), ("l1.norm1", torch.ones(56)), ("l1.mix.rel", torch.ones(16, 5))):
        with pytest.raises(registry.ModelFolderError):
            registry.load_folder_weights(K.write_folder(tmp_path / "turned", c.cfg, dict(c.w, **{name: t})), cfg, "cpu")


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_packed_weights_unpack_to_the_source(cases, name):
    from sllm_b200.models import fekolorn, registry
    c = cases(name)
    cfg = registry.read_folder_config(c.path, "fp32")
    got = dict(fekolorn.named_tensors(cfg, registry.load_folder_weights(c.path, cfg, "cpu")))
    assert set(got) == set(c.w) and all(torch.equal(got[n].float().view(c.w[n].shape), c.w[n]) for n in got)


def test_convert_and_generate_on_the_command_line(cases, tmp_path, capsys):
    from sllm_b200.cli import convert
    from sllm_b200.cli import main as cli
    from sllm_b200.formats import model_lock as ML
    c = cases("mixed")
    lock, gguf, dlock = tmp_path / "lock.json", str(tmp_path / "m.gguf"), str(tmp_path / "m.lock")
    lock.write_text(json.dumps(ML.make_model_lock(c.path, "local/fekolorn", "0" * 40, ["fekolorn"], {"family": "fekolorn"}, {"kind": "none"})))
    args = ["--lock", str(lock), "--cache", c.path, "--output", gguf, "--derived-lock", dlock, "--weight-format", "fp32"]
    assert convert.main(["--kind", "kegorax", *args]) != 0      # another family's folder
    assert convert.main(["--kind", "fekolorn", *args]) == 0
    capsys.readouterr()
    prompt = c.prompt(9, 5)
    assert cli.main(["decode", "--gguf", gguf, "--derived-lock", dlock, "--cpu", "--max-new-tokens", "4",
                     "--input-token-ids", ",".join(map(str, prompt))]) == 0
    rec = json.loads(capsys.readouterr().out.strip().splitlines()[-1])
    assert rec["output_tokens"] == _greedy(c, prompt, 4)


def test_random_shape_round_trips_through_gguf(tmp_path, capsys):
    from sllm_b200.cli import convert
    from sllm_b200.formats import gguf as G
    from sllm_b200.models import fekolorn, loader, registry
    gguf, dlock = str(tmp_path / "t.gguf"), str(tmp_path / "t.lock")
    for extra, layers in (([], 3), (["--layers", "2"], 2)):
        assert convert.main(["--kind", "random-llama", "--artifact", "tiny-fekolorn", "--output", gguf, "--derived-lock", dlock, *extra]) == 0
        cfg, w, family = loader.load_model_gguf(G.verify_gguf(gguf, G.read_derived_lock(dlock)), "cpu")
        assert family == "fekolorn" and cfg.weight_format == "bf16" and len(w.layers) == layers
        if not torch.cuda.is_available():
            ref = dict(fekolorn.named_tensors(cfg, registry.init_random_weights(cfg, "cpu", 0)))
            assert all(torch.equal(t, ref[n]) for n, t in fekolorn.named_tensors(cfg, w))


def test_argument_blocks_match_the_library():
    import ctypes as C
    from sllm_b200.ops import _lib
    if not _lib.kernels_available():
        pytest.skip("kernel library not built")
    for fn, cls in ((S._k().sllm_linear_state_abi, S.LinearStateArgs), (A._k().sllm_kv_abi, A.KvPrepareArgs),
                    (R._k().sllm_streams_abi, R.StreamArgs)):
        out = (C.c_int * 2)()
        assert fn(out, 2) == 2
        assert list(out) == [C.sizeof(cls), cls.eps.offset]
