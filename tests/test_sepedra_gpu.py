"""CUDA kernels of the gated recurrence, of attention over keys and values of different widths and of the dense-weight experts
against fp32 / fp64 PyTorch statements of the same op."""
import dataclasses

import pytest
import torch

import sepedra_oracle as O
from sllm_b200 import ops
from sllm_b200.engine.batch import ForwardBatch, make_prefill_batch
from sllm_b200.ops import kv_attention as A
from sllm_b200.ops import moe as M
from sllm_b200.ops import rglru as R
from sllm_b200.ops.core import LinearWeight

pytestmark = pytest.mark.gpu
DEV = "cuda"


def _bf(*shape, std=1.0):
    return (torch.randn(*shape, device=DEV) * std).to(torch.bfloat16)


def _ok():
    assert ops.device_status(torch.device(DEV)) == 0


def _close(got, want, rms=1e-2, peak=0.1):
    d = got.double().cpu() - want
    assert d.pow(2).mean().sqrt() < rms * want.pow(2).mean().sqrt() and d.abs().max() < peak * want.abs().max()


# ------------------------------------------------------------------------------------------ products, norms, routing
@pytest.mark.parametrize("m,n,k", [(1, 5, 64), (3, 130, 200), (70, 64, 2560), (300, 72, 128), (129, 1000, 72), (9, 12, 33)])
def test_unrounded_and_capped_products(m, n, k):
    torch.manual_seed(m)
    x, w = _bf(m, k), _bf(n, k)
    want = x.double() @ w.double().T
    y = ops.linear(x, LinearWeight("dense", w), out_fp32=True)
    assert y.dtype == torch.float32 and (y.double() - want).abs().max() < 1e-4 * want.abs().max()
    y = ops.linear(x, LinearWeight("dense", w), act="softcap", act_arg=7.0).double()
    assert (y - 7 * torch.tanh(want / 7)).abs().max() < 0.03
    y = ops.linear(x.float(), LinearWeight("dense", w.float()), act="softcap", act_arg=7.0).double()
    assert (y - 7 * torch.tanh(want / 7)).abs().max() < 1e-4
    _ok()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("d", [56, 61, 2048])
def test_residual_rows_without_an_input_norm(dtype, d):
    torch.manual_seed(d)
    table, ids = torch.randn(30, d, device=DEV).to(dtype), torch.tensor([3, 29, 0], dtype=torch.int32, device=DEV)
    x, z = ops.embed_group_norm(table, ids, None, 1e-5)
    assert torch.equal(z, table[ids.long()]) and torch.equal(x, z.float())
    y, w = torch.randn(7, d, device=DEV).to(dtype), torch.randn(d, device=DEV)
    terms = torch.tensor([[6, 0, 2], [1, -1, 1], [5, 4, 3]], dtype=torch.int32, device=DEV)
    yd = torch.cat([y.double(), torch.zeros(1, d, device=DEV).double()])
    want = x.double() + O.rms(yd[terms.long()].sum(1), 1e-5) * w.double()
    z = ops.add_group_norm(x, y, w, None, 1e-5, terms=terms, raw=True)
    assert (x.double() - want).abs().max() < 3e-5 and torch.equal(z, x.to(dtype))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("t", [1, 33, 200])
@pytest.mark.parametrize("d,E,top,count,keep", [(176, 10, 4, 5, 3), (61, 5, 2, 1, 1), (1024, 256, 32, 8, 4), (72, 1, 1, 1, 1)])
def test_router_from_unrounded_logits(dtype, t, d, E, top, count, keep):
    torch.manual_seed(d + t)
    x, w = torch.randn(t, d, device=DEV).to(dtype), torch.randn(E, d, device=DEV).to(dtype)
    idx, wt = M.router(x, LinearWeight("dense", w), top, True, count, keep)
    z = x.double() @ w.double().T
    p = torch.softmax(z, -1)
    assert torch.allclose(p.gather(1, idx.long()), wt.double(), rtol=2e-3, atol=1e-7)
    ref = M.route(z.float().cpu(), top, True, count, keep)[0]
    assert (idx.cpu() != ref).any(1).float().mean() < 0.03       # sums in another order: a close call may differ
    _ok()


# ------------------------------------------------------------------------------------------ experts
@pytest.mark.parametrize("T,d,ff,E,top", [(3, 184, 80, 11, 3), (40, 128, 136, 5, 2), (300, 256, 64, 3, 2), (700, 200, 200, 4, 3), (64, 64, 24, 40, 8),
                                           (9, 61, 30, 4, 2), (1, 512, 512, 1, 1)])
def test_grouped_experts(T, d, ff, E, top):
    torch.manual_seed(T)
    act = M.GatedAct(0.9, 1.702, 1.0)
    gates, ups, downs = ([_bf(*s, std=s[1] ** -0.5) for _ in range(E)] for s in ((ff, d), (ff, d), (d, ff)))
    x = _bf(T, d)
    # uneven loads: expert 0 takes most, some take nothing
    score = torch.rand(T, E, device=DEV) + torch.linspace(1.5, 0, E, device=DEV)
    idx = score.topk(top, -1).indices.int()
    w = torch.rand(T, top, device=DEV)
    want = torch.zeros(T, d, dtype=torch.float64)
    for e in range(E):
        p = {n: m[e].double().cpu() for n, m in (("gate", gates), ("up", ups), ("down", downs))}
        y = O.expert(x.double().cpu(), p, "", 0.9)
        for j in range(top):
            hit = (idx[:, j] == e).cpu()
            want[hit] += w[:, j].double().cpu()[hit, None] * y[hit]
    bank = M.ExpertBank.pack(gates, ups, downs, act)
    y, dst = M.bank_forward(x, idx, w, bank)
    got = sum(y.double()[dst[:, j].long()] for j in range(top))
    _close(got, want, 8e-3, 3e-2)
    if d % 8 == 0:                                       # both tile heights over the same rows
        off, src, dst, pw = M.permute(idx, w, 0, E)
        xp = M.gather(x, src, off)
        for rows, bn in ((32, 128), (128, 128), (128, 256)):
            a = M._grouped(xp, None, bank.gate_up, off, 0, None, act, bank.padded, T * top, rows, bn)
            y = M._grouped(a, None, bank.down, off, 1, pw, act, d, T * top, rows, bn)
            _close(sum(y.double()[dst[:, j].long()] for j in range(top)), want, 8e-3, 3e-2)
    bank = M.ExpertBank.pack([m.float() for m in gates], [m.float() for m in ups], [m.float() for m in downs], act)
    y, dst = M.bank_forward(x.float(), idx, w, bank)
    _close(sum(y.double()[dst[:, j].long()] for j in range(top)), want, 1e-5, 1e-4)
    _ok()


# ------------------------------------------------------------------------------------------ recurrence
def _rec(width, blocks, taps, dtype=torch.bfloat16, seed=0):
    torch.manual_seed(seed)
    spec = R.RglruSpec(width, blocks, taps)
    b = spec.block
    v = lambda *s: torch.randn(*s, device=DEV)
    w = R.RglruWeights.make(spec, bias_y=0.3 * v(width), bias_x=0.3 * v(width), conv_w=0.6 * v(taps, width), conv_b=0.3 * v(width),
                            gate_r=_bf(blocks, b, b, std=2 * b ** -0.5).to(dtype), gate_i=_bf(blocks, b, b, std=2 * b ** -0.5).to(dtype),
                            bias_r=v(width), bias_i=v(width), lam=1.5 * v(width) - 4)
    return spec, w


def _rec_want(proj, spec, w, past):
    """fp64 outputs and final state of one sequence from its start; ``proj`` all its rows."""
    W = spec.width
    p = proj.double().cpu()
    c = lambda t: t.double().cpu()
    u = O.causal_conv(p[:, W:2 * W] + c(w.bias_x), c(w.conv_w).T) + c(w.conv_b)
    d = {"ra": c(w.gate_r), "ri": c(w.gate_i), "ra.b": c(w.bias_r).view(spec.blocks, -1), "ri.b": c(w.bias_i).view(spec.blocks, -1),
         "lam": c(w.lam)}
    a, b = O.rglru_gates(u, d, "", spec.blocks)
    S, out = torch.zeros(W).double(), torch.empty_like(u)
    for t in range(u.shape[0]):
        S = a[t] * S + b[t]
        out[t] = S
    return out * O.gelu_tanh(p[:, :W] + c(w.bias_y)), S


@pytest.mark.parametrize("impl", [None, "cuda_core"])
@pytest.mark.parametrize("width,blocks,taps", [(384, 6, 4), (512, 2, 4), (320, 2, 3), (72, 9, 2), (160, 1, 1), (768, 3, 4), (96, 4, 4)])
def test_recurrence_over_portions_and_steps(impl, width, blocks, taps):
    """Portions around the tile's edges, then single tokens of all sequences, each slot going on where it was."""
    spec, w = _rec(width, blocks, taps)
    lens = [[1, 64, 5], [63, 2, 65], [200, 1, 64], [129, 3, 2]]
    total = [sum(x) + 3 for x in lens]
    proj = [_bf(n, 2 * width) for n in total]
    state, ring = torch.zeros(6, width, device=DEV), torch.zeros(6, taps, width, device=DEV)
    slots = [4, 0, 5, 2]
    out, at = [[] for _ in lens], [0] * 4
    table = torch.zeros((4, 1), dtype=torch.int32, device=DEV)
    for k in range(3):
        b = make_prefill_batch([[0] * x[k] for x in lens], table, DEV, at)
        b.slots = torch.tensor(slots, dtype=torch.int32, device=DEV)
        y = R.rglru(torch.cat([proj[i][at[i]:at[i] + lens[i][k]] for i in range(4)]), spec, w, state, ring, b, impl)
        r = 0
        for i in range(4):
            out[i].append(y[r:r + lens[i][k]])
            r, at[i] = r + lens[i][k], at[i] + lens[i][k]
    for _ in range(3):
        pos = torch.tensor(at, dtype=torch.int32, device=DEV)
        b = ForwardBatch(pos, pos, torch.arange(4, dtype=torch.int32, device=DEV), pos + 1, table,
                         row_off=torch.arange(5, dtype=torch.int32, device=DEV), slots=torch.tensor(slots, dtype=torch.int32, device=DEV))
        y = R.rglru(torch.stack([proj[i][at[i]] for i in range(4)]), spec, w, state, ring, b, impl)
        for i in range(4):
            out[i].append(y[i:i + 1])
            at[i] += 1
    for i in range(4):
        want, S = _rec_want(proj[i], spec, w, None)
        _close(torch.cat(out[i]), want, 1e-2, 0.03)
        _close(state[slots[i]], S, 6e-3, 0.02)
    assert state[[1, 3]].abs().max() == 0 and ring[[1, 3]].abs().max() == 0
    _ok()


@pytest.mark.parametrize("rows", [1, 16, 17, 64, 65, 150])
def test_recurrence_decode_batches(rows):
    """Many sequences at different positions, states and rings given, against one step of the equation."""
    spec, w = _rec(512, 2, 4)
    proj, state, ring = _bf(rows, 1024), torch.randn(rows + 3, 512, device=DEV), torch.randn(rows + 3, 4, 512, device=DEV)
    slots = torch.randperm(rows + 3, device=DEV)[:rows].int()
    pos = torch.randint(3, 900, (rows,), device=DEV).int()
    s0, r0 = state.clone(), ring.clone()
    b = ForwardBatch(pos, pos, torch.arange(rows, dtype=torch.int32, device=DEV), pos + 1, torch.zeros((rows, 1), dtype=torch.int32, device=DEV),
                     row_off=torch.arange(rows + 1, dtype=torch.int32, device=DEV), slots=slots)
    y = R.rglru(proj, spec, w, state, ring, b)
    for i in range(rows):
        s, p = int(slots[i]), int(pos[i])
        x = proj[i, 512:].float() + w.bias_x
        u = w.conv_b + w.conv_w[3] * x + sum(w.conv_w[3 - k] * r0[s, (p - k) % 4] for k in (1, 2, 3))
        a, t = R.terms(u[None], spec, w)
        S = a[0] * s0[s] + t[0]
        _close(state[s], S.double().cpu(), 1e-2, 0.05)
        _close(y[i], (S * torch.nn.functional.gelu(proj[i, :512].float() + w.bias_y, approximate="tanh")).double().cpu(), 1e-2, 0.05)
        assert torch.equal(ring[s, p % 4], x) and torch.equal(ring[s, (p + 1) % 4], r0[s, (p + 1) % 4])
    _ok()


# ------------------------------------------------------------------------------------------ attention
def _attn(heads, kv_heads, dim, vdim, rot=None, taps=4, window=0, dtype=torch.bfloat16, ends=(), page=16, seed=0):
    torch.manual_seed(seed)
    spec = A.KVSpec(heads, kv_heads, dim, vdim, 2.0 * dim ** -0.5, 5e3, dim // 2 * 2 if rot is None else rot, taps,
                    {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 200}, window=window)
    nb = (max(ends) + page - 1) // page
    up = lambda n: (n + 7) // 8 * 8
    k, v = (torch.randn(nb * len(ends) + 2, kv_heads, page, up(n), device=DEV).to(dtype) for n in (dim, vdim))
    table = torch.randperm(nb * len(ends) + 2)[:nb * len(ends)].view(len(ends), nb).int().to(DEV)
    return spec, A.KVPages(k, v, page), table


def _rows(plane, table, s, n, page):
    return plane[table[s, :(n + page - 1) // page].long()].transpose(1, 2).flatten(0, 1)[:n].double().cpu()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,rot,taps", [(4, 2, 64, 64, 64, 4), (6, 3, 20, 24, 12, 3), (3, 1, 128, 128, 32, 4), (2, 2, 10, 14, 6, 5),
                                                               (5, 5, 7, 9, 4, 2), (1, 1, 200, 136, 0, 1), (8, 4, 72, 40, 72, 7)])
def test_prepare_in_portions_and_steps(dtype, heads, kv_heads, dim, vdim, rot, taps):
    lens = [[9, 1, 20], [1, 2, 3], [40, 17, 1]]
    ends = [sum(x) + 2 for x in lens]
    spec, kv, table = _attn(heads, kv_heads, dim, vdim, rot, taps, dtype=dtype, ends=ends)
    C = spec.channels
    cw, f = torch.randn(taps, C, device=DEV), spec.inv_freq(DEV)
    proj = [torch.randn(n, C + 8, device=DEV).to(dtype) for n in ends]
    ring, slots = torch.full((5, taps, C), 7.0, device=DEV), torch.tensor([3, 0, 4], dtype=torch.int32, device=DEV)
    out, at = [[], [], []], [0] * 3
    for k in range(5):
        if k < 3:
            n = [x[k] for x in lens]
            b = make_prefill_batch([[0] * m for m in n], table, DEV, at)
        else:
            n = [1] * 3
            pos = torch.tensor(at, dtype=torch.int32, device=DEV)
            b = ForwardBatch(pos, pos, torch.arange(3, dtype=torch.int32, device=DEV), pos + 1, table,
                             row_off=torch.arange(4, dtype=torch.int32, device=DEV))
        b.slots = slots
        q = A.prepare(torch.cat([proj[i][at[i]:at[i] + n[i]] for i in range(3)]), spec, cw, f, 1e-5, kv, ring, b)
        assert q.shape[2] == spec.q_pad and q[..., dim:].abs().sum() == 0
        for i, part in enumerate(q[..., :dim].split(n)):
            out[i].append(part)
            at[i] += n[i]
    tol = 2e-5 if dtype == torch.float32 else 6e-3
    r = {"base": 5e3, "dims": spec.rot_dims, "scaling": spec.rot_scaling}
    for i in range(3):
        x = O.causal_conv(proj[i][:, :C].double().cpu(), cw.double().cpu().T)
        q = x[:, :heads * dim].view(-1, heads, dim)
        k = x[:, heads * dim:(heads + kv_heads) * dim].view(-1, kv_heads, dim)
        v = x[:, (heads + kv_heads) * dim:].view(-1, kv_heads, vdim)
        for got, want in ((torch.cat(out[i]), O.rms(O.rotate(q, r), 1e-5)),
                          (_rows(kv.k, table, i, ends[i], 16)[..., :dim], O.rms(O.rotate(k, r), 1e-5)),
                          (_rows(kv.v, table, i, ends[i], 16)[..., :vdim], v)):
            assert (got.double().cpu() - want).abs().max() < tol * max(1.0, float(want.abs().max())), i
    assert (ring[[1, 2]] == 7).all()


@pytest.mark.parametrize("heads,kv_heads,dim,vdim,window,lens,starts", [
    (4, 2, 64, 64, 0, [64], [0]), (3, 1, 72, 40, 0, [100, 300], [0, 50]), (8, 2, 128, 128, 0, [130, 5, 700, 64], [0, 3, 257, 1000]),
    (4, 4, 24, 104, 0, [513, 2, 90], [1000, 7, 0]), (2, 1, 192, 64, 0, [200], [0]), (4, 1, 128, 128, 70, [257, 129, 30], [127, 128, 200]),
    (6, 3, 256, 256, 0, [90, 2], [0, 40]), (5, 5, 10, 14, 0, [80], [9])])
@pytest.mark.parametrize("sink", [None, 0.0, 3.0])
def test_attention_of_long_and_short_portions(heads, kv_heads, dim, vdim, window, lens, starts, sink):
    ends = [s + n for s, n in zip(starts, lens)]
    spec, kv, table = _attn(heads, kv_heads, dim, vdim, ends=ends, window=window)
    b = make_prefill_batch([[0] * n for n in lens], table, DEV, starts)
    t = sum(lens)
    q = torch.zeros(t, heads, spec.q_pad, device=DEV, dtype=torch.bfloat16)
    q[..., :dim] = _bf(t, heads, dim)
    gate = _bf(t, heads * vdim + 16)[:, 8:8 + heads * vdim]
    sinks = None if sink is None else torch.full((heads,), sink, device=DEV)
    got = A.attention(q, gate, spec, kv, sinks, b)
    rows = A.paged_rows(q, gate, spec, kv, sinks, table, b.seq_index, b.kv_lens, b.max_kv)
    any_size = A.paged_rows(q, gate, spec, kv, sinks, table, b.seq_index, b.kv_lens, b.max_kv, impl="cuda_core_any")
    r0 = 0
    for s, (n, st) in enumerate(zip(lens, starts)):
        k, v = _rows(kv.k, table, s, st + n, 16)[..., :dim], _rows(kv.v, table, s, st + n, 16)[..., :vdim]
        k, v = (x.repeat_interleave(heads // kv_heads, 1) for x in (k, v))
        pos = torch.arange(st, st + n)
        sc = torch.einsum("ihd,jhd->hij", q[r0:r0 + n, :, :dim].double().cpu(), k) * spec.scale
        gap = pos[:, None] - torch.arange(st + n)[None]
        sc = sc.masked_fill((gap < 0) | ((gap >= window) if window else False), float("-inf"))
        if sink is not None:
            sc = torch.cat([sc, torch.full((heads, n, 1), sink).double()], -1)
        p = torch.softmax(sc, -1)[..., :st + n]
        want = torch.einsum("hij,jhv->ihv", p, v).reshape(n, -1) * torch.sigmoid(gate[r0:r0 + n].double().cpu())
        for y in (got, rows, any_size):
            _close(y[r0:r0 + n], want, 1.2e-2, 0.05)
        r0 += n
    _ok()


@pytest.mark.parametrize("dim", [24, 64, 128])
def test_one_loud_key_at_page_and_tile_edges(dim):
    """A key that takes all of the weight, at every distance around a page's and a tile's edge, as one row and in a portion."""
    n = 333
    spec, kv, table = _attn(2, 1, dim, dim, ends=[n])
    si, kl = torch.zeros(1, dtype=torch.int32, device=DEV), torch.tensor([n], dtype=torch.int32, device=DEV)
    b = make_prefill_batch([[0] * 70], table, DEV, [n - 70])
    q = torch.zeros(70, 2, spec.q_pad, device=DEV, dtype=torch.bfloat16)
    q[..., :dim] = _bf(1, 1, dim)
    quiet = kv.k.clone()
    sinks = torch.zeros(2, device=DEV)
    for gap in (0, 1, 15, 16, 17, 63, 64, 65, 127, 128, 129, n - 1, n - 2, n - 17):
        j = n - 1 - gap
        kv.k.copy_(quiet)
        kv.k[table[0, j // 16].long(), 0, j % 16, :dim] = (q[0, 0, :dim].float() * 8).bfloat16()
        loud = kv.v[table[0, j // 16].long(), 0, j % 16, :dim].double().cpu()
        for o in (A.paged_rows(q[-1:], None, spec, kv, sinks, table, si, kl, n)[0], A.attention(q, None, spec, kv, sinks, b)[-1]):
            assert (o.view(2, dim).double().cpu() - loud).abs().max() < 0.05 * loud.abs().max(), gap
    _ok()


def test_layers_that_borrow_keys_reuse_the_gathered_rows():
    spec, kv, table = _attn(4, 2, 64, 64, ends=[200])
    borrows = dataclasses.replace(spec, own_kv=False)
    other = A.KVPages(kv.k.clone().mul_(-1), kv.v.clone(), 16)
    b = make_prefill_batch([[0] * 200], table, DEV, [0])
    q = _bf(200, 4, 64)
    a1 = A.attention(q, None, spec, kv, None, b)
    rows = b.plans["gathered", 0][1]
    assert torch.equal(A.attention(q, None, borrows, kv, None, b), a1) and b.plans["gathered", 0][1] is rows
    a3 = A.attention(q, None, borrows, other, None, b)
    assert b.plans["gathered", 0][1] is not rows and (a3 - a1).abs().max() > 0.1


def test_whole_prompts_portions_and_captured_steps_agree(tmp_path):
    import sepedra_cases as S
    for name in ("wide", "grouped"):
        c = S.Case(tmp_path, name, 4)
        toks = c.prompt(330, 6)
        want = c.oracle(toks)
        eng = c.engine(DEV, "bf16", max_tokens=384)
        for cuts in ([330], [63], [64], [65, 200, 1], [150, 2, 100, 1], [300, 1]):
            assert S.agrees(S.run_cut(eng, toks, cuts), want, "bf16"), (name, cuts)
        _ok()
