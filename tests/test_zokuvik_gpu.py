"""CUDA kernels of the latent-attention, delta-rule and grouped-norm layers against fp32 PyTorch statements of the same op."""
import pytest
import torch

import zokuvik_oracle as O
from sllm_b200 import ops
from sllm_b200.engine.batch import make_prefill_batch
from sllm_b200.ops import latent as A
from sllm_b200.ops.core import LinearWeight

pytestmark = pytest.mark.gpu
DEV = "cuda"


def _bf(*shape, std=1.0):
    return (torch.randn(*shape, device=DEV) * std).to(torch.bfloat16)


def _ok():
    assert ops.device_status(torch.device(DEV)) == 0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("d,groups", [(96, 3), (60, 5), (2560, 1), (4096, 32), (77, 7), (520, 8)])
def test_group_norm_launch(dtype, d, groups):
    torch.manual_seed(d)
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    table, ids = torch.randn(50, d, device=DEV).to(dtype), torch.tensor([3, 49, 0, 7, 7], dtype=torch.int32, device=DEV)
    w1, w2 = torch.randn(d, device=DEV), torch.randn(d, device=DEV)
    ref = lambda x, w: O.group_norm(x.double(), w.double(), 1e-6, groups)
    x, z = ops.embed_group_norm(table, ids, w1, 1e-6, groups)
    assert torch.equal(x, table[ids.long()].float()) and z.dtype == dtype
    assert (z.double() - ref(x, w1)).abs().max() < tol * 5
    y = torch.randn(5, d, device=DEV).to(dtype)
    want = x.double() + ref(y, w2)
    z = ops.add_group_norm(x, y, w2, w1, 1e-6, groups)
    assert (x.double() - want).abs().max() < 2e-5 and (z.double() - ref(x, w1)).abs().max() < tol * 5
    assert ops.add_group_norm(x, y, w2, None, 1e-6, groups) is None
    rows = torch.tensor([4, 0], device=DEV)
    z = ops.group_norm(x, w1, 1e-6, groups, dtype, rows)
    assert z.shape[0] == 2 and (z.double() - ref(x[rows], w1)).abs().max() < tol * 5


@pytest.mark.parametrize("m,n,k", [(1, 5, 7), (3, 130, 64), (65, 70, 33), (200, 64, 129)])
def test_cuda_core_product(m, n, k):
    torch.manual_seed(m)
    x, w, r = torch.randn(m, k, device=DEV), torch.randn(n, k, device=DEV), torch.randn(m, n, device=DEV)
    want = x.double() @ w.double().T
    assert (ops.linear(x, LinearWeight("dense", w)).double() - want).abs().max() < 1e-4
    assert (ops.linear(x, LinearWeight("dense", w), r).double() - want - r.double()).abs().max() < 1e-4
    y = ops.linear(x, LinearWeight("dense", w), act="relu_sq").double()
    assert (y - torch.relu(want) ** 2).abs().max() < 2e-5 * (1 + want.abs().max() ** 2)
    if k % 8:
        xb, wb = x.bfloat16(), w.bfloat16()
        want = xb.double() @ wb.double().T
        assert (ops.linear(xb, LinearWeight("dense", wb)).double() - want).abs().max() < 2e-2 * want.abs().max()


@pytest.mark.parametrize("m", [1, 20, 100, 300])
def test_product_with_squared_relu_epilogue(m):
    torch.manual_seed(m)
    x, w = _bf(m, 200), _bf(328, 200, std=0.1)
    want = torch.relu(x.double() @ w.double().T) ** 2
    got = ops.linear(x, LinearWeight("dense", w), act="relu_sq").double()
    assert (got - want).abs().max() < 6e-3 * want.max()
    _ok()


def test_argmax_of_fp32_rows():
    torch.manual_seed(0)
    for n in (7, 211, 9001):
        x = torch.randn(3, n, device=DEV)
        x[1, n // 2] = x[1].max() + 1
        x[2, 1] = float("nan")
        got = ops.argmax(x).tolist()
        assert got[:2] == x[:2].argmax(-1).tolist() and got[2] == -1


# ------------------------------------------------------------------------------------------ attention kernels
def _setup(heads, rank, rot, lens, window, page, dim=16, vdim=16, seed=0):
    torch.manual_seed(seed)
    width = rank + rot
    spec = A.LatentSpec(heads, dim, rot, vdim, rank, width ** -0.5, 1e4, rot, True, window=window)
    nb = (max(lens) + page - 1) // page
    pages = _bf(nb * len(lens) + 2, page, (width + 7) // 8 * 8)
    table = torch.randperm(nb * len(lens) + 2)[:nb * len(lens)].view(len(lens), nb).int().to(DEV)
    return spec, A.LatentPages(pages, page), table


def _rows(kv, table, s, n, width):
    blks = table[s, :(n + kv.page_size - 1) // kv.page_size].long()
    return kv.pages[blks].flatten(0, 1)[:n, :width]


@pytest.mark.parametrize("heads,rank,rot,lens,window,page", [
    (6, 160, 48, [1, 65, 700], 0, 16), (20, 512, 64, [2048, 33], 0, 16), (3, 48, 24, [100, 17, 64, 5], 21, 16),
    (40, 256, 32, [513, 300], 100, 32), (33, 512, 64, [640, 128], 0, 8), (17, 512, 64, [64, 63, 129], 40, 16), (1, 16, 2, [3000], 0, 16)])
def test_page_streaming_attention(heads, rank, rot, lens, window, page):
    spec, kv, table = _setup(heads, rank, rot, lens, window, page)
    q = _bf(len(lens), heads, spec.width, std=3.0)
    si, kl = torch.arange(len(lens), device=DEV).int(), torch.tensor(lens, device=DEV).int()
    got = A.attend(q, spec, kv, table, si, kl, max(lens)).double()
    plain = A.attend(q, spec, kv, table, si, kl, impl="cuda_core").double()
    for s, n in enumerate(lens):
        rows = _rows(kv, table, s, n, spec.width)[max(0, n - window) if window else 0:].double()
        want = torch.softmax(q[s].double() @ rows.T * spec.scale, -1) @ rows[:, :rank]
        for y in (got[s], plain[s]):
            assert (y - want).abs().max() < 2e-2 * want.abs().max(), (s, n)
    _ok()


@pytest.mark.parametrize("impl", [None, "cuda_core"])
@pytest.mark.parametrize("window", [0, 1, 16, 71, 128])
def test_one_loud_key_at_page_and_window_edges(impl, window):
    """A key that takes all of the weight when it is visible, at every distance around a page's, a tile's and the
    window's edge."""
    n, page = 333, 16
    spec, kv, table = _setup(2, 64, 16, [n], window, page)
    q = _bf(1, 2, spec.width)
    si, kl = torch.zeros(1, dtype=torch.int32, device=DEV), torch.tensor([n], dtype=torch.int32, device=DEV)
    quiet = kv.pages.clone()
    for gap in sorted({0, 1, 15, 16, 17, 63, 64, 65, window - 1, window, window + 1, n - 1, n - 2, n - 17} - {-1}):
        j = n - 1 - gap
        kv.pages.copy_(quiet)
        row = q[0].float().sum(0) * 30
        kv.pages[table[0, j // page].long(), j % page, :spec.width] = row.bfloat16()
        o = A.attend(q, spec, kv, table, si, kl, n, impl=impl)[0].double()
        seen = window == 0 or gap < window
        loud = kv.pages[table[0, j // page].long(), j % page, :64].double()
        hit = (o - loud).abs().max() < 0.05 * loud.abs().max()
        assert bool(hit) == seen or (window == 1 and gap == 0), gap
    _ok()


@pytest.mark.parametrize("heads,dim,rot,vdim,rank,window,inter,lens,starts", [
    (6, 48, 32, 40, 160, 0, True, [64], [0]), (7, 24, 40, 56, 144, 90, False, [100, 300], [0, 50]),
    (3, 128, 64, 128, 512, 0, True, [130, 5, 700, 64], [0, 3, 257, 1000]), (2, 40, 24, 104, 96, 300, False, [513, 2, 90], [1000, 7, 0]),
    (5, 64, 2, 64, 64, 1, True, [200], [0]), (2, 128, 64, 128, 256, 128, True, [257, 129], [127, 128])])
def test_expanded_portions_beside_short_ones(heads, dim, rot, vdim, rank, window, inter, lens, starts):
    ends = [s + n for s, n in zip(starts, lens)]
    spec, kv, table = _setup(heads, rank, rot, ends, window, 16, dim, vdim)
    spec.interleaved, spec.scale = inter, (dim + rot) ** -0.5
    b = make_prefill_batch([[0] * n for n in lens], table, DEV, starts)
    t = sum(lens)
    q, ex, gate = _bf(t, heads * (dim + rot), std=2.0), _bf(heads * (dim + vdim), rank, std=rank ** -0.5), _bf(t, heads)
    uk, uv = ex[:heads * dim].view(heads, dim, rank), ex[heads * dim:].view(heads, vdim, rank)
    f = spec.inv_freq(DEV)
    got = A.attention(q, gate, spec, uk, uv.transpose(1, 2).contiguous(), LinearWeight("dense", ex), f, kv, b).double()
    x = q.double().view(t, heads, dim + rot)
    r0 = 0
    for s, (n, st) in enumerate(zip(lens, starts)):
        rows = _rows(kv, table, s, st + n, spec.width).double()
        k, v = torch.einsum("jc,hdc->hjd", rows[:, :rank], uk.double()), torch.einsum("jc,hvc->hjv", rows[:, :rank], uv.double())
        pos = torch.arange(st, st + n, device=DEV)
        qr = O.rotate(x[r0:r0 + n, :, dim:].cpu(), pos.cpu(), rot, 1e4, inter).to(DEV)
        sc = torch.einsum("ihd,hjd->hij", x[r0:r0 + n, :, :dim], k) + torch.einsum("ihr,jr->hij", qr, rows[:, rank:])
        gap = pos[:, None] - torch.arange(st + n, device=DEV)[None]
        see = (gap >= 0) & ((gap < window) if window else True)
        p = torch.softmax((sc * spec.scale).masked_fill(~see, float("-inf")), -1)
        want = torch.einsum("hij,hjv->ihv", p, v) * torch.sigmoid(gate[r0:r0 + n].double())[..., None]
        d = got[r0:r0 + n].view(n, heads, vdim) - want
        assert d.pow(2).mean().sqrt() < 1e-2 * want.pow(2).mean().sqrt() and d.abs().max() < 0.1 * want.abs().max(), s
        r0 += n
    _ok()


def test_portion_plan_covers_every_row_once():
    b = [0, 2, 70, 75, 75, 275, 476, 477]
    ports = A.plan_portions(b, [5, 0, 9, 3, 40, 0, 11], 50, DEV)
    assert [(p.lo, p.hi, p.spans is not None) for p in ports] == [(0, 2, False), (2, 70, True), (70, 75, False), (75, 476, True),
                                                                 (476, 477, False)]
    tiles = ports[3].tiles.tolist()
    assert sorted((t[0], t[1]) for t in tiles) == [(0, 128), (128, 72), (200, 128), (328, 73)]
    assert ports[3].spans.tolist() == [[4, 0, 240, 0], [5, 0, 201, 240]]


def test_whole_prompts_portions_and_captured_steps_agree(tmp_path):
    """The same request whole, through the expanded and absorbed forms of a portion, and decoded by captured steps."""
    import zokuvik_cases as Z
    c = Z.Case(tmp_path, "wide-heads", 4)
    toks = c.prompt(330, 6)
    want = c.oracle(toks)
    eng = c.engine(DEV, "bf16", max_tokens=384)
    for cuts in ([330], [63], [64], [65, 200, 1], [150, 2, 100, 1], [300, 1]):
        assert Z.error(Z.run_cut(eng, toks, cuts), want) < Z.TOL["bf16"], cuts
    _ok()
