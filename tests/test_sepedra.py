"""Sepedra against its plain restatement (tests/sepedra_oracle.py): every mechanism, whole prompts, portions, decoding,
mixed batches, pages and slots used again, the scheduler, files and the command line - on the CPU oracle path of the ops
and, where a GPU is present, on the CUDA kernels in fp32 and bf16."""
import json
import os

import pytest
import torch

import sepedra_cases as S
import sepedra_oracle as O
from sllm_b200.cache.paged import OutOfPages
from sllm_b200.ops import kv_attention as A
from sllm_b200.ops import moe as M
from sllm_b200.ops import rglru as R
from sllm_b200.ops.short_conv import causal_conv

RUNS = [("cpu", "fp32"), pytest.param("cuda", "fp32", marks=pytest.mark.gpu), pytest.param("cuda", "bf16", marks=pytest.mark.gpu)]


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
            made[name, seed] = S.Case(tmp_path_factory.mktemp("sp"), name, seed)
        return made[name, seed]
    return get


# ------------------------------------------------------------------------------------------ mechanisms
def test_scaled_frequencies_cover_all_three_bands():
    rot = {"base": 3e4, "dims": 56, "scaling": {"factor": 5.0, "low": 1.5, "high": 5.0, "original": 300}}
    got = A.rope_frequencies(rot["base"], rot["dims"], rot["scaling"])
    plain = A.rope_frequencies(rot["base"], rot["dims"])
    want = torch.tensor([O.frequency(i, rot) for i in range(28)], dtype=torch.float64)
    assert torch.allclose(got, want, rtol=1e-12)
    kept, slowed = got == plain, torch.isclose(got, plain / 5)
    assert kept.any() and slowed.any() and (~kept & ~slowed).any()
    assert torch.allclose(A.rope_frequencies(7e2, 10), torch.tensor([O.frequency(i, {"base": 7e2, "dims": 10}) for i in range(5)]).double())


@pytest.mark.parametrize("taps", [1, 2, 4, 7])
def test_short_convolution_in_portions(taps):
    u, w = torch.randn(23, 6), torch.randn(taps, 6)
    want = O.causal_conv(u.double(), w.t().double())
    for cuts in ([23], [1] * 23, [2] * 11 + [1], [5, 1, 9, 8]):
        ring = torch.full((3, taps, 6), 99.0)                 # what an earlier sequence left behind is not read
        got, at = [], 0
        for n in cuts:
            got.append(causal_conv(u[at:at + n], w, ring, torch.tensor([0, n]), torch.tensor([1]), torch.arange(at, at + n)))
            at += n
        assert torch.allclose(torch.cat(got).double(), want, atol=1e-5), cuts


def test_recurrence_terms():
    spec = R.RglruSpec(12, 3, 4)
    w = {"ra": torch.randn(3, 4, 4), "ri": torch.randn(3, 4, 4), "ra.b": torch.randn(3, 4), "ri.b": torch.randn(3, 4), "lam": torch.randn(12)}
    u = torch.randn(9, 12)
    z = torch.zeros(12)
    rec = R.RglruWeights.make(spec, bias_y=z, bias_x=z, conv_w=z, conv_b=z, gate_r=w["ra"], gate_i=w["ri"], bias_r=w["ra.b"].view(-1),
                              bias_i=w["ri.b"].view(-1), lam=w["lam"])
    for got, want in zip(R.terms(u, spec, rec), O.rglru_gates(u.double(), {k: v.double() for k, v in w.items()}, "", 3)):
        assert torch.allclose(got.double(), want, atol=1e-5)
    tiles = R.pack_gates(spec, w["ra"], w["ri"])
    assert tiles.shape == (3, 1, 2, 128, 64) and torch.equal(tiles[1, 0, 1, :4, :4], w["ri"][1]) and tiles[:, :, :, 4:].abs().max() == 0


def test_tiles_follow_the_sequences():
    t = R.plan_tiles([0, 1, 65, 65, 194], "cpu").tolist()
    assert [(a, b, c, d & 0xffffff, d >> 24) for a, b, c, d in t] == \
        [(0, 1, 0, 0, 1), (1, 64, 1, 0, 1), (65, 64, 3, 0, 0), (129, 64, 3, 1, 0), (193, 1, 3, 2, 1)]


@pytest.mark.parametrize("device", ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)])
@pytest.mark.parametrize("E,top,count,keep", [(15, 4, 5, 3), (8, 1, 8, 1), (64, 8, 8, 4), (5, 5, 1, 1), (200, 20, 10, 3), (6, 2, 2, 2)])
def test_group_limited_routing(device, E, top, count, keep):
    g = torch.Generator().manual_seed(E)
    z = torch.randn(40, E, generator=g) * 2
    idx, w = M.route(z.to(device), top, True, count, keep)
    free = M.route(z.to(device), top, True)[0]
    for t in range(40):
        want = O.route(z[t].double(), {"top": top, "groups": {"count": count, "keep": keep}})
        assert idx[t].tolist() == [e for e, _ in want]
        assert torch.allclose(w[t].double().cpu(), torch.stack([s for _, s in want]), rtol=1e-5)
        assert len({int(e) // (E // count) for e in idx[t]}) <= keep
    assert (idx != free).any().item() == (keep < count and top > 1)         # the limit decides for some token


def test_expert_bank_round_trip_and_clamps():
    g = torch.Generator().manual_seed(0)
    gates, ups, downs = ([torch.randn(*s, generator=g) for _ in range(3)] for s in ((70, 16), (70, 16), (16, 70)))
    bank = M.ExpertBank.pack(gates, ups, downs, M.GatedAct(0.8, 1.702, 1.0))
    assert bank.padded == 128 and bank.gate_up.shape == (3, 256, 16)
    for e in range(3):
        assert all(torch.equal(a, b) for a, b in zip(bank.matrices(e), (gates[e], ups[e], downs[e])))
    x, idx, w = torch.randn(5, 16, generator=g), torch.tensor([[0, 2], [1, 0], [2, 1], [0, 1], [1, 2]], dtype=torch.int32), torch.rand(5, 2)
    y, dst = M.bank_forward(x, idx, w, bank)
    got = M.combine(y, dst, None)
    wd = {f"e{e}.{n}": m[e].double() for e in range(3) for n, m in (("gate", gates), ("up", ups), ("down", downs))}
    for t in range(5):
        want = sum(w[t, j].double() * O.expert(x[t:t + 1].double(), wd, f"e{int(idx[t, j])}.", 0.8)[0] for j in range(2))
        assert torch.allclose(got[t].double(), want, atol=1e-4)
    h = x.double() @ gates[0].double().T
    assert (h > 0.8).any() and (h < -0.8).any()             # the gate is cut from above only, the up part on both sides


def test_summed_rows_join_the_residual_normed():
    from sllm_b200 import ops
    x, y, w = torch.randn(4, 12), torch.randn(9, 12), torch.randn(12)
    terms = torch.tensor([[0, 8], [3, -1], [2, 5], [7, 7]], dtype=torch.int32)
    s = torch.stack([y[0] + y[8], y[3], y[2] + y[5], 2 * y[7]])
    want = x.double() + O.rms(s.double(), 1e-5) * w.double()
    z = ops.add_group_norm(x, y, w, None, 1e-5, terms=terms, raw=True)
    assert torch.allclose(x.double(), want, atol=1e-5) and torch.equal(z, x) and z.data_ptr() != x.data_ptr()


# ------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("name", list(S.CASES))
def test_prompt_portions_and_decoding_agree_with_the_oracle(cases, name, device, dtype):
    c = cases(name)
    n = 150 if device == "cuda" else 50
    toks = c.prompt(n, 1)
    want = c.oracle(toks)
    eng = c.engine(device, dtype)
    whole = S.run_cut(eng, toks, [n])
    assert S.agrees(whole, want, dtype)
    assert S.agrees(whole[:4], want[:4], dtype)
    for cuts in ([2], [1], [3, 5, 2], [16], [17, 1, 64, 2], [n - 9, 1]):
        assert S.agrees(S.run_cut(eng, toks, cuts), want, dtype), cuts
    assert eng.cache.pool.stats()["free"] == eng.cache.pool.stats()["pages"] and len(eng.cache._free) == 4
    if device == "cuda":
        from sllm_b200 import ops
        assert ops.device_status(torch.device("cuda")) == 0


@pytest.mark.parametrize("device", ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)])
def test_routes_follow_the_residual(tmp_path, device):
    """Routers that read every channel of what the layers before them wrote (the other models' routes hang on the token)."""
    cfg = S.CASES["mixed"]
    c = S.Case(tmp_path, "free", cfg=cfg, weights=S.random_weights(cfg, 11, clear_routes=False))
    toks = c.prompt(60, 2)
    eng = c.engine(device, "fp32")
    for cuts in ([60], [7, 1]):
        assert S.agrees(S.run_cut(eng, toks, cuts), c.oracle(toks), "fp32")


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
            assert S.agrees(out[r:r + n], want[k][at[k]:at[k] + n], dtype), (step, k)
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
    with pytest.raises(ValueError):
        eng.step([a], [[0]])                                 # nothing new to run


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("dim,vdim", [(16, 16), (64, 64)])
def test_one_far_key_decides(tmp_path, device, dtype, dim, vdim):
    """A token that only one query looks for, at the first positions, at page borders and far away: the logits show whether
    position i sees position j, in prompts, portions and decoding, in the layer that holds the keys and in one that borrows
    them."""
    m = dict(heads=2, kv_heads=1, dim=dim, vdim=vdim, rot=4, conv=1, scale=24.0 / dim, base=1e6, scaling=None)
    cfg = S.config([S.attention(None, **m), S.attention(None, kv_from=0, **m)], width=64, vocab=40, cap=50.0)
    for li in (0, 1):
        w = S.random_weights(cfg, 5)
        w[f"l{1 - li}.mix.o"].zero_()                        # the other layer is inert (the norm of 0 is 0)
        for x in ("l0.mix.q.conv", "l1.mix.q.conv", "l0.mix.k.conv", "l0.mix.v.conv"):
            w[x].fill_(1.0)
        e = w["embed"].double()
        q = O.rms((e @ w[f"l{li}.mix.q"].double().T).view(-1, 2, dim)[:, 0], 1e-5)
        k = O.rms(e @ w["l0.mix.k"].double().T, 1e-5)
        sc = q @ k.T
        qi, kj = divmod(int(sc.argmax()), sc.shape[1])
        filler = int(sc[qi].argmin())
        c = S.Case(tmp_path, f"far{li}{device}{dtype}", cfg=cfg, weights=w)
        eng = c.engine(device, dtype)
        for j in (0, 1, 14, 15, 16, 31):
            for gap in (1, 16, 100):
                toks = [filler] * (j + gap + 1)
                toks[j], toks[-1] = kj, qi
                base = list(toks)
                base[j] = filler
                with_key, without = c.oracle(toks)[-1], c.oracle(base)[-1]
                assert float((with_key - without).pow(2).mean().sqrt() / without.pow(2).mean().sqrt()) > 0.2
                for cuts in ([len(toks)], [len(toks) - 1, 1], [2]):
                    got = S.run_cut(eng, toks, cuts)[-1:]
                    assert S.error(got, with_key[None]) < (0.1 if dtype == "bf16" else 1e-3), (li, j, gap, cuts)


@pytest.mark.parametrize("device,dtype", RUNS)
def test_the_sink_shows_at_the_first_tokens(tmp_path, monkeypatch, device, dtype):
    """With the sink left out of the oracle, the first tokens come out different by far more than the tolerance."""
    # (the norm of the sublayer's output hides a factor that all heads share; heads whose scores differ do not share it)
    cfg = S.config([S.attention(None, heads=4, kv_heads=2, dim=64, vdim=64, rot=64, scale=0.3, scaling=None)], width=64, vocab=50, cap=50.0)
    c = S.Case(tmp_path, f"sink{device}{dtype}", 2, cfg=cfg)
    toks = c.prompt(70, 3)
    want = c.oracle(toks)
    monkeypatch.setattr(O, "softmax_one", lambda s: torch.softmax(s, -1))
    wrong = O.forward(toks, cfg, c.w64)
    monkeypatch.undo()
    assert S.error(wrong[:3], want[:3]) > 0.25
    for cuts in ([70], [1]):
        assert S.error(S.run_cut(c.engine(device, dtype), toks, cuts)[:3], want[:3]) < (2e-2 if dtype == "bf16" else 1e-4)


@pytest.mark.parametrize("device,dtype", RUNS)
def test_long_decoding_keeps_the_state(cases, device, dtype):
    c = cases("odd" if dtype == "fp32" else "grouped", 2)
    n = 300 if device == "cuda" else 100
    toks = c.prompt(n, 4)
    assert S.agrees(S.run_cut(c.engine(device, dtype), toks, [5, 1]), c.oracle(toks), dtype)


# ------------------------------------------------------------------------------------------ serving
def _greedy(c, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(c.oracle(toks)[-1].argmax()))
    return toks[len(prompt):]


@pytest.mark.parametrize("device", ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)])
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
    assert S.agrees(eng.step([b], [[18]]), c.oracle(toks)[-1:], "fp32")
    a.tokens.append(toks[21])
    assert S.agrees(eng.step([a], [[0]]), c.oracle(toks[:22])[-1:], "fp32")


def test_page_export_round_trip(cases):
    eng = cases("mixed").engine("cpu", "fp32")
    a = eng.new_sequence([])
    a.tokens.extend(cases("mixed").prompt(37, 2))
    eng.step([a], [[]])
    img = eng.cache.export_pages(a.seq_id)
    b = eng.cache.import_pages(img)
    again = eng.cache.export_pages(b)
    assert img["length"] == again["length"] == 37 and torch.equal(img["values"], again["values"])
    assert eng.cache.bytes_per_token() == 4 * 2 * (24 + 24)     # one layer holds keys (20, padded) and values, two heads


@pytest.mark.parametrize("device", ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)])
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
    assert S.agrees(got[0], want[[0, 6]], "fp32") and S.agrees(got[1], want[11:], "fp32")


# ------------------------------------------------------------------------------------------ files, registry, command line
def test_config_is_read_and_refused(cases, tmp_path):
    from sllm_b200.models import registry
    from sllm_b200.models.config import NAMED
    c = cases("mixed")
    cfg = registry.read_folder_config(c.path, "fp32")
    assert (cfg.family, cfg.n_layers, cfg.vocab, cfg.logit_softcap) == ("sepedra", 4, 211, 20.0)
    assert NAMED["sepedra"]().family == "sepedra"
    L = c.cfg["layers"]

    def bad(i, **mixer):
        e = dict(L[i], mixer=dict(L[i]["mixer"], **mixer))
        return {"layers": L[:i] + [e] + L[i + 1:]}

    for change in ({"architecture": "Other"}, {"layers": [{"type": "x", "mixer": {}, "mlp": None}]}, bad(0, blocks=5), bad(1, kv_heads=4),
                   bad(2, kv_from=0), bad(2, kv_from=2), bad(2, kv_from=3), bad(2, vdim=16), bad(1, rot={"base": 10.0, "dims": 22}),
                   {"layers": [S.rglru(S.moe(experts=6, top=3, ff=8, count=3, keep=1), width=8, blocks=1)]},
                   {"layers": [S.rglru({"kind": "dense", "ff": 8}, width=8, blocks=1)]}):
        p = S.write_folder(tmp_path / "bad", dict(c.cfg, **change), {})
        with pytest.raises(registry.ModelFolderError):
            registry.read_folder_config(p)
    w = dict(c.w)
    del w["l1.mix.k.conv"]
    with pytest.raises(registry.ModelFolderError):
        registry.load_folder_weights(S.write_folder(tmp_path / "short", c.cfg, w), cfg, "cpu")
    w = dict(c.w, **{"l0.mlp.e3.down": c.w["l0.mlp.e3.down"].T.contiguous()})
    with pytest.raises(registry.ModelFolderError):
        registry.load_folder_weights(S.write_folder(tmp_path / "turned", c.cfg, w), cfg, "cpu")


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_packed_weights_unpack_to_the_source(cases, name):
    from sllm_b200.models import registry, sepedra
    c = cases(name)
    cfg = registry.read_folder_config(c.path, "fp32")
    got = dict(sepedra.named_tensors(cfg, registry.load_folder_weights(c.path, cfg, "cpu")))
    assert set(got) == set(c.w) and all(got[n].shape == c.w[n].shape and torch.equal(got[n].float(), c.w[n]) for n in got)


def test_convert_and_generate_on_the_command_line(cases, tmp_path, capsys):
    from sllm_b200.cli import convert
    from sllm_b200.cli import main as cli
    from sllm_b200.formats import model_lock as ML
    c = cases("mixed")
    lock, gguf, dlock = tmp_path / "lock.json", str(tmp_path / "m.gguf"), str(tmp_path / "m.lock")
    lock.write_text(json.dumps(ML.make_model_lock(c.path, "local/sepedra", "0" * 40, ["sepedra"], {"family": "sepedra"}, {"kind": "none"})))
    args = ["--lock", str(lock), "--cache", c.path, "--output", gguf, "--derived-lock", dlock, "--weight-format", "fp32"]
    assert convert.main(["--kind", "zokuvik", *args]) != 0      # another family's folder
    assert convert.main(["--kind", "sepedra", *args]) == 0
    capsys.readouterr()
    prompt = c.prompt(9, 5)
    assert cli.main(["decode", "--gguf", gguf, "--derived-lock", dlock, "--cpu", "--max-new-tokens", "4",
                     "--input-token-ids", ",".join(map(str, prompt))]) == 0
    rec = json.loads(capsys.readouterr().out.strip().splitlines()[-1])
    assert rec["output_tokens"] == _greedy(c, prompt, 4)


def test_random_shape_round_trips_through_gguf(tmp_path, capsys):
    from sllm_b200.cli import convert
    from sllm_b200.formats import gguf as G
    from sllm_b200.models import loader, registry, sepedra
    gguf, dlock = str(tmp_path / "t.gguf"), str(tmp_path / "t.lock")
    assert convert.main(["--kind", "random-llama", "--artifact", "tiny-sepedra", "--output", gguf, "--derived-lock", dlock]) == 0
    cfg, w, family = loader.load_model_gguf(G.verify_gguf(gguf, G.read_derived_lock(dlock)), "cpu")
    assert family == "sepedra" and cfg.weight_format == "bf16"
    if not torch.cuda.is_available():
        ref = dict(sepedra.named_tensors(cfg, registry.init_random_weights(cfg, "cpu", 0)))
        assert all(torch.equal(t, ref[n]) for n, t in sepedra.named_tensors(cfg, w))


def test_argument_blocks_match_the_library():
    import ctypes as C
    from sllm_b200.ops import _lib
    if not _lib.kernels_available():
        pytest.skip("kernel library not built")
    for fn, cls, last in ((R._k().sllm_rglru_abi, R.RglruArgs, "decode"), (A._k().sllm_kv_abi, A.KvPrepareArgs, "eps")):
        out = (C.c_int * 2)()
        assert fn(out, 2) == 2
        assert list(out) == [C.sizeof(cls), getattr(cls, last).offset]
