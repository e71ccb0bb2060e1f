"""Zokuvik against its plain restatement (tests/zokuvik_oracle.py): every mechanism, whole prompts, portions, decoding,
mixed batches, pages and slots used again, the scheduler, files and the command line - on the CPU oracle path of the ops
and, where a GPU is present, on the CUDA kernels in fp32 and bf16."""
import json
import math
import os

import pytest
import torch

import zokuvik_cases as Z
import zokuvik_oracle as O
from sllm_b200.cache.paged import OutOfPages
from sllm_b200.ops import delta as D
from sllm_b200.ops import latent as A

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
            made[name, seed] = Z.Case(tmp_path_factory.mktemp("zk"), name, seed)
        return made[name, seed]
    return get


# ------------------------------------------------------------------------------------------ mechanisms
@pytest.mark.parametrize("interleaved", [True, False])
def test_rotation_layouts(interleaved):
    x, pos = torch.randn(5, 3, 12), torch.tensor([0, 1, 7, 300, 4095])
    spec = A.LatentSpec(3, 4, 12, 4, 8, 1.0, 500.0, 10, interleaved)
    got = A.rotate(x, pos, spec.inv_freq("cpu"), 10, interleaved)
    want = O.rotate(x.double(), pos, 10, 500.0, interleaved)
    assert (got.double() - want).abs().max() < 2e-3          # fp32 angles up to 4095 rad
    assert (got.double() - want)[:3].abs().max() < 1e-5
    assert torch.equal(got[..., 10:], x[..., 10:])
    assert (got[1] - x[1]).abs().max() > 0.1


def test_group_norm_parts_are_independent():
    from sllm_b200 import ops
    x, w = torch.randn(4, 60), torch.randn(60)
    for groups in (1, 2, 5, 60):
        got = ops.group_norm(x, w, 1e-5, groups, torch.float32)
        assert torch.allclose(got.double(), O.group_norm(x.double(), w.double(), 1e-5, groups), atol=1e-5)
    y = x.clone()
    y[:, :12] *= 50
    a, b = ops.group_norm(x, w, 1e-5, 5, torch.float32), ops.group_norm(y, w, 1e-5, 5, torch.float32)
    assert torch.equal(a[:, 12:], b[:, 12:])


def test_delta_rule_update_matches_the_matrix_form():
    """diag(w) S - (a u)(u^T S) + k v^T is (diag(w) - (a u) u^T) S + k v^T, with the old state in both terms."""
    d = 7
    S, r, k, v = torch.randn(d, d).double(), *(torch.randn(d).double() for _ in range(3))
    w, a = torch.rand(d).double(), torch.rand(d).double()
    u = k / torch.sqrt((k * k).sum() + 1e-6)
    want = (torch.diag(w) - torch.outer(a * u, u)) @ S + torch.outer(k, v)
    got, o = O.delta_step(S, r, k, v, w, a)
    assert torch.allclose(got, want) and torch.allclose(o, want.T @ r)


@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("heads,dim", [(1, 16), (3, 24), (2, 33), (2, 128), (1, 200)])
def test_general_delta_layer(device, dtype, heads, dim):
    """The op on a flat batch of two sequences, prompt form then one token each, against the recurrence."""
    g = torch.Generator().manual_seed(dim)
    rnd = lambda *s: torch.randn(s, generator=g).to(torch.bfloat16).float()
    rank, n, dt = 9, heads * dim, torch.float32 if dtype == "fp32" else torch.bfloat16
    spec = D.DeltaSpec(heads, dim, rank)
    w = {"w2": rnd(n, rank), "w0": rnd(n), "a.b": rnd(n), "norm": rnd(n)}
    lens = [5, 18]
    streams = [rnd(m + 3, 5 * n + rank) for m in lens]       # projections r | k | v | a | g | w1 of each sequence

    def want(p):
        q = p.double()
        x = lambda i: q[:, i * n:(i + 1) * n].view(-1, heads, dim)
        low = torch.tanh(q[:, 5 * n:]) @ w["w2"].double().T + w["w0"].double()
        dec = torch.exp(-math.exp(-0.5) * torch.sigmoid(low)).view(-1, heads, dim)
        a = torch.sigmoid(q[:, 3 * n:4 * n] + w["a.b"].double()).view(-1, heads, dim)
        o = torch.zeros_like(dec)
        for h in range(heads):
            S = torch.zeros(dim, dim).double()
            for t in range(q.shape[0]):
                S, o[t, h] = O.delta_step(S, x(0)[t, h], x(1)[t, h], x(2)[t, h], dec[t, h], a[t, h])
        return O.rms(o, 1e-5).reshape(-1, n) * w["norm"].double() * torch.sigmoid(q[:, 4 * n:5 * n])

    from sllm_b200.ops.core import LinearWeight
    dev = torch.device(device)
    to = lambda t: t.to(dev)
    w2 = torch.zeros(n, 16)
    w2[:, :rank] = w["w2"]
    state = torch.zeros(4, heads, dim, dim, device=dev)
    slots = torch.tensor([2, 0], dtype=torch.int32, device=dev)
    run = lambda p, off, one: D.general_delta(p.to(dt).to(dev), spec, LinearWeight("dense", w2.to(dt).to(dev)), to(w["w0"]),
                                              to(w["a.b"]), to(w["norm"]), 1e-5, state,
                                              torch.tensor(off, dtype=torch.int32, device=dev), slots, one).double().cpu()
    got = [run(torch.cat([streams[0][:5], streams[1][:18]]), [0, 5, 23], False)]
    parts = [got[0][:5]], [got[0][5:]]
    for t in range(3):
        y = run(torch.stack([streams[0][5 + t], streams[1][18 + t]]), [0, 1, 2], True)
        parts[0].append(y[:1])
        parts[1].append(y[1:])
    tol = 2e-5 if dtype == "fp32" else 4e-2
    for p, s in zip(parts, streams):
        ref = want(s)
        assert (torch.cat(p) - ref).abs().max() < tol * ref.abs().max()
    assert state[1].abs().max() == 0 and state[3].abs().max() == 0      # slots of nobody stay as they were


# ------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("device,dtype", RUNS)
@pytest.mark.parametrize("name", list(Z.CASES))
def test_prompt_portions_and_decoding_agree_with_the_oracle(cases, name, device, dtype):
    c = cases(name)
    n = 150 if device == "cuda" else 60
    toks = c.prompt(n, 1)
    want = c.oracle(toks)
    eng = c.engine(device, dtype)
    whole = Z.run_cut(eng, toks, [n])
    assert Z.error(whole, want) < Z.TOL[dtype]
    assert Z.error(whole[:4], want[:4]) < Z.TOL[dtype]
    for cuts in ([2], [1], [3, 5, 2], [16], [17, 1, 64, 2], [n - 9, 1]):
        got = Z.run_cut(eng, toks, cuts)
        assert Z.error(got, want) < Z.TOL[dtype], cuts
    assert eng.cache.pool.stats()["free"] == eng.cache.pool.stats()["pages"] and len(eng.cache._free) == 4
    if device == "cuda":
        from sllm_b200 import ops
        assert ops.device_status(torch.device("cuda")) == 0


@pytest.mark.parametrize("device,dtype", RUNS)
def test_batches_of_unequal_requests_equal_each_alone(cases, device, dtype):
    """Portions of some requests beside single tokens of others, requests that pause, and pages and slots that are taken
    again by later requests, in a pool that just fits the live ones."""
    c = cases("mixed", 3)
    lens = {"a": 45, "b": 3, "c": 61, "d": 30, "e": 52, "f": 17}
    toks = {k: c.prompt(n, 7 + i) for i, (k, n) in enumerate(lens.items())}
    want = {k: c.oracle(t) for k, t in toks.items()}
    eng = c.engine(device, dtype, max_tokens=240)            # live: at most a, c, d, e
    schedule = [{"a": 20, "b": 2, "c": 2}, {"a": 1, "b": 1, "c": 33}, {"c": 5, "d": 16}, {"a": 1, "d": 1, "c": 1}, {"a": 7, "d": 2},
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
            assert Z.error(out[r:r + n], want[k][at[k]:at[k] + n]) < Z.TOL[dtype], (step, k)
            r, at[k] = r + n, at[k] + n
            if at[k] == lens[k]:
                eng.free_sequence(live.pop(k))
    assert eng.cache.pool.stats()["high_water"] <= 15


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
def test_window_edge_far_key_and_first_tokens(tmp_path, device, dtype):
    """A token that only one query looks for: with the embedding of token 1 aligned to the key of token 2, the logits show
    whether position i still sees position j.  Checked just inside and just outside the window, over page borders, in
    prompts and decoding, and for a full-attention layer at any distance."""
    win = 23
    cfg = Z.config([Z.windowed(None, heads=2, dim=16, rot=8, vdim=16, rank=32, window=win, scale=1.0),
                    Z.latent(None, heads=2, dim=16, rot=8, vdim=16, rank=32, q_rank=24, scale=1.0)], width=64, vocab=40)
    for li in (0, 1):
        w = Z.random_weights(cfg, 5)
        p = f"l{li}.mix."
        # rotated parts silent: only the unrotated score decides; W_dkv of the other layer zero: that layer is inert
        R = 8
        w[p + "dkv"][-R:] = 0
        w[f"l{1 - li}.mix.o"].zero_()
        q_of = "dq" if li else "q"
        w[p + q_of] *= 4
        want_w = {k: v.double() for k, v in w.items()}
        # find a (query token, key token) pair with the highest score over the vocabulary
        e = O.group_norm(want_w["embed"], want_w[f"l{li}.norm1"], 1e-6, 1)
        m = cfg["layers"][li]["mixer"]
        q = ((O.rms(e @ want_w[p + "dq"].T, 1e-6) * want_w[p + "dq.norm"]) @ want_w[p + "uq"].T) if li else e @ want_w[p + "q"].T
        q = q.view(-1, 2, 24)[:, 0, :16]
        k = ((O.rms((e @ want_w[p + "dkv"].T)[:, :32], 1e-6) * want_w[p + "dkv.norm"]) @ want_w[p + "uk"].T).view(-1, 2, 16)[:, 0]
        sc = q @ k.T
        qi, kj = divmod(int(sc.argmax()), sc.shape[1])
        filler = int(sc[qi].argmin())
        c = Z.Case(tmp_path, f"edge{li}{device}{dtype}", cfg=cfg, weights=w)
        eng = c.engine(device, dtype)
        for j in (0, 1, 14, 15, 16, 31):
            for gap in ((win - 1, win) if li == 0 else (1, 16, 100)):
                toks = [filler] * (j + gap + 1)
                toks[j], toks[-1] = kj, qi
                base = list(toks)
                base[j] = filler
                with_key, without = c.oracle(toks)[-1], c.oracle(base)[-1]
                seen = li == 1 or gap < win
                moved = float((with_key - without).pow(2).mean().sqrt() / without.pow(2).mean().sqrt())
                assert (moved > 0.3) == seen                 # the test's own weights make the edge visible
                for cuts in ([len(toks)], [len(toks) - 1, 1], [2]):
                    got = Z.run_cut(eng, toks, cuts)[-1:]
                    assert Z.error(got, with_key[None]) < (0.15 if dtype == "bf16" else 1e-3), (li, j, gap, cuts)


@pytest.mark.parametrize("device,dtype", RUNS)
def test_long_decoding_keeps_the_state(cases, device, dtype):
    c = cases("delta-first", 2)
    n = 300 if device == "cuda" else 120
    toks = c.prompt(n, 4)
    got = Z.run_cut(c.engine(device, dtype), toks, [5, 1])
    assert Z.error(got, c.oracle(toks)) < Z.TOL[dtype]


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
    want = [_greedy(c, p, 6) for p in prompts]
    eng = c.engine(device, "fp32")
    assert eng.generate(prompts, 6) == want
    loop = EngineLoop(eng, max_batch=3, prefill_chunk_tokens=7)
    out, done = [[] for _ in prompts], [threading.Event() for _ in prompts]
    try:
        for i, p in enumerate(prompts):
            loop.submit(GenRequest(prompt=p, max_new_tokens=6, on_token=lambda t, s, i=i: out[i].append(t),
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
    got = eng.step([b], [[18]])
    assert Z.error(got, c.oracle(toks)[-1:]) < Z.TOL["fp32"]
    a.tokens.append(toks[21])
    assert Z.error(eng.step([a], [[0]]), c.oracle(toks[:22])[-1:]) < Z.TOL["fp32"]


def test_fork_without_a_state_starts_over(cases):
    """A source that holds pages but no state slot (a prefix-cache entry) shares nothing with a recurrent model."""
    from sllm_b200.engine.engine import Sequence
    c = cases("mixed")
    toks = c.prompt(25, 8)
    eng = c.engine("cpu", "fp32")
    a = eng.new_sequence([])
    a.tokens.extend(toks[:20])
    eng.step([a], [[]])
    entry = Sequence(prompt=toks[:20], seq_id=eng.fork_kv(a, 20), num_computed=20)
    b = eng.fork_sequence(entry, toks)
    assert b.num_computed == 0
    assert Z.error(eng.step([b], [[24]]), c.oracle(toks)[-1:]) < Z.TOL["fp32"]


def test_page_export_round_trip(cases):
    eng = cases("mixed").engine("cpu", "fp32")
    a = eng.new_sequence([])
    a.tokens.extend(cases("mixed").prompt(37, 2))
    eng.step([a], [[]])
    img = eng.cache.export_pages(a.seq_id)
    b = eng.cache.import_pages(img)
    again = eng.cache.export_pages(b)
    assert img["length"] == again["length"] == 37 and torch.equal(img["values"], again["values"])


@pytest.mark.parametrize("device", ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)])
def test_trace_session_writes_logits(cases, tmp_path, device):
    from sllm_b200.cli.trace import TraceError, TraceSession
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
    assert Z.error(got[0], want[[0, 6]]) < Z.TOL["fp32"] and Z.error(got[1], want[11:]) < Z.TOL["fp32"]
    with pytest.raises(TraceError):
        t.run({"step": 3, "entries": [{"id": "x", "tokens": [c.cfg["vocab"]], "want": []}], "end": []})


# ------------------------------------------------------------------------------------------ files, registry, command line
def test_config_is_read_and_refused(cases, tmp_path):
    from sllm_b200.models import registry
    from sllm_b200.models.config import NAMED
    c = cases("mixed")
    cfg = registry.read_folder_config(c.path, "fp32")
    assert (cfg.family, cfg.n_layers, cfg.vocab, cfg.norm_groups) == ("zokuvik", 3, 211, 3)
    assert NAMED["zokuvik"]().family == "zokuvik"
    for change in ({"architecture": "Other"}, {"layers": [{"type": "x", "mixer": {}, "mlp": None}]},
                   {"norm": {"eps": 1e-5, "groups": 7}}):
        p = Z.write_folder(tmp_path / "bad", dict(c.cfg, **change), {})
        with pytest.raises(registry.ModelFolderError):
            registry.read_folder_config(p)
    w = dict(c.w)
    del w["l1.mix.w2"]
    with pytest.raises(registry.ModelFolderError):
        registry.load_folder_weights(Z.write_folder(tmp_path / "short", c.cfg, w), cfg, "cpu")
    w = dict(c.w, **{"l2.mix.uk": c.w["l2.mix.uk"].T.contiguous()})
    with pytest.raises(registry.ModelFolderError):
        registry.load_folder_weights(Z.write_folder(tmp_path / "turned", c.cfg, w), cfg, "cpu")


def test_packed_weights_unpack_to_the_source(cases):
    from sllm_b200.models import registry, zokuvik
    c = cases("mixed")
    cfg = registry.read_folder_config(c.path, "fp32")
    w = registry.load_folder_weights(c.path, cfg, "cpu")
    got = dict(zokuvik.named_tensors(cfg, w))
    assert set(got) == set(c.w) and all(torch.equal(got[n].float(), c.w[n]) for n in got)


def test_convert_and_generate_on_the_command_line(cases, tmp_path, capsys):
    from sllm_b200.cli import convert
    from sllm_b200.cli import main as cli
    from sllm_b200.formats import model_lock as ML
    c = cases("mixed")
    lock, gguf, dlock = tmp_path / "lock.json", str(tmp_path / "m.gguf"), str(tmp_path / "m.lock")
    doc = ML.make_model_lock(c.path, "local/zokuvik", "0" * 40, ["zokuvik"], {"family": "zokuvik"}, {"kind": "none"})
    lock.write_text(json.dumps(doc))
    assert convert.main(["--kind", "zokuvik", "--lock", str(lock), "--cache", c.path, "--output", gguf, "--derived-lock", dlock,
                         "--weight-format", "fp32"]) == 0
    capsys.readouterr()
    prompt = c.prompt(9, 5)
    assert cli.main(["decode", "--gguf", gguf, "--derived-lock", dlock, "--cpu", "--max-new-tokens", "5",
                     "--input-token-ids", ",".join(map(str, prompt))]) == 0
    rec = json.loads(capsys.readouterr().out.strip().splitlines()[-1])
    assert rec["output_tokens"] == _greedy(c, prompt, 5)


def test_random_shape_round_trips_through_gguf(tmp_path, capsys):
    from sllm_b200.cli import convert
    from sllm_b200.formats import gguf as G
    from sllm_b200.models import loader, registry, zokuvik
    gguf, dlock = str(tmp_path / "t.gguf"), str(tmp_path / "t.lock")
    assert convert.main(["--kind", "random-llama", "--artifact", "tiny-zokuvik", "--output", gguf, "--derived-lock", dlock]) == 0
    cfg, w, family = loader.load_model_gguf(G.verify_gguf(gguf, G.read_derived_lock(dlock)), "cpu")
    assert family == "zokuvik" and cfg.weight_format == "bf16"
    if not torch.cuda.is_available():
        ref = dict(zokuvik.named_tensors(cfg, registry.init_random_weights(cfg, "cpu", 0)))
        assert all(torch.equal(t, ref[n]) for n, t in zokuvik.named_tensors(cfg, w))


def test_delta_argument_block_matches_the_library():
    import ctypes as C
    from sllm_b200.ops import _lib
    if not _lib.kernels_available():
        pytest.skip("kernel library not built")
    out = (C.c_int * 2)()
    assert D._k().sllm_delta_abi(out, 2) == 2
    assert list(out) == [C.sizeof(D.DeltaArgs), D.DeltaArgs.eps.offset]
