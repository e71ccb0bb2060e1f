#!/usr/bin/env python
"""Headline benchmark: decode throughput of the Llama-3-8B-shape model (block-scaled FP8 weights,
FP8 paged KV cache, page 16), batch 32, 2048-token prompts, on N B200s of one node (TP = N).

    python bench.py --gpus N --steps K --warmup W            # this framework
    python bench.py --impl reference --gpus N ...             # the reference (unavailable: HIP/Rust only)

One "step" is one decode step of the whole batch (batch output tokens).  `value` is device-timed
(CUDA events around K graph-replayed steps with on-device token feedback); `e2e` times K calls of the
public `Engine.decode` API, each copying that step's input tokens/positions from pinned host memory
and reading the sampled tokens back.  Synthetic data: seeded uniform-random prompts, seeded ~N(0, 0.02)
weights.  Each decode step streams the whole weight set (8 GB >> 126 MB L2), so no L2 flush is needed.
"""
from __future__ import annotations

import argparse
import json
import os
import statistics
import subprocess
import sys
import tempfile
import time

# Published decode rate of the reference used as the `vs_baseline` denominator: Qwen3.5-4B FP8 W8A8 on
# MI300X, 17-in/17-out, batch 1 (ci/matrix/phase36-mi300x-session-d-summary-v1.json, row phase36-d-fp8-*).
# The reference serialises concurrent requests, so its aggregate rate at any batch equals this number.
REFERENCE_PUBLISHED_TOK_S = 56.62


def parse_args():
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=128)
    ap.add_argument("--warmup", type=int, default=8)
    ap.add_argument("--impl", default="own", choices=["own", "reference", "torch"],
                    help="own: this engine; reference: the unmodified reference (unavailable here); torch: the "
                         "unfused plain-PyTorch + NCCL comparator under baseline/")
    ap.add_argument("--batch", type=int, default=32)
    ap.add_argument("--prompt", type=int, default=2048)
    ap.add_argument("--model", default="llama3-8b")
    ap.add_argument("--weights", default=None, help="weight format override (default: fp8 for the dense models)")
    ap.add_argument("--kv", default=None, help="KV-cache format override")
    ap.add_argument("--synthetic-kv", action="store_true",
                    help="decode-only measurement: mark the prompt's KV pages as computed without running the prefill "
                         "(used for shapes whose prefill is not the subject, e.g. the MoE decode config)")
    ap.add_argument("--spec-width", type=int, default=0,
                    help="speculative decoding: draft tokens per step from a llama-draft model (acceptance forced by a "
                         "seeded Bernoulli(0.7) mask so that the full verify compute always runs)")
    ap.add_argument("--tp-impl", default="fused", choices=["fused", "nccl"])
    ap.add_argument("--parallelism", default="tp", choices=["tp", "dp"],
                    help="N > 1: tp = one model sharded over the GPUs (fused GEMM + all-reduce; the layout the benchmark "
                         "configuration names), dp = one replica per GPU, each decoding batch / N of the sequences (no "
                         "communication inside a step)")
    ap.add_argument("--no-replica-run", action="store_true",
                    help="N > 1, dense models under 16 GiB of weights: skip the second measurement of the same global batch "
                         "as one replica per GPU (reported under `replica_layout`)")
    ap.add_argument("--act4", action="store_true",
                    help="4-bit-weight models: quantise activations to the weights' 4-bit format and run the GEMMs on the "
                         "block-scaled tensor-core kernel (W4A4) instead of W4A16")
    ap.add_argument("--layers", type=int, default=0, help="profiling only: override the layer count")
    ap.add_argument("--compare", default=None, choices=["zokuvik", "sepedra", "kegorax", "fekolorn"],
                    help="instead of the headline workload: prompt and decode throughput and per-kernel roofline fractions of "
                         "a design beside the framework's closest model at equal sizes (one GPU)")
    ap.add_argument("--no-batch1", action="store_true", help="skip the extra batch-1 measurement")
    return ap.parse_args()


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while a region runs."""
    Q = ("index,clocks.sm,clocks.max.sm,power.draw,clocks_event_reasons.active,"
         "clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
         "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self, gpu_index: int):
        self.gpu = gpu_index
        self.proc = None
        self.path = None

    def start(self):
        try:
            f = tempfile.NamedTemporaryFile("w", suffix=".csv", delete=False)
            self.path = f.name
            self.proc = subprocess.Popen(["nvidia-smi", f"--query-gpu={self.Q}", "--format=csv,noheader,nounits",
                                          "-lms", "20", "-i", str(self.gpu)], stdout=f, stderr=subprocess.DEVNULL)
        except Exception:
            self.proc = None

    def stop(self) -> dict:
        if self.proc is None:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": ["unsampled"]}
        time.sleep(0.15)
        self.proc.terminate()
        try:
            self.proc.wait(timeout=5)
        except Exception:
            self.proc.kill()
        sm, smax, reasons, power = [], [], set(), []
        try:
            for line in open(self.path):
                p = [x.strip() for x in line.split(",")]
                if len(p) < 9:
                    continue
                try:
                    sm.append(float(p[1])); smax.append(float(p[2])); power.append(float(p[3]))
                except ValueError:
                    continue
                for name, v in zip(("hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"), p[5:9]):
                    if v.lower().startswith("active"):
                        reasons.add(name)
            os.unlink(self.path)
        except Exception:
            pass
        return {"sm_mhz": statistics.median(sm) if sm else None, "sm_max_mhz": max(smax) if smax else None,
                "power_w_max": max(power) if power else None, "samples": len(sm), "reasons": sorted(reasons)}


def run_reference(args):
    print(json.dumps({
        "impl": "reference",
        "unavailable": "reference is Rust + HIP for AMD gfx1030/gfx1201/gfx942 only (no CUDA path, no cargo/hipcc "
                       "here); installing the reference with pip fails at metadata generation (test-contract package "
                       "with no importable modules)"}))
    return 0


def run_torch_baseline(args):
    """Same model shape, prompt and step count through baseline/torch_llama.py (bf16 library GEMMs, SDPA, NCCL)."""
    import torch
    import torch.distributed as dist
    sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
    from baseline.torch_llama import TorchLlama
    from sllm_b200.models import config as mc
    world = int(os.environ.get("WORLD_SIZE", "1"))
    rank = int(os.environ.get("RANK", "0"))
    local_rank = int(os.environ.get("LOCAL_RANK", "0"))
    torch.cuda.set_device(local_rank)
    device = torch.device("cuda", local_rank)
    if world > 1:
        os.environ.setdefault("MASTER_ADDR", "127.0.0.1")
        dist.init_process_group("nccl", device_id=device)
    cfg = mc.NAMED[args.model]()
    if args.layers > 0:
        cfg.n_layers = args.layers
    cfg.max_context = ((args.prompt + args.warmup + args.steps + 64 + 255) // 256) * 256
    model = TorchLlama(cfg, device, seed=0, tp_size=world, tp_rank=rank, max_batch=args.batch)
    g = torch.Generator().manual_seed(1234)
    prompts = torch.randint(0, cfg.vocab, (args.batch, args.prompt), generator=g)
    pinned = torch.empty((args.batch, 1), dtype=torch.int64, pin_memory=True)
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)

    def sync():
        if world > 1:
            dist.barrier()
        torch.cuda.synchronize()

    sync()
    e0.record()
    nxt = None
    for i in range(0, args.batch, 8):      # prefill in groups of 8 like the engine arm
        part = model_forward_rows(model, prompts[i:i + 8].to(device), i, 0)
        nxt = part if nxt is None else torch.cat([nxt, part])
    e1.record()
    sync()
    prefill_ms = e0.elapsed_time(e1)
    pos = args.prompt
    for _ in range(args.warmup):
        nxt = model.forward(nxt.view(-1, 1), pos)
        pos += 1
    clocks = ClockSampler(local_rank)
    if rank == 0:
        clocks.start()
    sync()
    t0 = time.perf_counter()
    e0.record()
    for _ in range(args.steps):
        pinned.copy_(nxt.view(-1, 1))                     # D2H of the step's result
        tok = pinned.to(device, non_blocking=True)        # H2D of the next step's input from pinned memory
        nxt = model.forward(tok, pos)
        pos += 1
    e1.record()
    sync()
    wall_ms = (time.perf_counter() - t0) * 1e3
    ms = max(e0.elapsed_time(e1), wall_ms)
    if world > 1:
        t = torch.tensor([ms], device=device, dtype=torch.float64)
        dist.all_reduce(t, op=dist.ReduceOp.MAX)
        ms = float(t.item())
    clk = clocks.stop() if rank == 0 else None
    if rank == 0:
        value = args.batch * args.steps / (ms / 1e3)
        print(json.dumps({
            "metric": "decode_output_tokens_per_s", "value": round(value, 2), "unit": "tok/s", "n_gpus": args.gpus,
            "steps": args.steps, "warmup": args.warmup, "ms_per_step": round(ms / args.steps, 4), "higher_is_better": True,
            "scaling": "strong", "vs_baseline": round(value / REFERENCE_PUBLISHED_TOK_S, 2), "dtype": "bf16",
            "data": "synthetic: seeded uniform-random prompts, seeded N(0,0.02) random-init weights",
            "config": {"model": f"{cfg.name}-bf16", "global_batch": args.batch, "seq_len": args.prompt,
                       "output_tokens": args.steps, "kv_cache": "bf16-contiguous", "parallelism": f"tp{args.gpus}-nccl"},
            "clocks": clk, "e2e": {"value": round(value, 2), "unit": "tok/s", "ms_per_step": round(ms / args.steps, 4),
                                   "h2d_bytes_per_step": args.batch * 8, "d2h_bytes_per_step": args.batch * 8,
                                   "api": "baseline.torch_llama.TorchLlama.forward"},
            "gpu_launches": 0, "ttft_ms_batch_prefill": round(prefill_ms, 2), "impl": "torch-unfused-baseline"}))
    sys.stdout.flush()
    if world > 1:
        dist.barrier()
        dist.destroy_process_group()
        os._exit(0)
    return 0


def run_speculative(args, cfg, device, tp, world, rank, barrier, max_over_ranks, clocks):
    """Speculative decoding: the target (tensor parallel over all ranks) verifies `spec_width` tokens drafted by a
    llama-draft model that runs on every rank (TP=1); acceptance is forced by a seeded Bernoulli(0.7) mask so that the
    full verify compute always runs; the comparison is target-only decoding of the same batch on the same box."""
    import torch
    from sllm_b200.engine.engine import build_engine
    from sllm_b200.engine.speculative import ExternalDraftProvider, SpeculativeDecoder
    from sllm_b200.models import config as mc
    eng = build_engine(cfg, device, seed=0, max_batch=args.batch, tp=tp)
    dcfg = mc.NAMED["llama-draft"]()
    dcfg.max_context = cfg.max_context
    deng = build_engine(dcfg, device, seed=7, max_batch=args.batch)
    g = torch.Generator().manual_seed(1234)
    prompts = torch.randint(0, cfg.vocab, (args.batch, args.prompt), generator=g).tolist()

    def fresh():
        seqs = [eng.new_sequence(p) for p in prompts]
        for i in range(0, args.batch, 8):
            for s, t in zip(seqs[i:i + 8], eng.prefill(seqs[i:i + 8])):
                s.tokens.append(t)
        return seqs

    # target-only reference on the same box
    seqs = fresh()
    for _ in range(args.warmup):
        for s, t in zip(seqs, eng.decode(seqs)):
            s.tokens.append(t)
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    barrier()
    e0.record()
    for _ in range(args.steps):
        for s, t in zip(seqs, eng.decode(seqs)):
            s.tokens.append(t)
    e1.record()
    barrier()
    base_ms = max_over_ranks(e0.elapsed_time(e1))
    for s in seqs:
        eng.free_sequence(s)
    # speculative
    dec = SpeculativeDecoder(eng, ExternalDraftProvider(deng, args.spec_width, cfg.vocab), args.spec_width, forced_accept_p=0.7,
                             seed=99)
    seqs = fresh()
    for _ in range(args.warmup):
        dec.step(seqs)
    if rank == 0:
        clocks.start()
    emitted0 = dec.acct.emitted
    barrier()
    e0.record()
    for _ in range(args.steps):
        dec.step(seqs)
    e1.record()
    barrier()
    ms = max_over_ranks(e0.elapsed_time(e1))
    clk = clocks.stop() if rank == 0 else None
    tokens = dec.acct.emitted - emitted0
    if rank == 0:
        value = tokens / (ms / 1e3)
        base = args.batch * args.steps / (base_ms / 1e3)
        print(json.dumps({
            "metric": "speculative_decode_output_tokens_per_s", "value": round(value, 2), "unit": "tok/s", "n_gpus": args.gpus,
            "steps": args.steps, "warmup": args.warmup, "ms_per_step": round(ms / args.steps, 4), "higher_is_better": True,
            "scaling": "strong", "vs_baseline": round(value / REFERENCE_PUBLISHED_TOK_S, 2), "dtype": f"{args.weights} target, bf16 draft",
            "data": "synthetic: seeded uniform-random prompts, random-init weights; acceptance forced by a seeded Bernoulli(0.7) mask",
            "config": {"model": f"{cfg.name}-{args.weights}", "draft": "llama-draft-bf16", "global_batch": args.batch,
                       "seq_len": args.prompt, "draft_width": args.spec_width, "parallelism": f"target tp{args.gpus}, draft tp1"},
            "clocks": clk, "target_only_tok_s": round(base, 2), "speedup_vs_target_only": round(value / base, 3),
            "acceptance": dec.acct.to_dict(), "gpu_launches": int(eng.kernel_launches + deng.kernel_launches), "impl": "own"}))
    sys.stdout.flush()
    if world > 1:
        torch.cuda.synchronize()
        if tp is not None:
            tp.close()
        import torch.distributed as dist
        dist.barrier()
        dist.destroy_process_group()
        os._exit(0)
    return 0


def model_forward_rows(model, tokens, row0: int, start: int):
    """Prefill of a group of rows into their slice of the contiguous KV cache."""
    k_full, v_full = model.k, model.v
    n = tokens.shape[0]
    model.k = [k[row0:row0 + n] for k in k_full]
    model.v = [v[row0:row0 + n] for v in v_full]
    try:
        return model.forward(tokens, start)
    finally:
        model.k, model.v = k_full, v_full


def _estimate_weight_bytes(cfg) -> float:
    """Resident weight bytes of a dense decoder of this shape in its weight format (embedding and head included)."""
    per = {"fp32": 4.0, "bf16": 2.0, "fp8": 1.0 + 4.0 / 128, "nvfp4": 0.5 + 1.0 / 16, "mxfp4": 0.5 + 1.0 / 32}.get(cfg.weight_format, 2.0)
    d = cfg.d_model
    layer = (cfg.q_size + 2 * cfg.kv_size) * d + d * cfg.q_size + 3 * cfg.ffn * d
    return cfg.n_layers * layer * per + (1 if cfg.tie_embeddings else 2) * cfg.vocab * d * per


def main():
    args = parse_args()
    if args.impl == "reference":
        return run_reference(args)
    if args.impl == "torch":
        return run_torch_baseline(args)

    import torch
    import torch.distributed as dist

    world = int(os.environ.get("WORLD_SIZE", "1"))
    rank = int(os.environ.get("RANK", "0"))
    local_rank = int(os.environ.get("LOCAL_RANK", "0"))
    if world != args.gpus and world > 1:
        raise SystemExit(f"--gpus {args.gpus} but WORLD_SIZE={world}")
    torch.cuda.set_device(local_rank)
    device = torch.device("cuda", local_rank)
    if world > 1:
        os.environ.setdefault("MASTER_ADDR", "127.0.0.1")
        dist.init_process_group("nccl", device_id=device)

    from sllm_b200 import build
    build.build_all()
    from sllm_b200.engine.engine import build_engine
    from sllm_b200.models import config as mc
    from sllm_b200.ops import _lib

    if args.compare:
        import importlib
        module = {"zokuvik": "family_bench", "sepedra": "sepedra_bench", "kegorax": "kegorax_bench",
                  "fekolorn": "fekolorn_bench"}[args.compare]
        return importlib.import_module(f"sllm_b200.utils.{module}").main(args)
    if args.act4:
        from sllm_b200.ops import w4 as _w4
        _w4.set_w4a4(True)
    cfg = mc.NAMED[args.model]()
    if cfg.family != "moe":
        cfg.weight_format, cfg.kv_format = args.weights or "fp8", args.kv or "fp8"
    else:
        cfg.weight_format, cfg.kv_format = args.weights or cfg.weight_format, args.kv or cfg.kv_format
    args.weights, args.kv = cfg.weight_format, cfg.kv_format
    if args.layers > 0:
        cfg.n_layers = args.layers
        cfg.name += f"-{args.layers}layers-PROFILING-ONLY"
    total_ctx = args.prompt + args.warmup + 2 * args.steps + 64
    cfg.max_context = ((total_ctx + 255) // 256) * 256
    weight_gib = _estimate_weight_bytes(cfg) / 2 ** 30
    layout = args.parallelism
    if layout == "dp" and (world == 1 or args.batch % world or cfg.family == "moe"):
        layout = "tp"
    also_replicas = (layout == "tp" and world > 1 and cfg.family != "moe" and weight_gib < 16 and args.batch % world == 0
                     and args.spec_width == 0 and not args.no_replica_run)
    replicas = world if layout == "dp" else 1
    tp = None
    if world > 1 and layout == "tp":
        from sllm_b200.parallel.tp import make_tp
        tp = make_tp(world, rank, device, impl=args.tp_impl, max_tokens=max(args.batch, 128), d_model=cfg.d_model)
    ep = None
    if world > 1 and layout == "tp" and cfg.family == "moe":
        from sllm_b200.parallel.ep import FusedEP, NcclEP
        ep = FusedEP(world, rank, device, max(args.batch, 128), cfg.d_model) if args.tp_impl == "fused" \
            else NcclEP(world, rank, device)

    def barrier():
        if world > 1:
            dist.barrier()
        torch.cuda.synchronize()

    def max_over_ranks(ms: float) -> float:
        if world == 1:
            return ms
        t = torch.tensor([ms], device=device, dtype=torch.float64)
        dist.all_reduce(t, op=dist.ReduceOp.MAX)
        return float(t.item())

    def measure(batch: int, steps: int, warmup: int, sample_clocks: bool, sharded: bool = True):
        eng = build_engine(cfg, device, seed=0, max_batch=batch, tp=tp if sharded else None, ep=ep if sharded else None)
        g = torch.Generator().manual_seed(1234)
        prompts = torch.randint(0, cfg.vocab, (batch, args.prompt), generator=g).tolist()
        seqs = [eng.new_sequence(p) for p in prompts]
        # ---- prefill (TTFT), in groups of 8 sequences to bound activation memory
        barrier()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        if args.synthetic_kv:
            for s in seqs:
                eng.cache.pool.reserve(s.seq_id, len(s.tokens))
                eng.cache.pool.commit(s.seq_id, len(s.tokens))
                s.num_computed = len(s.tokens)
                s.tokens.append(int(s.tokens[-1]))
        else:
            for i in range(0, batch, 8):
                grp = seqs[i:i + 8]
                first = eng.prefill(grp)
                for s, t in zip(grp, first):
                    s.tokens.append(t)
        e1.record()
        barrier()
        prefill_ms = max_over_ranks(e0.elapsed_time(e1))
        # ---- warm-up through the public API (captures the CUDA graph)
        for _ in range(warmup):
            toks = eng.decode(seqs)
            for s, t in zip(seqs, toks):
                s.tokens.append(t)
        clocks = ClockSampler(local_rank)
        if sample_clocks and rank == 0:
            clocks.start()
        # ---- end-to-end: K calls of Engine.decode (pinned H2D of inputs + D2H of tokens every step)
        h2d0, d2h0, l0 = eng.h2d_bytes, eng.d2h_bytes, eng.kernel_launches
        barrier()
        t0 = time.perf_counter()
        e0.record()
        for _ in range(steps):
            toks = eng.decode(seqs)
            for s, t in zip(seqs, toks):
                s.tokens.append(t)
        e1.record()
        barrier()
        e2e_wall_ms = (time.perf_counter() - t0) * 1e3
        e2e_ms = max_over_ranks(max(e0.elapsed_time(e1), e2e_wall_ms))
        h2d = (eng.h2d_bytes - h2d0) / steps
        d2h = (eng.d2h_bytes - d2h0) / steps
        launches_per_step = (eng.kernel_launches - l0) // steps
        # ---- device-only: K graph replays with on-device token feedback
        n = eng._padded(batch)
        pool = eng.cache.pool
        for s in seqs:
            pool.reserve(s.seq_id, len(s.tokens) + steps + 1)
        pool.fill_block_table([s.seq_id for s in seqs], eng.h_table)
        eng.d_table[:batch].copy_(eng.h_table[:batch])
        eng._table_key = None
        graph = eng._graphs[(n, True)]
        barrier()
        e0.record()
        for _ in range(steps):
            eng.d_tokens[:n].copy_(eng.d_out[:n])
            eng.d_positions[:n].add_(1)
            eng.d_kv_lens[:n].add_(1)
            graph.replay()
        e1.record()
        barrier()
        dev_ms = max_over_ranks(e0.elapsed_time(e1))
        clk = clocks.stop() if (sample_clocks and rank == 0) else None
        status = int(__import__("sllm_b200").ops.device_status(device))
        for s in seqs:
            eng.free_sequence(s)
        res = dict(batch=batch, prefill_ms=prefill_ms, e2e_ms=e2e_ms, dev_ms=dev_ms, h2d=h2d, d2h=d2h,
                   launches_per_step=launches_per_step, clocks=clk, status=status)
        del eng
        torch.cuda.empty_cache()
        return res

    if args.spec_width > 0:
        return run_speculative(args, cfg, device, tp, world, rank, barrier, max_over_ranks, ClockSampler(local_rank))
    # data parallel: every rank is a replica decoding its share of the sequences; the step time is the slowest rank's
    main_res = measure(args.batch // replicas, args.steps, args.warmup, True)
    replica_res = measure(args.batch // world, args.steps, args.warmup, False, sharded=False) if also_replicas else None
    extra = None
    if not args.no_batch1 and args.batch != 1:
        extra = measure(1, min(args.steps, 64), max(3, min(args.warmup, 4)), False)

    if rank == 0:
        k = args.steps
        value = args.batch * k / (main_res["dev_ms"] / 1e3)
        e2e_value = args.batch * k / (main_res["e2e_ms"] / 1e3)
        out = {
            "metric": "decode_output_tokens_per_s",
            "value": round(value, 2),
            "unit": "tok/s",
            "n_gpus": args.gpus,
            "steps": k,
            "warmup": args.warmup,
            "ms_per_step": round(main_res["dev_ms"] / k, 4),
            "higher_is_better": True,
            "scaling": "strong",
            "vs_baseline": round(value / REFERENCE_PUBLISHED_TOK_S, 2),
            "vs_baseline_denominator": "56.62 tok/s: the reference's published FP8 decode rate (Qwen3.5-4B, one request, "
                                       "MI300X); another model, batch and GPU, so context rather than a like-for-like ratio",
            "dtype": ("fp8_e4m3_block128_weights+fp8_kv (bf16 activations, fp32 accumulate)" if args.weights == "fp8" else
                      f"{args.weights} weights ({cfg.expert_format} experts) + {args.kv} kv, bf16 activations, fp32 accumulate"
                      if cfg.family == "moe" else f"{args.weights} weights + {args.kv} kv, bf16 activations, fp32 accumulate") +
                     ("; 4-bit GEMMs take 4-bit block-scaled activations (W4A4)" if args.act4 else ""),
            "data": "synthetic: seeded uniform-random prompts, seeded N(0,0.02) random-init weights" +
                    ("; KV pages of the prompt marked computed without a prefill (decode-only measurement)"
                     if args.synthetic_kv else ""),
            "config": {"model": f"{cfg.name}-{args.weights}", "global_batch": args.batch,
                       "seq_len": args.prompt, "output_tokens": k, "kv_cache": f"{args.kv}-paged-16",
                       "parallelism": (f"dp{args.gpus}" if layout == "dp" else
                                       (f"tp{args.gpus}+ep{args.gpus}" if cfg.family == "moe" else f"tp{args.gpus}") +
                                       (f"-{args.tp_impl}" if args.gpus > 1 else "")),
                       "parallelism_note": ("one replica per GPU, each decoding global_batch / N sequences; launches and "
                                            "copied bytes are job totals" if layout == "dp" else
                                            "one model sharded over the GPUs"),
                       "l2": "each step streams the full weight set (>> 126 MB L2); no flush needed"},
            "clocks": main_res["clocks"],
            "e2e": {"value": round(e2e_value, 2), "unit": "tok/s", "ms_per_step": round(main_res["e2e_ms"] / k, 4),
                    "h2d_bytes_per_step": int(main_res["h2d"]) * replicas, "d2h_bytes_per_step": int(main_res["d2h"]) * replicas,
                    "api": "sllm_b200.engine.Engine.decode"},
            "gpu_launches": int(main_res["launches_per_step"] * k) * replicas,
            "ttft_ms_batch_prefill": round(main_res["prefill_ms"], 2),
            "itl_ms": round(main_res["e2e_ms"] / k, 4),
            "device_status": main_res["status"],
            "fallbacks": _lib.fallbacks(),
            "impl": "own",
        }
        if replica_res is not None:
            kk = args.steps
            out["replica_layout"] = {
                "parallelism": f"dp{args.gpus}",
                "note": "the same global batch as one replica per GPU, each decoding global_batch / N sequences; no "
                        "communication inside a step; launches and copied bytes are job totals",
                "value": round(args.batch * kk / (replica_res["dev_ms"] / 1e3), 2), "unit": "tok/s",
                "ms_per_step": round(replica_res["dev_ms"] / kk, 4),
                "e2e": {"value": round(args.batch * kk / (replica_res["e2e_ms"] / 1e3), 2), "unit": "tok/s",
                        "h2d_bytes_per_step": int(replica_res["h2d"]) * world, "d2h_bytes_per_step": int(replica_res["d2h"]) * world},
                "gpu_launches": int(replica_res["launches_per_step"] * kk) * world, "device_status": replica_res["status"]}
        if extra:
            ks = min(args.steps, 64)
            out["batch1"] = {"tok_s_device": round(ks / (extra["dev_ms"] / 1e3), 2),
                             "tok_s_e2e": round(ks / (extra["e2e_ms"] / 1e3), 2),
                             "ttft_ms": round(extra["prefill_ms"], 2)}
        print(json.dumps(out))
    sys.stdout.flush()
    if world > 1:
        torch.cuda.synchronize()
        if ep is not None:
            ep.close()
        if tp is not None:
            tp.close()
        dist.barrier()
        dist.destroy_process_group()
        os._exit(0)
    return 0


if __name__ == "__main__":
    sys.exit(main())
