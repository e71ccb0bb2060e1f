"""`trace_run`: replays a trace of token ids through a model folder's engine, step by step, and writes logits.

Standard input holds one JSON object a line:
    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["b"]}
A step runs the tokens it brings, all entries as one batch (`Engine.step`); the logits of the wanted places go to
<out>/<step>.f32 as little-endian fp32 [wanted, vocab]; requests named in `end` give their pages and state slot back.
After every step a line `done <step>` is printed.  Nothing is sampled.  Runs on the GPU only.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

MAX_LIVE = 4                 # requests that hold a state slot at any time
DTYPES = {"bfloat16": "bf16", "float32": "fp32"}


class TraceError(RuntimeError):
    pass


class TraceSession:
    def __init__(self, engine, out_dir: str):
        self.engine, self.out_dir = engine, out_dir
        self.live: dict = {}

    def run(self, rec: dict) -> int:
        """One step; returns its number."""
        import numpy as np
        n = int(rec["step"])
        seqs, wanted, seen = [], [], set()
        for e in rec["entries"]:
            rid, toks = str(e["id"]), [int(t) for t in e["tokens"]]
            if rid in seen:
                raise TraceError(f"step {n}: request {rid!r} appears twice")
            if not toks or any(not 0 <= t < self.engine.cfg.vocab for t in toks):
                raise TraceError(f"step {n}: request {rid!r}: no tokens, or a token outside the vocabulary")
            seen.add(rid)
            s = self.live.get(rid)
            if s is None:
                s = self.live[rid] = self.engine.new_sequence([])
            s.tokens.extend(toks)
            seqs.append(s)
            wanted.append([int(p) for p in e["want"]])
        if seqs:
            logits = self.engine.step(seqs, wanted)
            if any(wanted):
                data = logits.float().cpu().numpy().astype("<f4")
                tmp = os.path.join(self.out_dir, f".{n}.part")
                with open(tmp, "wb") as f:
                    f.write(np.ascontiguousarray(data).tobytes())
                os.replace(tmp, os.path.join(self.out_dir, f"{n}.f32"))
        for rid in rec.get("end", ()):
            s = self.live.pop(str(rid), None)
            if s is None:
                raise TraceError(f"step {n}: unknown request {rid!r} in end")
            self.engine.free_sequence(s)
        return n


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", required=True, choices=sorted(DTYPES))
    ap.add_argument("--out", required=True, help="folder for the logits of each step")
    ap.add_argument("--max-tokens", required=True, type=int, help="tokens that live requests hold together at any time")
    a = ap.parse_args(argv)
    import torch
    from .. import build
    from ..engine.engine import load_engine
    from ..models import registry
    from ..ops import _lib
    cfg = registry.read_folder_config(a.model, dtype=DTYPES[a.dtype])
    if a.max_tokens < 1:
        raise TraceError("--max-tokens must be positive")
    if not torch.cuda.is_available():
        raise TraceError("no CUDA device is available")
    build.build_host()
    build.build_family(cfg.family)
    _lib.set_fail_closed(True)
    step_tokens = (a.max_tokens + 63) // 64 * 64
    engine = load_engine(a.model, "cuda:0", DTYPES[a.dtype], max_tokens=step_tokens, max_batch=MAX_LIVE, max_seqs=MAX_LIVE)
    session = TraceSession(engine, a.out)
    for line in sys.stdin:
        if line.strip():
            n = session.run(json.loads(line))
            sys.stdout.write(f"done {n}\n")
            sys.stdout.flush()
    return 0
