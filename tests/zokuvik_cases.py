"""Small Zokuvik configurations with random weights, written as model folders, and their oracle weights."""
from __future__ import annotations

import json
import os
import struct

import torch

import zokuvik_oracle as O


def latent(ff, *, heads, dim, rot, vdim, rank, q_rank, scale=None, base=1e4):
    return {"type": "latent_attention", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "q_rank": q_rank,
                      "scale": scale or (dim + rot) ** -0.5, "rot": {"base": base, "dims": rot}}}


def windowed(ff, *, heads, dim, rot, vdim, rank, window, scale=None, base=1e4):
    return {"type": "latent_attention_2", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "mask": {"size": window},
                      "scale": scale or (dim + rot) ** -0.5, "rot": {"base": base, "dims": rot}}}


def delta(ff, *, heads, dim):
    return {"type": "general_delta", "mlp": None if ff is None else {"kind": "dense", "ff": ff}, "mixer": {"heads": heads, "dim": dim}}


def config(layers, *, width, vocab, groups=1, eps=1e-6):
    return {"architecture": "Zokuvik", "width": width, "vocab": vocab, "norm": {"eps": eps, "groups": groups}, "layers": layers}


# sizes that are uneven on purpose: head counts of 1, 3 and 5, no power of two, a group count that does not divide 8,
# norms with one group, a model whose first layer has no feed-forward
CASES = {
    "mixed": config([latent(72, heads=3, dim=16, rot=24, vdim=40, rank=48, q_rank=56, base=3e3),
                     delta(None, heads=3, dim=24),
                     windowed(88, heads=5, dim=24, rot=8, vdim=16, rank=64, window=19, scale=0.21, base=7e2)],
                    width=96, vocab=211, groups=3, eps=1e-5),
    "delta-first": config([delta(64, heads=1, dim=33), windowed(None, heads=1, dim=8, rot=16, vdim=8, rank=24, window=1),
                           delta(40, heads=2, dim=56), latent(56, heads=4, dim=8, rot=2, vdim=24, rank=16, q_rank=24)],
                          width=80, vocab=96),
    "odd": config([windowed(36, heads=2, dim=10, rot=6, vdim=14, rank=20, window=40), delta(20, heads=3, dim=10),
                   latent(None, heads=2, dim=6, rot=10, vdim=18, rank=28, q_rank=22)], width=60, vocab=77, groups=5),
    "wide-heads": config([latent(96, heads=2, dim=128, rot=64, vdim=128, rank=256, q_rank=96),
                          windowed(96, heads=2, dim=64, rot=64, vdim=104, rank=136, window=70),
                          delta(None, heads=1, dim=128)], width=128, vocab=128, groups=2),
}


def random_weights(cfg: dict, seed: int, rank: int = 12) -> dict:
    """name -> fp32 tensor whose values are bf16 numbers."""
    g = torch.Generator().manual_seed(seed)
    d = cfg["width"]
    w: dict = {}

    def put(name, *shape, std=None):
        x = torch.randn(shape, generator=g)
        if std is None:
            std = shape[-1] ** -0.5
        w[name] = (x * std).to(torch.bfloat16).float()

    def norm(name, n):
        w[name] = (1 + 0.3 * torch.randn(n, generator=g)).to(torch.bfloat16).float()

    put("embed", cfg["vocab"], d, std=1.0)
    for i, e in enumerate(cfg["layers"]):
        p, q, m = f"l{i}.", f"l{i}.mix.", e["mixer"]
        norm(p + "norm1", d)
        norm(p + "norm1b", d)
        H, D = m["heads"], m["dim"]
        if e["type"] == "general_delta":
            for x in ("r", "k", "v", "a", "g"):
                put(q + x, H * D, d)
            put(q + "w1", rank, d)
            put(q + "w2", H * D, rank, std=1.0)
            put(q + "w0", H * D, std=1.5)
            put(q + "a.b", H * D, std=1.0)
            norm(q + "norm", H * D)
            put(q + "o", d, H * D)
        else:
            R, V, C = m["rot_dim"], m["vdim"], m["kv_rank"]
            if "q_rank" in m:
                put(q + "dq", m["q_rank"], d)
                norm(q + "dq.norm", m["q_rank"])
                put(q + "uq", H * (D + R), m["q_rank"], std=2 * m["q_rank"] ** -0.5)
                put(q + "g", H, d)
            else:
                put(q + "q", H * (D + R), d, std=2 * d ** -0.5)
            put(q + "dkv", C + R, d)
            norm(q + "dkv.norm", C)
            put(q + "uk", H * D, C)
            put(q + "uv", H * V, C)
            put(q + "o", d, H * V)
        if e["mlp"] is not None:
            norm(p + "norm2", d)
            norm(p + "norm2b", d)
            put(p + "mlp.up", e["mlp"]["ff"], d)
            put(p + "mlp.down", d, e["mlp"]["ff"])
    norm("final.norm", d)
    put("head", cfg["vocab"], d)
    return w


def write_folder(path, cfg: dict, w: dict) -> str:
    path = str(path)
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    head, blobs, off = {}, [], 0
    for name, t in w.items():
        raw = t.to(torch.bfloat16).contiguous().view(torch.int16).numpy().tobytes()
        head[name] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [off, off + len(raw)]}
        blobs.append(raw)
        off += len(raw)
    h = json.dumps(head).encode()
    with open(os.path.join(path, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h + b"".join(blobs))
    return path


class Case:
    """A model folder, its oracle, and engines of it."""

    def __init__(self, tmp, name: str, seed: int = 0, cfg: dict = None, weights: dict = None):
        self.cfg = cfg or CASES[name]
        self.w = weights or random_weights(self.cfg, seed)
        self.path = write_folder(os.path.join(str(tmp), name), self.cfg, self.w)
        self.w64 = {k: v.double() for k, v in self.w.items()}

    def engine(self, device, dtype, max_tokens=512, max_seqs=4, graphs=True):
        from sllm_b200.engine.engine import load_engine
        return load_engine(self.path, device, dtype, max_tokens=max_tokens, max_batch=4, max_seqs=max_seqs, use_cuda_graphs=graphs)

    def oracle(self, tokens) -> torch.Tensor:
        return O.forward(tokens, self.cfg, self.w64)

    def prompt(self, n: int, seed: int) -> list:
        g = torch.Generator().manual_seed(1000 + seed)
        return torch.randint(0, self.cfg["vocab"], (n,), generator=g).tolist()


TOL = {"fp32": 3e-5, "bf16": 9e-2}          # rms of the logit difference over the rms of the logits


def error(got: torch.Tensor, want: torch.Tensor) -> float:
    d = got.double().cpu() - want
    return float((d.pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt()).max())


def run_cut(engine, tokens: list, cuts: list) -> torch.Tensor:
    """Logits of every position of one request fed in portions of the given sizes (the last size repeats)."""
    s = engine.new_sequence([])
    out, at, k = [], 0, 0
    while at < len(tokens):
        n = min(cuts[min(k, len(cuts) - 1)], len(tokens) - at)
        s.tokens.extend(tokens[at:at + n])
        out.append(engine.step([s], [list(range(n))]).double().cpu())
        at, k = at + n, k + 1
    engine.free_sequence(s)
    return torch.cat(out)
