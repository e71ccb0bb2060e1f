"""Small Fekolorn configurations with random weights, written as model folders, and their oracle weights."""
from __future__ import annotations

import os

import torch

import fekolorn_oracle as O
from zokuvik_cases import error, run_cut, write_folder          # noqa: F401  (shared helpers of the folder-based families)


def dense(ff):
    return {"kind": "dense", "ff": ff}


def _att(att, scale):
    heads, kv_heads, dim, vdim = att
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or 1.5 * dim ** -0.5}


def attention(mlp, *, att, window, far, v_mix=True, scale=None):
    """att: (heads, kv_heads, dim, vdim)."""
    return {"type": "attention", "mlp": mlp, "mixer": dict(_att(att, scale), mask={"size": window}, bias_max=far, v_mix=v_mix)}


def parallel(mlp, *, att, delta, conv, rot, base=3e3, scales=(0.8, 0.6), scale=None):
    """delta: (heads, kv_heads, dim, vdim) of the recurrence."""
    left = dict(_att(att, scale), rot={"base": base, "dims": rot})
    right = dict(zip(("heads", "kv_heads", "dim", "vdim"), delta), conv=conv)
    return {"type": "parallel", "mlp": mlp, "mixer": {"left": left, "right": right, "left_scale": scales[0], "right_scale": scales[1]}}


def config(layers, *, width, vocab, streams, eps=1e-5, scale=3.0, bigram=(53, 31, 7)):
    return {"architecture": "Fekolorn", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers, "streams": streams,
            "embedding": {"scale": scale, "bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))}}


# sizes that are uneven on purpose: keys and values of different widths, partial and no rotation, filters of 1, 2, 3 and 5 taps,
# heads that no vector access fits, layers without feed-forward, with and without mixed values, biases that reach further than the
# window and less far, one, two, three, four and six streams
CASES = {
    "mixed": config([parallel(dense(72), att=(4, 2, 24, 16), delta=(4, 2, 12, 20), conv=3, rot=12),
                     attention(dense(40), att=(6, 2, 20, 24), window=19, far=30),
                     attention(None, att=(4, 2, 16, 24), window=26, far=9),
                     parallel(None, att=(3, 1, 12, 12), delta=(3, 1, 12, 12), conv=2, rot=4, scales=(1.0, -0.5)),
                     attention(dense(36), att=(5, 1, 12, 8), window=7, far=12, v_mix=False)], width=56, vocab=211, streams=3),
    "odd": config([attention(dense(37), att=(3, 3, 7, 9), window=9, far=5),
                   parallel(dense(18), att=(5, 5, 6, 10), delta=(3, 1, 7, 9), conv=5, rot=0),
                   parallel(None, att=(2, 1, 10, 5), delta=(1, 1, 33, 5), conv=1, rot=6),
                   attention(None, att=(3, 1, 5, 27), window=1, far=8)], width=61, vocab=77, streams=1, scale=1.0, bigram=(1, 3, 5)),
    "wide": config([parallel(dense(160), att=(4, 2, 128, 128), delta=(4, 2, 64, 128), conv=4, rot=64),
                    attention(dense(200), att=(4, 1, 64, 64), window=70, far=130),
                    attention(dense(136), att=(2, 2, 128, 32), window=40, far=32)], width=128, vocab=128, streams=4),
    "grouped": config([attention(dense(88), att=(8, 1, 72, 40), window=33, far=100),
                       parallel(None, att=(8, 4, 64, 64), delta=(6, 3, 40, 24), conv=2, rot=64, base=5e5),
                       attention(dense(48), att=(12, 2, 48, 20), window=50, far=64)], width=96, vocab=100, streams=2, bigram=(999, 1, 1)),
    "states": config([parallel(dense(64), att=(2, 1, 136, 40), delta=(2, 2, 136, 40), conv=4, rot=128),
                      parallel(dense(80), att=(2, 2, 16, 16), delta=(2, 1, 16, 160), conv=2, rot=2)], width=72, vocab=90, streams=6),
    "windows": config([attention(dense(56), att=(2, 1, 32, 32), window=24, far=20, v_mix=False),
                       attention(dense(56), att=(4, 4, 16, 16), window=11, far=300)], width=40, vocab=64, streams=2),
}
BIAS_ROWS = {"mixed": 16, "odd": 6, "grouped": 32, "windows": 10}


def random_weights(cfg: dict, seed: int, rows: int = 12) -> dict:
    """name -> fp32 tensor whose values are bf16 numbers; ``rows``: of every distance-bias table."""
    g = torch.Generator().manual_seed(seed)
    d, n = cfg["width"], cfg["streams"]
    w: dict = {}

    def put(name, *shape, std=None, mean=0.0):
        x = torch.randn(shape, generator=g)
        w[name] = (mean + x * (shape[-1] ** -0.5 if std is None else std)).to(torch.bfloat16).float()

    def connection(name):
        put(name + ".in", n, std=0.3, mean=1.0 / n)
        put(name + ".out", n, std=0.3, mean=0.8)
        put(name + ".mix", n, n, std=0.2)
        w[name + ".mix"] = (w[name + ".mix"] + 0.9 * torch.eye(n)).to(torch.bfloat16).float()

    put("embed", cfg["vocab"], d, std=0.7)
    put("bigram", cfg["embedding"]["bigram"]["buckets"] + 1, d, std=0.7)
    for i, e in enumerate(cfg["layers"]):
        p, q, m = f"l{i}.", f"l{i}.mix.", e["mixer"]
        put(p + "norm1", std=0.2, mean=1.0)
        connection(p + "hc1")
        l, a = (q, m) if e["type"] == "attention" else (q + "left.", m["left"])
        H, G = a["heads"], a["kv_heads"]
        for x, r in (("q", H * a["dim"]), ("k", G * a["dim"]), ("v", G * a["vdim"])):
            put(l + x, r, d)
        put(l + "sink", H, std=1.5)
        put(l + "o", d, H * a["vdim"])
        if e["type"] == "attention":
            put(q + "q.norm", H * a["dim"], std=0.3, mean=1.0)
            put(q + "k.norm", G * a["dim"], std=0.3, mean=1.0)
            put(q + "rel", rows, H, std=1.0)
            if m["v_mix"]:
                put(q + "vmix", std=0.1, mean=0.4)
        else:
            r, s = q + "right.", m["right"]
            H, G, D, V = s["heads"], s["kv_heads"], s["dim"], s["vdim"]
            for x, k in (("q", G * D), ("k", G * D), ("v", H * V)):
                put(r + x, k, d)
                put(f"{r}{x}.conv", k, s["conv"], std=0.7)
            put(r + "a", H, d)
            put(r + "b", H, d)
            put(r + "A_log", H, std=0.7)
            put(r + "dt_bias", H, std=1.0, mean=-2.0)
            put(r + "norm", V, std=0.3, mean=1.0)
            put(r + "g", H * V, d)
            put(r + "o", d, H * V)
        if e["mlp"] is not None:
            ff = e["mlp"]["ff"]
            put(p + "norm2", std=0.2, mean=1.0)
            connection(p + "hc2")
            put(p + "mlp.up", ff, d)
            put(p + "mlp.down", d, ff)
            put(p + "mlp.act", 4, std=0.5)
    put("final.norm", std=0.2, mean=1.0)
    put("head", cfg["vocab"], d)
    return w


class Case:
    """A model folder, its oracle, and engines of it."""

    def __init__(self, tmp, name: str, seed: int = 0, cfg: dict = None, weights: dict = None):
        self.cfg = cfg or CASES[name]
        self.w = weights or random_weights(self.cfg, seed, BIAS_ROWS.get(name, 12))
        self.path = write_folder(os.path.join(str(tmp), name), self.cfg, self.w)
        self.w64 = {k: v.double() for k, v in self.w.items()}
        self._known: dict = {}

    def engine(self, device, dtype, max_tokens=512, max_seqs=4, graphs=True):
        from sllm_b200.engine.engine import load_engine
        return load_engine(self.path, device, dtype, max_tokens=max_tokens, max_batch=4, max_seqs=max_seqs, use_cuda_graphs=graphs)

    def oracle(self, tokens) -> torch.Tensor:
        key = tuple(tokens)
        if key not in self._known:
            self._known[key] = O.forward(tokens, self.cfg, self.w64)
        return self._known[key]

    def prompt(self, n: int, seed: int) -> list:
        g = torch.Generator().manual_seed(1000 + seed)
        return torch.randint(0, self.cfg["vocab"], (n,), generator=g).tolist()


TOL = {"fp32": 5e-5, "bf16": 9e-2}          # rms of the logit difference over the rms of the logits


def agrees(got: torch.Tensor, want: torch.Tensor, dtype: str) -> bool:
    return error(got, want) < TOL[dtype]
