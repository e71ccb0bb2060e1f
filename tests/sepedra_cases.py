"""Small Sepedra configurations with random weights, written as model folders, and their oracle weights."""
from __future__ import annotations

import os

import torch

import sepedra_oracle as O
from zokuvik_cases import error, run_cut, write_folder          # noqa: F401  (shared helpers of the folder-based families)


def moe(*, experts, top, ff, limit=2.5, count=1, keep=1):
    r = {"experts": experts, "top": top}
    if count > 1:
        r["groups"] = {"count": count, "keep": keep}
    return {"kind": "moe", "router": r, "expert": {"ff": ff, "limit": limit}}


def rglru(mlp, *, width, blocks, conv=4):
    return {"type": "rglru", "mlp": mlp, "mixer": {"width": width, "blocks": blocks, "conv": conv}}


SCALING = {"factor": 6.0, "low": 1.0, "high": 3.0, "original": 96}


def attention(mlp, *, heads, kv_heads, dim, vdim, rot, conv=4, scale=None, base=5e3, scaling=SCALING, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "scale": scale or 2.0 * dim ** -0.5,
         "rot": {"base": base, "dims": rot}}
    if scaling is not None:
        m["rot"]["scaling"] = scaling
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mlp": mlp, "mixer": m}


def config(layers, *, width, vocab, eps=1e-5, cap=20.0):
    return {"architecture": "Sepedra", "width": width, "vocab": vocab, "norm": {"eps": eps}, "logit_softcap": cap, "layers": layers}


# sizes that are uneven on purpose: keys and values of different widths, partial rotation, filters of 1, 2, 3 and 5 taps,
# blocks that no vector access fits, one expert, layers without experts, keys shared over several layers
_ATT = dict(heads=6, kv_heads=2, dim=20, vdim=24, rot=12, conv=3)
_TALL = dict(heads=4, kv_heads=2, dim=128, vdim=128, rot=128)
_EIGHT = dict(heads=8, kv_heads=1, dim=64, vdim=64, rot=32)
CASES = {
    "mixed": config([rglru(moe(experts=6, top=2, ff=40, count=3, keep=2), width=72, blocks=3, conv=3),
                     attention(moe(experts=4, top=3, ff=24, limit=0.7), **_ATT), attention(None, kv_from=1, **_ATT),
                     rglru(moe(experts=8, top=3, ff=72, count=2, keep=1), width=48, blocks=2)], width=56, vocab=211),
    "odd": config([attention(None, heads=3, kv_heads=3, dim=10, vdim=14, rot=6, conv=5, scaling=None),
                   rglru(moe(experts=5, top=1, ff=18), width=21, blocks=3, conv=2), rglru(None, width=35, blocks=1, conv=1),
                   attention(moe(experts=1, top=1, ff=30, limit=1.1), heads=1, kv_heads=1, dim=6, vdim=18, rot=2, conv=1)],
                  width=60, vocab=77, cap=9.0),
    "wide": config([rglru(moe(experts=16, top=4, ff=96, count=4, keep=2), width=320, blocks=2),
                    attention(moe(experts=12, top=5, ff=136, count=6, keep=3), **_TALL), rglru(None, width=256, blocks=1, conv=2),
                    attention(moe(experts=3, top=2, ff=64), kv_from=1, **_TALL)], width=128, vocab=128),
    "grouped": config([attention(moe(experts=9, top=2, ff=48, count=3, keep=1), **_EIGHT), attention(None, kv_from=0, **_EIGHT),
                       rglru(None, width=64, blocks=8, conv=3), attention(None, kv_from=0, **_EIGHT),
                       attention(moe(experts=7, top=7, ff=64), heads=3, kv_heads=1, dim=72, vdim=40, rot=8, conv=2)],
                      width=96, vocab=100, cap=40.0),
    # no attention at all; a filter and a block beyond the tensor-core form of the recurrence; no soft cap
    "states": config([rglru(None, width=64, blocks=1, conv=6), rglru(moe(experts=6, top=2, ff=80, count=2, keep=1), width=264, blocks=1)],
                     width=72, vocab=90, cap=None),
}


CODE = 8             # leading channels of the residual that keep the token's embedding


def _decide_routes(cfg: dict, w: dict, g: torch.Generator) -> None:
    """Makes every routing decision a clear one: no sublayer writes the first channels (their norm weights are zero), the
    routers read only those, and a token's values there are drawn again until no choice of any layer is close.  (With a close
    call, two correct computations may use different experts, and everything after that token differs.)"""
    routers = [(w[f"l{i}.mlp.router"], e["mlp"]["router"]) for i, e in enumerate(cfg["layers"]) if e["mlp"] is not None]
    for name, t in w.items():
        if ".norm" in name and name != "final.norm":
            t[:CODE] = 0
    for t, _ in routers:
        t[:, CODE:] = 0
        t *= 4

    def clear(code):
        for t, r in routers:
            z, gr = t[:, :CODE].double() @ code.double(), r.get("groups") or {"count": 1, "keep": 1}
            best = z.view(gr["count"], -1).max(-1).values
            order = torch.sort(best, descending=True).values
            if gr["keep"] < gr["count"]:
                if order[gr["keep"] - 1] - order[gr["keep"]] < 0.02:
                    return False
                shut = (best < order[gr["keep"] - 1]).repeat_interleave(z.numel() // gr["count"])
                z = z.masked_fill(shut, float("-inf"))
            order = torch.sort(z, descending=True).values
            if r["top"] < z.numel() and order[r["top"] - 1] - order[r["top"]] < 0.02:
                return False
        return True

    for row in w["embed"]:
        while not clear(row[:CODE]):
            row[:CODE] = torch.randn(CODE, generator=g).to(torch.bfloat16).float()


def random_weights(cfg: dict, seed: int, clear_routes: bool = True) -> dict:
    """name -> fp32 tensor whose values are bf16 numbers."""
    g = torch.Generator().manual_seed(seed)
    d = cfg["width"]
    w: dict = {}

    def put(name, *shape, std=None, mean=0.0):
        x = torch.randn(shape, generator=g)
        w[name] = (mean + x * (shape[-1] ** -0.5 if std is None else std)).to(torch.bfloat16).float()

    put("embed", cfg["vocab"], d, std=1.0)
    for i, e in enumerate(cfg["layers"]):
        p, q, m = f"l{i}.", f"l{i}.mix.", e["mixer"]
        put(p + "norm1", d, std=0.3, mean=1.0)
        if e["type"] == "rglru":
            n, b = m["width"], m["width"] // m["blocks"]
            for x in ("y", "x"):
                put(q + x, n, d)
                put(q + x + ".b", n, std=0.3)
            put(q + "conv", n, m["conv"], std=0.7)
            put(q + "conv.b", n, std=0.3)
            for x in ("ra", "ri"):
                put(q + x, m["blocks"], b, b, std=2 * b ** -0.5)
                put(q + x + ".b", m["blocks"], b, std=0.5)
            put(q + "lam", n, std=1.5, mean=-4.0)
            put(q + "o", d, n)
        else:
            rows = {"q": m["heads"] * m["dim"], "k": m["kv_heads"] * m["dim"], "v": m["kv_heads"] * m["vdim"]}
            for x in ("q",) if "kv_from" in m else ("q", "k", "v"):
                put(q + x, rows[x], d)
                put(q + x + ".conv", rows[x], m["conv"], std=0.7)
            put(q + "g", m["heads"] * m["vdim"], d)
            put(q + "o", d, m["heads"] * m["vdim"])
        if e["mlp"] is not None:
            put(p + "norm2", d, std=0.3, mean=1.0)
            ff, E = e["mlp"]["expert"]["ff"], e["mlp"]["router"]["experts"]
            put(p + "mlp.router", E, d, std=2 * d ** -0.5)
            for k in range(E):
                for x, shape in (("gate", (ff, d)), ("up", (ff, d)), ("down", (d, ff))):
                    put(f"{p}mlp.e{k}.{x}", *shape)
    put("final.norm", d, std=0.3, mean=1.0)
    put("head", cfg["vocab"], d, std=6 * d ** -0.5)
    if clear_routes:
        _decide_routes(cfg, w, g)
    return w


class Case:
    """A model folder, its oracle, and engines of it."""

    def __init__(self, tmp, name: str, seed: int = 0, cfg: dict = None, weights: dict = None):
        self.cfg = cfg or CASES[name]
        self.w = weights or random_weights(self.cfg, seed)
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


TOL = {"fp32": 3e-5, "bf16": 9e-2}          # rms of the logit difference over the rms of the logits


def agrees(got: torch.Tensor, want: torch.Tensor, dtype: str) -> bool:
    return error(got, want) < TOL[dtype]
