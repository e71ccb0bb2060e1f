"""Small Kegorax configurations with random weights, written as model folders, and their oracle weights."""
from __future__ import annotations

import os

import torch

import kegorax_oracle as O
from zokuvik_cases import error, run_cut, write_folder          # noqa: F401  (shared helpers of the folder-based families)


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(*, experts, top, ff, scale=1.7, count=1, keep=1):
    r = {"experts": experts, "top": top, "scale": scale}
    if count > 1:
        r["groups"] = {"count": count, "keep": keep}
    return {"kind": "moe", "router": r, "expert": {"ff": ff}}


def _left(att, scale):
    heads, kv_heads, dim, vdim = att
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or 1.5 * dim ** -0.5}


def parallel(mlp, *, att, chunk, lin, rot, base=3e3, tau=8.0, scale=None):
    """att: (heads, kv_heads, dim, vdim) of the attention; lin: (heads, dim, vdim) of the recurrence."""
    left = dict(_left(att, scale), mask={"size": chunk}, rot={"base": base, "dims": rot})
    return {"type": "parallel", "mlp": mlp, "mixer": {"left": left, "right": dict(zip(("heads", "dim", "vdim"), lin), tau=tau)}}


def parallel_2(mlp, *, att, window, keep, ret, decay, scales=(0.8, 0.6), scale=None):
    left = dict(_left(att, scale), mask={"size": window, "keep_first": keep})
    right = dict(zip(("heads", "dim", "vdim"), ret), decay=decay)
    return {"type": "parallel_2", "mlp": mlp, "mixer": {"left": left, "right": right, "left_scale": scales[0], "right_scale": scales[1]}}


def delta(mlp, *, heads, kv_heads, dim, vdim, conv):
    return {"type": "channel_delta", "mlp": mlp, "mixer": dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv)}


def config(layers, *, width, vocab, loop=None, eps=1e-5, scale=3.0):
    c = {"architecture": "Kegorax", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


# sizes that are uneven on purpose: keys and values of different widths, partial and no rotation, filters of 1, 2, 3 and 5 taps,
# heads that no vector access fits, one expert, layers without feed-forward, blocks at the start, in the middle, at the end, of
# one layer, of one pass, and none
CASES = {
    "mixed": config([parallel_2(dense(72), att=(6, 2, 20, 24), window=19, keep=3, ret=(3, 12, 20), decay=[0.8, 0.95, 0.995]),
                     parallel(moe(experts=6, top=2, ff=40, count=3, keep=2), att=(4, 2, 24, 16), chunk=21, lin=(2, 20, 12), rot=12),
                     delta(None, heads=4, kv_heads=2, dim=12, vdim=20, conv=3),
                     parallel(None, att=(3, 1, 12, 12), chunk=17, lin=(3, 12, 12), rot=4, tau=2.0)], width=56, vocab=211, loop=(1, 3, 3)),
    "odd": config([delta(dense(36), heads=3, kv_heads=1, dim=7, vdim=9, conv=5),
                   parallel_2(moe(experts=5, top=1, ff=18, scale=0.6), att=(3, 3, 10, 14), window=9, keep=0, ret=(1, 10, 6), decay=[1.0],
                              scales=(1.0, -0.5)),
                   parallel(moe(experts=1, top=1, ff=30), att=(5, 5, 6, 18), chunk=10, lin=(5, 6, 10), rot=0),
                   delta(None, heads=1, kv_heads=1, dim=33, vdim=5, conv=1)], width=60, vocab=77, scale=1.0),
    "wide": config([delta(moe(experts=16, top=4, ff=96, count=4, keep=2), heads=4, kv_heads=2, dim=64, vdim=128, conv=4),
                    parallel_2(dense(160), att=(4, 2, 128, 128), window=70, keep=20, ret=(2, 128, 64), decay=[0.9, 0.999]),
                    parallel(moe(experts=12, top=5, ff=136, count=6, keep=3), att=(4, 1, 64, 64), chunk=96, lin=(2, 64, 136), rot=32)],
                   width=128, vocab=128, loop=(1, 3, 2)),
    "grouped": config([parallel(dense(88), att=(8, 1, 64, 64), chunk=50, lin=(1, 24, 40), rot=64, tau=16.0),
                       parallel_2(None, att=(8, 4, 72, 40), window=33, keep=40, ret=(4, 16, 16), decay=[0.5, 0.9, 0.99, 0.9999]),
                       delta(moe(experts=9, top=2, ff=48, count=3, keep=1), heads=6, kv_heads=3, dim=40, vdim=24, conv=2)],
                      width=96, vocab=100, loop=(0, 1, 4)),
    # no attention; one pass
    "states": config([delta(dense(64), heads=2, kv_heads=2, dim=136, vdim=40, conv=4),
                      delta(moe(experts=6, top=3, ff=80, count=2, keep=1), heads=2, kv_heads=1, dim=16, vdim=160, conv=2)],
                     width=72, vocab=90, loop=(1, 2, 1)),
}


CODE = 8             # leading channels of the residual that keep the token's embedding


def _decide_routes(cfg: dict, w: dict, g: torch.Generator) -> None:
    """Makes every routing decision a clear one: no sublayer writes the first channels, the routers read only those, and a token's
    values there are large (so that a norm's divisor hangs mostly on them) and drawn again until no choice of any layer is close
    for the divisors that can occur.  (With a close call, two correct computations may use different experts, and everything
    after that token differs.)"""
    d = cfg["width"]
    routers = [(i, e["mlp"]["router"]) for i, e in enumerate(cfg["layers"]) if e["mlp"] is not None and e["mlp"]["kind"] == "moe"]
    for name, t in w.items():
        if name.endswith((".o", ".down")):
            t[:CODE] = 0
    if "loop.step" in w:
        w["loop.step"][:, :CODE] = 0
    w["final.norm"][:CODE] = 0
    for i, _ in routers:
        w[f"l{i}.mlp.router"][:, CODE:] = 0

    def clear(code):
        top = (d / float((code.double() ** 2).sum())) ** 0.5
        for i, r in routers:
            gr = r.get("groups") or {"count": 1, "keep": 1}
            picks = set()
            for c in (0.4, 0.5, 0.6, 0.7, 0.8, 0.9, 1.0):
                z = (w[f"l{i}.mlp.router"][:, :CODE].double() * w[f"l{i}.norm2"][:CODE].double()) @ (c * top * code.double())
                s = torch.sigmoid(z) + w[f"l{i}.mlp.correction"].double()
                best = s.view(gr["count"], -1)
                best = best.topk(min(2, best.shape[1]), -1).values.sum(-1)
                order = torch.sort(best, descending=True).values
                if gr["keep"] < gr["count"]:
                    if order[gr["keep"] - 1] - order[gr["keep"]] < 0.01:
                        return False
                    s = s.masked_fill((best < order[gr["keep"] - 1]).repeat_interleave(s.numel() // gr["count"]), float("-inf"))
                order = torch.sort(s, descending=True)
                if r["top"] < s.numel() and order.values[r["top"] - 1] - order.values[r["top"]] < 0.01:
                    return False
                picks.add(tuple(sorted(order.indices[:r["top"]].tolist())))
            if len(picks) > 1:
                return False
        return True

    for row in w["embed"]:
        for _ in range(20000):
            row[:CODE] = (4 * torch.randn(CODE, generator=g)).to(torch.bfloat16).float()
            if clear(row[:CODE]):
                break
        else:
            raise AssertionError("no clear code")


def random_weights(cfg: dict, seed: int, clear_routes: bool = True, rank: int = 12) -> dict:
    """name -> fp32 tensor whose values are bf16 numbers."""
    g = torch.Generator().manual_seed(seed)
    d = cfg["width"]
    w: dict = {}

    def put(name, *shape, std=None, mean=0.0):
        x = torch.randn(shape, generator=g)
        w[name] = (mean + x * (shape[-1] ** -0.5 if std is None else std)).to(torch.bfloat16).float()

    put("embed", cfg["vocab"], d, std=0.7)
    if "loop" in cfg:
        put("loop.step", cfg["loop"]["times"], d, std=0.7)
    for i, e in enumerate(cfg["layers"]):
        p, q, m = f"l{i}.", f"l{i}.mix.", e["mixer"]
        put(p + "norm1", d, std=0.3, mean=1.0)
        r, sm = (q, m) if e["type"] == "channel_delta" else (q + "right.", m["right"])
        H, D, V = sm["heads"], sm["dim"], sm["vdim"]
        G = sm.get("kv_heads", H)
        for x, n in (("q", G * D), ("k", G * D), ("v", H * V)):
            put(r + x, n, d)
            if e["type"] == "channel_delta":
                put(f"{r}{x}.conv", n, m["conv"], std=0.7)
        put(r + "o", d, H * V)
        if e["type"] == "channel_delta":
            for x, n in (("a", H * D), ("g", H * V)):
                put(f"{r}{x}1", rank + (x == "g"), d)
                put(f"{r}{x}2", n, rank + (x == "g"), std=0.5)
            put(r + "b", H, d)
            put(r + "A_log", H, std=0.7)
            put(r + "dt_bias", H * D, std=1.0, mean=-2.0)
            put(r + "norm", V, std=0.3, mean=1.0)
        else:
            put(r + "g", H * V, d)
            l, a = q + "left.", m["left"]
            rows = {"q": a["heads"] * a["dim"], "k": a["kv_heads"] * a["dim"], "v": a["kv_heads"] * a["vdim"]}
            for x in ("q", "k", "v"):
                put(l + x, rows[x], d)
            put(l + "o", d, a["heads"] * a["vdim"])
            if e["type"] == "parallel":
                put(r + "a1", rank, d)
                put(r + "a2", H * D, rank, std=0.5)
                put(r + "a2.b", H * D, std=1.0, mean=1.0)
                put(r + "norm", V, std=0.3, mean=1.0)
                put(l + "sink", a["heads"], std=1.5)
                put(l + "g", a["heads"], d)
                put(l + "out", d, std=0.3, mean=1.0)
                put(r + "out", d, std=0.3, mean=1.0)
            else:
                for x in ("q", "k", "v"):
                    put(f"{l}{x}.b", rows[x], std=0.5)
                put(l + "q.norm", a["dim"], std=0.3, mean=1.0)
                put(l + "k.norm", a["dim"], std=0.3, mean=1.0)
        if e["mlp"] is None:
            continue
        put(p + "norm2", d, std=0.3, mean=1.0)
        if e["mlp"]["kind"] == "dense":
            ff = e["mlp"]["ff"]
            put(p + "mlp.gate", ff, d)
            put(p + "mlp.up", ff, d)
            put(p + "mlp.down", d, ff)
            continue
        ff, E = e["mlp"]["expert"]["ff"], e["mlp"]["router"]["experts"]
        put(p + "mlp.router", E, d, std=0.25)
        put(p + "mlp.correction", E, std=0.2)
        for k in range(E):
            for x, shape in (("gate", (ff, d)), ("up", (ff, d)), ("down", (d, ff))):
                put(f"{p}mlp.e{k}.{x}", *shape)
    put("final.norm", d, std=0.3, mean=1.0)
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


TOL = {"fp32": 5e-5, "bf16": 9e-2}          # rms of the logit difference over the rms of the logits


def agrees(got: torch.Tensor, want: torch.Tensor, dtype: str) -> bool:
    return error(got, want) < TOL[dtype]
