"""Kegorax: a decoder whose configuration lists its layers one by one, each layer with sizes of its own, and may run a block
of them several times in a row with the same weights.

  parallel        attention inside chunks of positions (rotary half-split pairs, learned sink, output gate per head) beside
                  gated linear attention; both outputs are normed and averaged
  parallel_2      windowed attention with kept first positions (biases, query / key norms, distance slopes, one added to the
                  denominator) beside retention; a weighted sum
  channel_delta   delta rule with a decay per key channel, short convolutions on q, k and v, low-rank output gate

x <- x + mixer(norm1(x)), x <- x + ff(norm2(x)); the feed-forward is a gated GELU layer, routed experts chosen by corrected
sigmoid scores from the best groups, or absent.  Before each pass of the block a vector of its own joins the residual, before
each but the first the embedding as well; every pass has its own pages and states.  The residual is 32-bit.  All of a
layer's input projections are one GEMM; every addition to the residual, with what a pass adds and the next sublayer's norm,
is one launch (ops.add_group_norm).  The output matrix is the embedding.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Callable, Iterator, Optional

import torch

from .. import ops
from ..engine.batch import ForwardBatch
from ..ops import kv_attention as A
from ..ops import linear_state as S
from ..ops import moe as M
from ..ops.core import LinearWeight
from .config import ModelConfig
from .llama import NoTP
from .packing import SourceTensors

ARCHITECTURE = "Kegorax"
MIXERS = ("parallel", "parallel_2", "channel_delta")
GROUP_TOP = 2                              # a group of experts scores the sum of this many of its largest choice scores
MAX_EXPERTS, MAX_TOP = 256, 32


# ------------------------------------------------------------------------------------------ configuration
def attention_spec(entry: dict) -> Optional[A.KVSpec]:
    if entry["type"] == "channel_delta":
        return None
    m, chunked = entry["mixer"]["left"], entry["type"] == "parallel"
    heads, kv_heads, dim, vdim = (int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
    if heads < 1 or kv_heads < 1 or heads % kv_heads or dim < 1 or vdim < 1:
        raise ValueError("attention: positive sizes, and kv_heads must divide heads")
    size = int(m["mask"]["size"])
    if size < 1:
        raise ValueError("attention: mask.size must be positive")
    kw = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=float(m["scale"]), interleaved=False, gate_heads=True)
    if not chunked:
        keep = int(m["mask"].get("keep_first") or 0)
        if keep < 0:
            raise ValueError("attention: mask.keep_first must not be negative")
        return A.KVSpec(rot_base=1.0, rot_dims=0, window=size, keep_first=keep, **kw)
    dims = int(m["rot"]["dims"])
    if dims % 2 or not 0 <= dims <= dim:
        raise ValueError("attention: rot.dims must be even and at most dim")
    return A.KVSpec(rot_base=float(m["rot"]["base"]), rot_dims=dims, chunk=size, qk_norm=False, **kw)


def _state_mixer(entry: dict) -> dict:
    return entry["mixer"] if entry["type"] == "channel_delta" else entry["mixer"]["right"]


def state_sizes(entry: dict) -> tuple:
    """(heads, query / key heads, dim, vdim) of a layer's recurrence."""
    m = _state_mixer(entry)
    heads, dim, vdim = (int(m[k]) for k in ("heads", "dim", "vdim"))
    kv_heads = int(m["kv_heads"]) if entry["type"] == "channel_delta" else heads
    if min(heads, kv_heads, dim, vdim) < 1 or heads % kv_heads:
        raise ValueError("recurrence: positive sizes, and kv_heads must divide heads")
    if entry["type"] == "channel_delta" and int(m["conv"]) < 1:
        raise ValueError("channel_delta: conv must be positive")
    if entry["type"] == "parallel" and not float(m["tau"]) > 0:
        raise ValueError("parallel: tau must be positive")
    if entry["type"] == "parallel_2" and len(m["decay"]) != heads:
        raise ValueError("parallel_2: one decay per head")
    return heads, kv_heads, dim, vdim


@dataclass
class MoeSpec:
    """Sizes and constants of one layer's experts."""
    experts: int
    top: int
    ff: int
    scale: float
    groups: int = 1
    keep: int = 1


def moe_spec(entry: dict) -> Optional[MoeSpec]:
    m = entry["mlp"]
    if m is None or m["kind"] == "dense":
        return None
    if m["kind"] != "moe":
        raise ValueError(f"unknown feed-forward kind {m['kind']!r}")
    r, g = m["router"], m["router"].get("groups") or {"count": 1, "keep": 1}
    s = MoeSpec(int(r["experts"]), int(r["top"]), int(m["expert"]["ff"]), float(r["scale"]), int(g["count"]), int(g["keep"]))
    if not 1 <= s.experts <= MAX_EXPERTS or not 1 <= s.top <= min(s.experts, MAX_TOP):
        raise ValueError(f"experts: 1 to {MAX_EXPERTS}, of which a token uses 1 to {MAX_TOP}")
    if s.groups < 1 or s.experts % s.groups or not 1 <= s.keep <= s.groups or s.keep * (s.experts // s.groups) < s.top:
        raise ValueError("expert groups: count must divide the experts, and the kept groups must hold `top` of them")
    return s


def layer_runs(layers: int, loop: Optional[dict]) -> list:
    """[(layer, pass)] in running order; ``pass`` is the number of the loop's pass on its first layer, else None."""
    if loop is None:
        return [(i, None) for i in range(layers)]
    a, z = loop["start"], loop["stop"]
    out = [(i, None) for i in range(a)]
    for t in range(loop["times"]):
        out += [(i, t if i == a else None) for i in range(a, z)]
    return out + [(i, None) for i in range(z, layers)]


def config_from_source(d: dict, name: str = "kegorax", dtype: str = "bf16", max_context: int = 8192) -> ModelConfig:
    """ModelConfig of a parsed config.json."""
    if d.get("architecture") != ARCHITECTURE:
        raise ValueError(f"architecture {d.get('architecture')!r} is not {ARCHITECTURE}")
    entries = d["layers"]
    loop = d.get("loop")
    if loop is not None:
        loop = {k: int(loop[k]) for k in ("start", "stop", "times")}
        if not 0 <= loop["start"] < loop["stop"] <= len(entries) or loop["times"] < 1:
            raise ValueError("loop: start < stop within the layers, and at least one pass")
    cfg = ModelConfig(name=name, family="kegorax", n_layers=len(entries), d_model=int(d["width"]), vocab=int(d["vocab"]),
                      rms_eps=float(d["norm"]["eps"]), embedding_scale=float(d["embedding"]["scale"]), tie_embeddings=True,
                      layer_specs=entries, layer_loop=loop, weight_format=dtype, kv_format=dtype, max_context=max_context, n_kv_heads=1)
    for e in entries:
        if e["type"] not in MIXERS:
            raise ValueError(f"unknown mixer type {e['type']!r}")
        s, moe = attention_spec(e), moe_spec(e)
        state_sizes(e)
        if s is not None:
            cfg.n_heads, cfg.n_kv_heads, cfg.head_dim = s.heads, s.kv_heads, s.dim
        if moe is not None:
            cfg.n_experts, cfg.top_k, cfg.expert_ffn = moe.experts, moe.top, moe.ff
        elif e["mlp"] is not None:
            cfg.ffn = max(cfg.ffn if cfg.ffn != ModelConfig.ffn else 0, int(e["mlp"]["ff"]))
    return cfg


def source_shapes(cfg: ModelConfig, rank: Callable[[str], int]) -> dict:
    """name -> shape of every source tensor; ``rank(name)`` is the inner size of the low-rank product whose first factor has that
    name (the only sizes that the configuration does not carry)."""
    d = cfg.d_model
    out = {"embed": (cfg.vocab, d)}
    if cfg.layer_loop is not None:
        out["loop.step"] = (cfg.layer_loop["times"], d)
    for i, e in enumerate(cfg.layer_specs):
        p, q = f"l{i}.", f"l{i}.mix."
        out[p + "norm1"] = (d,)
        H, G, D, V = state_sizes(e)
        r = q if e["type"] == "channel_delta" else q + "right."
        out[r + "q"], out[r + "k"], out[r + "v"], out[r + "o"] = (G * D, d), (G * D, d), (H * V, d), (d, H * V)
        if e["type"] != "parallel_2":
            ra = rank(r + "a1")
            out[r + "a1"], out[r + "a2"], out[r + "norm"] = (ra, d), (H * D, ra), (V,)
        if e["type"] == "channel_delta":
            rg, taps = rank(r + "g1"), int(e["mixer"]["conv"])
            for x in ("q", "k", "v"):
                out[f"{r}{x}.conv"] = (out[r + x][0], taps)
            out[r + "g1"], out[r + "g2"] = (rg, d), (H * V, rg)
            out[r + "b"], out[r + "A_log"], out[r + "dt_bias"] = (H, d), (H,), (H * D,)
        else:
            out[r + "g"] = (H * V, d)
            s, l = attention_spec(e), q + "left."
            out[l + "q"], out[l + "k"], out[l + "v"] = (s.q_cols, d), (s.kv_heads * s.dim, d), (s.kv_heads * s.vdim, d)
            out[l + "o"] = (d, s.out_cols)
            if e["type"] == "parallel":
                out[r + "a2.b"] = (H * D,)
                out[l + "sink"], out[l + "g"] = (s.heads,), (s.heads, d)
                out[l + "out"] = out[r + "out"] = (d,)
            else:
                for x in ("q", "k", "v"):
                    out[f"{l}{x}.b"] = (out[l + x][0],)
                out[l + "q.norm"] = out[l + "k.norm"] = (s.dim,)
        if e["mlp"] is None:
            continue
        moe = moe_spec(e)
        out[p + "norm2"] = (d,)
        if moe is None:
            ff = int(e["mlp"]["ff"])
            out[p + "mlp.gate"], out[p + "mlp.up"], out[p + "mlp.down"] = (ff, d), (ff, d), (d, ff)
        else:
            out[p + "mlp.router"], out[p + "mlp.correction"] = (moe.experts, d), (moe.experts,)
            for k in range(moe.experts):
                x = f"{p}mlp.e{k}."
                out[x + "gate"], out[x + "up"], out[x + "down"] = (moe.ff, d), (moe.ff, d), (d, moe.ff)
    out["final.norm"] = (d,)
    return out


# ------------------------------------------------------------------------------------------ resident weights
@dataclass
class KegoraxLayer:
    norm1: torch.Tensor                        # vectors are fp32
    in_proj: LinearWeight                      # all projections of the layer's input; every part starts at a multiple of 8 rows
    rows: list                                 # [(source name after "mix.", first row, rows)] of in_proj
    state: S.StateSpec
    sw: S.StateWeights
    o: LinearWeight                            # of the recurrence
    a_log: Optional[torch.Tensor] = None
    attn: Optional[A.KVSpec] = None
    gate_col: int = -1                         # first column of the attention's output gate (-1: none)
    o_attn: Optional[LinearWeight] = None
    inv_freq: Optional[torch.Tensor] = None
    bias: Optional[torch.Tensor] = None        # [channels of q | k | v]
    q_norm: Optional[torch.Tensor] = None
    k_norm: Optional[torch.Tensor] = None
    sinks: Optional[torch.Tensor] = None       # [heads]: scores that join the denominator only
    slopes: Optional[torch.Tensor] = None
    attn_out: Optional[torch.Tensor] = None    # norms of the two outputs (None: they join as they are)
    state_out: Optional[torch.Tensor] = None
    attn_coef: float = 0.0
    state_coef: float = 1.0
    norm2: Optional[torch.Tensor] = None
    gate_up: Optional[LinearWeight] = None
    down: Optional[LinearWeight] = None
    moe: Optional[MoeSpec] = None
    router: Optional[LinearWeight] = None
    scores: Optional[M.SigmoidScores] = None
    bank: Optional[M.ExpertBank] = None


@dataclass
class KegoraxWeights:
    embed: torch.Tensor
    layers: list
    final_norm: torch.Tensor
    lm_head: LinearWeight                      # the embedding
    steps: Optional[torch.Tensor] = None       # fp32 [passes, width]
    vocab_offset: int = 0


def pack_weights(cfg: ModelConfig, get: Callable, device) -> KegoraxWeights:
    """``get(name)`` returns a source tensor (any float type, any device)."""
    device = torch.device(device)
    src = SourceTensors(cfg, get, source_shapes(cfg, lambda n: int(get(n).shape[0])), device)
    shapes, fetch, raw, mat, vec, taps = src.shapes, src.fetch, src.raw, src.mat, src.vec, src.taps
    layers = []
    for i, e in enumerate(cfg.layer_specs):
        p, q = f"l{i}.", f"l{i}.mix."
        H, G, D, V = state_sizes(e)
        m = _state_mixer(e)
        kw: dict = dict(norm1=vec(p + "norm1"))
        if e["type"] == "channel_delta":
            in_proj, rows = src.packed(q, [["q", "k", "v"], ["b"], ["a1"], ["g1"]])
            r, at = "", {n: a for n, a, _ in rows}
            kw["a_log"] = vec(q + "A_log")
            sw = S.StateWeights(w_a=src.second_factor(q + "a2"), w_g=src.second_factor(q + "g2"), bias=vec(q + "dt_bias"),
                                rate=torch.exp(kw["a_log"].double()).float(), conv_w=taps(*(f"{q}{x}.conv" for x in ("q", "k", "v"))),
                                norm=vec(q + "norm"))
            st = S.StateSpec(S.DELTA, H, G, D, V, {"q": at["q"], "k": at["k"], "v": at["v"], "g": at["g1"], "a": at["a1"], "b": at["b"]},
                             q_scale=D ** -0.5, taps=int(m["conv"]), rank_a=shapes[q + "a1"][0], rank_g=shapes[q + "g1"][0])
        else:
            chunked, r = e["type"] == "parallel", "right."
            parts = [["left.q", "left.k", "left.v"]] + ([["left.g"]] if chunked else []) + [[r + x] for x in ("q", "k", "v", "g")]
            in_proj, rows = src.packed(q, parts + ([[r + "a1"]] if chunked else []))
            at = {n: a for n, a, _ in rows}
            cols = {x: at[r + x] for x in ("q", "k", "v", "g")}
            s = attention_spec(e)
            kw.update(attn=s, o_attn=mat(q + "left.o"))
            if chunked:
                sw = S.StateWeights(w_a=src.second_factor(q + r + "a2"), bias=vec(q + r + "a2.b"), norm=vec(q + r + "norm"))
                st = S.StateSpec(S.GATED, H, H, D, V, dict(cols, a=at[r + "a1"]), q_scale=D ** -0.5, tau=float(m["tau"]),
                                 rank_a=shapes[q + r + "a1"][0])
                kw.update(gate_col=at["left.g"], inv_freq=s.inv_freq(device), sinks=vec(q + "left.sink"), attn_out=vec(q + "left.out"),
                          state_out=vec(q + r + "out"), attn_coef=0.5, state_coef=0.5)
            else:
                sw = S.StateWeights(rate=torch.tensor([float(x) for x in m["decay"]], device=device))
                st = S.StateSpec(S.FIXED, H, H, D, V, cols, k_scale=D ** -0.5)
                kw.update(bias=vec(*(f"{q}left.{x}.b" for x in ("q", "k", "v"))), q_norm=vec(q + "left.q.norm"), k_norm=vec(q + "left.k.norm"),
                          sinks=torch.zeros(s.heads, device=device), slopes=A.distance_slopes(s.heads, device),
                          attn_coef=float(e["mixer"]["left_scale"]), state_coef=float(e["mixer"]["right_scale"]))
        kw.update(in_proj=in_proj, rows=rows, state=st, sw=sw, o=mat(q + r + "o"))
        moe = moe_spec(e)
        if e["mlp"] is not None:
            kw["norm2"] = vec(p + "norm2")
        if moe is not None:
            part = lambda x: [raw(f"{p}mlp.e{k}.{x}") for k in range(moe.experts)]
            kw.update(moe=moe, router=mat(p + "mlp.router"), scores=M.SigmoidScores(vec(p + "mlp.correction"), moe.scale),
                      bank=M.ExpertBank.pack(part("gate"), part("up"), part("down"), M.GatedAct()))
        elif e["mlp"] is not None:
            kw.update(gate_up=mat(p + "mlp.gate", p + "mlp.up"), down=mat(p + "mlp.down"))
        layers.append(KegoraxLayer(**kw))
    embed = raw("embed").contiguous()
    steps = None if cfg.layer_loop is None else fetch("loop.step").to(device=device, dtype=torch.float32).contiguous()
    return KegoraxWeights(embed, layers, vec("final.norm"), LinearWeight("dense", embed), steps)


def named_tensors(cfg: ModelConfig, w: KegoraxWeights) -> Iterator:
    """(source name, tensor) of every tensor: the inverse of ``pack_weights``."""
    yield "embed", w.embed
    if w.steps is not None:
        yield "loop.step", w.steps
    for i, (e, l) in enumerate(zip(cfg.layer_specs, w.layers)):
        p, q = f"l{i}.", f"l{i}.mix."
        yield p + "norm1", l.norm1
        for name, r0, n in l.rows:
            yield q + name, l.in_proj.w[r0:r0 + n]
        s, sw, delta = l.state, l.sw, e["type"] == "channel_delta"
        r = q if delta else q + "right."
        yield r + "o", l.o.w
        if s.form != S.FIXED:
            yield r + "a2", sw.w_a.w[:, :s.rank_a]
            yield r + ("dt_bias" if delta else "a2.b"), sw.bias
            yield r + "norm", sw.norm
        if delta:
            yield r + "g2", sw.w_g.w[:, :s.rank_g]
            yield r + "A_log", l.a_log
            c0 = 0
            for x, n in (("q", s.kv_heads * s.dim), ("k", s.kv_heads * s.dim), ("v", s.out_cols)):
                yield f"{r}{x}.conv", sw.conv_w[:, c0:c0 + n].t().contiguous()
                c0 += n
        else:
            yield q + "left.o", l.o_attn.w
            if s.form == S.GATED:
                yield q + "left.sink", l.sinks
                yield q + "left.out", l.attn_out
                yield r + "out", l.state_out
            else:
                a = l.attn
                for x, b in zip(("q", "k", "v"), l.bias.split([a.q_cols, a.kv_heads * a.dim, a.kv_heads * a.vdim])):
                    yield f"{q}left.{x}.b", b
                yield q + "left.q.norm", l.q_norm
                yield q + "left.k.norm", l.k_norm
        if l.norm2 is not None:
            yield p + "norm2", l.norm2
        if l.moe is not None:
            yield p + "mlp.router", l.router.w
            yield p + "mlp.correction", l.scores.correction
            for k in range(l.moe.experts):
                for name, t in zip(("gate", "up", "down"), l.bank.matrices(k)):
                    yield f"{p}mlp.e{k}.{name}", t
        elif l.gate_up is not None:
            ff = l.down.w.shape[1]
            yield p + "mlp.gate", l.gate_up.w[:ff]
            yield p + "mlp.up", l.gate_up.w[ff:]
            yield p + "mlp.down", l.down.w
    yield "final.norm", w.final_norm


def init_random_kegorax_weights(cfg: ModelConfig, device, seed: int = 0, rank: int = 64) -> KegoraxWeights:
    """Seeded weights of the configured shape, drawn tensor by tensor on the target device (a generator per tensor, so the
    order of use does not matter): matrices ~N(0, 1 / fan-in), norms near 1, decays mostly between 0.9 and 1."""
    device = torch.device(device)
    shapes = source_shapes(cfg, lambda n: rank)
    index = {n: k for k, n in enumerate(shapes)}

    def get(name):
        shape = shapes[name]
        gen = torch.Generator(device=device)
        gen.manual_seed(seed * 100003 + index[name])
        x = torch.randn(shape, generator=gen, device=device, dtype=torch.float32)
        if ".norm" in name or name.endswith(".out"):
            return 1.0 + 0.05 * x
        if name.endswith("dt_bias"):
            return x - 3.0
        if name.endswith("A_log"):
            return 0.5 * x
        if name.endswith("a2.b"):
            return x + 1.0
        if name.endswith(".sink"):
            return x
        if name.endswith(".b") and len(shape) == 1 or name.endswith("correction") or name == "loop.step":
            return 0.1 * x
        return x * shape[-1] ** -0.5
    return pack_weights(cfg, get, device)


# ------------------------------------------------------------------------------------------ model
@dataclass
class _Run:
    """One run of a layer: what follows it on the residual."""
    layer: KegoraxLayer
    after: Optional[torch.Tensor]              # norm of the next run's input
    again: bool = False                        # the next run starts a pass: its vector joins,
    embed: bool = False                        # and the embedding
    step: Optional[torch.Tensor] = field(default=None)


class KegoraxModel:
    """Stateless forward over a ForwardBatch; pages and states (one set per run of a layer) live in the KVLayeredCache passed
    in."""

    def __init__(self, cfg: ModelConfig, weights: KegoraxWeights, tp=None):
        if tp is not None and tp.size != 1:
            raise ValueError("the kegorax family runs on one GPU")
        self.cfg, self.w = cfg, weights
        self.tp = tp or NoTP()
        self.dtype = weights.embed.dtype
        order = layer_runs(cfg.n_layers, cfg.layer_loop)
        self.first_step = None if order[0][1] is None else weights.steps[order[0][1]]
        self.runs: list = []
        for j, (i, _) in enumerate(order):
            nxt, t = order[j + 1] if j + 1 < len(order) else (None, None)
            self.runs.append(_Run(weights.layers[i], None if nxt is None else weights.layers[nxt].norm1, t is not None,
                                  t is not None and t > 0, None if t is None else weights.steps[t]))

    @property
    def local_kv_heads(self) -> int:
        return self.cfg.n_kv_heads

    def _attention(self, proj, lw: KegoraxLayer, j: int, b: ForwardBatch, cache):
        s, kv = lw.attn, cache.layer(j)
        q = A.prepare(proj, s, None, lw.inv_freq, self.cfg.rms_eps, kv, None, b, bias=lw.bias, q_norm=lw.q_norm, k_norm=lw.k_norm)
        gate = None if lw.gate_col < 0 else proj[:, lw.gate_col:lw.gate_col + s.heads]
        return ops.linear(A.attention(q, gate, s, kv, lw.sinks, b, lw.slopes), lw.o_attn)

    def _recurrence(self, proj, lw: KegoraxLayer, j: int, b: ForwardBatch, cache):
        ring = cache.state(j, 1) if lw.state.form == S.DELTA else None
        return ops.linear(S.linear_state(proj, lw.state, lw.sw, self.cfg.rms_eps, cache.state(j), ring, b), lw.o)

    def hidden(self, b: ForwardBatch, cache) -> torch.Tensor:
        cfg, w, eps = self.cfg, self.w, self.cfg.rms_eps
        if b.row_off is None or b.slots is None:
            raise ValueError("the kegorax family needs row offsets and state slots in the batch")
        if b.embeds is not None:
            raise ValueError("the kegorax family takes token ids only")
        x, z = ops.embed_group_norm(w.embed, b.tokens, self.runs[0].layer.norm1 if self.runs else None, eps, scale=cfg.embedding_scale,
                                    step=self.first_step)
        for j, run in enumerate(self.runs):
            lw = run.layer
            again = None
            if run.again:
                again = ops.Again(w.embed, b.tokens, cfg.embedding_scale, run.step) if run.embed else ops.Again(step=run.step)
            proj = ops.linear(z, lw.in_proj)
            y = self._recurrence(proj, lw, j, b, cache)
            out = dict(w_out=lw.norm2) if lw.norm2 is not None else dict(w_out=run.after, again=again)
            if lw.attn is not None:
                ya = self._attention(proj, lw, j, b, cache)
                z = ops.add_group_norm(x, ya, lw.attn_out, eps=eps, coef=lw.attn_coef, second=(y, lw.state_out, lw.state_coef), **out)
            else:
                z = ops.add_group_norm(x, y, None, eps=eps, **out)
            if lw.norm2 is None:
                continue
            if lw.moe is not None:
                m = lw.moe
                idx, wt = M.router(z, lw.router, m.top, groups=m.groups, keep=m.keep, group_top=GROUP_TOP, sigmoid=lw.scores)
                y, terms = M.bank_forward(z, idx, wt, lw.bank)
                z = ops.add_group_norm(x, y, None, run.after, eps, terms=terms, again=again)
            else:
                y = ops.linear(ops.gated_act(ops.linear(z, lw.gate_up), "gelu_tanh"), lw.down)
                z = ops.add_group_norm(x, y, None, run.after, eps, again=again)
        return x

    def final_hidden(self, h: torch.Tensor, rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        """Final-normed rows of the residual stream in the activation type."""
        return ops.group_norm(h, self.w.final_norm, self.cfg.rms_eps, 1, self.dtype, rows)

    def logits(self, h: torch.Tensor, b: ForwardBatch) -> torch.Tensor:
        return ops.linear(self.final_hidden(h, b.logit_rows), self.w.lm_head)

    def _keep(self, h: torch.Tensor) -> torch.Tensor:
        self.last_hidden = h
        return h

    def forward(self, b: ForwardBatch, cache) -> torch.Tensor:
        return self.logits(self._keep(self.hidden(b, cache)), b)

    def greedy(self, b: ForwardBatch, cache) -> torch.Tensor:
        return ops.argmax(self.forward(b, cache))


def make_cache(cfg: ModelConfig, model: KegoraxModel, num_pages: int, device, max_seqs: int):
    """Planes and states are numbered by run: a layer of the loop has one set per pass."""
    from ..cache.layered import KVLayeredCache
    planes, states = {}, {}
    for j, run in enumerate(model.runs):
        s, a = run.layer.state, run.layer.attn
        states[j] = [(s.heads, s.dim, s.vdim)] + ([(s.taps, s.channels)] if s.form == S.DELTA else [])
        if a is not None:
            planes[j] = [(a.kv_heads, a.dim), (a.kv_heads, a.vdim)]
    return KVLayeredCache(cfg, num_pages, device, max_seqs, planes, states)


# ------------------------------------------------------------------------------------------ named shapes
def shape_from_entries(name: str, entries: list, *, width: int, vocab: int, loop: Optional[dict] = None, eps: float = 1e-6,
                       scale: float = 1.0, max_context: int = 8192) -> ModelConfig:
    return config_from_source({"architecture": ARCHITECTURE, "layers": entries, "width": width, "vocab": vocab, "norm": {"eps": eps},
                               "embedding": {"scale": scale}, "loop": loop}, name=name, max_context=max_context)


def _dense_entry(ff: int) -> dict:
    return {"kind": "dense", "ff": ff}


def _moe_entry(experts: int, top: int, ff: int, count: int, keep: int, scale: float) -> dict:
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "groups": {"count": count, "keep": keep},
                                                            "scale": scale}}


def kegorax_shape(layers: int = 32, width: int = 2048, heads: int = 16, ff: int = 6144, experts: int = 64, top: int = 8,
                  expert_ff: int = 1024, times: int = 1) -> ModelConfig:
    """A size whose layers resemble a served model's (benchmarks, random weights), in groups of four: three delta-rule layers -
    two with a dense feed-forward, one with experts - and one parallel layer, of the two kinds in turn.  Heads of 128
    channels; attention has a quarter as many key / value heads.  ``times``: passes of the middle half of the layers."""
    moe, dense = _moe_entry(experts, top, expert_ff, 8, 4, 2.5), _dense_entry(ff)
    att = dict(heads=heads, kv_heads=max(1, heads // 4), dim=128, vdim=128, scale=128 ** -0.5)
    sizes = dict(heads=heads, dim=128, vdim=128)
    delta = dict(sizes, kv_heads=heads, conv=4)
    par = {"left": dict(att, mask={"size": 2048}, rot={"base": 5e5, "dims": 64}), "right": dict(sizes, tau=16.0)}
    par2 = {"left": dict(att, mask={"size": 1024, "keep_first": 4}), "left_scale": 0.7, "right_scale": 0.7,
            "right": dict(sizes, decay=[1 - 2.0 ** (-5 - 7 * h / max(1, heads - 1)) for h in range(heads)])}
    entries = []
    for i in range(layers):
        if i % 4 != 3:
            entries.append({"type": "channel_delta", "mixer": delta, "mlp": moe if i % 4 == 2 else dense})
        elif (i // 4) % 2 == 0:
            entries.append({"type": "parallel", "mixer": par, "mlp": moe})
        else:
            entries.append({"type": "parallel_2", "mixer": par2, "mlp": dense})
    loop = {"start": layers // 4, "stop": layers - layers // 4, "times": times} if times > 1 else None
    return shape_from_entries("kegorax", entries, width=width, vocab=151936, loop=loop, scale=width ** 0.5)


def tiny_kegorax() -> ModelConfig:
    """CPU-checkable: all mixers, a looped block, a layer without feed-forward, uneven sizes."""
    return shape_from_entries("tiny-kegorax", [
        {"type": "parallel", "mlp": _moe_entry(6, 2, 24, 3, 2, 1.5), "mixer": {
            "left": dict(heads=4, kv_heads=2, dim=20, vdim=12, scale=0.3, mask={"size": 24}, rot={"base": 3e3, "dims": 12}),
            "right": dict(heads=3, dim=12, vdim=20, tau=8.0)}},
        {"type": "channel_delta", "mlp": _dense_entry(40), "mixer": dict(heads=4, kv_heads=2, dim=12, vdim=20, conv=3)},
        {"type": "parallel_2", "mlp": None, "mixer": {
            "left": dict(heads=3, kv_heads=1, dim=12, vdim=16, scale=0.4, mask={"size": 19, "keep_first": 3}),
            "right": dict(heads=2, dim=20, vdim=12, decay=[0.9, 0.99]), "left_scale": 0.8, "right_scale": 0.6}}],
        width=56, vocab=320, loop={"start": 0, "stop": 2, "times": 2}, scale=2.0, max_context=512)
