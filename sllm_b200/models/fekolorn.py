"""Fekolorn: a decoder whose residual is several parallel streams and whose configuration lists its layers one by one.

  attention   windowed attention without rotation: query / key norms over all heads at once, learned biases over the distance,
              learned sinks, values mixed with those of the first layer that mixes
  parallel    full attention (rotary half-split pairs, normed values, learned sinks) beside a gated delta rule with one decay per
              head, short convolutions and a SiLU output gate; a weighted sum of both outputs

Every sublayer reads a weighted sum of the streams and writes back while they mix (ops/streams.py); norms have a single weight.
The feed-forward is W_down act(W_up h), act a polynomial of normed powers.  The embedding of a token is joined by one of the
(previous token, token) pair; the previous token is part of a sequence's state.  All of a layer's input projections are one GEMM;
every meeting of a sublayer with the streams, with the next sublayer's norm, is one launch.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Callable, Iterator, Optional

import torch

from .. import ops
from ..engine.batch import ForwardBatch
from ..ops import kv_attention as A
from ..ops import linear_state as S
from ..ops import streams as R
from ..ops.core import LinearWeight
from .config import ModelConfig
from .llama import NoTP
from .packing import SourceTensors

ARCHITECTURE = "Fekolorn"
MIXERS = ("attention", "parallel")
LAST_TOKEN = "last_token"                  # key of the cache's state that carries a sequence's last token


# ------------------------------------------------------------------------------------------ configuration
def attention_spec(entry: dict) -> A.KVSpec:
    windowed = entry["type"] == "attention"
    m = entry["mixer"] if windowed else entry["mixer"]["left"]
    heads, kv_heads, dim, vdim = (int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
    if min(heads, kv_heads, dim, vdim) < 1 or heads % kv_heads:
        raise ValueError("attention: positive sizes, and kv_heads must divide heads")
    kw = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=float(m["scale"]), interleaved=False)
    if windowed:
        size = int(m["mask"]["size"])
        if size < 1 or not float(m["bias_max"]) > 0:
            raise ValueError("attention: mask.size and bias_max must be positive")
        return A.KVSpec(rot_base=1.0, rot_dims=0, window=size, norm_all=True, **kw)
    dims = int(m["rot"]["dims"])
    if dims % 2 or not 0 <= dims <= dim:
        raise ValueError("attention: rot.dims must be even and at most dim")
    return A.KVSpec(rot_base=float(m["rot"]["base"]), rot_dims=dims, qk_norm=False, v_norm=True, **kw)


def mixes_values(entry: dict) -> bool:
    return entry["type"] == "attention" and bool(entry["mixer"].get("v_mix"))


def state_sizes(entry: dict) -> tuple:
    """(heads, query / key heads, dim, vdim, taps) of a parallel layer's recurrence."""
    out = tuple(int(entry["mixer"]["right"][k]) for k in ("heads", "kv_heads", "dim", "vdim", "conv"))
    if min(out) < 1 or out[0] % out[1]:
        raise ValueError("recurrence: positive sizes, and kv_heads must divide heads")
    return out


def config_from_source(d: dict, name: str = "fekolorn", dtype: str = "bf16", max_context: int = 8192) -> ModelConfig:
    """ModelConfig of a parsed config.json."""
    if d.get("architecture") != ARCHITECTURE:
        raise ValueError(f"architecture {d.get('architecture')!r} is not {ARCHITECTURE}")
    entries, emb = d["layers"], d["embedding"]
    bigram = emb.get("bigram")
    if bigram is not None:
        bigram = {k: int(bigram[k]) for k in ("buckets", "mul_prev", "mul_cur")}
        if bigram["buckets"] < 1:
            raise ValueError("embedding.bigram: buckets must be positive")
    cfg = ModelConfig(name=name, family="fekolorn", n_layers=len(entries), d_model=int(d["width"]), vocab=int(d["vocab"]),
                      rms_eps=float(d["norm"]["eps"]), embedding_scale=float(emb["scale"]), layer_specs=entries,
                      streams=int(d["streams"]), bigram=bigram, weight_format=dtype, kv_format=dtype, max_context=max_context, n_kv_heads=1)
    if not entries or not 1 <= cfg.streams <= R.MAX_STREAMS:
        raise ValueError(f"at least one layer, and 1 to {R.MAX_STREAMS} streams")
    if cfg.vocab > R.MAX_TOKEN:
        raise ValueError(f"the vocabulary is limited to {R.MAX_TOKEN} tokens")
    values = set()
    for e in entries:
        if e["type"] not in MIXERS:
            raise ValueError(f"unknown mixer type {e['type']!r}")
        s = attention_spec(e)
        cfg.n_heads, cfg.n_kv_heads, cfg.head_dim = s.heads, s.kv_heads, s.dim
        if e["type"] == "parallel":
            state_sizes(e)
        elif mixes_values(e):
            values.add(s.kv_heads * s.vdim)
        if e["mlp"] is not None:
            if e["mlp"]["kind"] != "dense":
                raise ValueError(f"unknown feed-forward kind {e['mlp']['kind']!r}")
            cfg.ffn = max(cfg.ffn if cfg.ffn != ModelConfig.ffn else 0, int(e["mlp"]["ff"]))
    if len(values) > 1:
        raise ValueError("layers that mix values must have equally many of them")
    return cfg


def source_shapes(cfg: ModelConfig, bias_rows: Callable[[str], int]) -> dict:
    """name -> shape of every source tensor; ``bias_rows(name)`` is the number of rows of the distance-bias table of that name (the
    only sizes that the configuration does not carry)."""
    d, n = cfg.d_model, cfg.streams
    out = {"embed": (cfg.vocab, d)}
    if cfg.bigram is not None:
        out["bigram"] = (cfg.bigram["buckets"] + 1, d)
    for i, e in enumerate(cfg.layer_specs):
        p, q, a = f"l{i}.", f"l{i}.mix.", attention_spec(e)
        l = q if e["type"] == "attention" else q + "left."
        out[p + "norm1"] = ()
        out[l + "q"], out[l + "k"], out[l + "v"] = (a.q_cols, d), (a.kv_heads * a.dim, d), (a.kv_heads * a.vdim, d)
        out[l + "sink"], out[l + "o"] = (a.heads,), (d, a.out_cols)
        if e["type"] == "attention":
            out[q + "q.norm"], out[q + "k.norm"] = (a.q_cols,), (a.kv_heads * a.dim,)
            out[q + "rel"] = (bias_rows(q + "rel"), a.heads)
            if mixes_values(e):
                out[q + "vmix"] = ()
        else:
            H, G, D, V, taps = state_sizes(e)
            r = q + "right."
            for x, rows in (("q", G * D), ("k", G * D), ("v", H * V)):
                out[r + x], out[f"{r}{x}.conv"] = (rows, d), (rows, taps)
            out[r + "b"] = out[r + "a"] = (H, d)
            out[r + "A_log"] = out[r + "dt_bias"] = (H,)
            out[r + "norm"], out[r + "g"], out[r + "o"] = (V,), (H * V, d), (d, H * V)
        subs = ("hc1",)
        if e["mlp"] is not None:
            ff, subs = int(e["mlp"]["ff"]), ("hc1", "hc2")
            out[p + "norm2"] = ()
            out[p + "mlp.up"], out[p + "mlp.down"], out[p + "mlp.act"] = (ff, d), (d, ff), (4,)
        for x in subs:
            out[f"{p}{x}.in"], out[f"{p}{x}.out"], out[f"{p}{x}.mix"] = (n,), (n,), (n, n)
    out["final.norm"], out["head"] = (), (cfg.vocab, d)
    return out


# ------------------------------------------------------------------------------------------ resident weights
@dataclass
class FekolornLayer:
    norm1: torch.Tensor                        # vectors are fp32; norms have one number
    conn1: R.Connection
    in_proj: LinearWeight                      # all projections of the layer's input; every part starts at a multiple of 8 rows
    rows: list                                 # [(source name after "mix.", first row, rows)] of in_proj
    attn: A.KVSpec
    o: LinearWeight
    sinks: torch.Tensor
    inv_freq: Optional[torch.Tensor] = None
    q_norm: Optional[torch.Tensor] = None
    k_norm: Optional[torch.Tensor] = None
    rel: Optional[torch.Tensor] = None         # [rows, heads], and what the kernels read of it
    dist: Optional[A.DistanceBias] = None
    v_mix: Optional[float] = None              # share of the first mixing layer's values (None: the layer does not mix)
    state: Optional[S.StateSpec] = None        # of the recurrence beside the attention
    sw: Optional[S.StateWeights] = None
    a_log: Optional[torch.Tensor] = None
    o_state: Optional[LinearWeight] = None
    attn_coef: float = 1.0
    state_coef: float = 0.0
    norm2: Optional[torch.Tensor] = None
    conn2: Optional[R.Connection] = None
    up: Optional[LinearWeight] = None
    down: Optional[LinearWeight] = None
    act: Optional[torch.Tensor] = None         # [4]


@dataclass
class FekolornWeights:
    embed: torch.Tensor
    pair: Optional[R.PairEmbedding]
    layers: list
    final_norm: torch.Tensor
    lm_head: LinearWeight
    vocab_offset: int = 0


def pack_weights(cfg: ModelConfig, get: Callable, device) -> FekolornWeights:
    """``get(name)`` returns a source tensor (any float type, any device)."""
    src = SourceTensors(cfg, get, source_shapes(cfg, lambda n: int(get(n).shape[0])), device)
    vec, mat = src.vec, src.mat
    connection = lambda x: R.Connection(src.f32(x + ".in"), src.f32(x + ".mix"), src.f32(x + ".out"))
    layers = []
    for i, e in enumerate(cfg.layer_specs):
        p, q, a = f"l{i}.", f"l{i}.mix.", attention_spec(e)
        kw: dict = dict(norm1=vec(p + "norm1"), conn1=connection(p + "hc1"), attn=a)
        if e["type"] == "attention":
            in_proj, rows = src.packed(q, [["q", "k", "v"]])
            rel = src.f32(q + "rel")
            kw.update(q_norm=vec(q + "q.norm"), k_norm=vec(q + "k.norm"), rel=rel, sinks=vec(q + "sink"), o=mat(q + "o"),
                      dist=A.DistanceBias.make(rel, float(e["mixer"]["bias_max"]), a.window))
            if mixes_values(e):
                kw["v_mix"] = float(src.f32(q + "vmix"))
        else:
            H, G, D, V, taps = state_sizes(e)
            r = q + "right."
            in_proj, rows = src.packed(q, [["left.q", "left.k", "left.v"], ["right.q", "right.k", "right.v"], ["right.g"],
                                           ["right.a"], ["right.b"]])
            at = {n: k for n, k, _ in rows}
            kw["a_log"] = vec(r + "A_log")
            kw.update(inv_freq=a.inv_freq(src.device), sinks=vec(q + "left.sink"), o=mat(q + "left.o"), o_state=mat(r + "o"),
                      attn_coef=float(e["mixer"]["left_scale"]), state_coef=float(e["mixer"]["right_scale"]),
                      state=S.StateSpec(S.HEAD_DELTA, H, G, D, V, {x: at["right." + x] for x in ("q", "k", "v", "g", "a", "b")},
                                        q_scale=D ** -0.5, taps=taps),
                      sw=S.StateWeights(bias=vec(r + "dt_bias"), rate=torch.exp(kw["a_log"].double()).float(), norm=vec(r + "norm"),
                                        conv_w=src.taps(*(f"{r}{x}.conv" for x in ("q", "k", "v")))))
        if e["mlp"] is not None:
            kw.update(norm2=vec(p + "norm2"), conn2=connection(p + "hc2"), up=mat(p + "mlp.up"), down=mat(p + "mlp.down"),
                      act=vec(p + "mlp.act"))
        layers.append(FekolornLayer(in_proj=in_proj, rows=rows, **kw))
    pair = None
    if cfg.bigram is not None:
        pair = R.PairEmbedding(src.raw("bigram").contiguous(), cfg.bigram["mul_prev"], cfg.bigram["mul_cur"])
    return FekolornWeights(src.raw("embed").contiguous(), pair, layers, vec("final.norm"), mat("head"))


def named_tensors(cfg: ModelConfig, w: FekolornWeights) -> Iterator:
    """(source name, tensor) of every tensor: the inverse of ``pack_weights``."""
    yield "embed", w.embed
    if w.pair is not None:
        yield "bigram", w.pair.table
    for i, l in enumerate(w.layers):
        p, q = f"l{i}.", f"l{i}.mix."
        yield p + "norm1", l.norm1
        for name, r0, n in l.rows:
            yield q + name, l.in_proj.w[r0:r0 + n]
        a, s = (q, None) if l.state is None else (q + "left.", l.state)
        yield a + "sink", l.sinks
        yield a + "o", l.o.w
        if s is None:
            yield q + "q.norm", l.q_norm
            yield q + "k.norm", l.k_norm
            yield q + "rel", l.rel
            if l.v_mix is not None:
                yield q + "vmix", torch.tensor([l.v_mix])
        else:
            r, c0 = q + "right.", 0
            for x, n in (("q", s.kv_heads * s.dim), ("k", s.kv_heads * s.dim), ("v", s.out_cols)):
                yield f"{r}{x}.conv", l.sw.conv_w[:, c0:c0 + n].t().contiguous()
                c0 += n
            yield r + "A_log", l.a_log
            yield r + "dt_bias", l.sw.bias
            yield r + "norm", l.sw.norm
            yield r + "o", l.o_state.w
        subs = [("hc1", l.conn1)]
        if l.norm2 is not None:
            subs.append(("hc2", l.conn2))
            yield p + "norm2", l.norm2
            yield p + "mlp.up", l.up.w
            yield p + "mlp.down", l.down.w
            yield p + "mlp.act", l.act
        for x, c in subs:
            yield f"{p}{x}.in", c.read
            yield f"{p}{x}.mix", c.mix
            yield f"{p}{x}.out", c.out
    yield "final.norm", w.final_norm
    yield "head", w.lm_head.w


def init_random_fekolorn_weights(cfg: ModelConfig, device, seed: int = 0, bias_rows: int = 32) -> FekolornWeights:
    """Seeded weights of the configured shape, drawn tensor by tensor on the target device (a generator per tensor, so the
    order of use does not matter): matrices ~N(0, 1 / fan-in), norms near 1, decays mostly between 0.9 and 1, streams that
    mix a little."""
    device = torch.device(device)
    shapes = source_shapes(cfg, lambda n: bias_rows)
    index = {n: k for k, n in enumerate(shapes)}

    def get(name):
        shape = shapes[name]
        gen = torch.Generator(device=device)
        gen.manual_seed(seed * 100003 + index[name])
        x = torch.randn(shape, generator=gen, device=device, dtype=torch.float32)
        last = name.rsplit(".", 1)[-1]
        if last in ("norm", "norm1", "norm2", "out"):
            return 1.0 + 0.05 * x
        if last == "in":
            return (1.0 + 0.05 * x) / cfg.streams
        if last == "mix" and ".hc" in name:
            return torch.eye(cfg.streams, device=device) + 0.05 * x
        if last == "vmix":
            return 0.3 + 0.05 * x
        if last == "act":
            return torch.tensor([0.6, 0.3, 0.3, 0.0], device=device) + 0.05 * x
        if last == "dt_bias":
            return x - 3.0
        if last == "A_log":
            return 0.5 * x
        if last in ("sink", "rel"):
            return x
        return x * shape[-1] ** -0.5
    return pack_weights(cfg, get, device)


# ------------------------------------------------------------------------------------------ model
class FekolornModel:
    """Stateless forward over a ForwardBatch; pages, states and every sequence's last token live in the KVLayeredCache passed
    in.  The residual is [T, streams, width]."""

    def __init__(self, cfg: ModelConfig, weights: FekolornWeights, tp=None):
        if tp is not None and tp.size != 1:
            raise ValueError("the fekolorn family runs on one GPU")
        self.cfg, self.w = cfg, weights
        self.tp = tp or NoTP()
        self.dtype = weights.embed.dtype
        # (read weights, norm) of every sublayer in running order, and nothing behind the last
        self.reads = [r for l in weights.layers
                      for r in [(l.conn1.read, l.norm1)] + ([] if l.norm2 is None else [(l.conn2.read, l.norm2)])] + [(None, None)]

    @property
    def local_kv_heads(self) -> int:
        return self.cfg.n_kv_heads

    def _mixer(self, z, lw: FekolornLayer, i: int, b: ForwardBatch, cache, first):
        """(attention output, output of the recurrence or None, the layer's own values)."""
        a, kv, eps = lw.attn, cache.layer(i), self.cfg.rms_eps
        proj = ops.linear(z, lw.in_proj)
        v0 = a.q_cols + a.kv_heads * a.dim
        mix = None if lw.v_mix is None or first is None else (first, lw.v_mix)
        q = A.prepare(proj, a, None, lw.inv_freq, eps, kv, None, b, q_norm=lw.q_norm, k_norm=lw.k_norm, mix=mix)
        y = ops.linear(A.attention(q, None, a, kv, lw.sinks, b, dist=lw.dist), lw.o)
        y2 = None
        if lw.state is not None:
            y2 = ops.linear(S.linear_state(proj, lw.state, lw.sw, eps, cache.state(i), cache.state(i, 1), b), lw.o_state)
        return y, y2, proj[:, v0:v0 + a.kv_heads * a.vdim]

    def hidden(self, b: ForwardBatch, cache) -> torch.Tensor:
        cfg, w, eps = self.cfg, self.w, self.cfg.rms_eps
        if b.row_off is None or b.slots is None:
            raise ValueError("the fekolorn family needs row offsets and state slots in the batch")
        if b.embeds is not None:
            raise ValueError("the fekolorn family takes token ids only")
        reads = iter(self.reads)
        read, norm = next(reads)
        last = None if w.pair is None else cache.state(LAST_TOKEN)
        x, z = R.start_streams(w.embed, b, cfg.embedding_scale, w.pair, last, cfg.streams, read, norm, eps)
        first = None
        for i, lw in enumerate(w.layers):
            y, y2, own = self._mixer(z, lw, i, b, cache, first)
            if first is None and lw.v_mix is not None:
                first = own
            read, norm = next(reads)
            z = R.join_streams(x, y, lw.conn1, read, norm, eps, lw.attn_coef, None if y2 is None else (y2, lw.state_coef))
            if lw.norm2 is not None:
                y = ops.linear(ops.poly_norm(ops.linear(z, lw.up), lw.act, eps), lw.down)
                read, norm = next(reads)
                z = R.join_streams(x, y, lw.conn2, read, norm, eps)
        return x

    def final_hidden(self, h: torch.Tensor, rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        """Final-normed rows of the residual (the sum of its streams) in the activation type."""
        return R.read_streams(h, self.w.final_norm, self.cfg.rms_eps, self.dtype, rows)

    def logits(self, h: torch.Tensor, b: ForwardBatch) -> torch.Tensor:
        return ops.linear(self.final_hidden(h, b.logit_rows), self.w.lm_head)

    def _keep(self, h: torch.Tensor) -> torch.Tensor:
        self.last_hidden = h
        return h

    def forward(self, b: ForwardBatch, cache) -> torch.Tensor:
        return self.logits(self._keep(self.hidden(b, cache)), b)

    def greedy(self, b: ForwardBatch, cache) -> torch.Tensor:
        return ops.argmax(self.forward(b, cache))


def make_cache(cfg: ModelConfig, model: FekolornModel, num_pages: int, device, max_seqs: int):
    from ..cache.layered import KVLayeredCache
    planes, states = {}, {}
    for i, l in enumerate(model.w.layers):
        a, s = l.attn, l.state
        planes[i] = [(a.kv_heads, a.dim), (a.kv_heads, a.vdim)]
        if s is not None:
            states[i] = [(s.heads, s.dim, s.vdim), (s.taps, s.channels)]
    if cfg.bigram is not None:
        states[LAST_TOKEN] = [(1,)]
    return KVLayeredCache(cfg, num_pages, device, max_seqs, planes, states)


# ------------------------------------------------------------------------------------------ named shapes
def shape_from_entries(name: str, entries: list, *, width: int, vocab: int, streams: int, bigram: Optional[dict], eps: float = 1e-6,
                       scale: float = 1.0, max_context: int = 8192) -> ModelConfig:
    return config_from_source({"architecture": ARCHITECTURE, "layers": entries, "width": width, "vocab": vocab, "norm": {"eps": eps},
                               "embedding": {"scale": scale, "bigram": bigram}, "streams": streams}, name=name, max_context=max_context)


def _bigram(buckets: int) -> dict:
    return {"buckets": buckets, "mul_prev": 31, "mul_cur": 17}


def fekolorn_shape(layers: int = 32, width: int = 2048, heads: int = 16, ff: int = 6144, streams: int = 2) -> ModelConfig:
    """A size whose layers resemble a served model's (benchmarks, random weights), in groups of four: three parallel layers and one
    with windowed attention.  Heads of 128 channels; attention has a quarter as many key / value heads."""
    att = dict(heads=heads, kv_heads=max(1, heads // 4), dim=128, vdim=128, scale=128 ** -0.5)
    window = dict(att, mask={"size": 1024}, bias_max=512, v_mix=True)
    par = {"left": dict(att, rot={"base": 5e5, "dims": 64}), "left_scale": 0.7, "right_scale": 0.7,
           "right": dict(heads=heads, kv_heads=heads, dim=128, vdim=128, conv=4)}
    mlp = {"kind": "dense", "ff": ff}
    entries = [{"type": "attention", "mixer": window, "mlp": mlp} if i % 4 == 3 else {"type": "parallel", "mixer": par, "mlp": mlp}
               for i in range(layers)]
    return shape_from_entries("fekolorn", entries, width=width, vocab=151936, streams=streams, bigram=_bigram(65521), scale=width ** 0.5)


def tiny_fekolorn() -> ModelConfig:
    """CPU-checkable: both mixers, mixed values, a layer without feed-forward, three streams, uneven sizes."""
    att = lambda **kw: dict(heads=4, kv_heads=2, dim=20, vdim=12, scale=0.3, **kw)
    par = {"left": dict(heads=3, kv_heads=1, dim=12, vdim=16, scale=0.4, rot={"base": 3e3, "dims": 8}), "left_scale": 0.8,
           "right": dict(heads=4, kv_heads=2, dim=12, vdim=20, conv=3), "right_scale": 0.6}
    return shape_from_entries("tiny-fekolorn", [
        {"type": "parallel", "mixer": par, "mlp": {"kind": "dense", "ff": 40}},
        {"type": "attention", "mixer": att(mask={"size": 24}, bias_max=20, v_mix=True), "mlp": None},
        {"type": "attention", "mixer": att(mask={"size": 17}, bias_max=40, v_mix=True), "mlp": {"kind": "dense", "ff": 56}}],
        width=56, vocab=320, streams=3, bigram=_bigram(101), scale=2.0, max_context=512)
