"""Sepedra: a decoder whose configuration lists its layers one by one - gated linear recurrences and attention with a sink,
each layer with sizes of its own - with group-limited routed experts and one RMSNorm per sublayer, on its output.

  rglru       y | x from the input, short convolution on x, block-diagonal gates, per-channel fp32 state, GELU output gate
  attention   short convolutions on q, k and v, interleaved rotary pairs with scaled frequencies, unweighted query / key
              norms, one added to the softmax denominator, sigmoid output gate per channel; a layer may take the keys and
              values of an earlier one

x <- x + norm1(mixer(x)), x <- x + norm2(experts(x)); the sublayers read x itself and a layer may have no experts.  The
residual is 32-bit; every norm, its addition and the rounding of the next sublayer's input are one launch
(ops.add_group_norm), which also sums the routed rows of a token.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Callable, Iterator, Optional

import torch

from .. import ops
from ..engine.batch import ForwardBatch
from ..ops import kv_attention as A
from ..ops import moe as M
from ..ops import rglru as R
from ..ops.core import LinearWeight
from .config import ModelConfig
from .llama import NoTP

ARCHITECTURE = "Sepedra"
MIXERS = ("rglru", "attention")
EXPERT_ALPHA, EXPERT_SHIFT = 1.702, 1.0
MAX_EXPERTS, MAX_TOP = 256, 32


# ------------------------------------------------------------------------------------------ configuration
def attention_spec(entry: dict) -> A.KVSpec:
    m = entry["mixer"]
    dim, dims = int(m["dim"]), int(m["rot"]["dims"])
    heads, kv_heads = int(m["heads"]), int(m["kv_heads"])
    if dims % 2 or not 0 <= dims <= dim:
        raise ValueError("attention: rot.dims must be even and at most dim")
    if heads < 1 or kv_heads < 1 or heads % kv_heads:
        raise ValueError("attention: kv_heads must divide heads")
    return A.KVSpec(heads=heads, kv_heads=kv_heads, dim=dim, vdim=int(m["vdim"]), scale=float(m["scale"]),
                    rot_base=float(m["rot"]["base"]), rot_dims=dims, rot_scaling=m["rot"].get("scaling"), taps=int(m["conv"]),
                    own_kv=m.get("kv_from") is None)


def rglru_spec(entry: dict) -> R.RglruSpec:
    m = entry["mixer"]
    s = R.RglruSpec(int(m["width"]), int(m["blocks"]), int(m["conv"]))
    if s.blocks < 1 or s.width % s.blocks:
        raise ValueError("rglru: blocks must divide width")
    return s


@dataclass
class MoeSpec:
    """Sizes and constants of one layer's experts."""
    experts: int
    top: int
    ff: int
    limit: float
    groups: int = 1
    keep: int = 1


def moe_spec(entry: dict) -> Optional[MoeSpec]:
    m = entry["mlp"]
    if m is None:
        return None
    if m["kind"] != "moe":
        raise ValueError(f"unknown feed-forward kind {m['kind']!r}")
    r, g = m["router"], m["router"].get("groups") or {"count": 1, "keep": 1}
    s = MoeSpec(int(r["experts"]), int(r["top"]), int(m["expert"]["ff"]), float(m["expert"]["limit"]), int(g["count"]), int(g["keep"]))
    if not 1 <= s.experts <= MAX_EXPERTS or not 1 <= s.top <= min(s.experts, MAX_TOP):
        raise ValueError(f"experts: 1 to {MAX_EXPERTS}, of which a token uses 1 to {MAX_TOP}")
    if s.groups < 1 or s.experts % s.groups or not 1 <= s.keep <= s.groups or s.keep * (s.experts // s.groups) < s.top:
        raise ValueError("expert groups: count must divide the experts, and the kept groups must hold `top` of them")
    return s


def config_from_source(d: dict, name: str = "sepedra", dtype: str = "bf16", max_context: int = 8192) -> ModelConfig:
    """ModelConfig of a parsed config.json."""
    if d.get("architecture") != ARCHITECTURE:
        raise ValueError(f"architecture {d.get('architecture')!r} is not {ARCHITECTURE}")
    entries = d["layers"]
    cfg = ModelConfig(name=name, family="sepedra", n_layers=len(entries), d_model=int(d["width"]), vocab=int(d["vocab"]),
                      rms_eps=float(d["norm"]["eps"]), logit_softcap=float(d.get("logit_softcap") or 0.0), layer_specs=entries,
                      weight_format=dtype, kv_format=dtype, max_context=max_context, n_kv_heads=1)
    specs: list = []
    for i, e in enumerate(entries):
        moe = moe_spec(e)
        if moe is not None:
            cfg.n_experts, cfg.top_k, cfg.expert_ffn = moe.experts, moe.top, moe.ff
        if e["type"] not in MIXERS:
            raise ValueError(f"unknown mixer type {e['type']!r}")
        s = rglru_spec(e) if e["type"] == "rglru" else attention_spec(e)
        specs.append(s)
        if e["type"] != "attention":
            continue
        cfg.n_heads, cfg.n_kv_heads, cfg.head_dim = s.heads, s.kv_heads, s.dim
        if not s.own_kv:
            j = int(e["mixer"]["kv_from"])
            src = specs[j] if 0 <= j < i else None
            if not isinstance(src, A.KVSpec) or not src.own_kv or (src.kv_heads, src.dim, src.vdim) != (s.kv_heads, s.dim, s.vdim):
                raise ValueError(f"layer {i}: kv_from must name an earlier attention layer of the same key and value sizes")
    return cfg


def source_shapes(cfg: ModelConfig) -> dict:
    """name -> shape of every source tensor."""
    d = cfg.d_model
    out = {"embed": (cfg.vocab, d)}
    for i, e in enumerate(cfg.layer_specs):
        p, q = f"l{i}.", f"l{i}.mix."
        out[p + "norm1"] = (d,)
        if e["type"] == "rglru":
            s = rglru_spec(e)
            for x in ("y", "x"):
                out[q + x], out[q + x + ".b"] = (s.width, d), (s.width,)
            out[q + "conv"], out[q + "conv.b"] = (s.width, s.taps), (s.width,)
            for x in ("ra", "ri"):
                out[q + x], out[q + x + ".b"] = (s.blocks, s.block, s.block), (s.blocks, s.block)
            out[q + "lam"], out[q + "o"] = (s.width,), (d, s.width)
        else:
            s = attention_spec(e)
            rows = {"q": s.q_cols, "k": s.kv_heads * s.dim, "v": s.kv_heads * s.vdim}
            for x in ("q", "k", "v") if s.own_kv else ("q",):
                out[q + x], out[q + x + ".conv"] = (rows[x], d), (rows[x], s.taps)
            out[q + "g"], out[q + "o"] = (s.out_cols, d), (d, s.out_cols)
        moe = moe_spec(e)
        if moe is not None:
            out[p + "norm2"], out[p + "mlp.router"] = (d,), (moe.experts, d)
            for k in range(moe.experts):
                r = f"{p}mlp.e{k}."
                out[r + "gate"] = out[r + "up"] = (moe.ff, d)
                out[r + "down"] = (d, moe.ff)
    out["final.norm"], out["head"] = (d,), (cfg.vocab, d)
    return out


# ------------------------------------------------------------------------------------------ resident weights
@dataclass
class SepedraLayer:
    norm1: torch.Tensor                        # norm vectors are fp32
    in_proj: LinearWeight                      # rglru: [y | x]; attention: [q | k | v | g] or [q | g]; rows padded to 8
    o: LinearWeight
    rglru: Optional[R.RglruSpec] = None
    rec: Optional[R.RglruWeights] = None
    attn: Optional[A.KVSpec] = None
    kv_layer: int = -1                         # whose pages an attention layer reads
    conv_w: Optional[torch.Tensor] = None      # fp32 [taps, channels]
    inv_freq: Optional[torch.Tensor] = None
    sinks: Optional[torch.Tensor] = None       # fp32 [heads], zero: a score of 0 joins every denominator
    norm2: Optional[torch.Tensor] = None
    moe: Optional[MoeSpec] = None
    router: Optional[LinearWeight] = None
    bank: Optional[M.ExpertBank] = None


@dataclass
class SepedraWeights:
    embed: torch.Tensor
    layers: list
    final_norm: torch.Tensor
    lm_head: LinearWeight
    vocab_offset: int = 0


def pack_weights(cfg: ModelConfig, get: Callable, device) -> SepedraWeights:
    """``get(name)`` returns a source tensor (any float type, any device)."""
    device = torch.device(device)
    dt = torch.float32 if cfg.weight_format == "fp32" else torch.bfloat16
    shapes = source_shapes(cfg)

    def fetch(name: str) -> torch.Tensor:
        t = get(name)
        if tuple(t.shape) != shapes[name]:
            raise ValueError(f"{name}: shape {tuple(t.shape)}, expected {shapes[name]}")
        return t

    def raw(name):
        return fetch(name).to(device=device, dtype=dt)

    def mat(*names) -> LinearWeight:
        w = torch.cat([raw(n) for n in names], dim=0)
        pad = (-w.shape[0]) % 8 if len(names) > 1 else 0
        return LinearWeight("dense", (torch.cat([w, w.new_zeros((pad, w.shape[1]))]) if pad else w).contiguous())

    def vec(name):
        return fetch(name).to(device=device, dtype=torch.float32).reshape(-1).contiguous()

    def taps(*names):
        return torch.cat([fetch(n).to(device=device, dtype=torch.float32) for n in names]).t().contiguous()

    layers = []
    for i, e in enumerate(cfg.layer_specs):
        p, q = f"l{i}.", f"l{i}.mix."
        if e["type"] == "rglru":
            s = rglru_spec(e)
            rec = R.RglruWeights.make(s, bias_y=vec(q + "y.b"), bias_x=vec(q + "x.b"), conv_w=taps(q + "conv"), conv_b=vec(q + "conv.b"),
                                      gate_r=raw(q + "ra").contiguous(), gate_i=raw(q + "ri").contiguous(), bias_r=vec(q + "ra.b"),
                                      bias_i=vec(q + "ri.b"), lam=vec(q + "lam"))
            kw = dict(rglru=s, rec=rec, in_proj=mat(q + "y", q + "x"))
        else:
            s = attention_spec(e)
            conv = [q + x for x in (("q", "k", "v") if s.own_kv else ("q",))]
            kw = dict(attn=s, kv_layer=i if s.own_kv else int(e["mixer"]["kv_from"]), in_proj=mat(*conv, q + "g"),
                      conv_w=taps(*(c + ".conv" for c in conv)), inv_freq=s.inv_freq(device), sinks=torch.zeros(s.heads, device=device))
        moe = moe_spec(e)
        if moe is not None:
            part = lambda x: [raw(f"{p}mlp.e{k}.{x}") for k in range(moe.experts)]
            kw.update(moe=moe, norm2=vec(p + "norm2"), router=mat(p + "mlp.router"),
                      bank=M.ExpertBank.pack(part("gate"), part("up"), part("down"), M.GatedAct(moe.limit, EXPERT_ALPHA, EXPERT_SHIFT)))
        layers.append(SepedraLayer(norm1=vec(p + "norm1"), o=mat(q + "o"), **kw))
    return SepedraWeights(raw("embed").contiguous(), layers, vec("final.norm"), mat("head"), 0)


def named_tensors(cfg: ModelConfig, w: SepedraWeights) -> Iterator:
    """(source name, tensor) of every tensor: the inverse of ``pack_weights``."""
    yield "embed", w.embed
    for i, l in enumerate(w.layers):
        p, q = f"l{i}.", f"l{i}.mix."
        yield p + "norm1", l.norm1
        if l.rglru is not None:
            s, r = l.rglru, l.rec
            rows = [("y", s.width), ("x", s.width)]
            blocked = (s.blocks, s.block)
            for name, t in (("y.b", r.bias_y), ("x.b", r.bias_x), ("conv", r.conv_w.t().contiguous()), ("conv.b", r.conv_b),
                            ("ra", r.gate_r), ("ra.b", r.bias_r.view(blocked)), ("ri", r.gate_i), ("ri.b", r.bias_i.view(blocked)),
                            ("lam", r.lam)):
                yield q + name, t
        else:
            s = l.attn
            rows = [("q", s.q_cols)] + ([("k", s.kv_heads * s.dim), ("v", s.kv_heads * s.vdim)] if s.own_kv else [])
            c0 = 0
            for name, n in rows:
                yield f"{q}{name}.conv", l.conv_w[:, c0:c0 + n].t().contiguous()
                c0 += n
            rows.append(("g", s.out_cols))
        r0 = 0
        for name, n in rows:
            yield q + name, l.in_proj.w[r0:r0 + n]
            r0 += n
        yield q + "o", l.o.w
        if l.moe is not None:
            yield p + "norm2", l.norm2
            yield p + "mlp.router", l.router.w
            for k in range(l.moe.experts):
                for name, t in zip(("gate", "up", "down"), l.bank.matrices(k)):
                    yield f"{p}mlp.e{k}.{name}", t
    yield "final.norm", w.final_norm
    yield "head", w.lm_head.w


def init_random_sepedra_weights(cfg: ModelConfig, device, seed: int = 0) -> SepedraWeights:
    """Seeded weights of the configured shape, drawn tensor by tensor on the target device (a generator per tensor, so the
    order of use does not matter): matrices ~N(0, 1 / fan-in), norms near 1, decays between about 0.9 and 0.999."""
    device = torch.device(device)
    shapes = source_shapes(cfg)
    index = {n: k for k, n in enumerate(shapes)}

    def get(name):
        shape = shapes[name]
        gen = torch.Generator(device=device)
        gen.manual_seed(seed * 100003 + index[name])
        x = torch.randn(shape, generator=gen, device=device, dtype=torch.float32)
        if ".norm" in name:
            return 1.0 + 0.05 * x
        if name.endswith(".lam"):
            return x - 4.0
        if name.endswith(".b"):
            return 0.1 * x
        return x if name == "embed" else x * shape[-1] ** -0.5
    return pack_weights(cfg, get, device)


# ------------------------------------------------------------------------------------------ model
class SepedraModel:
    """Stateless forward over a ForwardBatch; pages and states live in the KVLayeredCache passed in."""

    def __init__(self, cfg: ModelConfig, weights: SepedraWeights, tp=None):
        if tp is not None and tp.size != 1:
            raise ValueError("the sepedra family runs on one GPU")
        self.cfg, self.w = cfg, weights
        self.tp = tp or NoTP()
        self.dtype = weights.embed.dtype

    @property
    def local_kv_heads(self) -> int:
        return self.cfg.n_kv_heads

    def _attention(self, z, lw: SepedraLayer, i: int, b: ForwardBatch, cache):
        s = lw.attn
        proj = ops.linear(z, lw.in_proj)
        kv = cache.layer(lw.kv_layer)
        q = A.prepare(proj, s, lw.conv_w, lw.inv_freq, self.cfg.rms_eps, kv if s.own_kv else None, cache.state(i), b)
        gate = proj[:, s.channels:s.channels + s.out_cols]
        return ops.linear(A.attention(q, gate, s, kv, lw.sinks, b), lw.o)

    def _rglru(self, z, lw: SepedraLayer, i: int, b: ForwardBatch, cache):
        y = R.rglru(ops.linear(z, lw.in_proj), lw.rglru, lw.rec, cache.state(i, 0), cache.state(i, 1), b)
        return ops.linear(y, lw.o)

    def hidden(self, b: ForwardBatch, cache) -> torch.Tensor:
        eps = self.cfg.rms_eps
        if b.row_off is None or b.slots is None:
            raise ValueError("the sepedra family needs row offsets and state slots in the batch")
        if b.embeds is not None:
            raise ValueError("the sepedra family takes token ids only")
        x, z = ops.embed_group_norm(self.w.embed, b.tokens, None, eps)
        for i, lw in enumerate(self.w.layers):
            y = (self._rglru if lw.rglru is not None else self._attention)(z, lw, i, b, cache)
            z = ops.add_group_norm(x, y, lw.norm1, None, eps, raw=True)
            if lw.moe is not None:
                m = lw.moe
                idx, wt = M.router(z, lw.router, m.top, True, m.groups, m.keep)
                y, terms = M.bank_forward(z, idx, wt, lw.bank)
                z = ops.add_group_norm(x, y, lw.norm2, None, eps, terms=terms, raw=True)
        return x

    def final_hidden(self, h: torch.Tensor, rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        """Final-normed rows of the residual stream in the activation type."""
        return ops.group_norm(h, self.w.final_norm, self.cfg.rms_eps, 1, self.dtype, rows)

    def logits(self, h: torch.Tensor, b: ForwardBatch) -> torch.Tensor:
        cap = self.cfg.logit_softcap
        z = self.final_hidden(h, b.logit_rows)
        return ops.linear(z, self.w.lm_head, act="softcap", act_arg=cap) if cap > 0 else ops.linear(z, self.w.lm_head)

    def _keep(self, h: torch.Tensor) -> torch.Tensor:
        self.last_hidden = h
        return h

    def forward(self, b: ForwardBatch, cache) -> torch.Tensor:
        return self.logits(self._keep(self.hidden(b, cache)), b)

    def greedy(self, b: ForwardBatch, cache) -> torch.Tensor:
        return ops.argmax(self.forward(b, cache))


def make_cache(cfg: ModelConfig, model: SepedraModel, num_pages: int, device, max_seqs: int):
    from ..cache.layered import KVLayeredCache
    planes, states = {}, {}
    for i, l in enumerate(model.w.layers):
        if l.rglru is not None:
            states[i] = [(l.rglru.width,), (l.rglru.taps, l.rglru.width)]
        else:
            states[i] = [(l.attn.taps, l.attn.channels)]
            if l.attn.own_kv:
                planes[i] = [(l.attn.kv_heads, l.attn.dim), (l.attn.kv_heads, l.attn.vdim)]
    return KVLayeredCache(cfg, num_pages, device, max_seqs, planes, states)


# ------------------------------------------------------------------------------------------ named shapes
def shape_from_entries(name: str, entries: list, *, width: int, vocab: int, eps: float = 1e-6, logit_softcap: float = 30.0,
                       max_context: int = 8192) -> ModelConfig:
    return config_from_source({"architecture": ARCHITECTURE, "layers": entries, "width": width, "vocab": vocab, "norm": {"eps": eps},
                               "logit_softcap": logit_softcap}, name=name, max_context=max_context)


def _rglru_entry(mlp: Optional[dict], width: int, blocks: int, conv: int = 4) -> dict:
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}, "mlp": mlp}


def _attention_entry(mlp: Optional[dict], **mixer) -> dict:
    return {"type": "attention", "mixer": {k: v for k, v in mixer.items() if v is not None}, "mlp": mlp}


def _moe_entry(experts: int, top: int, ff: int, limit: float, count: int, keep: int) -> dict:
    return {"kind": "moe", "router": {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}},
            "expert": {"ff": ff, "limit": limit}}


def sepedra_shape(layers: int = 32, width: int = 2048, heads: int = 16, experts: int = 64, top: int = 8, ff: int = 512) -> ModelConfig:
    """A size whose layers resemble a served model's (benchmarks, random weights): every fourth layer is attention with heads
    of 128 channels and a quarter as many key / value heads - every second of them takes the keys and values of the one before
    -, the others are recurrences as wide as the model in blocks of 256."""
    moe = _moe_entry(experts, top, ff, 7.0, 8, 4)
    rot = {"base": 5e5, "dims": 128, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}
    entries = [_attention_entry(moe, heads=heads, kv_heads=max(1, heads // 4), dim=128, vdim=128, conv=4, scale=128 ** -0.5, rot=rot,
                                kv_from=i - 4 if (i // 4) % 2 else None)
               if i % 4 == 3 else _rglru_entry(moe, width, max(1, width // 256)) for i in range(layers)]
    return shape_from_entries("sepedra", entries, width=width, vocab=151936)


def tiny_sepedra() -> ModelConfig:
    """CPU-checkable: both mixers, shared keys and values, a layer without experts, uneven sizes."""
    rot = {"base": 3e3, "dims": 12, "scaling": {"factor": 4.0, "low": 1.0, "high": 3.0, "original": 64}}
    att = dict(heads=6, kv_heads=2, dim=20, vdim=24, conv=3, scale=0.3, rot=rot)
    return shape_from_entries("tiny-sepedra", [
        _rglru_entry(_moe_entry(6, 2, 40, 1.5, 3, 2), 72, 3), _attention_entry(None, **att),
        _attention_entry(_moe_entry(5, 3, 24, 3.0, 1, 1), **att, kv_from=1)], width=56, vocab=320, max_context=512)
