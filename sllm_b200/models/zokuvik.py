"""Zokuvik: a decoder whose configuration lists its layers one by one - two forms of latent attention and a generalised
delta rule, each layer with sizes of its own - with grouped RMSNorms before and after every sublayer on a 32-bit residual.

  latent_attention    queries through a latent, interleaved rotary pairs, all earlier positions, sigmoid output gate per head
  latent_attention_2  queries straight from the input, split-half rotary pairs, sliding window
  general_delta       r | k | v | a | g and a low-rank decay from the input, delta-rule state per head, normed and gated output

x <- x + norm1b(mixer(norm1(x))), x <- x + norm2b(W_down relu(W_up norm2(x))^2); a layer may have no feed-forward.
Each layer's input projections are one GEMM; every norm pair around the residual is one launch (ops.add_group_norm); the
feed-forward's activation rides in its first product's epilogue.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Callable, Iterator, Optional

import torch

from .. import ops
from ..engine.batch import ForwardBatch
from ..ops import delta as D
from ..ops import latent as A
from ..ops.core import LinearWeight
from .config import ModelConfig
from .llama import NoTP

ARCHITECTURE = "Zokuvik"

# what a mixer type means; sizes come from the layer's entry
_LATENT_FORMS = {
    "latent_attention": dict(query_latent=True, gated=True, interleaved=True, windowed=False),
    "latent_attention_2": dict(query_latent=False, gated=False, interleaved=False, windowed=True),
}
_DELTA_FORM = "general_delta"


# ------------------------------------------------------------------------------------------ configuration
def latent_spec(entry: dict) -> A.LatentSpec:
    m, form = entry["mixer"], _LATENT_FORMS[entry["type"]]
    dims = int(m["rot"]["dims"])
    if dims % 2 or dims > int(m["rot_dim"]):
        raise ValueError(f"{entry['type']}: rot.dims must be even and at most rot_dim")
    window = int(m["mask"]["size"]) if form["windowed"] else 0
    if form["windowed"] and window < 1:
        raise ValueError(f"{entry['type']}: mask.size must be positive")
    return A.LatentSpec(heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]), vdim=int(m["vdim"]),
                        kv_rank=int(m["kv_rank"]), scale=float(m["scale"]), rot_base=float(m["rot"]["base"]), rot_dims=dims,
                        interleaved=form["interleaved"], q_rank=int(m["q_rank"]) if form["query_latent"] else 0,
                        window=window, gated=form["gated"])


def config_from_source(d: dict, name: str = "zokuvik", dtype: str = "bf16", max_context: int = 8192) -> ModelConfig:
    """ModelConfig of a parsed config.json."""
    if d.get("architecture") != ARCHITECTURE:
        raise ValueError(f"architecture {d.get('architecture')!r} is not {ARCHITECTURE}")
    specs = d["layers"]
    for e in specs:
        if e["type"] not in _LATENT_FORMS and e["type"] != _DELTA_FORM:
            raise ValueError(f"unknown mixer type {e['type']!r}")
        if e["mlp"] is not None and e["mlp"]["kind"] != "dense":
            raise ValueError(f"unknown feed-forward kind {e['mlp']['kind']!r}")
    width, groups = int(d["width"]), int(d["norm"]["groups"])
    if groups < 1 or width % groups:
        raise ValueError("the norm groups must divide the width")
    cfg = ModelConfig(name=name, family="zokuvik", n_layers=len(specs), d_model=width, vocab=int(d["vocab"]),
                      rms_eps=float(d["norm"]["eps"]), norm_groups=groups, layer_specs=specs, weight_format=dtype,
                      kv_format=dtype, max_context=max_context, n_kv_heads=1)
    for e in specs:
        if e["type"] in _LATENT_FORMS:
            s = latent_spec(e)
            cfg.n_heads, cfg.head_dim = s.heads, s.width
            break
    cfg.ffn = max((int(e["mlp"]["ff"]) for e in specs if e["mlp"] is not None), default=0)
    return cfg


def source_shapes(cfg: ModelConfig, decay_rank: Callable[[int], int]) -> dict:
    """name -> shape of every source tensor; decay_rank(layer) is the inner size of a general_delta layer's decay
    projection (the only size that the configuration does not carry)."""
    d = cfg.d_model
    out = {"embed": (cfg.vocab, d)}
    for i, e in enumerate(cfg.layer_specs):
        p, m = f"l{i}.", e["mixer"]
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if e["mlp"] is not None else ()):
            out[p + n] = (d,)
        q = p + "mix."
        if e["type"] in _LATENT_FORMS:
            s = latent_spec(e)
            if s.q_rank:
                out[q + "dq"], out[q + "dq.norm"] = (s.q_rank, d), (s.q_rank,)
                out[q + "uq"] = (s.heads * (s.dim + s.rot_dim), s.q_rank)
            else:
                out[q + "q"] = (s.heads * (s.dim + s.rot_dim), d)
            out[q + "dkv"], out[q + "dkv.norm"] = (s.width, d), (s.kv_rank,)
            out[q + "uk"], out[q + "uv"] = (s.heads * s.dim, s.kv_rank), (s.heads * s.vdim, s.kv_rank)
            if s.gated:
                out[q + "g"] = (s.heads, d)
            out[q + "o"] = (d, s.heads * s.vdim)
        else:
            n, r = int(m["heads"]) * int(m["dim"]), decay_rank(i)
            for x in ("r", "k", "v", "a", "g"):
                out[q + x] = (n, d)
            out[q + "w1"], out[q + "w2"] = (r, d), (n, r)
            out[q + "w0"] = out[q + "a.b"] = out[q + "norm"] = (n,)
            out[q + "o"] = (d, n)
        if e["mlp"] is not None:
            ff = int(e["mlp"]["ff"])
            out[p + "mlp.up"], out[p + "mlp.down"] = (ff, d), (d, ff)
    out["final.norm"], out["head"] = (d,), (cfg.vocab, d)
    return out


# ------------------------------------------------------------------------------------------ resident weights
@dataclass
class ZokuvikLayer:
    kind: str                                  # mixer type
    norm1: torch.Tensor                        # norm vectors are fp32
    norm1b: torch.Tensor
    in_proj: LinearWeight                      # latent: [dq or q | dkv | g]; delta: [r | k | v | a | g | w1]; rows padded to 8
    o: LinearWeight
    norm2: Optional[torch.Tensor] = None
    norm2b: Optional[torch.Tensor] = None
    up: Optional[LinearWeight] = None
    down: Optional[LinearWeight] = None
    latent: Optional[A.LatentSpec] = None
    inv_freq: Optional[torch.Tensor] = None
    uq: Optional[LinearWeight] = None
    q_norm: Optional[torch.Tensor] = None
    kv_norm: Optional[torch.Tensor] = None
    expand: Optional[LinearWeight] = None      # [heads * dim | heads * vdim, kv_rank]: W_uk, then W_uv
    uk: Optional[torch.Tensor] = None          # [heads, dim, kv_rank], a view of ``expand``
    uvt: Optional[torch.Tensor] = None         # [heads, kv_rank, vdim]
    delta: Optional[D.DeltaSpec] = None
    w2: Optional[LinearWeight] = None          # [heads * dim, rank padded to 8]
    w0: Optional[torch.Tensor] = None
    a_bias: Optional[torch.Tensor] = None
    out_norm: Optional[torch.Tensor] = None


@dataclass
class ZokuvikWeights:
    embed: torch.Tensor
    layers: list
    final_norm: torch.Tensor
    lm_head: LinearWeight
    vocab_offset: int = 0


def _pad_rows(w: torch.Tensor) -> torch.Tensor:
    pad = (-w.shape[0]) % 8
    return w if not pad else torch.cat([w, w.new_zeros((pad, w.shape[1]))], dim=0)


def pack_weights(cfg: ModelConfig, get: Callable, device) -> ZokuvikWeights:
    """``get(name)`` returns a source tensor (any float type, any device)."""
    device = torch.device(device)
    dt = torch.float32 if cfg.weight_format == "fp32" else torch.bfloat16
    shapes: dict = {}

    def fetch(name: str) -> torch.Tensor:
        t = get(name)
        if tuple(t.shape) != shapes[name]:
            raise ValueError(f"{name}: shape {tuple(t.shape)}, expected {shapes[name]}")
        return t

    def mat(*names, pad: bool = False) -> LinearWeight:
        w = torch.cat([fetch(n).to(device=device, dtype=dt) for n in names], dim=0)
        return LinearWeight("dense", (_pad_rows(w) if pad else w).contiguous())

    def vec(name):
        return fetch(name).to(device=device, dtype=torch.float32).contiguous()

    ranks = {i: int(get(f"l{i}.mix.w1").shape[0]) for i, e in enumerate(cfg.layer_specs) if e["type"] == _DELTA_FORM}
    shapes.update(source_shapes(cfg, ranks.__getitem__))
    layers = []
    for i, e in enumerate(cfg.layer_specs):
        p, q = f"l{i}.", f"l{i}.mix."
        kw = dict(kind=e["type"], norm1=vec(p + "norm1"), norm1b=vec(p + "norm1b"), o=mat(q + "o"))
        if e["mlp"] is not None:
            kw.update(norm2=vec(p + "norm2"), norm2b=vec(p + "norm2b"), up=mat(p + "mlp.up"), down=mat(p + "mlp.down"))
        if e["type"] in _LATENT_FORMS:
            s = latent_spec(e)
            names = [q + ("dq" if s.q_rank else "q"), q + "dkv"] + ([q + "g"] if s.gated else [])
            kw.update(latent=s, in_proj=mat(*names, pad=True), kv_norm=vec(q + "dkv.norm"), inv_freq=s.inv_freq(device),
                      expand=mat(q + "uk", q + "uv"))
            nk = s.heads * s.dim
            kw.update(uk=kw["expand"].w[:nk].view(s.heads, s.dim, s.kv_rank),
                      uvt=kw["expand"].w[nk:].view(s.heads, s.vdim, s.kv_rank).transpose(1, 2).contiguous())
            if s.q_rank:
                kw.update(uq=mat(q + "uq"), q_norm=vec(q + "dq.norm"))
        else:
            s = D.DeltaSpec(int(e["mixer"]["heads"]), int(e["mixer"]["dim"]), ranks[i])
            w2 = mat(q + "w2").w
            rank_pad = (s.rank + 7) // 8 * 8
            w2p = w2.new_zeros((w2.shape[0], rank_pad))
            w2p[:, :s.rank] = w2
            kw.update(delta=s, in_proj=mat(*(q + x for x in ("r", "k", "v", "a", "g", "w1")), pad=True),
                      w2=LinearWeight("dense", w2p), w0=vec(q + "w0"), a_bias=vec(q + "a.b"), out_norm=vec(q + "norm"))
        layers.append(ZokuvikLayer(**kw))
    embed = fetch("embed").to(device=device, dtype=dt).contiguous()
    return ZokuvikWeights(embed, layers, vec("final.norm"), mat("head"), 0)


def named_tensors(cfg: ModelConfig, w: ZokuvikWeights) -> Iterator:
    """(source name, tensor) of every tensor: the inverse of ``pack_weights``."""
    yield "embed", w.embed
    for i, (e, l) in enumerate(zip(cfg.layer_specs, w.layers)):
        p, q = f"l{i}.", f"l{i}.mix."
        yield p + "norm1", l.norm1
        yield p + "norm1b", l.norm1b
        if l.latent is not None:
            s = l.latent
            rows = [("dq", s.q_rank) if s.q_rank else ("q", s.heads * (s.dim + s.rot_dim)), ("dkv", s.width)]
            rows += [("g", s.heads)] if s.gated else []
            if s.q_rank:
                yield q + "uq", l.uq.w
                yield q + "dq.norm", l.q_norm
            yield q + "dkv.norm", l.kv_norm
            yield q + "uk", l.uk.reshape(s.heads * s.dim, s.kv_rank)
            yield q + "uv", l.uvt.transpose(1, 2).reshape(s.heads * s.vdim, s.kv_rank)
        else:
            s = l.delta
            rows = [(x, s.size) for x in ("r", "k", "v", "a", "g")] + [("w1", s.rank)]
            yield q + "w2", l.w2.w[:, :s.rank]
            yield q + "w0", l.w0
            yield q + "a.b", l.a_bias
            yield q + "norm", l.out_norm
        r0 = 0
        for name, n in rows:
            yield q + name, l.in_proj.w[r0:r0 + n]
            r0 += n
        yield q + "o", l.o.w
        if l.up is not None:
            yield p + "norm2", l.norm2
            yield p + "norm2b", l.norm2b
            yield p + "mlp.up", l.up.w
            yield p + "mlp.down", l.down.w
    yield "final.norm", w.final_norm
    yield "head", w.lm_head.w


def init_random_zokuvik_weights(cfg: ModelConfig, device, seed: int = 0, decay_rank: int = 64) -> ZokuvikWeights:
    """Seeded weights of the configured shape: matrices ~N(0, 1 / fan-in), norms near 1, drawn tensor by tensor on the
    target device (a generator per tensor, so the order of use does not matter)."""
    device = torch.device(device)
    shapes = source_shapes(cfg, lambda i: decay_rank)
    index = {n: k for k, n in enumerate(shapes)}

    def get(name):
        shape = shapes[name]
        gen = torch.Generator(device=device)
        gen.manual_seed(seed * 100003 + index[name])
        x = torch.randn(shape, generator=gen, device=device, dtype=torch.float32)
        if name.endswith("norm") or ".norm" in name:
            return 1.0 + 0.05 * x
        if len(shape) == 1:
            return 0.5 * x
        return x if name == "embed" else x * shape[1] ** -0.5
    return pack_weights(cfg, get, device)


# ------------------------------------------------------------------------------------------ model
class ZokuvikModel:
    """Stateless forward over a ForwardBatch; pages and states live in the LatentHybridCache passed in."""

    def __init__(self, cfg: ModelConfig, weights: ZokuvikWeights, tp=None):
        if tp is not None and tp.size != 1:
            raise ValueError("the zokuvik family runs on one GPU")
        self.cfg, self.w = cfg, weights
        self.tp = tp or NoTP()
        self.dtype = weights.embed.dtype

    @property
    def local_kv_heads(self) -> int:
        return 1

    def _latent(self, z, lw: ZokuvikLayer, b: ForwardBatch, kv):
        s = lw.latent
        proj = ops.linear(z, lw.in_proj)
        q_cols = s.q_rank or s.heads * (s.dim + s.rot_dim)
        cq = A.append(proj, 0, q_cols, s, lw.q_norm, lw.kv_norm, self.cfg.rms_eps, lw.inv_freq, kv, b.positions, b.seq_index,
                      b.block_table)
        q = ops.linear(cq, lw.uq) if s.q_rank else proj[:, :q_cols]
        gate = proj[:, q_cols + s.width:q_cols + s.width + s.heads] if s.gated else None
        return ops.linear(A.attention(q, gate, s, lw.uk, lw.uvt, lw.expand, lw.inv_freq, kv, b), lw.o)

    def _delta(self, z, lw: ZokuvikLayer, b: ForwardBatch, state):
        proj = ops.linear(z, lw.in_proj)
        one_each = b.num_tokens == b.slots.numel() and b.row_off_host is None
        y = D.general_delta(proj, lw.delta, lw.w2, lw.w0, lw.a_bias, lw.out_norm, self.cfg.rms_eps, state, b.row_off, b.slots, one_each)
        return ops.linear(y, lw.o)

    def hidden(self, b: ForwardBatch, cache) -> torch.Tensor:
        cfg, layers = self.cfg, self.w.layers
        eps, groups = cfg.rms_eps, cfg.norm_groups
        if b.row_off is None or b.slots is None:
            raise ValueError("the zokuvik family needs row offsets and state slots in the batch")
        if b.embeds is not None:
            raise ValueError("the zokuvik family takes token ids only")
        x, z = ops.embed_group_norm(self.w.embed, b.tokens, layers[0].norm1, eps, groups)
        for i, lw in enumerate(layers):
            y = self._latent(z, lw, b, cache.layer(i)) if lw.latent is not None else self._delta(z, lw, b, cache.state(i))
            after = layers[i + 1].norm1 if i + 1 < len(layers) else None
            z = ops.add_group_norm(x, y, lw.norm1b, lw.norm2 if lw.up is not None else after, eps, groups)
            if lw.up is not None:
                y = ops.linear(ops.linear(z, lw.up, act="relu_sq"), lw.down)
                z = ops.add_group_norm(x, y, lw.norm2b, after, eps, groups)
        return x

    def final_hidden(self, h: torch.Tensor, rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        """Final-normed rows of the residual stream in the activation type."""
        return ops.group_norm(h, self.w.final_norm, self.cfg.rms_eps, self.cfg.norm_groups, self.dtype, rows)

    def logits(self, h: torch.Tensor, b: ForwardBatch) -> torch.Tensor:
        return ops.linear(self.final_hidden(h, b.logit_rows), self.w.lm_head)

    def _keep(self, h: torch.Tensor) -> torch.Tensor:
        self.last_hidden = h
        return h

    def forward(self, b: ForwardBatch, cache) -> torch.Tensor:
        return self.logits(self._keep(self.hidden(b, cache)), b)

    def greedy(self, b: ForwardBatch, cache) -> torch.Tensor:
        return ops.argmax(self.forward(b, cache))


def make_cache(cfg: ModelConfig, model: ZokuvikModel, num_pages: int, device, max_seqs: int):
    from ..cache.latent import LatentHybridCache
    ls = model.w.layers
    return LatentHybridCache(cfg, num_pages, device, max_seqs,
                             {i: l.latent.width for i, l in enumerate(ls) if l.latent is not None},
                             {i: (l.delta.heads, l.delta.dim) for i, l in enumerate(ls) if l.delta is not None})


# ------------------------------------------------------------------------------------------ named shapes
def _entry(kind: str, ff: Optional[int], **mixer) -> dict:
    return {"type": kind, "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def shape_from_entries(name: str, entries: list, *, width: int, vocab: int, groups: int, eps: float = 1e-6,
                       max_context: int = 8192) -> ModelConfig:
    return config_from_source({"architecture": ARCHITECTURE, "layers": entries, "width": width, "vocab": vocab,
                               "norm": {"eps": eps, "groups": groups}}, name=name, max_context=max_context)


def zokuvik_shape(layers: int = 32, width: int = 2560, heads: int = 20, ff: int = 9216, window: int = 1024) -> ModelConfig:
    """A size whose layers resemble a served model's (benchmarks, random weights): every fourth layer is latent attention
    with heads of 128 + 64 channels and a latent of 512 - full and windowed ones in turn - the others are delta rules with
    heads of 128."""
    att = dict(heads=heads, dim=128, rot_dim=64, vdim=128, kv_rank=512, scale=192 ** -0.5)
    kinds = [_entry("latent_attention", ff, q_rank=1024, rot={"base": 1e6, "dims": 64}, **att),
             _entry("latent_attention_2", ff, rot={"base": 1e4, "dims": 64}, mask={"size": window}, **att)]
    delta = _entry("general_delta", ff, heads=heads, dim=128)
    entries = [kinds[(i // 4) % 2] if i % 4 == 3 else delta for i in range(layers)]
    return shape_from_entries("zokuvik", entries, width=width, vocab=151936, groups=1)


def tiny_zokuvik() -> ModelConfig:
    """CPU-checkable: one layer of every kind, a layer without feed-forward, uneven sizes."""
    return shape_from_entries("tiny-zokuvik", [
        _entry("general_delta", 80, heads=3, dim=24),
        _entry("latent_attention", None, heads=3, dim=16, rot_dim=24, vdim=40, kv_rank=48, q_rank=56, scale=0.2,
               rot={"base": 3e3, "dims": 24}),
        _entry("latent_attention_2", 104, heads=5, dim=24, rot_dim=8, vdim=16, kv_rank=64, scale=0.17, mask={"size": 21},
               rot={"base": 7e2, "dims": 8})], width=96, vocab=320, groups=3, max_context=512)
