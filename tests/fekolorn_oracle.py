"""Plain restatement of the Fekolorn design, one function per mechanism, whole sequences only, no cache.

It shares no code with the package: weights come as a dictionary name -> tensor, the configuration as the parsed
config.json, and everything is computed in the dtype of the weights (tests use float64).  It is slow on purpose: every
function is the equation it implements.
"""
from __future__ import annotations

import math

import torch


# ---------------------------------------------------------------- norms, activations
def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def poly_norm(z: torch.Tensor, coef: torch.Tensor, eps: float) -> torch.Tensor:
    """Three normed powers of z and a constant, weighted by coef [4]."""
    a, b, c, e = coef
    return a * rms(z, eps) + b * rms(z ** 2, eps) + c * rms(z ** 3, eps) + e


# ---------------------------------------------------------------- embedding
def bigram_row(prev, cur: int, spec: dict) -> int:
    """Row of the bigram table; prev is None at the start of a sequence."""
    if prev is None:
        return spec["buckets"]
    return (prev * spec["mul_prev"] + cur * spec["mul_cur"]) % spec["buckets"]


def embedding(tokens, cfg: dict, w: dict) -> torch.Tensor:
    spec = cfg["embedding"]
    out = []
    for i, t in enumerate(tokens):
        row = bigram_row(tokens[i - 1] if i else None, t, spec["bigram"])
        out.append(w["embed"][t] * spec["scale"] + w["bigram"][row])
    return torch.stack(out)


# ---------------------------------------------------------------- positions
def rotate(x: torch.Tensor, rot: dict) -> torch.Tensor:
    """x [T, heads, dim]: channels i and i + dims / 2 turn by position * base^(-2 i / dims)."""
    out, n = x.clone(), rot["dims"] // 2
    pos = torch.arange(x.shape[0], dtype=torch.float64)
    for i in range(n):
        a = pos * float(rot["base"]) ** (-2.0 * i / rot["dims"])
        c, s = torch.cos(a).to(x.dtype)[:, None], torch.sin(a).to(x.dtype)[:, None]
        u, v = x[..., i], x[..., i + n]
        out[..., i] = u * c - v * s
        out[..., i + n] = v * c + u * s
    return out


def bucket(n: int, rows: int, far: float) -> int:
    """Row of the distance-bias table for distance n: one row per distance up to half the table, then logarithmic, the last row
    at distance `far` and beyond."""
    near = rows // 2
    if n < near:
        return n
    return min(rows - 1, near + math.floor(math.log(n / near) / math.log(far / near) * (rows - near)))


def sees_window(i: int, j: int, size: int) -> bool:
    return 0 <= i - j < size


def visible(t: int, rule) -> torch.Tensor:
    return torch.tensor([[rule(i, j) for j in range(t)] for i in range(t)], dtype=torch.bool).view(t, t)


# ---------------------------------------------------------------- softmax attention
def softmax_sink(s: torch.Tensor, sink: float) -> torch.Tensor:
    """exp(s_j) / (exp(sink) + sum exp(s)) over the last dimension."""
    top = torch.clamp(s.max(-1, keepdim=True).values, min=float(sink))
    e = torch.exp(s - top)
    return e / (torch.exp(float(sink) - top) + e.sum(-1, keepdim=True))


def distance_bias(rel: torch.Tensor, far: float, t: int) -> torch.Tensor:
    """[H, t, t]: rel[bucket(i - j), h] for j <= i."""
    rows = torch.tensor([bucket(n, rel.shape[0], far) for n in range(t)])
    gap = (torch.arange(t)[:, None] - torch.arange(t)[None, :]).clamp(min=0)
    return rel[rows[gap]].permute(2, 0, 1)


def attend(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, seen: torch.Tensor, sinks, bias=None) -> torch.Tensor:
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim]; bias [H, T, T] joins the scaled scores."""
    t, H, G = q.shape[0], q.shape[1], k.shape[1]
    o = torch.empty(t, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        if bias is not None:
            s = s + bias[h]
        o[:, h] = softmax_sink(s.masked_fill(~seen, float("-inf")), sinks[h]) @ v[:, g]
    return o


def mixed_values(v: torch.Tensor, first, lam) -> torch.Tensor:
    """v between a layer's own values and the first such layer's (None: this is that layer)."""
    return v if first is None else (1 - lam) * v + lam * first


def window_attention(h: torch.Tensor, w: dict, p: str, m: dict, eps: float, first) -> tuple:
    """(output, the layer's own values [T, G * vdim]); first: the values to mix in, or None."""
    t, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = (rms(h @ w[p + "q"].T, eps) * w[p + "q.norm"]).view(t, H, m["dim"])
    k = (rms(h @ w[p + "k"].T, eps) * w[p + "k.norm"]).view(t, G, m["dim"])
    own = h @ w[p + "v"].T
    v = mixed_values(own, first, w.get(p + "vmix")).view(t, G, m["vdim"])
    seen = visible(t, lambda i, j: sees_window(i, j, m["mask"]["size"]))
    o = attend(q, k, v, m["scale"], seen, w[p + "sink"], distance_bias(w[p + "rel"], m["bias_max"], t))
    return o.reshape(t, -1) @ w[p + "o"].T, own


def rotary_attention(h: torch.Tensor, w: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    t, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = rotate((h @ w[p + "q"].T).view(t, H, m["dim"]), m["rot"])
    k = rotate((h @ w[p + "k"].T).view(t, G, m["dim"]), m["rot"])
    v = rms((h @ w[p + "v"].T).view(t, G, m["vdim"]), eps)
    o = attend(q, k, v, m["scale"], visible(t, lambda i, j: j <= i), w[p + "sink"])
    return o.reshape(t, -1) @ w[p + "o"].T


# ---------------------------------------------------------------- gated delta rule
def causal_conv(u: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """u [T, C], w [C, taps]; the last column of w meets the current token, zeros lie before the start."""
    taps = w.shape[1]
    y = torch.zeros_like(u)
    for t in range(u.shape[0]):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                y[t] += w[:, j] * u[s]
    return y


def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def head_decay(h: torch.Tensor, w: dict, p: str) -> torch.Tensor:
    return torch.exp(-torch.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))


def delta_states(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: torch.Tensor, beta: torch.Tensor) -> torch.Tensor:
    """S <- decay S, then S <- S + k (beta (v - S^T k))^T, o = S^T q.  q, k [T, H, dim], v [T, H, vdim], decay, beta [T, H]."""
    S = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=q.dtype)
    o = torch.empty_like(v)
    for t in range(q.shape[0]):
        S = decay[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = torch.einsum("hkv,hk->hv", S, q[t])
    return o


def gated_delta(h: torch.Tensor, w: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    t, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(h @ w[p + x].T, w[p + x + ".conv"])) for x in ("q", "k", "v"))
    q, k = unit(q.view(t, G, D)) * D ** -0.5, unit(k.view(t, G, D))
    q, k = (x.repeat_interleave(H // G, dim=1) for x in (q, k))
    o = delta_states(q, k, v.view(t, H, V), head_decay(h, w, p), torch.sigmoid(h @ w[p + "b"].T))
    return ((rms(o, eps) * w[p + "norm"]).reshape(t, -1) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


# ---------------------------------------------------------------- streams
def read(streams: list, weights) -> torch.Tensor:
    return sum(a * x for a, x in zip(weights, streams))


def write(streams: list, y: torch.Tensor, mix: torch.Tensor, out) -> list:
    """New stream t: what flows into it from every old stream (mix [from, to]) and its share of y."""
    n = len(streams)
    return [sum(mix[s, t] * streams[s] for s in range(n)) + out[t] * y for t in range(n)]


# ---------------------------------------------------------------- model
def forward(tokens, cfg: dict, w: dict, layers_out: list = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence."""
    tokens, eps = [int(t) for t in tokens], cfg["norm"]["eps"]
    streams = [embedding(tokens, cfg, w) for _ in range(cfg["streams"])]
    first = None
    for i, spec in enumerate(cfg["layers"]):
        p, m = f"l{i}.", spec["mixer"]
        h = rms(read(streams, w[p + "hc1.in"]), eps) * w[p + "norm1"]
        if spec["type"] == "attention":
            y, own = window_attention(h, w, p + "mix.", m, eps, first if m.get("v_mix") else None)
            if first is None and m.get("v_mix"):
                first = own
        else:
            y = m["left_scale"] * rotary_attention(h, w, p + "mix.left.", m["left"], eps) + \
                m["right_scale"] * gated_delta(h, w, p + "mix.right.", m["right"], eps)
        streams = write(streams, y, w[p + "hc1.mix"], w[p + "hc1.out"])
        if spec["mlp"] is not None:
            h = rms(read(streams, w[p + "hc2.in"]), eps) * w[p + "norm2"]
            y = poly_norm(h @ w[p + "mlp.up"].T, w[p + "mlp.act"], eps) @ w[p + "mlp.down"].T
            streams = write(streams, y, w[p + "hc2.mix"], w[p + "hc2.out"])
        if layers_out is not None:
            layers_out.append(sum(streams))
    return (rms(sum(streams), eps) * w["final.norm"]) @ w["head"].T
