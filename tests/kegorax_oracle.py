"""Plain restatement of the Kegorax design, one function per mechanism, whole sequences only, no cache.

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


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


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


def slope(h: int, heads: int) -> float:
    return 2.0 ** (-8.0 * (h + 1) / heads)


def sees_chunk(i: int, j: int, size: int) -> bool:
    return j <= i and i // size == j // size


def sees_window(i: int, j: int, size: int, keep: int) -> bool:
    return j <= i and (i - j < size or j < keep)


def visible(t: int, rule) -> torch.Tensor:
    return torch.tensor([[rule(i, j) for j in range(t)] for i in range(t)], dtype=torch.bool).view(t, t)


# ---------------------------------------------------------------- softmax attention
def softmax_sink(s: torch.Tensor, sink: float) -> torch.Tensor:
    """exp(s_j) / (exp(sink) + sum exp(s)) over the last dimension."""
    top = torch.clamp(s.max(-1, keepdim=True).values, min=float(sink))
    e = torch.exp(s - top)
    return e / (torch.exp(float(sink) - top) + e.sum(-1, keepdim=True))


def attend(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, seen: torch.Tensor, sinks, slopes=None) -> torch.Tensor:
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim] -> [T, H, vdim]."""
    t, H, G = q.shape[0], q.shape[1], k.shape[1]
    gap = (torch.arange(t)[:, None] - torch.arange(t)[None, :]).to(q.dtype)
    o = torch.empty(t, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        if slopes is not None:
            s = s - slopes[h] * gap
        o[:, h] = softmax_sink(s.masked_fill(~seen, float("-inf")), sinks[h]) @ v[:, g]
    return o


def chunk_attention(h: torch.Tensor, w: dict, p: str, m: dict) -> torch.Tensor:
    t, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = rotate((h @ w[p + "q"].T).view(t, H, m["dim"]), m["rot"])
    k = rotate((h @ w[p + "k"].T).view(t, G, m["dim"]), m["rot"])
    v = (h @ w[p + "v"].T).view(t, G, m["vdim"])
    seen = visible(t, lambda i, j: sees_chunk(i, j, m["mask"]["size"]))
    o = attend(q, k, v, m["scale"], seen, w[p + "sink"])
    o = o * torch.sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(t, -1) @ w[p + "o"].T


def window_attention(h: torch.Tensor, w: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    t, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = rms((h @ w[p + "q"].T + w[p + "q.b"]).view(t, H, m["dim"]), eps) * w[p + "q.norm"]
    k = rms((h @ w[p + "k"].T + w[p + "k.b"]).view(t, G, m["dim"]), eps) * w[p + "k.norm"]
    v = (h @ w[p + "v"].T + w[p + "v.b"]).view(t, G, m["vdim"])
    seen = visible(t, lambda i, j: sees_window(i, j, m["mask"]["size"], m["mask"]["keep_first"]))
    o = attend(q, k, v, m["scale"], seen, [0.0] * H, [slope(x, H) for x in range(H)])
    return o.reshape(t, -1) @ w[p + "o"].T


# ---------------------------------------------------------------- recurrences
def linear_states(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: torch.Tensor) -> torch.Tensor:
    """S <- diag(decay_t) S + k v^T, o = S^T q.  q, k, decay [T, H, dim], v [T, H, vdim]."""
    S = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=q.dtype)
    o = torch.empty_like(v)
    for t in range(q.shape[0]):
        S = decay[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hkv,hk->hv", S, q[t])
    return o


def delta_states(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: torch.Tensor, beta: torch.Tensor) -> torch.Tensor:
    """S <- diag(decay_t) S, then S <- S + k (beta (v - S^T k))^T, o = S^T q.  beta [T, H]."""
    S = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=q.dtype)
    o = torch.empty_like(v)
    for t in range(q.shape[0]):
        S = decay[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = torch.einsum("hkv,hk->hv", S, q[t])
    return o


def gated_linear(h: torch.Tensor, w: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    t, H, D = h.shape[0], m["heads"], m["dim"]
    q = (h @ w[p + "q"].T).view(t, H, D) * D ** -0.5
    k = (h @ w[p + "k"].T).view(t, H, D)
    v = (h @ w[p + "v"].T).view(t, H, m["vdim"])
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]
    o = linear_states(q, k, v, (torch.sigmoid(z) ** (1.0 / m["tau"])).view(t, H, D))
    o = (rms(o, eps) * w[p + "norm"]).reshape(t, -1)
    return (o * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def retention(h: torch.Tensor, w: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    t, H, D = h.shape[0], m["heads"], m["dim"]
    q = (h @ w[p + "q"].T).view(t, H, D)
    k = (h @ w[p + "k"].T).view(t, H, D) * D ** -0.5
    v = (h @ w[p + "v"].T).view(t, H, m["vdim"])
    o = linear_states(q, k, v, torch.tensor(m["decay"], dtype=h.dtype)[None, :, None].expand(t, H, D))
    return (rms(o, eps).reshape(t, -1) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


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


def channel_decay(h: torch.Tensor, w: dict, p: str, heads: int, dim: int) -> torch.Tensor:
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]
    sp = torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))
    return torch.exp(-torch.exp(w[p + "A_log"])[None, :, None] * sp.view(h.shape[0], heads, dim))


def channel_delta(h: torch.Tensor, w: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    t, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(h @ w[p + x].T, w[p + x + ".conv"])) for x in ("q", "k", "v"))
    q, k = unit(q.view(t, G, D)) * D ** -0.5, unit(k.view(t, G, D))
    q, k = (x.repeat_interleave(H // G, dim=1) for x in (q, k))
    o = delta_states(q, k, v.view(t, H, V), channel_decay(h, w, p, H, D), torch.sigmoid(h @ w[p + "b"].T))
    gate = torch.sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T).view(t, H, V)
    return (rms(o, eps) * w[p + "norm"] * gate).reshape(t, -1) @ w[p + "o"].T


# ---------------------------------------------------------------- mixers of a layer
def mixer(kind: str, h: torch.Tensor, w: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    if kind == "channel_delta":
        return channel_delta(h, w, p, m, eps)
    if kind == "parallel":
        left, right = chunk_attention(h, w, p + "left.", m["left"]), gated_linear(h, w, p + "right.", m["right"], eps)
        return 0.5 * (rms(left, eps) * w[p + "left.out"] + rms(right, eps) * w[p + "right.out"])
    left, right = window_attention(h, w, p + "left.", m["left"], eps), retention(h, w, p + "right.", m["right"], eps)
    return m["left_scale"] * left + m["right_scale"] * right


# ---------------------------------------------------------------- feed-forward
def dense(h: torch.Tensor, w: dict, p: str) -> torch.Tensor:
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def expert(h: torch.Tensor, w: dict, p: str) -> torch.Tensor:
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(z: torch.Tensor, correction: torch.Tensor, r: dict) -> list:
    """[(expert, weight)] of one token with logits z [E], the largest choice score first."""
    s = torch.sigmoid(z)
    c = (s + correction).tolist()
    gr = r.get("groups") or {"count": 1, "keep": 1}
    size = len(c) // gr["count"]
    score = [sum(sorted(c[g * size:(g + 1) * size], reverse=True)[:2]) for g in range(gr["count"])]
    best = sorted(range(gr["count"]), key=lambda g: -score[g])[:gr["keep"]]
    allowed = [e for e in range(len(c)) if e // size in best]
    return [(e, s[e] * r["scale"]) for e in sorted(allowed, key=lambda e: -c[e])[:r["top"]]]


def experts(h: torch.Tensor, w: dict, p: str, spec: dict) -> torch.Tensor:
    z = h @ w[p + "router"].T
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in route(z[t], w[p + "correction"], spec["router"]):
            y[t] += s * expert(h[t:t + 1], w, f"{p}e{e}.")[0]
    return y


# ---------------------------------------------------------------- model
def order(cfg: dict) -> list:
    """[(layer, pass)] in the order in which they run; pass is None outside the loop."""
    loop = cfg.get("loop")
    n = len(cfg["layers"])
    if not loop:
        return [(i, None) for i in range(n)]
    out = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        out += [(i, t) for i in range(loop["start"], loop["stop"])]
    return out + [(i, None) for i in range(loop["stop"], n)]


def forward(tokens, cfg: dict, w: dict, layers_out: list = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence."""
    emb = w["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    x, eps = emb, cfg["norm"]["eps"]
    for i, t in order(cfg):
        if t is not None and i == cfg["loop"]["start"]:
            if t > 0:
                x = x + emb
            x = x + w["loop.step"][t]
        p, spec = f"l{i}.", cfg["layers"][i]
        x = x + mixer(spec["type"], rms(x, eps) * w[p + "norm1"], w, p + "mix.", spec["mixer"], eps)
        if spec["mlp"] is not None:
            h = rms(x, eps) * w[p + "norm2"]
            x = x + (dense(h, w, p + "mlp.") if spec["mlp"]["kind"] == "dense" else experts(h, w, p + "mlp.", spec["mlp"]))
        if layers_out is not None:
            layers_out.append(x)
    return (rms(x, eps) * w["final.norm"]) @ w["embed"].T
