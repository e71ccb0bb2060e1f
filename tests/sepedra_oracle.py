"""Plain restatement of the Sepedra design, one function per mechanism, whole sequences only, no cache.

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


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


# ---------------------------------------------------------------- short convolution
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


# ---------------------------------------------------------------- rotation
def frequency(i: int, rot: dict) -> float:
    """Turning rate of pair i, with the banded scaling of long-context models."""
    f = float(rot["base"]) ** (-2.0 * i / rot["dims"])
    sc = rot.get("scaling")
    if not sc:
        return f
    wave = 2 * math.pi / f
    if wave < sc["original"] / sc["high"]:
        return f
    if wave > sc["original"] / sc["low"]:
        return f / sc["factor"]
    s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
    return (1 - s) * f / sc["factor"] + s * f


def rotate(x: torch.Tensor, rot: dict) -> torch.Tensor:
    """x [T, H, D] at positions 0 .. T - 1; channels 2i and 2i + 1 of the first rot.dims turn together."""
    out = x.clone()
    pos = torch.arange(x.shape[0], dtype=torch.float64)
    for i in range(rot["dims"] // 2):
        a = pos * frequency(i, rot)
        c, s = torch.cos(a).to(x.dtype)[:, None], torch.sin(a).to(x.dtype)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


# ---------------------------------------------------------------- gated linear recurrence
def rglru_gates(u: torch.Tensor, w: dict, p: str, blocks: int):
    """(decay a, input term b) of the recurrence S <- a S + b for every token."""
    t, n = u.shape
    x = u.view(t, blocks, n // blocks)
    r = torch.sigmoid(torch.einsum("tbi,boi->tbo", x, w[p + "ra"]) + w[p + "ra.b"]).reshape(t, n)
    g = torch.sigmoid(torch.einsum("tbi,boi->tbo", x, w[p + "ri"]) + w[p + "ri.b"]).reshape(t, n)
    a = torch.exp(-8 * r * torch.log1p(torch.exp(w[p + "lam"])))
    return a, torch.sqrt(1 - a * a) * g * u


def rglru(h: torch.Tensor, w: dict, p: str, m: dict) -> torch.Tensor:
    y = gelu_tanh(h @ w[p + "y"].T + w[p + "y.b"])
    u = causal_conv(h @ w[p + "x"].T + w[p + "x.b"], w[p + "conv"]) + w[p + "conv.b"]
    a, b = rglru_gates(u, w, p, m["blocks"])
    S, out = torch.zeros_like(u[0]), torch.empty_like(u)
    for t in range(h.shape[0]):
        S = a[t] * S + b[t]
        out[t] = S
    return (out * y) @ w[p + "o"].T


# ---------------------------------------------------------------- attention
def keys_values(h: torch.Tensor, w: dict, p: str, m: dict, eps: float):
    t, G = h.shape[0], m["kv_heads"]
    k = causal_conv(h @ w[p + "k"].T, w[p + "k.conv"]).view(t, G, m["dim"])
    v = causal_conv(h @ w[p + "v"].T, w[p + "v.conv"]).view(t, G, m["vdim"])
    return rms(rotate(k, m["rot"]), eps), v


def softmax_one(s: torch.Tensor) -> torch.Tensor:
    """exp(s_j) / (1 + sum exp(s)) over the last dimension."""
    top = torch.clamp(s.max(-1, keepdim=True).values, min=0)
    e = torch.exp(s - top)
    return e / (torch.exp(-top) + e.sum(-1, keepdim=True))


def attention(h: torch.Tensor, w: dict, p: str, m: dict, eps: float, kv) -> torch.Tensor:
    """kv: (keys [T, G, dim], values [T, G, vdim]) of this layer or of the one it takes them from."""
    t, H, G = h.shape[0], m["heads"], m["kv_heads"]
    k, v = kv
    q = causal_conv(h @ w[p + "q"].T, w[p + "q.conv"]).view(t, H, m["dim"])
    q = rms(rotate(q, m["rot"]), eps)
    o = torch.empty(t, H, v.shape[2], dtype=h.dtype)
    for x in range(H):
        g = x // (H // G)
        s = (q[:, x] @ k[:, g].T) * m["scale"]
        s = s.masked_fill(torch.arange(t)[None, :] > torch.arange(t)[:, None], float("-inf"))
        o[:, x] = softmax_one(s) @ v[:, g]
    return (o.reshape(t, -1) * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


# ---------------------------------------------------------------- experts
def expert(h: torch.Tensor, w: dict, p: str, limit: float) -> torch.Tensor:
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ w[p + "down"].T


def route(z: torch.Tensor, r: dict) -> list:
    """[(expert, weight)] of one token with logits z [E]."""
    s = torch.softmax(z, -1)
    E = z.shape[0]
    gr = r.get("groups") or {"count": 1, "keep": 1}
    size = E // gr["count"]
    best = sorted(range(gr["count"]), key=lambda g: -float(s[g * size:(g + 1) * size].max()))[:gr["keep"]]
    allowed = [e for e in range(E) if e // size in best]
    chosen = sorted(allowed, key=lambda e: -float(s[e]))[:r["top"]]
    return [(e, s[e]) for e in chosen]


def experts(h: torch.Tensor, w: dict, p: str, spec: dict) -> torch.Tensor:
    z = h @ w[p + "router"].T
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in route(z[t], spec["router"]):
            y[t] += s * expert(h[t:t + 1], w, f"{p}e{e}.", spec["expert"]["limit"])[0]
    return y


# ---------------------------------------------------------------- model
def forward(tokens, cfg: dict, w: dict, layers_out: list = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence."""
    x = w["embed"][torch.as_tensor(tokens)]
    eps, held = cfg["norm"]["eps"], {}
    for i, spec in enumerate(cfg["layers"]):
        p, m = f"l{i}.", spec["mixer"]
        if spec["type"] == "rglru":
            y = rglru(x, w, p + "mix.", m)
        else:
            src = m.get("kv_from")
            if src is None:
                held[i] = keys_values(x, w, p + "mix.", m, eps)
                src = i
            y = attention(x, w, p + "mix.", m, eps, held[src])
        x = x + rms(y, eps) * w[p + "norm1"]
        if spec["mlp"] is not None:
            x = x + rms(experts(x, w, p + "mlp.", spec["mlp"]), eps) * w[p + "norm2"]
        if layers_out is not None:
            layers_out.append(x)
    z = (rms(x, eps) * w["final.norm"]) @ w["head"].T
    cap = cfg.get("logit_softcap")
    return cap * torch.tanh(z / cap) if cap else z
