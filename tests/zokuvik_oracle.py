"""Plain restatement of the Zokuvik design, one function per mechanism, whole sequences only, no cache.

It shares no code with the package: weights come as a dictionary name -> tensor, the configuration as the parsed
config.json, and everything is computed in the dtype of the weights (tests use float64 or float32).  It is slow on
purpose: every function is the equation it implements.
"""
from __future__ import annotations

import json
import math
import struct

import torch


def read_safetensors(path: str, dtype=torch.float64) -> dict:
    """name -> tensor of a safetensors file that holds BF16 / F32 tensors."""
    with open(path, "rb") as f:
        raw = f.read()
    n = struct.unpack("<Q", raw[:8])[0]
    head = json.loads(raw[8:8 + n])
    out = {}
    for name, e in head.items():
        if name == "__metadata__":
            continue
        a, b = e["data_offsets"]
        dt = {"BF16": torch.bfloat16, "F32": torch.float32}[e["dtype"]]
        out[name] = torch.frombuffer(bytearray(raw[8 + n + a:8 + n + b]), dtype=dt).view(e["shape"]).to(dtype)
    return out


# ---------------------------------------------------------------- norms
def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def group_norm(x: torch.Tensor, w: torch.Tensor, eps: float, groups: int) -> torch.Tensor:
    t, d = x.shape
    return rms(x.view(t, groups, d // groups), eps).reshape(t, d) * w


# ---------------------------------------------------------------- rotation
def rotate(x: torch.Tensor, pos: torch.Tensor, dims: int, base: float, interleaved: bool) -> torch.Tensor:
    """x [T, H, R]; the first `dims` channels turn, in pairs (2i, 2i+1) or (i, i + dims/2)."""
    out = x.clone()
    for i in range(dims // 2):
        a = pos.to(torch.float64) * float(base) ** (-2.0 * i / dims)
        c, s = torch.cos(a).to(x.dtype)[:, None], torch.sin(a).to(x.dtype)[:, None]
        iu, iv = (2 * i, 2 * i + 1) if interleaved else (i, i + dims // 2)
        u, v = x[..., iu], x[..., iv]
        out[..., iu] = u * c - v * s
        out[..., iv] = v * c + u * s
    return out


# ---------------------------------------------------------------- latent attention
def latent_attention(h: torch.Tensor, w: dict, p: str, m: dict, eps: float, interleaved: bool) -> torch.Tensor:
    """The two latent-attention mixers.  A query latent is used when `<p>dq` exists, an output gate when `<p>g` does,
    a sliding window when the mixer has `mask`."""
    t = h.shape[0]
    H, D, R, V, C = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(t)
    if p + "dq" in w:
        q = (rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]) @ w[p + "uq"].T
    else:
        q = h @ w[p + "q"].T
    q = q.view(t, H, D + R)
    q_n, q_r = q[..., :D], rotate(q[..., D:], pos, m["rot"]["dims"], m["rot"]["base"], interleaved)
    kv = h @ w[p + "dkv"].T
    c = rms(kv[:, :C], eps) * w[p + "dkv.norm"]
    k_r = rotate(kv[:, None, C:], pos, m["rot"]["dims"], m["rot"]["base"], interleaved)[:, 0]
    k_n = (c @ w[p + "uk"].T).view(t, H, D)
    v = (c @ w[p + "uv"].T).view(t, H, V)
    s = (torch.einsum("ihd,jhd->hij", q_n, k_n) + torch.einsum("ihr,jr->hij", q_r, k_r)) * m["scale"]
    gap = pos[:, None] - pos[None, :]
    seen = gap >= 0
    if "mask" in m:
        seen = seen & (gap < m["mask"]["size"])
    s = s.masked_fill(~seen, float("-inf"))
    o = torch.einsum("hij,jhv->ihv", torch.softmax(s, dim=-1), v)
    if p + "g" in w:
        o = o * torch.sigmoid(h @ w[p + "g"].T)[..., None]
    return o.reshape(t, H * V) @ w[p + "o"].T


# ---------------------------------------------------------------- generalised delta rule
def delta_step(S, r, k, v, decay, a):
    """One token of one head: S [key, value]; returns (new S, output)."""
    u = k / torch.sqrt((k * k).sum() + 1e-6)
    S = decay[:, None] * S - (a * u)[:, None] * (u @ S)[None, :] + k[:, None] * v[None, :]
    return S, S.T @ r


def delta_inputs(h, w, p):
    r, k, v = h @ w[p + "r"].T, h @ w[p + "k"].T, h @ w[p + "v"].T
    x = torch.tanh(h @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"]
    decay = torch.exp(-math.exp(-0.5) * torch.sigmoid(x))
    a = torch.sigmoid(h @ w[p + "a"].T + w[p + "a.b"])
    return r, k, v, decay, a


def general_delta(h: torch.Tensor, w: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    t = h.shape[0]
    H, D = m["heads"], m["dim"]
    r, k, v, decay, a = (x.view(t, H, D) for x in delta_inputs(h, w, p))
    S = torch.zeros(H, D, D, dtype=h.dtype)
    o = torch.empty(t, H, D, dtype=h.dtype)
    for i in range(t):
        u = k[i] / torch.sqrt((k[i] * k[i]).sum(-1, keepdim=True) + 1e-6)
        S = decay[i][..., None] * S - (a[i] * u)[..., None] * torch.einsum("hk,hkv->hv", u, S)[:, None, :] \
            + k[i][..., None] * v[i][:, None, :]
        o[i] = torch.einsum("hkv,hk->hv", S, r[i])
    y = rms(o, eps).reshape(t, H * D) * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)
    return y @ w[p + "o"].T


# ---------------------------------------------------------------- feed-forward, layer, model
def feed_forward(h: torch.Tensor, w: dict, p: str) -> torch.Tensor:
    return torch.relu(h @ w[p + "up"].T) ** 2 @ w[p + "down"].T


def mixer(h, w, p, spec, eps):
    kind, m = spec["type"], spec["mixer"]
    if kind == "latent_attention":
        return latent_attention(h, w, p, m, eps, interleaved=True)
    if kind == "latent_attention_2":
        return latent_attention(h, w, p, m, eps, interleaved=False)
    if kind == "general_delta":
        return general_delta(h, w, p, m, eps)
    raise ValueError(kind)


def layer(x, w, i, spec, eps, groups):
    p = f"l{i}."
    gn = lambda z, name: group_norm(z, w[p + name], eps, groups)
    x = x + gn(mixer(gn(x, "norm1"), w, p + "mix.", spec, eps), "norm1b")
    if spec["mlp"] is not None:
        x = x + gn(feed_forward(gn(x, "norm2"), w, p + "mlp."), "norm2b")
    return x


def forward(tokens, cfg: dict, w: dict, layers_out: list = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence."""
    x = w["embed"][torch.as_tensor(tokens)]
    eps, groups = cfg["norm"]["eps"], cfg["norm"]["groups"]
    for i, spec in enumerate(cfg["layers"]):
        x = layer(x, w, i, spec, eps, groups)
        if layers_out is not None:
            layers_out.append(x)
    return group_norm(x, w["final.norm"], eps, groups) @ w["head"].T
