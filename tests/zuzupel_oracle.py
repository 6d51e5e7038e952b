"""Plain, slow implementation of the Zuzupel design (CPU, torch, one function per mechanism).

Works on a configuration dictionary and a flat name -> tensor dictionary, token by token where the mechanism is
sequential, with no caches, no fusion and nothing shared with the package.  ``dtype`` is the arithmetic type
(float64 by default: the oracle's own rounding then never matters).

Notation: h is a sublayer's input [T, W]; p is a mixer's tensor prefix (it ends with a dot).
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

Tensors = Dict[str, torch.Tensor]


# --------------------------------------------------------------------------- small pieces
def rms(x: torch.Tensor, w, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def layer_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def sigmoid(z: torch.Tensor) -> torch.Tensor:
    return 1 / (1 + torch.exp(-z))


def log_sigmoid(z: torch.Tensor) -> torch.Tensor:
    return -softplus(-z)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * sigmoid(z)


def softplus(z: torch.Tensor) -> torch.Tensor:
    return z.clamp(min=0) + torch.log1p(torch.exp(-z.abs()))


def relu2(z: torch.Tensor) -> torch.Tensor:
    return z.clamp(min=0) ** 2


def causal_conv(x: torch.Tensor, k: torch.Tensor) -> torch.Tensor:
    """Per-channel causal convolution without a bias; the last column of ``k`` [channels, taps] meets the current token."""
    taps = k.shape[1]
    out = torch.zeros_like(x)
    for back in range(min(taps, x.shape[0])):
        out[back:] += k[:, taps - 1 - back] * x[: x.shape[0] - back]
    return out


# --------------------------------------------------------------------------- recurrences over one head
def delta_rule(q, k, v, beta, g):
    """q, k, g [T, D], v [T, V], beta [T].  The state's rows fade by g, then it is corrected towards v at k."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype)
    out = torch.zeros_like(v)
    for t in range(q.shape[0]):
        S = g[t][:, None] * S
        S = S + torch.outer(k[t], beta[t] * (v[t] - k[t] @ S))
        out[t] = q[t] @ S
    return out


def wkv_rule(r, k, v, w, u):
    """r, k, w [T, D], v [T, V], u [D].  The current token enters the read-out through u, the state without it."""
    S = torch.zeros(r.shape[1], v.shape[1], dtype=r.dtype)
    out = torch.zeros_like(v)
    for t in range(r.shape[0]):
        kv = torch.outer(k[t], v[t])
        out[t] = r[t] @ (S + u[:, None] * kv)
        S = w[t][:, None] * S + kv
    return out


def mlstm_rule(q, k, v, i, f):
    """q, k [T, D], v [T, V], log gates i, f [T]: stabilised matrix memory with a normaliser."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype)
    n = torch.zeros(q.shape[1], dtype=q.dtype)
    m = torch.zeros((), dtype=q.dtype)
    out = torch.zeros_like(v)
    for t in range(q.shape[0]):
        new = torch.maximum(f[t] + m, i[t])
        a, b = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        S, n, m = a * S + b * torch.outer(k[t], v[t]), a * n + b * k[t], new
        out[t] = (q[t] @ S) / (torch.maximum((n @ q[t]).abs(), torch.exp(-m)) + 1e-6)
    return out


# --------------------------------------------------------------------------- mixers
def channel_delta(h, w: Tensors, p: str, m: dict, eps: float):
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def branch(n):
        return silu(causal_conv(h @ w[p + n].T, w[p + n + ".conv"]))

    q, k = unit(branch("q").view(T, G, D)) * D ** -0.5, unit(branch("k").view(T, G, D))
    v = branch("v").view(T, H, V)
    beta = sigmoid(h @ w[p + "b"].T)
    rate = softplus((h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]).view(T, H, D)
    g = torch.exp(-torch.exp(w[p + "A_log"])[:, None] * rate)
    o = torch.stack([delta_rule(q[:, j * G // H], k[:, j * G // H], v[:, j], beta[:, j], g[:, j]) for j in range(H)], 1)
    gate = sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T).view(T, H, V)
    return (rms(o, w[p + "norm"], eps) * gate).reshape(T, H * V) @ w[p + "o"].T


def wkv(h, w: Tensors, p: str, m: dict, eps: float):
    T, H, D = h.shape[0], m["heads"], m["dim"]
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])

    def mix(s):
        return h + (before - h) * w[p + "mu." + s]

    r, k, v = ((mix(s) @ w[p + s].T).view(T, H, D) for s in "rkv")
    gate = silu(mix("g") @ w[p + "g"].T)
    decay = torch.exp(-torch.exp(torch.tanh(mix("w") @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"])).view(T, H, D)
    o = torch.stack([wkv_rule(r[:, j], k[:, j], v[:, j], decay[:, j], w[p + "u"][j]) for j in range(H)], 1)
    return (rms(o, 1, eps).reshape(T, H * D) * w[p + "norm"] * gate) @ w[p + "o"].T


def rotate(x, rot: dict):
    """x [T, heads, dim]: the first ``dims`` of every head turned by position, halves paired."""
    half = rot["dims"] // 2
    f = torch.tensor([rot["base"] ** (-2 * i / rot["dims"]) / rot["scaling"]["factor"] for i in range(half)], dtype=x.dtype)
    a = torch.arange(x.shape[0], dtype=x.dtype)[:, None, None] * f
    u, v, rest = x[..., :half], x[..., half: 2 * half], x[..., 2 * half:]
    return torch.cat([u * torch.cos(a) - v * torch.sin(a), v * torch.cos(a) + u * torch.sin(a), rest], -1)


def visible(i: int, size: int) -> range:
    """Keys that position i sees: those of its own chunk up to itself."""
    return range(i // size * size, i + 1)


def chunk_attention(h, w: Tensors, p: str, m: dict, eps: float):
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T + w[p + "q.b"]).view(T, H, D)
    k = (h @ w[p + "k"].T + w[p + "k.b"]).view(T, G, D)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).view(T, G, V)
    q, k = rotate(rms(q, w[p + "q.norm"], eps), m["rot"]), rotate(rms(k, w[p + "k.norm"], eps), m["rot"])
    out = torch.zeros(T, H, V, dtype=h.dtype)
    for i in range(T):
        js = visible(i, m["mask"]["size"])
        for j in range(H):
            g = j * G // H
            s = k[js.start:js.stop, g] @ q[i, j] * m["scale"]
            e = torch.exp(s - s.max())
            out[i, j] = (e / e.sum()) @ v[js.start:js.stop, g]
    return out.reshape(T, H * V) @ w[p + "o"].T


def mlstm(h, w: Tensors, p: str, m: dict, eps: float):
    T, H, D, V, cap = h.shape[0], m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q, k = (h @ w[p + "q"].T).view(T, H, D) * D ** -0.5, (h @ w[p + "k"].T).view(T, H, D)
    v = (h @ w[p + "v"].T).view(T, H, V)
    i = cap * torch.tanh((h @ w[p + "i"].T + w[p + "i.b"]) / cap)
    f = log_sigmoid(cap * torch.tanh((h @ w[p + "f"].T + w[p + "f.b"]) / cap))
    o = torch.stack([mlstm_rule(q[:, j], k[:, j], v[:, j], i[:, j], f[:, j]) for j in range(H)], 1)
    return (rms(o, 1, eps).reshape(T, H * V) * w[p + "norm"] * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def parallel(h, w: Tensors, p: str, m: dict, eps: float):
    left = rms(chunk_attention(h, w, p + "left.", m["left"], eps), w[p + "left.out"], eps)
    right = rms(mlstm(h, w, p + "right.", m["right"], eps), w[p + "right.out"], eps)
    return (left + right) / 2


MIXERS = {"channel_delta": channel_delta, "wkv": wkv, "parallel": parallel}


# --------------------------------------------------------------------------- model
def owner(cfg: dict, i: int) -> int:
    """The layer whose tensors layer i uses."""
    j = cfg["layers"][i].get("weights_of")
    return i if j is None else owner(cfg, j)


def forward(cfg: dict, weights: Tensors, tokens: List[int], dtype=torch.float64, trace: Optional[list] = None) -> torch.Tensor:
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.tensor(tokens)]
    for i in range(len(cfg["layers"])):
        j = owner(cfg, i)
        layer, p = cfg["layers"][j], f"l{j}."
        x = x + layer_norm(MIXERS[layer["type"]](x, w, p + "mix.", layer["mixer"], eps), w[p + "norm1"], eps)
        if layer.get("mlp"):
            x = x + layer_norm(relu2(x @ w[p + "mlp.up"].T) @ w[p + "mlp.down"].T, w[p + "norm2"], eps)
        if trace is not None:
            trace.append(x.clone())
    return layer_norm(x, w["final.norm"], eps) @ w["head"].T
