"""Plain, slow implementation of the Tumatar design (CPU, torch, one function per mechanism).

Works on a configuration dictionary and a flat name -> tensor dictionary, token by token where the mechanism is
sequential, with no caches, no fusion and nothing shared with the package.  ``dtype`` is the arithmetic type
(float64 by default: the oracle's own rounding then never matters).

Notation: h is a sublayer's normed input [T, W]; p is a layer's tensor prefix.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

Tensors = Dict[str, torch.Tensor]


def rms(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def sigmoid(z: torch.Tensor) -> torch.Tensor:
    return 1 / (1 + torch.exp(-z))


def latent_attention(h: torch.Tensor, w: Tensors, p: str, m: dict, eps: float) -> torch.Tensor:
    """Queries through a latent, keys and values of every head from one normed latent per token, causal softmax,
    heads gated element by element by the sublayer's input.  No positions enter."""
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    cq = rms(h @ w[p + "dq"].T, w[p + "dq.norm"], eps)
    q = (cq @ w[p + "uq"].T).view(T, H, D)
    c = rms(h @ w[p + "dkv"].T, w[p + "dkv.norm"], eps)
    k = (c @ w[p + "uk"].T).view(T, H, D)
    v = (c @ w[p + "uv"].T).view(T, H, V)
    out = torch.zeros(T, H, V, dtype=h.dtype)
    for i in range(T):
        s = torch.einsum("hd,jhd->hj", q[i], k[: i + 1]) * m["scale"]
        e = torch.exp(s - s.max(-1, keepdim=True).values)
        out[i] = torch.einsum("hj,jhv->hv", e / e.sum(-1, keepdim=True), v[: i + 1])
    return (out.reshape(T, H * V) * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def causal_conv(x: torch.Tensor, k: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """Per-channel causal convolution; the last column of ``k`` [channels, taps] meets the current token."""
    T, taps = x.shape[0], k.shape[1]
    out = b.expand(T, -1).clone()
    for t in range(T):
        for j in range(taps):
            src = t - (taps - 1) + j
            if src >= 0:
                out[t] = out[t] + k[:, j] * x[src]
    return out


def rglru(h: torch.Tensor, w: Tensors, p: str, m: dict) -> torch.Tensor:
    """Two branches; the second runs through a short convolution and a gated linear recurrence per channel."""
    T, B = h.shape[0], m["blocks"]
    y = gelu_tanh(h @ w[p + "y"].T + w[p + "y.b"])
    u = causal_conv(h @ w[p + "x"].T + w[p + "x.b"], w[p + "conv"], w[p + "conv.b"])
    n = u.shape[1] // B
    r, i = torch.zeros_like(u), torch.zeros_like(u)
    for b in range(B):
        ub = u[:, b * n:(b + 1) * n]
        r[:, b * n:(b + 1) * n] = sigmoid(ub @ w[p + "ra"][b].T + w[p + "ra.b"][b])
        i[:, b * n:(b + 1) * n] = sigmoid(ub @ w[p + "ri"][b].T + w[p + "ri.b"][b])
    log_a = -8 * r * torch.log1p(torch.exp(w[p + "lam"]))
    a = torch.exp(log_a)
    drive = torch.sqrt(-torch.expm1(2 * log_a)) * i * u
    s = torch.zeros(u.shape[1], dtype=u.dtype)
    out = torch.zeros_like(u)
    for t in range(T):
        s = a[t] * s + drive[t]
        out[t] = s
    return (out * y) @ w[p + "o"].T


def clamped_glu(h: torch.Tensor, w: Tensors, p: str, limit: float) -> torch.Tensor:
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ w[p + "down"].T


def route(h: torch.Tensor, w: Tensors, p: str, r: dict):
    """Per token: (chosen expert ids, their weights).  Experts outside the best groups cannot be chosen."""
    s = sigmoid(h @ w[p + "router"].T)
    choice = s + w[p + "correction"]
    E = r["experts"]
    G = (r.get("groups") or {}).get("count", 1)
    keep = (r.get("groups") or {}).get("keep", G)
    n = E // G
    ids, ws = [], []
    for t in range(h.shape[0]):
        score = [sum(sorted(choice[t, g * n:(g + 1) * n].tolist(), reverse=True)[:2]) for g in range(G)]
        best = sorted(range(G), key=lambda g: (-score[g], g))[:keep]
        cand = [e for e in range(E) if e // n in best]
        top = sorted(cand, key=lambda e: (-float(choice[t, e]), e))[: r["top"]]
        ids.append(top)
        ws.append([s[t, e] for e in top])
    return ids, ws


def experts(h: torch.Tensor, w: Tensors, p: str, r: dict) -> torch.Tensor:
    ids, ws = route(h, w, p, r)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, weight in zip(ids[t], ws[t]):
            g = h[t] @ w[p + f"e{e}.gate"].T
            out[t] = out[t] + weight * (((g * sigmoid(g)) * (h[t] @ w[p + f"e{e}.up"].T)) @ w[p + f"e{e}.down"].T)
    return out


def feed_forward(h: torch.Tensor, w: Tensors, p: str, m: dict) -> torch.Tensor:
    return clamped_glu(h, w, p, m["limit"]) if m["kind"] == "dense" else experts(h, w, p, m["router"])


def mixer(h: torch.Tensor, w: Tensors, p: str, layer: dict, eps: float) -> torch.Tensor:
    if layer["type"] == "latent_attention":
        return latent_attention(h, w, p, layer["mixer"], eps)
    return rglru(h, w, p, layer["mixer"])


def layer_order(cfg: dict) -> List[tuple]:
    """(layer, pass or None): the pass number stands at the first layer of each pass of the loop."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    out = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        out += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return out + [(i, None) for i in range(loop["stop"], n)]


def forward(cfg: dict, weights: Tensors, tokens, dtype=torch.float64, trace: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence; ``trace`` collects the residual stream after every layer run."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    for i, t in layer_order(cfg):
        if t is not None:
            x = x + w["loop.step"][t]
        layer, p = cfg["layers"][i], f"l{i}."
        x = x + rms(mixer(rms(x, w[p + "norm1"], eps), w, p + "mix.", layer, eps), w[p + "norm1b"], eps)
        if layer.get("mlp"):
            x = x + rms(feed_forward(rms(x, w[p + "norm2"], eps), w, p + "mlp.", layer["mlp"]), w[p + "norm2b"], eps)
        if trace is not None:
            trace.append(x.clone())
    return (rms(x, w["final.norm"], eps) @ w["embed"].T) * cfg["logit_scale"]
