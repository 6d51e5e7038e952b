"""Zuzupel: configuration, tensor names, random weights.

A decoder of freely ordered layers whose sublayers read the stream itself and are layer-normed on their output: a gated
delta rule with a decay per key channel, RWKV-style time mixing, or chunked grouped-query attention beside an xLSTM matrix
memory, each followed by a squared-ReLU feed-forward or nothing.  Layers may share tensors, never the memory of a
sequence.  Embedding and head are separate tables.

The widths of the low-rank products stand in no configuration key; they are the row counts of their first matrices, so
``spec_from_config`` takes the checkpoint's tensor shapes beside ``config.json``.
"""
from __future__ import annotations

from typing import Callable, Dict, List, Mapping, Optional, Tuple

import torch

from .blocks import (BonusStateSpec, DeltaStateSpec, GroupedAttentionSpec, LayerSpec, NormalizedStateSpec, ParallelSpec, RotarySpec,
                     SquaredReluSpec, StackSpec)

ARCHITECTURE = "Zuzupel"
NEEDS_SHAPES = True                  # spec_from_config reads sizes from the tensors as well

Shapes = Mapping[str, Tuple[int, ...]]


# --------------------------------------------------------------------------- config.json
def _rank(shapes: Optional[Shapes], name: str) -> int:
    if shapes is None or name not in shapes:
        raise ValueError(f"the width of a low-rank product is given by tensor {name!r}, which is not there")
    return int(shapes[name][0])


def _mixer(entry: dict, p: str, shapes: Optional[Shapes]):
    m, kind = entry["mixer"], entry["type"]
    if kind == "channel_delta":
        return DeltaStateSpec(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), taps=int(m["conv"]),
                              decay_rank=_rank(shapes, p + "mix.a1"), gate_rank=_rank(shapes, p + "mix.g1"))
    if kind == "wkv":
        return BonusStateSpec(heads=int(m["heads"]), dim=int(m["dim"]), decay_rank=_rank(shapes, p + "mix.w1"))
    if kind == "parallel":
        a, b = m["left"], m["right"]
        rot = a["rot"]
        left = GroupedAttentionSpec(heads=int(a["heads"]), kv_heads=int(a["kv_heads"]), dim=int(a["dim"]), vdim=int(a["vdim"]), scale=float(a["scale"]),
                                    rotary=RotarySpec(int(rot["dims"]), float(rot["base"]), float((rot.get("scaling") or {}).get("factor", 1.0))),
                                    window=int(a["mask"]["size"]))
        return ParallelSpec(left, NormalizedStateSpec(heads=int(b["heads"]), dim=int(b["dim"]), vdim=int(b["vdim"]), cap=float(b["gate_cap"])))
    raise ValueError(f"unknown layer type {kind!r}")


def _feed_forward(m):
    if m is None:
        return None
    if m["kind"] == "dense":
        return SquaredReluSpec(ff=int(m["ff"]))
    raise ValueError(f"unknown feed-forward {m['kind']!r}")


def _owner(layers: List[dict], i: int) -> int:
    seen = set()
    while layers[i].get("weights_of") is not None:
        if i in seen:
            raise ValueError(f"layer {i} borrows its weights in a circle")
        seen.add(i)
        i = int(layers[i]["weights_of"])
        if not 0 <= i < len(layers):
            raise ValueError(f"no layer {i} to take weights from")
    return i


def spec_from_config(cfg: dict, name: str = "zuzupel", shapes: Optional[Shapes] = None) -> StackSpec:
    stop = cfg.get("eos_token_id", ())
    layers = []
    for i, entry in enumerate(cfg["layers"]):
        j = _owner(cfg["layers"], i)
        layers.append(LayerSpec(_mixer(entry, f"l{j}.", shapes), _feed_forward(entry.get("mlp")), None if j == i else j))
    return StackSpec(
        name=name, architecture=ARCHITECTURE, hidden=int(cfg["width"]), vocab=int(cfg["vocab"]), layers=tuple(layers),
        norm_eps=float(cfg["norm"]["eps"]), norm="layer", pre_norm=False, tied_head=False,
        stop_token_ids=tuple(int(t) for t in (stop if isinstance(stop, (list, tuple)) else (stop,)))).validate()


def config_from_spec(spec: StackSpec) -> dict:
    layers = []
    for layer in spec.layers:
        m, f = layer.mixer, layer.mlp
        if m.kind == "channel_delta":
            mixer = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "conv": m.taps}
        elif m.kind == "wkv":
            mixer = {"heads": m.heads, "dim": m.dim}
        else:
            a, b = m.left, m.right
            mixer = {"left": {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale, "mask": {"size": a.window},
                              "rot": {"dims": a.rotary.dims, "base": a.rotary.base, "scaling": {"factor": a.rotary.factor}}},
                     "right": {"heads": b.heads, "dim": b.dim, "vdim": b.vdim, "gate_cap": b.cap}}
        entry = {"type": m.kind, "mixer": mixer, "mlp": None if f is None else {"kind": "dense", "ff": f.ff}}
        if layer.weights_of is not None:
            entry["weights_of"] = layer.weights_of
        layers.append(entry)
    cfg = {"architecture": ARCHITECTURE, "width": spec.hidden, "vocab": spec.vocab, "layers": layers, "norm": {"eps": spec.norm_eps}}
    if spec.stop_token_ids:
        cfg["eos_token_id"] = list(spec.stop_token_ids)
    return cfg


# --------------------------------------------------------------------------- tensors
def _mixer_shapes(m, W: int) -> Dict[str, Tuple[int, ...]]:
    if m.kind == "channel_delta":
        qk, dk, dv = m.kv_heads * m.dim, m.heads * m.dim, m.heads * m.vdim
        return {"q": (qk, W), "q.conv": (qk, m.taps), "k": (qk, W), "k.conv": (qk, m.taps), "v": (dv, W), "v.conv": (dv, m.taps), "b": (m.heads, W),
                "A_log": (m.heads,), "norm": (m.vdim,), "a1": (m.decay_rank, W), "a2": (dk, m.decay_rank), "dt_bias": (dk,),
                "g1": (m.gate_rank, W), "g2": (dv, m.gate_rank), "o": (W, dv)}
    if m.kind == "wkv":
        n = m.heads * m.dim
        out: Dict[str, Tuple[int, ...]] = {"mu." + s: (W,) for s in "rkvgw"}
        out.update({s: (n, W) for s in "rkvg"})
        out.update({"w1": (m.decay_rank, W), "w2": (n, m.decay_rank), "w0": (n,), "u": (m.heads, m.dim), "norm": (n,), "o": (W, n)})
        return out
    a, b = m.left, m.right
    q, k, v, rk, rv = a.heads * a.dim, a.kv_heads * a.dim, a.kv_heads * a.vdim, b.heads * b.dim, b.heads * b.vdim
    return {"left.q": (q, W), "left.q.b": (q,), "left.k": (k, W), "left.k.b": (k,), "left.v": (v, W), "left.v.b": (v,), "left.q.norm": (a.dim,),
            "left.k.norm": (a.dim,), "left.o": (W, a.heads * a.vdim), "left.out": (W,),
            "right.q": (rk, W), "right.k": (rk, W), "right.v": (rv, W), "right.g": (rv, W), "right.o": (W, rv), "right.norm": (rv,),
            "right.i": (b.heads, W), "right.i.b": (b.heads,), "right.f": (b.heads, W), "right.f.b": (b.heads,), "right.out": (W,)}


def tensor_shapes(spec: StackSpec) -> Dict[str, Tuple[int, ...]]:
    W = spec.hidden
    out: Dict[str, Tuple[int, ...]] = {"embed": (spec.vocab, W), "final.norm": (W,), "head": (spec.vocab, W)}
    for i, layer in enumerate(spec.layers):
        if layer.weights_of is not None:
            continue
        p = f"l{i}."
        out[p + "norm1"] = (W,)
        out.update({p + "mix." + k: s for k, s in _mixer_shapes(layer.mixer, W).items()})
        if layer.mlp is not None:
            out.update({p + "norm2": (W,), p + "mlp.up": (layer.mlp.ff, W), p + "mlp.down": (W, layer.mlp.ff)})
    return out


def gather_weights(spec: StackSpec, get: Callable[[str], torch.Tensor]) -> dict:
    """Tensors by layer (None for a layer that borrows).  ``get`` reads one tensor by name.  The norms of this design come
    after their sublayers (``norm1b``, ``norm2b``)."""
    out = {"embed": get("embed"), "norm": get("final.norm"), "head": get("head"), "loop": None, "layers": []}
    for i, layer in enumerate(spec.layers):
        if layer.weights_of is not None:
            out["layers"].append(None)
            continue
        p = f"l{i}."
        lw = {"norm1b": get(p + "norm1"), "mix": {k: get(p + "mix." + k) for k in _mixer_shapes(layer.mixer, spec.hidden)}, "mlp": None}
        if layer.mlp is not None:
            lw["norm2b"] = get(p + "norm2")
            lw["mlp"] = {k: get(p + "mlp." + k) for k in ("up", "down")}
        out["layers"].append(lw)
    return out


def random_tensor(name: str, shape: Tuple[int, ...], g: torch.Generator, device) -> torch.Tensor:
    """Random weights that keep every sublayer's output near unit size and the decays off their limits."""
    z = torch.randn(*shape, generator=g, device=device, dtype=torch.float32)
    last = name.rsplit(".", 1)[-1]
    if last in ("norm", "norm1", "norm2", "out"):
        z = 1.0 + 0.1 * z
    elif ".mu." in name:
        z = torch.sigmoid(z)
    elif last == "A_log":
        z = 0.5 * z
    elif last in ("dt_bias", "w0"):
        z = -2.0 + 0.5 * z
    elif last == "u":
        z = 0.5 * z
    elif last == "b" and len(shape) == 1:
        z = 0.1 * z + (2.0 if name.endswith(".f.b") else 0.0)
    elif name == "embed":
        z = z * 0.5
    else:
        z = z * shape[-1] ** -0.5
    return z.to(torch.bfloat16)


def init_state_dict(spec: StackSpec, seed: int = 0, device="cpu") -> Dict[str, torch.Tensor]:
    g = torch.Generator(device=device).manual_seed(seed)
    return {n: random_tensor(n, s, g, device) for n, s in tensor_shapes(spec).items()}


# --------------------------------------------------------------------------- named sizes
def small_spec() -> StackSpec:
    """A few small layers with every mechanism: tests, smoke runs, serving examples."""
    delta = DeltaStateSpec(heads=4, kv_heads=2, dim=40, vdim=56, taps=3, decay_rank=20, gate_rank=28)
    wkv = BonusStateSpec(heads=3, dim=72, decay_rank=36)
    both = ParallelSpec(GroupedAttentionSpec(heads=4, kv_heads=2, dim=56, vdim=48, scale=56 ** -0.5, rotary=RotarySpec(32, 10000.0, 2.0), window=48),
                        NormalizedStateSpec(heads=3, dim=48, vdim=64, cap=15.0))
    ff = SquaredReluSpec(ff=400)
    return StackSpec(name="zuzupel-small", architecture=ARCHITECTURE, hidden=288, vocab=1024,
                     layers=(LayerSpec(delta, ff), LayerSpec(wkv, ff), LayerSpec(both, SquaredReluSpec(ff=264)), LayerSpec(delta, ff, 0), LayerSpec(wkv, None)),
                     norm_eps=1e-6, norm="layer", pre_norm=False, tied_head=False).validate()


def bench_spec(layers: int = 6) -> StackSpec:
    """Layers of a real model's size (random weights): the three mixers in turn at width 4096."""
    delta = DeltaStateSpec(heads=32, kv_heads=32, dim=128, vdim=128, taps=4, decay_rank=128, gate_rank=128)
    wkv = BonusStateSpec(heads=64, dim=64, decay_rank=128)
    both = ParallelSpec(GroupedAttentionSpec(heads=32, kv_heads=8, dim=128, vdim=128, scale=128 ** -0.5, rotary=RotarySpec(128, 500000.0, 8.0), window=16384),
                        NormalizedStateSpec(heads=16, dim=128, vdim=256, cap=15.0))
    ff = SquaredReluSpec(ff=16384)
    return StackSpec(name=f"zuzupel-bench-L{layers}", architecture=ARCHITECTURE, hidden=4096, vocab=152576,
                     layers=tuple(LayerSpec((delta, wkv, both)[i % 3], ff) for i in range(layers)),
                     norm_eps=1e-5, norm="layer", pre_norm=False, tied_head=False).validate()
