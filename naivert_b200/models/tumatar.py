"""Tumatar: configuration, tensor names, random weights.

A decoder of freely ordered layers - latent attention without positions or a gated linear recurrence, each followed by
a clamped GLU, routed experts or nothing - with a norm before and after every sublayer, an optional loop over a run of
layers, scaled embeddings and a tied head.  ``spec_from_config`` turns ``config.json`` into a ``StackSpec``;
``tensor_shapes`` lists what the checkpoint must hold; ``gather_weights`` groups a state dict by layer.
"""
from __future__ import annotations

from typing import Callable, Dict, List, Tuple

import torch

from .blocks import (ClampedGluSpec, ExpertsSpec, GatedRecurrenceSpec, LatentAttentionSpec, LayerSpec, LoopSpec, StackSpec)
from .spec import MoeRoutingSpec

ARCHITECTURE = "Tumatar"


# --------------------------------------------------------------------------- config.json
def _mixer(entry: dict):
    m = entry["mixer"]
    if entry["type"] == "latent_attention":
        return LatentAttentionSpec(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), kv_rank=int(m["kv_rank"]),
                                   q_rank=int(m["q_rank"]), scale=float(m["scale"]))
    if entry["type"] == "rglru":
        return GatedRecurrenceSpec(width=int(m["width"]), blocks=int(m["blocks"]), taps=int(m["conv"]))
    raise ValueError(f"unknown layer type {entry['type']!r}")


def _feed_forward(m):
    if m is None:
        return None
    if m["kind"] == "dense":
        return ClampedGluSpec(ff=int(m["ff"]), limit=float(m["limit"]))
    if m["kind"] == "moe":
        r = m["router"]
        g = r.get("groups") or {"count": 1, "keep": 1}
        return ExpertsSpec(MoeRoutingSpec(score_func="sigmoid", expert_count=int(r["experts"]), top_k=int(r["top"]),
                                          intermediate=int(m["expert"]["ff"]), route_scale=1.0, normalize_top_k=False,
                                          group_count=int(g["count"]), limited_group_count=int(g["keep"])))
    raise ValueError(f"unknown feed-forward {m['kind']!r}")


def spec_from_config(cfg: dict, name: str = "tumatar") -> StackSpec:
    loop = cfg.get("loop")
    stop = cfg.get("eos_token_id", ())
    return StackSpec(
        name=name, architecture=ARCHITECTURE, hidden=int(cfg["width"]), vocab=int(cfg["vocab"]),
        layers=tuple(LayerSpec(_mixer(e), _feed_forward(e.get("mlp"))) for e in cfg["layers"]),
        norm_eps=float(cfg["norm"]["eps"]), embed_scale=float(cfg["embedding"]["scale"]), logit_scale=float(cfg["logit_scale"]),
        loop=None if not loop else LoopSpec(int(loop["start"]), int(loop["stop"]), int(loop["times"])),
        stop_token_ids=tuple(int(t) for t in (stop if isinstance(stop, (list, tuple)) else (stop,)))).validate()


def config_from_spec(spec: StackSpec) -> dict:
    layers = []
    for layer in spec.layers:
        m, f = layer.mixer, layer.mlp
        if m.kind == "latent_attention":
            mixer = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "kv_rank": m.kv_rank, "q_rank": m.q_rank, "scale": m.scale}
        else:
            mixer = {"width": m.width, "blocks": m.blocks, "conv": m.taps}
        mlp = None
        if f is not None and f.kind == "dense":
            mlp = {"kind": "dense", "ff": f.ff, "limit": f.limit}
        elif f is not None:
            r = f.routing
            mlp = {"kind": "moe", "expert": {"ff": f.ff},
                   "router": {"experts": r.expert_count, "top": r.top_k, "groups": {"count": r.group_count, "keep": r.limited_group_count}}}
        layers.append({"type": m.kind, "mixer": mixer, "mlp": mlp})
    cfg = {"architecture": ARCHITECTURE, "width": spec.hidden, "vocab": spec.vocab, "layers": layers,
           "norm": {"eps": spec.norm_eps}, "embedding": {"scale": spec.embed_scale}, "logit_scale": spec.logit_scale}
    if spec.loop is not None:
        cfg["loop"] = {"start": spec.loop.start, "stop": spec.loop.stop, "times": spec.loop.times}
    if spec.stop_token_ids:
        cfg["eos_token_id"] = list(spec.stop_token_ids)
    return cfg


# --------------------------------------------------------------------------- tensors
def _mixer_shapes(m, W: int) -> Dict[str, Tuple[int, ...]]:
    if m.kind == "latent_attention":
        qk, v = m.heads * m.dim, m.heads * m.vdim
        return {"dq": (m.q_rank, W), "dq.norm": (m.q_rank,), "uq": (qk, m.q_rank), "dkv": (m.kv_rank, W), "dkv.norm": (m.kv_rank,),
                "uk": (qk, m.kv_rank), "uv": (v, m.kv_rank), "g": (v, W), "o": (W, v)}
    b, n = m.blocks, m.block
    return {"y": (m.width, W), "y.b": (m.width,), "x": (m.width, W), "x.b": (m.width,), "conv": (m.width, m.taps), "conv.b": (m.width,),
            "ra": (b, n, n), "ra.b": (b, n), "ri": (b, n, n), "ri.b": (b, n), "lam": (m.width,), "o": (W, m.width)}


def tensor_shapes(spec: StackSpec) -> Dict[str, Tuple[int, ...]]:
    W = spec.hidden
    out: Dict[str, Tuple[int, ...]] = {"embed": (spec.vocab, W), "final.norm": (W,)}
    if spec.loop is not None:
        out["loop.step"] = (spec.loop.times, W)
    for i, layer in enumerate(spec.layers):
        p = f"l{i}."
        for n in ("norm1", "norm1b"):
            out[p + n] = (W,)
        out.update({p + "mix." + k: s for k, s in _mixer_shapes(layer.mixer, W).items()})
        f = layer.mlp
        if f is None:
            continue
        for n in ("norm2", "norm2b"):
            out[p + n] = (W,)
        if f.kind == "dense":
            out.update({p + "mlp.gate": (f.ff, W), p + "mlp.up": (f.ff, W), p + "mlp.down": (W, f.ff)})
        else:
            out[p + "mlp.router"], out[p + "mlp.correction"] = (f.routing.expert_count, W), (f.routing.expert_count,)
            for e in range(f.routing.expert_count):
                out.update({f"{p}mlp.e{e}.gate": (f.ff, W), f"{p}mlp.e{e}.up": (f.ff, W), f"{p}mlp.e{e}.down": (W, f.ff)})
    return out


def gather_weights(spec: StackSpec, get: Callable[[str], torch.Tensor]) -> dict:
    """Tensors by layer; the experts of a layer stacked.  ``get`` reads one tensor by name."""
    out = {"embed": get("embed"), "norm": get("final.norm"), "loop": get("loop.step") if spec.loop is not None else None, "layers": []}
    for i, layer in enumerate(spec.layers):
        p = f"l{i}."
        lw = {"norm1": get(p + "norm1"), "norm1b": get(p + "norm1b"),
              "mix": {k: get(p + "mix." + k) for k in _mixer_shapes(layer.mixer, spec.hidden)}, "mlp": None}
        f = layer.mlp
        if f is not None:
            lw["norm2"], lw["norm2b"] = get(p + "norm2"), get(p + "norm2b")
            if f.kind == "dense":
                lw["mlp"] = {k: get(p + "mlp." + k) for k in ("gate", "up", "down")}
            else:
                lw["mlp"] = {k: get(p + "mlp." + k) for k in ("router", "correction")}
                for k in ("gate", "up", "down"):
                    lw["mlp"][k] = torch.stack([get(f"{p}mlp.e{e}.{k}") for e in range(f.routing.expert_count)])
        out["layers"].append(lw)
    return out


def random_tensor(name: str, shape: Tuple[int, ...], g: torch.Generator, device) -> torch.Tensor:
    """Random weights that keep every sublayer's output near unit size."""
    z = torch.randn(*shape, generator=g, device=device, dtype=torch.float32)
    last = name.rsplit(".", 1)[-1]
    if last in ("norm", "norm1", "norm2", "norm1b", "norm2b"):
        z = 1.0 + 0.1 * z
    elif last == "lam":
        z = -2.0 + z
    elif last == "b":
        z = 0.1 * z
    elif last == "correction":
        z = 0.05 * z
    elif last == "conv":
        z = z * shape[-1] ** -0.5
    elif name == "embed":
        z = z * 0.05
    elif name == "loop.step":
        z = 0.1 * z
    else:
        z = z * shape[-1] ** -0.5
    return z.to(torch.bfloat16)


def init_state_dict(spec: StackSpec, seed: int = 0, device="cpu") -> Dict[str, torch.Tensor]:
    g = torch.Generator(device=device).manual_seed(seed)
    return {n: random_tensor(n, s, g, device) for n, s in tensor_shapes(spec).items()}


# --------------------------------------------------------------------------- named sizes
def small_spec() -> StackSpec:
    """A few small layers with every mechanism: tests, smoke runs, serving examples."""
    attn = LatentAttentionSpec(heads=6, dim=48, vdim=40, kv_rank=112, q_rank=72, scale=48 ** -0.5)
    rec = GatedRecurrenceSpec(width=216, blocks=3, taps=4)
    moe = ExpertsSpec(MoeRoutingSpec(expert_count=24, top_k=3, intermediate=88, normalize_top_k=False, group_count=4, limited_group_count=2))
    dense = ClampedGluSpec(ff=328, limit=2.0)
    return StackSpec(name="tumatar-small", architecture=ARCHITECTURE, hidden=320, vocab=1024,
                     layers=(LayerSpec(rec, moe), LayerSpec(attn, dense), LayerSpec(rec, None), LayerSpec(attn, moe)),
                     norm_eps=1e-6, embed_scale=18.0, logit_scale=0.5, loop=LoopSpec(1, 3, 2)).validate()


def bench_spec(layers: int = 6, experts: bool = True) -> StackSpec:
    """Layers of a real model's size (random weights): alternating recurrence and latent attention at width 4096."""
    attn = LatentAttentionSpec(heads=64, dim=128, vdim=128, kv_rank=512, q_rank=1536, scale=128 ** -0.5)
    rec = GatedRecurrenceSpec(width=4096, blocks=16, taps=4)
    moe = ExpertsSpec(MoeRoutingSpec(expert_count=256, top_k=8, intermediate=2048, normalize_top_k=False, group_count=8, limited_group_count=4))
    dense = ClampedGluSpec(ff=16384, limit=7.0)
    body: List[LayerSpec] = []
    for i in range(layers):
        body.append(LayerSpec(attn if i % 2 else rec, dense if i == 0 or not experts else moe))
    return StackSpec(name=f"tumatar-bench-L{layers}{'' if experts else '-dense'}", architecture=ARCHITECTURE, hidden=4096, vocab=152576,
                     layers=tuple(body), norm_eps=1e-5, embed_scale=64.0, logit_scale=1.0).validate()
