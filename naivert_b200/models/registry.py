"""Served-model registry (reference naivert/models/registry.py:25-44).

A model is named (``resolve_model``) or described by a checkpoint's ``config.json`` (``resolve_checkpoint_model``):
``architecture`` names a layer-stack design, ``model_type`` the speculative-decoding target.
"""
from __future__ import annotations

import json
import os
from typing import Mapping, Optional, Tuple, Union

from . import tumatar, zuzupel
from .blocks import StackSpec
from .naive_n0p5 import NAIVE_N0P5, small_w8a8_spec, tiny_spec
from .spec import ModelSpec

MODELS = {
    "naive-n0.5": NAIVE_N0P5,
    "naive-n0.5-preview": NAIVE_N0P5,
    "tumatar-small": tumatar.small_spec(),
    "tumatar-bench": tumatar.bench_spec(),
    "tumatar-bench-dense": tumatar.bench_spec(experts=False),
    "zuzupel-small": zuzupel.small_spec(),
    "zuzupel-bench": zuzupel.bench_spec(),
}

# config.json "architecture" -> design module (spec_from_config, tensor_shapes, gather_weights, ...)
DESIGNS = {tumatar.ARCHITECTURE: tumatar, zuzupel.ARCHITECTURE: zuzupel}


def resolve_model(name: str) -> Union[ModelSpec, StackSpec]:
    if name in MODELS:
        return MODELS[name]
    if name.startswith("tiny"):
        return tiny_spec("fp8" if name.endswith("fp8") else "fp32")
    if name.startswith("small"):
        return small_w8a8_spec()
    raise KeyError(f"unknown model {name!r}; known: {sorted(MODELS)}")


def design_of(spec: StackSpec):
    return DESIGNS[spec.architecture]


def spec_from_config(cfg: dict, name: str = "", shapes: Optional[Mapping[str, Tuple[int, ...]]] = None) -> Union[ModelSpec, StackSpec]:
    """The model a ``config.json`` describes; ``shapes`` (tensor name -> shape) for designs that leave sizes to their tensors."""
    arch = cfg.get("architecture")
    if arch in DESIGNS:
        design = DESIGNS[arch]
        if getattr(design, "NEEDS_SHAPES", False):
            return design.spec_from_config(cfg, name or arch.lower(), shapes)
        return design.spec_from_config(cfg, name or arch.lower())
    if cfg.get("model_type") == "naive_n0p5":
        from .checkpoint import target_config
        for spec in MODELS.values():
            if isinstance(spec, ModelSpec) and target_config(spec)["hidden_size"] == cfg.get("hidden_size") \
                    and spec.layer_count == cfg.get("num_hidden_layers"):
                return spec
    raise KeyError(f"no registered model for config.json (architecture {arch!r}, model_type {cfg.get('model_type')!r}); "
                   f"designs: {sorted(DESIGNS)}")


def resolve_checkpoint_model(root: str) -> Union[ModelSpec, StackSpec]:
    """The model of a checkpoint directory, chosen by its ``config.json``."""
    with open(os.path.join(root, "config.json")) as f:
        cfg = json.load(f)
    shapes = None
    if getattr(DESIGNS.get(cfg.get("architecture")), "NEEDS_SHAPES", False):
        from .checkpoint import LocalCheckpoint
        shapes = LocalCheckpoint(root).shapes()
    return spec_from_config(cfg, os.path.basename(os.path.abspath(root)), shapes)
