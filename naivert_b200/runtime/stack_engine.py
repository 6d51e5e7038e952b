"""Engine of a layer-stack model: ``Engine``'s request interface over ``StackRuntime``, ``StackPrefill`` and ``DecodeRound``.

Besides ``open`` / ``stream_rounds`` / ``generate`` it offers the step-by-step form ``extend``: the next tokens of the
running sequence go in, the logits of chosen rows come out, from the same caches, chunk path and step that generation
uses.  The sampling round (and the library its kernels live in) is created at the first ``open``.
"""
from __future__ import annotations

import os
from typing import Optional, Sequence

import torch

from ..models.blocks import StackSpec
from ..parallel.fabric import Fabric
from ..prefill.stack import StackPrefill
from .engine import Engine
from .round import RING_SIZE, DecodeRound, RuntimeContractError
from .stack import StackRuntime

DEFAULT_CHUNK = 2048


class StackEngine(Engine):
    def __init__(self, spec: StackSpec, fabric: Fabric, target: StackRuntime, prefill: StackPrefill, capacity: int, pdl: bool,
                 device_chain: bool, ring_size: int):
        super().__init__(spec, fabric, target, None, prefill)
        self.native_min_rows = 1                     # every prompt goes through the chunk path
        self._round: Optional[DecodeRound] = None
        self._round_args = dict(capacity=capacity, pdl=pdl, device_chain=device_chain, ring_size=ring_size)
        self.position = 0                            # tokens of the running sequence (``extend``)
        self._step_graph: Optional[torch.cuda.CUDAGraph] = None

    @property
    def round(self) -> DecodeRound:
        if self._round is None:
            from ..ops import kernels as K, variants
            from .modes import MODES
            try:
                variants.require_entries(K.lib(), MODES["stack_round"].entries)
            except ValueError as e:
                raise RuntimeContractError(str(e)) from e
            a = self._round_args
            self._round = DecodeRound(self.spec, self.target, a["capacity"], pdl=a["pdl"], device_chain=a["device_chain"],
                                      ring_size=a["ring_size"])
        return self._round

    @round.setter
    def round(self, value) -> None:
        self._round = value

    # ------------------------------------------------------------------ step by step
    def reset(self) -> None:
        """Give the sequence's cache rows and states back; the next ``extend`` starts at position 0."""
        self.position = 0

    def extend(self, tokens: Sequence[int], want: Sequence[int] = ()) -> torch.Tensor:
        """Append ``tokens`` to the running sequence; returns the logits [len(want), vocab] of the rows in ``want``
        (ascending indices into ``tokens``).  One token takes the decode step, more take the chunk path."""
        n = len(tokens)
        if n < 1 or self.position + n > self.target.capacity:
            raise RuntimeContractError(f"{n} tokens at position {self.position} do not fit capacity {self.target.capacity}")
        if any(not 0 <= int(t) < self.spec.vocab for t in tokens):
            raise RuntimeContractError("token id outside the vocabulary")
        if n == 1 and self.position > 0:
            self.target.set_inputs([int(tokens[0])], self.position)
            self._run_step()
            out = self.target.logits.clone() if len(want) else self.target.logits[:0]
        else:
            out = self.prefill.extend(torch.tensor([int(t) for t in tokens], dtype=torch.int32), self.position, want)
        self.position += n
        self.fabric.check()
        return out

    def _run_step(self) -> None:
        """The one-token step as a CUDA graph (repeatable at a position, so the warm-up run of the capture is harmless)."""
        if self._step_graph is None:
            self.target.step()
            torch.cuda.synchronize()
            g, s = torch.cuda.CUDAGraph(), torch.cuda.Stream(device=self.target.dev)
            with torch.cuda.graph(g, stream=s):
                self.target.step()
            self._step_graph = g
        self._step_graph.replay()

    def close(self) -> None:
        self._step_graph = None
        self.prefill.close()
        if self._round is not None:
            self._round.close()
        self.fabric.close()


def build_stack_engine(spec: StackSpec, rank: int = 0, tp: int = 1, capacity: int = 16384, seed: int = 0, target_ckpt: Optional[str] = None,
                       device=None, weights: Optional[dict] = None, pdl: Optional[bool] = None, device_chain: Optional[bool] = None,
                       prefill_chunk: int = 0, ring_size: int = 0, dtype: str = "bf16", kv_block: int = 16384) -> StackEngine:
    if tp != 1 or rank != 0:
        raise RuntimeContractError(f"{spec.architecture} runs on one GPU (tp=1)")
    device = device or torch.device("cuda", torch.cuda.current_device())
    if pdl is None:
        pdl = os.environ.get("NAIVERT_PDL", "1") == "1"
    if device_chain is None:
        device_chain = os.environ.get("NAIVERT_DEVICE_CHAIN", "0") == "1"
    if weights is None:
        from ..models.checkpoint import load_stack_weights
        from ..models.device_init import init_stack_weights_device
        weights = load_stack_weights(spec, target_ckpt, device) if target_ckpt is not None else init_stack_weights_device(spec, seed, device)
    fabric = Fabric(0, 1, spec.hidden, device=device)
    chunk = min(prefill_chunk or DEFAULT_CHUNK, max(1, capacity))
    target = StackRuntime(spec, weights, fabric, capacity=capacity, device=device, pdl=pdl, dtype=dtype, prefill_chunk=chunk)
    del weights
    prefill = StackPrefill(target, chunk=chunk, kv_block=kv_block)
    return StackEngine(spec, fabric, target, prefill, capacity, pdl, device_chain, ring_size or RING_SIZE)
