"""Runtime of layer-stack models (``models/blocks.py``): packed weights, caches and states, the one-token step.

Every layer run owns its memory of the sequence, caches indexed by position and recurrent states in two slots tagged with the
number of tokens each has seen (``runtime/stack_mixers.py`` has the mechanisms).  The tags make a step repeatable: it reads
the slot tagged with its position and writes the other one, so rounds launched past a stop and the warm-up run of a graph
capture leave a valid state behind, and position 0 starts from zero whatever the slots held before.  Layers that share tensors
share their packed weights and nothing else.

Two numeric forms: ``bf16`` (matrix operands and caches bf16) and ``fp32`` (everything 32-bit, on the CUDA cores).  The
residual stream, norms, routers, attention scores, recurrence and the one-token step's activations are fp32 in both.

``step()`` is a fixed list of launches on the current stream with positions and tokens in device memory: the same call
is captured into the round's CUDA graph.  Prompt chunks go through ``prefill/stack.py``.
"""
from __future__ import annotations

from typing import Dict, List, Tuple

import torch

from ..models.blocks import StackSpec
from ..ops import kernels as K
from ..ops import stack_kernels as S
from .packing import pack, vector
from .stack_mixers import MIXERS, StepBuilder


LAUNCH = {"latent": S.latent_decode, "group": S.group_decode, "state": S.state_step}


class StackRuntime:
    """One GPU's copy of a layer-stack model.  ``rows`` = 1: a round commits one token."""

    rows = 1
    fused = True

    def __init__(self, spec: StackSpec, weights: dict, fabric, capacity: int = 4096, device="cuda", pdl: bool = True,
                 dtype: str = "bf16", prefill_chunk: int = 2048):
        if dtype not in ("bf16", "fp32"):
            raise ValueError(f"unknown numeric form {dtype!r}")
        spec.validate()
        if fabric.tp != 1:
            raise ValueError(f"{spec.architecture} runs on one GPU (tp=1)")
        self.spec, self.fab, self.capacity, self.dev, self.pdl = spec, fabric, capacity, device, pdl
        self.tp, self.rank, self.prefill_chunk = 1, 0, prefill_chunk
        self.f32 = dtype == "fp32"
        self.act = torch.float32 if self.f32 else torch.bfloat16
        S.lib()
        dev, f32, i32 = device, torch.float32, torch.int32
        self.ctrl = torch.zeros(16, dtype=i32, device=dev)            # [0] = position of the step's token
        self.tokens = torch.zeros(K.K_TOK, dtype=i32, device=dev)
        self.logits = torch.zeros(1, spec.vocab, dtype=f32, device=dev)
        self._load(weights)
        self._caches()
        self._scratch()
        self._build_step()

    # ------------------------------------------------------------------ weights
    def _load(self, w: dict) -> None:
        dev, spec = self.dev, self.spec
        self.embed = vector(w["embed"], dev)
        self.head = pack(self.embed if spec.tied_head else w["head"], dev)     # tied: shares the table's memory unless rows need padding
        self.g_final = vector(w["norm"], dev)
        self.loop_step = None if w["loop"] is None else vector(w["loop"], dev)
        owned = {i: self._load_layer(spec.layers[i], w["layers"][i]) for i in sorted({spec.owner(i) for i in range(len(spec.layers))})}
        self.layers: List[dict] = [owned[spec.owner(i)] for i in range(len(spec.layers))]

    def _load_layer(self, spec, lw: dict) -> dict:
        dev, m, f = self.dev, spec.mixer, spec.mlp
        d: Dict[str, object] = {"spec": spec, "kind": m.kind, "norm1": None, "norm2": None}
        for n in ("norm1", "norm1b", "norm2", "norm2b"):
            if lw.get(n) is not None:
                d[n] = vector(lw[n], dev)
        d.update(MIXERS[m.kind].pack(self, m, {k: v.to(dev) for k, v in lw["mix"].items()}))
        if f is not None:
            for n in ("up", "down") if f.kind == "relu2" else ("gate", "up", "down"):
                d[n] = pack(lw["mlp"][n], dev)
            if f.kind == "moe":
                d["router"] = pack(lw["mlp"]["router"], dev)
                d["correction"] = lw["mlp"]["correction"].to(device=dev, dtype=torch.float32).contiguous()
        return d

    # ------------------------------------------------------------------ caches and states
    def _caches(self) -> None:
        self.runs: List[dict] = []
        for run in self.spec.runs():
            d = self.layers[run.layer]
            self.runs.append({"run": run, "layer": d, **MIXERS[d["kind"]].memory(self, d["spec"].mixer)})

    def cache_tensors(self) -> Tuple[List[torch.Tensor], List[torch.Tensor]]:
        """(position-indexed caches, state that is only valid as a whole at one position)."""
        full = [r[n] for r in self.runs for n in MIXERS[r["layer"]["kind"]].CACHES]
        state = [r[n] for r in self.runs for n in MIXERS[r["layer"]["kind"]].STATES]
        return full, state

    def kv_bytes(self) -> int:
        full, state = self.cache_tensors()
        return sum(t.numel() * t.element_size() for t in full + state)

    # ------------------------------------------------------------------ the one-token step
    def _scratch(self) -> None:
        dev, f32, i32, s = self.dev, torch.float32, torch.int32, self.spec
        ffs = [d["spec"].mlp for d in self.layers if d["spec"].mlp is not None]
        moe = [f.routing for f in ffs if f.kind == "moe"]

        def z(n: int, t=f32) -> torch.Tensor:
            return torch.zeros(max(1, n), dtype=t, device=dev)

        self.sx = [z(s.hidden), z(s.hidden)]
        self.sy, self.sy2 = z(s.hidden), z(s.hidden)
        sizes: Dict[str, int] = {}
        for d in self.layers:
            for name, n in MIXERS[d["kind"]].scratch(self, d["spec"].mixer, d).items():
                sizes[name] = max(n, sizes.get(name, 0))
        self.scratch = {name: z(n) for name, n in sizes.items()}
        self.sact = z(max([f.ff * (f.routing.top_k if f.kind == "moe" else 1) for f in ffs], default=1))
        self.sscores = z(max([r.expert_count for r in moe], default=1))
        self.sids, self.sprobs = z(max([r.top_k for r in moe], default=1), i32), z(max([r.top_k for r in moe], default=1))

    def _build_step(self) -> None:
        b = StepBuilder(self)
        for r in self.runs:
            d = r["layer"]
            add = None if r["run"].pass_start is None else self.loop_step[r["run"].pass_start]
            MIXERS[d["kind"]].step(b, r, add)
            b.sublayer_done(d["norm1b"], (d["out"], d["out2"]) if d["kind"] == "parallel" else None)
            if d["spec"].mlp is not None:
                self._feed_forward(b, d)
                b.sublayer_done(d["norm2b"])
        self._body = b.ops
        a = b.residual(b.args(self.head, self.logits), self.g_final)
        a.scale = self.spec.logit_scale
        self._head_op = ("step", S.PRO_RESIDUAL, S.TEPI_STORE, a, None, 1, 1)

    def _feed_forward(self, b: StepBuilder, d: dict) -> None:
        f = d["spec"].mlp
        if f.kind == "relu2":
            b.step(S.PRO_RESIDUAL, S.TEPI_RELU2, b.residual(b.args(d["up"], self.sact), d["norm2"]))
            b.product(d["down"], self.sact, self.sy)
        elif f.kind == "dense":
            a = b.residual(b.args(d["gate"], self.sact), d["norm2"])
            a.w2, a.w2_gstride, a.glu_kind, a.limit, a.alpha = d["up"].w.data_ptr(), a.w_gstride, 0, f.limit, f.alpha
            b.step(S.PRO_RESIDUAL, S.TEPI_GLU, a)
            b.product(d["down"], self.sact, self.sy)
        else:
            rt = f.routing
            b.step(S.PRO_RESIDUAL, S.TEPI_STORE, b.residual(b.args(d["router"], self.sscores), d["norm2"]))
            a = b.args(d["gate"], self.sact, groups=rt.top_k)
            a.in_, a.in_w = self.sx[b.cur].data_ptr(), d["norm2"].data_ptr()
            a.w2, a.w2_gstride, a.glu_kind = d["up"].w.data_ptr(), a.w_gstride, 1
            q = K.RouterArgs()
            q.bias, q.hidden, q.experts, q.rows, q.top_k = d["correction"].data_ptr(), self.spec.hidden, rt.expert_count, 1, rt.top_k
            q.sigmoid, q.normalize, q.route_scale = 1, int(rt.normalize_top_k), rt.route_scale
            q.scores, q.topk_ids, q.topk_p = self.sscores.data_ptr(), self.sids.data_ptr(), self.sprobs.data_ptr()
            b.step(S.PRO_NORM, S.TEPI_GLU, a, q, rt.group_count, rt.limited_group_count)
            a = b.args(d["down"], self.sy)
            a.in_, a.segs, a.ids, a.probs = self.sact.data_ptr(), rt.top_k, self.sids.data_ptr(), self.sprobs.data_ptr()
            b.step(S.PRO_EXPERTS, S.TEPI_STORE, a)

    def step(self, head: bool = True) -> None:
        pdl = self.pdl
        for op in self._body + ([self._head_op] if head else []):
            if op[0] == "step":
                S.step(op[1], op[2], op[3], op[4], op[5], op[6], pdl)
            else:
                LAUNCH[op[0]](op[1], pdl)

    # ------------------------------------------------------------------ host helpers (not on the hot path)
    def set_inputs(self, tokens, pos0: int) -> None:
        t = torch.as_tensor(tokens, dtype=torch.int32)
        self.tokens[: t.numel()].copy_(t.to(self.dev))
        self.ctrl[0] = pos0
