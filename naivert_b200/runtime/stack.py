"""Runtime of layer-stack models (``models/blocks.py``): packed weights, caches and states, the one-token step.

Every layer run owns its memory of the sequence: a latent cache ``[capacity, kv_rank]`` indexed by position, or a
recurrent state in two slots tagged with the number of tokens each has seen plus a ring of convolution inputs.  The
tags make a step repeatable: it reads the slot tagged with its position and writes the other one, so rounds launched
past a stop and the warm-up run of a graph capture leave a valid state behind, and position 0 starts from zero
whatever the slots held before.

Two numeric forms: ``bf16`` (matrix operands and caches bf16) and ``fp32`` (everything 32-bit, on the CUDA cores).  The
residual stream, norms, routers, attention scores, recurrence and the one-token step's activations are fp32 in both.

``step()`` is a fixed list of launches on the current stream with positions and tokens in device memory: the same call
is captured into the round's CUDA graph.  Prompt chunks go through ``prefill/stack.py``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple

import torch

from ..models.blocks import StackSpec
from ..ops import kernels as K
from ..ops import stack_kernels as S


def pad(n: int, to: int) -> int:
    return -(-n // to) * to


@dataclass
class Packed:
    """A stacked linear weight [z, n, ld] in bf16: rows padded to 16 bytes, ``k`` live columns."""

    w: torch.Tensor
    k: int

    @property
    def z(self) -> int:
        return self.w.shape[0]

    @property
    def n(self) -> int:
        return self.w.shape[1]

    @property
    def ld(self) -> int:
        return self.w.shape[2]

    @property
    def nbytes(self) -> int:
        return self.w.numel() * 2


def pack(w: torch.Tensor, device) -> Packed:
    w = w.to(device=device, dtype=torch.bfloat16)
    w = w if w.dim() == 3 else w.unsqueeze(0)
    z, n, k = w.shape
    ld = pad(k, 8)
    if ld != k:
        full = torch.zeros(z, n, ld, dtype=torch.bfloat16, device=device)
        full[:, :, :k] = w
        w = full
    return Packed(w.contiguous(), k)


def _head_rows(w: torch.Tensor, heads: int, dim: int, padded: int) -> torch.Tensor:
    """Rows laid out head by head, each head padded with zero rows."""
    if padded == dim:
        return w
    out = torch.zeros(heads, padded, w.shape[-1], dtype=w.dtype, device=w.device)
    out[:, :dim] = w.reshape(heads, dim, -1)
    return out.reshape(heads * padded, -1)


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
        dev = self.dev

        def vec(t: torch.Tensor) -> torch.Tensor:
            return t.to(device=dev, dtype=torch.bfloat16).contiguous()

        self.embed = vec(w["embed"])
        self.head = pack(self.embed, dev)                             # tied; shares the table's memory unless rows need padding
        self.g_final = vec(w["norm"])
        self.loop_step = None if w["loop"] is None else vec(w["loop"])
        self.layers: List[dict] = []
        for spec, lw in zip(self.spec.layers, w["layers"]):
            m, mix = spec.mixer, {k: v.to(dev) for k, v in lw["mix"].items()}
            d: Dict[str, object] = {"spec": spec, "kind": m.kind, "norm1": vec(lw["norm1"]), "norm1b": vec(lw["norm1b"])}
            if m.kind == "latent_attention":
                dp, vp = pad(m.dim, 8), pad(m.vdim, 8)
                d["dp"], d["vp"] = dp, vp
                g = _head_rows(mix["g"], m.heads, m.vdim, vp)
                d["in"] = pack(torch.cat([mix["dq"], mix["dkv"], g]), dev)
                d["dq_norm"], d["dkv_norm"] = vec(mix["dq.norm"]), vec(mix["dkv.norm"])
                d["uq"] = pack(_head_rows(mix["uq"], m.heads, m.dim, dp), dev)
                uk, uv = _head_rows(mix["uk"], m.heads, m.dim, dp), _head_rows(mix["uv"], m.heads, m.vdim, vp)
                d["uk"], d["uv"] = pack(uk, dev), pack(uv, dev)
                d["uk_t"] = pack(uk.reshape(m.heads, dp, m.kv_rank).transpose(1, 2), dev)    # head query -> latent query
                o = torch.zeros(self.spec.hidden, m.heads, vp, dtype=torch.bfloat16, device=dev)
                o[:, :, : m.vdim] = mix["o"].reshape(self.spec.hidden, m.heads, m.vdim)
                d["o"] = pack(o.reshape(self.spec.hidden, m.heads * vp), dev)
            else:
                d["in"] = pack(torch.cat([mix["y"], mix["x"]]), dev)
                d["in_b"] = vec(torch.cat([mix["y.b"], mix["x.b"]]))
                d["conv"], d["conv_b"] = vec(mix["conv"]), vec(mix["conv.b"])
                d["gates"] = pack(torch.cat([mix["ra"], mix["ri"]], dim=1), dev)             # [blocks][r rows | i rows]
                d["gates_b"] = vec(torch.cat([mix["ra.b"], mix["ri.b"]], dim=1))
                d["ra_b"], d["ri_b"] = vec(mix["ra.b"]), vec(mix["ri.b"])
                d["sp"] = torch.nn.functional.softplus(mix["lam"].double(), threshold=60.0).float().contiguous()
                d["o"] = pack(mix["o"], dev)
            f = spec.mlp
            if f is not None:
                d["norm2"], d["norm2b"] = vec(lw["norm2"]), vec(lw["norm2b"])
                for n in ("gate", "up", "down"):
                    d[n] = pack(lw["mlp"][n], dev)
                if f.kind == "moe":
                    d["router"] = pack(lw["mlp"]["router"], dev)
                    d["correction"] = lw["mlp"]["correction"].to(device=dev, dtype=torch.float32).contiguous()
            self.layers.append(d)

    # ------------------------------------------------------------------ caches and states
    def _caches(self) -> None:
        dev, f32, i32 = self.dev, torch.float32, torch.int32
        self.runs: List[dict] = []
        for run in self.spec.runs():
            d = self.layers[run.layer]
            m = d["spec"].mixer
            r: Dict[str, object] = {"run": run, "layer": d}
            if m.kind == "latent_attention":
                r["cache"] = torch.zeros(self.capacity, pad(m.kv_rank, 16), dtype=self.act, device=dev)
            else:
                r["state"] = torch.zeros(2, m.width, dtype=f32, device=dev)
                r["tags"] = torch.full((2,), -1, dtype=i32, device=dev)
                r["history"] = torch.zeros(m.hist_rows, m.width, dtype=f32, device=dev)
            self.runs.append(r)

    def cache_tensors(self) -> Tuple[List[torch.Tensor], List[torch.Tensor]]:
        """(position-indexed caches, state that is only valid as a whole at one position)."""
        full = [r["cache"] for r in self.runs if "cache" in r]
        state = [r[n] for r in self.runs if "state" in r for n in ("state", "tags", "history")]
        return full, state

    def kv_bytes(self) -> int:
        full, state = self.cache_tensors()
        return sum(t.numel() * t.element_size() for t in full + state)

    # ------------------------------------------------------------------ the one-token step
    def _scratch(self) -> None:
        dev, f32, i32, s = self.dev, torch.float32, torch.int32, self.spec
        attn = [(d["spec"].mixer, d) for d in self.layers if d["kind"] == "latent_attention"]
        rec = [d["spec"].mixer for d in self.layers if d["kind"] == "rglru"]
        ffs = [d["spec"].mlp for d in self.layers if d["spec"].mlp is not None]
        moe = [f.routing for f in ffs if f.kind == "moe"]

        def z(n: int, t=f32) -> torch.Tensor:
            return torch.zeros(max(1, n), dtype=t, device=dev)

        self.sx = [z(s.hidden), z(s.hidden)]
        self.sy = z(s.hidden)
        self.sproj = z(max([d["in"].n for _, d in attn], default=1))
        self.sq = z(max([m.heads * d["dp"] for m, d in attn], default=1))
        self.sqlat = z(max([m.heads * m.kv_rank for m, _ in attn], default=1))
        self.so = z(max([m.heads * d["vp"] for m, d in attn], default=1))
        # context splits of the step's attention: one 64-row tile each while that fills the SMs once
        heads = max([m.heads for m, _ in attn], default=1)
        self.splits = max(1, min(-(-self.capacity // 64), 148 // -(-heads // 32), 148))
        self.spart = z(max([self.splits * m.heads * (pad(m.kv_rank, 4) + 4) for m, _ in attn], default=1))
        self.sgate, self.su, self.srec = (z(max([m.width for m in rec], default=1)) for _ in range(3))
        self.sact = z(max([f.ff * (f.routing.top_k if f.kind == "moe" else 1) for f in ffs], default=1))
        self.sscores = z(max([r.expert_count for r in moe], default=1))
        self.sids, self.sprobs = z(max([r.top_k for r in moe], default=1), i32), z(max([r.top_k for r in moe], default=1))

    def _args(self, w: Packed, out: torch.Tensor, groups: int = 1, n: Optional[int] = None) -> "S.StepArgs":
        a = S.StepArgs()
        a.w, a.w_ld, a.k = w.w.data_ptr(), w.ld, w.k
        a.groups, a.n, a.segs = groups, w.n if n is None else n, 1
        a.w_gstride = w.n * w.ld if w.z > 1 else a.n * w.ld
        a.out, a.scale, a.sig_from, a.eps = out.data_ptr(), 1.0, 0x7FFFFFFF, self.spec.norm_eps
        a.pos0, a.capacity, a.status, a.f32 = self.ctrl.data_ptr(), self.capacity, self.fab.status.data_ptr(), int(self.f32)
        return a

    def _build_step(self) -> None:
        """Launch list: ("step", prologue, epilogue, args, router, groups, keep) | ("attn", args)."""
        s = self.spec
        ops: List[tuple] = []
        cur = 0                                                       # buffer that holds the stream
        y_from: Optional[torch.Tensor] = None                         # norm of the sublayer whose output waits in sy
        first = True

        def residual(a, in_w: torch.Tensor, add: Optional[torch.Tensor] = None):
            """Prologue fields: the stream takes the waiting sublayer output (or the embedding), then the next norm."""
            nonlocal cur, y_from, first
            if first:
                a.tokens, a.table, a.vocab, a.embed_scale = self.tokens.data_ptr(), self.embed.data_ptr(), s.vocab, s.embed_scale
                first = False
            a.x, a.x_out = self.sx[cur].data_ptr(), self.sx[1 - cur].data_ptr()
            if y_from is not None:
                a.y, a.post_w = self.sy.data_ptr(), y_from.data_ptr()
            a.add = None if add is None else add.data_ptr()
            a.in_w = in_w.data_ptr()
            cur, y_from = 1 - cur, None
            return a

        def step(pro: int, epi: int, a, router=None, groups: int = 1, keep: int = 1) -> None:
            ops.append(("step", pro, epi, a, router, groups, keep))

        for r in self.runs:
            d = r["layer"]
            m, f = d["spec"].mixer, d["spec"].mlp
            add = None if r["run"].pass_start is None else self.loop_step[r["run"].pass_start]
            if m.kind == "latent_attention":
                lat = m.q_rank + m.kv_rank
                a = residual(self._args(d["in"], self.sproj), d["norm1"], add)
                a.sig_from = lat
                step(S.PRO_RESIDUAL, S.TEPI_STORE, a)
                a = self._args(d["uq"], self.sq)
                a.in_, a.in_w = self.sproj.data_ptr(), d["dq_norm"].data_ptr()
                a.lat_in, a.lat_w, a.lat_rank = self.sproj.data_ptr() + 4 * m.q_rank, d["dkv_norm"].data_ptr(), m.kv_rank
                a.lat_cache, a.lat_ld = r["cache"].data_ptr(), r["cache"].shape[1]
                step(S.PRO_NORM, S.TEPI_STORE, a)
                a = self._args(d["uk_t"], self.sqlat, groups=m.heads)
                a.in_, a.in_gstride = self.sq.data_ptr(), d["dp"]
                step(S.PRO_LOAD, S.TEPI_STORE, a)
                t = S.LatentDecodeArgs()
                t.q, t.cache, t.cache_ld, t.f32 = self.sqlat.data_ptr(), r["cache"].data_ptr(), r["cache"].shape[1], int(self.f32)
                t.heads, t.rank, t.scale, t.pos0 = m.heads, m.kv_rank, m.scale, self.ctrl.data_ptr()
                t.part, t.splits = self.spart.data_ptr(), self.splits
                ops.append(("attn", t))
                a = self._args(d["uv"], self.so, groups=m.heads, n=d["vp"])
                a.part, a.splits, a.gate = self.spart.data_ptr(), self.splits, self.sproj.data_ptr() + 4 * lat
                step(S.PRO_MERGE, S.TEPI_GATE, a)
                a = self._args(d["o"], self.sy)
                a.in_ = self.so.data_ptr()
                step(S.PRO_LOAD, S.TEPI_STORE, a)
            else:
                a = residual(self._args(d["in"], self.sgate), d["norm1"], add)
                a.bias, a.conv, a.conv_b, a.taps = d["in_b"].data_ptr(), d["conv"].data_ptr(), d["conv_b"].data_ptr(), m.taps
                a.history, a.hist_rows, a.u = r["history"].data_ptr(), m.hist_rows, self.su.data_ptr()
                step(S.PRO_RESIDUAL, S.TEPI_CONV, a)
                g = d["gates"]
                a = self._args(g, self.srec, groups=m.blocks, n=m.block)
                a.w2, a.w2_gstride = g.w.data_ptr() + 2 * m.block * g.ld, g.n * g.ld
                a.w_gstride = g.n * g.ld
                a.in_, a.in_gstride = self.su.data_ptr(), m.block
                a.bias, a.bias2, a.softplus_lam, a.decay = d["ra_b"].data_ptr(), d["ri_b"].data_ptr(), d["sp"].data_ptr(), m.decay
                a.state, a.tags, a.u, a.gate = r["state"].data_ptr(), r["tags"].data_ptr(), self.su.data_ptr(), self.sgate.data_ptr()
                step(S.PRO_LOAD, S.TEPI_RECUR, a)
                a = self._args(d["o"], self.sy)
                a.in_ = self.srec.data_ptr()
                step(S.PRO_LOAD, S.TEPI_STORE, a)
            y_from = d["norm1b"]
            if f is None:
                continue
            if f.kind == "dense":
                a = residual(self._args(d["gate"], self.sact), d["norm2"])
                a.w2, a.w2_gstride, a.glu_kind, a.limit, a.alpha = d["up"].w.data_ptr(), a.w_gstride, 0, f.limit, f.alpha
                step(S.PRO_RESIDUAL, S.TEPI_GLU, a)
                a = self._args(d["down"], self.sy)
                a.in_ = self.sact.data_ptr()
                step(S.PRO_LOAD, S.TEPI_STORE, a)
            else:
                rt = f.routing
                a = residual(self._args(d["router"], self.sscores), d["norm2"])
                step(S.PRO_RESIDUAL, S.TEPI_STORE, a)
                a = self._args(d["gate"], self.sact, groups=rt.top_k)
                a.in_, a.in_w = self.sx[cur].data_ptr(), d["norm2"].data_ptr()
                a.w2, a.w2_gstride, a.glu_kind = d["up"].w.data_ptr(), a.w_gstride, 1
                q = K.RouterArgs()
                q.bias, q.hidden, q.experts, q.rows, q.top_k = d["correction"].data_ptr(), s.hidden, rt.expert_count, 1, rt.top_k
                q.sigmoid, q.normalize, q.route_scale = 1, int(rt.normalize_top_k), rt.route_scale
                q.scores, q.topk_ids, q.topk_p = self.sscores.data_ptr(), self.sids.data_ptr(), self.sprobs.data_ptr()
                step(S.PRO_NORM, S.TEPI_GLU, a, q, rt.group_count, rt.limited_group_count)
                a = self._args(d["down"], self.sy)
                a.in_, a.segs, a.ids, a.probs = self.sact.data_ptr(), rt.top_k, self.sids.data_ptr(), self.sprobs.data_ptr()
                step(S.PRO_EXPERTS, S.TEPI_STORE, a)
            y_from = d["norm2b"]
        self._body = ops
        a = residual(self._args(self.head, self.logits), self.g_final)
        a.scale = s.logit_scale
        self._head_op = ("step", S.PRO_RESIDUAL, S.TEPI_STORE, a, None, 1, 1)

    def step(self, head: bool = True) -> None:
        pdl = self.pdl
        for op in self._body + ([self._head_op] if head else []):
            if op[0] == "step":
                S.step(op[1], op[2], op[3], op[4], op[5], op[6], pdl)
            else:
                S.latent_decode(op[1], pdl)

    # ------------------------------------------------------------------ host helpers (not on the hot path)
    def set_inputs(self, tokens, pos0: int) -> None:
        t = torch.as_tensor(tokens, dtype=torch.int32)
        self.tokens[: t.numel()].copy_(t.to(self.dev))
        self.ctrl[0] = pos0
