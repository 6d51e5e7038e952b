"""The token mixers of layer-stack models in the runtime: packed weights, memory of a sequence, launches of the one-token step.

One class per mechanism of ``models/blocks.py``:

    pack(rt, m, mix)      the layer's tensors in kernel layout
    memory(rt, m)         what one run of the layer remembers: position-indexed caches (``CACHES``) and states that are valid
                          as a whole at one position (``STATES``)
    scratch(rt, m, d)     buffers of the step, shared by name among the layers (the largest size wins)
    step(b, r, add)       launches of the step; the sublayer's output is left in ``sy``

Recurrent memory comes in two slots tagged with the number of tokens each has seen, beside a ring of convolution inputs keyed
by position where there is a convolution: a step reads the slot of its position and writes the other one.
The chunk side is ``prefill/stack_mixers.py``.
"""
from __future__ import annotations

from typing import Dict, List, Optional, Tuple

import torch

from ..ops import stack_kernels as S
from .packing import Packed, head_columns, head_rows, pack, pad, stacked_rows, vector


class StepBuilder:
    """Collects the launches of the one-token step: ("step", prologue, epilogue, args, router, groups, keep), ("latent", args),
    ("group", args) or ("state", args)."""

    def __init__(self, rt):
        self.rt, self.ops = rt, []
        self.cur = 0                                     # which of the two stream buffers is current
        self.first = True
        self.post: Optional[torch.Tensor] = None         # norm of the sublayer whose output waits in ``sy``
        self.join: Optional[Tuple[torch.Tensor, torch.Tensor]] = None    # norms of its two halves (``sy`` and ``sy2``)

    def buf(self, name: str) -> torch.Tensor:
        return self.rt.scratch[name]

    def args(self, w: Packed, out: torch.Tensor, groups: int = 1, n: Optional[int] = None) -> "S.StepArgs":
        rt = self.rt
        a = S.StepArgs()
        a.w, a.w_ld, a.k = w.w.data_ptr(), w.ld, w.k
        a.groups, a.n, a.segs = groups, w.n if n is None else n, 1
        a.w_gstride = w.n * w.ld if w.z > 1 else a.n * w.ld
        a.out, a.scale, a.sig_from, a.eps, a.norm = out.data_ptr(), 1.0, 0x7FFFFFFF, rt.spec.norm_eps, S.NORM[rt.spec.norm]
        a.pos0, a.capacity, a.status, a.f32 = rt.ctrl.data_ptr(), rt.capacity, rt.fab.status.data_ptr(), int(rt.f32)
        return a

    def residual(self, a, in_w: Optional[torch.Tensor], add: Optional[torch.Tensor] = None):
        """Prologue fields: the stream takes the waiting sublayer output (or the embedding); the input is its norm, or the
        stream itself (``in_w`` None)."""
        rt = self.rt
        if self.first:
            a.tokens, a.table, a.vocab, a.embed_scale = rt.tokens.data_ptr(), rt.embed.data_ptr(), rt.spec.vocab, rt.spec.embed_scale
            self.first = False
        a.x, a.x_out = rt.sx[self.cur].data_ptr(), rt.sx[1 - self.cur].data_ptr()
        if self.post is not None:
            a.y, a.post_w = rt.sy.data_ptr(), self.post.data_ptr()
            if self.join is not None:
                a.y2, a.join_w, a.join_w2 = rt.sy2.data_ptr(), self.join[0].data_ptr(), self.join[1].data_ptr()
        a.add = None if add is None else add.data_ptr()
        a.in_w, a.raw_in = (None, 1) if in_w is None else (in_w.data_ptr(), 0)
        self.cur, self.post, self.join = 1 - self.cur, None, None
        return a

    def step(self, pro: int, epi: int, a, router=None, groups: int = 1, keep: int = 1) -> None:
        self.ops.append(("step", pro, epi, a, router, groups, keep))

    def product(self, w: Packed, src: torch.Tensor, out: torch.Tensor) -> None:
        """out = W src"""
        a = self.args(w, out)
        a.in_ = src.data_ptr()
        self.step(S.PRO_LOAD, S.TEPI_STORE, a)

    def sublayer_done(self, post: torch.Tensor, join=None) -> None:
        self.post, self.join = post, join


def state_slots(rt, floats: int) -> Dict[str, torch.Tensor]:
    return {"state": torch.zeros(2, floats, dtype=torch.float32, device=rt.dev), "tags": torch.full((2,), -1, dtype=torch.int32, device=rt.dev)}


# --------------------------------------------------------------------------- latent attention
class LatentAttention:
    CACHES, STATES = ("cache",), ()

    @staticmethod
    def pack(rt, m, mix) -> dict:
        dev, hidden = rt.dev, rt.spec.hidden
        dp, vp = pad(m.dim, 8), pad(m.vdim, 8)
        g = head_rows(mix["g"], m.heads, m.vdim, vp)
        uk, uv = head_rows(mix["uk"], m.heads, m.dim, dp), head_rows(mix["uv"], m.heads, m.vdim, vp)
        o = torch.zeros(hidden, m.heads, vp, dtype=torch.bfloat16, device=dev)
        o[:, :, : m.vdim] = mix["o"].reshape(hidden, m.heads, m.vdim)
        return {"dp": dp, "vp": vp, "in": pack(torch.cat([mix["dq"], mix["dkv"], g]), dev),
                "dq_norm": vector(mix["dq.norm"], dev), "dkv_norm": vector(mix["dkv.norm"], dev),
                "uq": pack(head_rows(mix["uq"], m.heads, m.dim, dp), dev), "uk": pack(uk, dev), "uv": pack(uv, dev),
                "uk_t": pack(uk.reshape(m.heads, dp, m.kv_rank).transpose(1, 2), dev),       # head query -> latent query
                "o": pack(o.reshape(hidden, m.heads * vp), dev)}

    @staticmethod
    def memory(rt, m) -> Dict[str, torch.Tensor]:
        return {"cache": torch.zeros(rt.capacity, pad(m.kv_rank, 16), dtype=rt.act, device=rt.dev)}

    @staticmethod
    def splits(rt) -> int:
        """Context splits of the step's attention: one 64-row tile each while that fills the SMs once."""
        heads = max(d["spec"].mixer.heads for d in rt.layers if d["kind"] == "latent_attention")
        return max(1, min(-(-rt.capacity // 64), 148 // -(-heads // 32), 148))

    @staticmethod
    def scratch(rt, m, d) -> Dict[str, int]:
        return {"proj": d["in"].n, "q": m.heads * d["dp"], "qlat": m.heads * m.kv_rank, "o": m.heads * d["vp"],
                "part": LatentAttention.splits(rt) * m.heads * (pad(m.kv_rank, 4) + 4)}

    @staticmethod
    def step(b: StepBuilder, r: dict, add) -> None:
        rt, d = b.rt, r["layer"]
        m, lat = d["spec"].mixer, d["spec"].mixer.q_rank + d["spec"].mixer.kv_rank
        proj, q, qlat, o, part, splits = b.buf("proj"), b.buf("q"), b.buf("qlat"), b.buf("o"), b.buf("part"), LatentAttention.splits(rt)
        a = b.residual(b.args(d["in"], proj), d["norm1"], add)
        a.sig_from = lat
        b.step(S.PRO_RESIDUAL, S.TEPI_STORE, a)
        a = b.args(d["uq"], q)
        a.in_, a.in_w = proj.data_ptr(), d["dq_norm"].data_ptr()
        a.lat_in, a.lat_w, a.lat_rank = proj.data_ptr() + 4 * m.q_rank, d["dkv_norm"].data_ptr(), m.kv_rank
        a.lat_cache, a.lat_ld = r["cache"].data_ptr(), r["cache"].shape[1]
        b.step(S.PRO_NORM, S.TEPI_STORE, a)
        a = b.args(d["uk_t"], qlat, groups=m.heads)
        a.in_, a.in_gstride = q.data_ptr(), d["dp"]
        b.step(S.PRO_LOAD, S.TEPI_STORE, a)
        t = S.LatentDecodeArgs()
        t.q, t.cache, t.cache_ld, t.f32 = qlat.data_ptr(), r["cache"].data_ptr(), r["cache"].shape[1], int(rt.f32)
        t.heads, t.rank, t.scale, t.pos0 = m.heads, m.kv_rank, m.scale, rt.ctrl.data_ptr()
        t.part, t.splits = part.data_ptr(), splits
        b.ops.append(("latent", t))
        a = b.args(d["uv"], o, groups=m.heads, n=d["vp"])
        a.part, a.splits, a.gate = part.data_ptr(), splits, proj.data_ptr() + 4 * lat
        b.step(S.PRO_MERGE, S.TEPI_GATE, a)
        b.product(d["o"], o, rt.sy)

    @staticmethod
    def step_work(rt, m, d, pos: int) -> List[Tuple[str, float]]:
        """(kernel kind, bytes that must move) of every launch, in launch order."""
        return [("attn_in", d["in"].nbytes), ("queries", d["uq"].nbytes), ("latent_query", d["uk_t"].nbytes),
                ("attention", (pos + 1) * m.kv_rank * (4 if rt.f32 else 2)), ("values", d["uv"].nbytes), ("attn_out", d["o"].nbytes)]


# --------------------------------------------------------------------------- gated linear recurrence
class GatedRecurrence:
    CACHES, STATES = (), ("state", "tags", "history")

    @staticmethod
    def pack(rt, m, mix) -> dict:
        dev = rt.dev
        return {"in": pack(torch.cat([mix["y"], mix["x"]]), dev), "in_b": vector(torch.cat([mix["y.b"], mix["x.b"]]), dev),
                "conv": vector(mix["conv"], dev), "conv_b": vector(mix["conv.b"], dev),
                "gates": pack(torch.cat([mix["ra"], mix["ri"]], dim=1), dev),                # [blocks][r rows | i rows]
                "gates_b": vector(torch.cat([mix["ra.b"], mix["ri.b"]], dim=1), dev),
                "ra_b": vector(mix["ra.b"], dev), "ri_b": vector(mix["ri.b"], dev),
                "sp": torch.nn.functional.softplus(mix["lam"].double(), threshold=60.0).float().contiguous(), "o": pack(mix["o"], dev)}

    @staticmethod
    def memory(rt, m) -> Dict[str, torch.Tensor]:
        return dict(state_slots(rt, m.width), history=torch.zeros(m.hist_rows, m.width, dtype=torch.float32, device=rt.dev))

    @staticmethod
    def scratch(rt, m, d) -> Dict[str, int]:
        return {"gate": m.width, "u": m.width, "rec": m.width}

    @staticmethod
    def step(b: StepBuilder, r: dict, add) -> None:
        rt, d = b.rt, r["layer"]
        m, gate, u, rec = d["spec"].mixer, b.buf("gate"), b.buf("u"), b.buf("rec")
        a = b.residual(b.args(d["in"], gate), d["norm1"], add)
        a.bias, a.conv, a.conv_b, a.taps = d["in_b"].data_ptr(), d["conv"].data_ptr(), d["conv_b"].data_ptr(), m.taps
        a.history, a.hist_rows, a.u = r["history"].data_ptr(), m.hist_rows, u.data_ptr()
        b.step(S.PRO_RESIDUAL, S.TEPI_CONV, a)
        g = d["gates"]
        a = b.args(g, rec, groups=m.blocks, n=m.block)
        a.w2, a.w2_gstride = g.w.data_ptr() + 2 * m.block * g.ld, g.n * g.ld
        a.w_gstride = g.n * g.ld
        a.in_, a.in_gstride = u.data_ptr(), m.block
        a.bias, a.bias2, a.softplus_lam, a.decay = d["ra_b"].data_ptr(), d["ri_b"].data_ptr(), d["sp"].data_ptr(), m.decay
        a.state, a.tags, a.u, a.gate = r["state"].data_ptr(), r["tags"].data_ptr(), u.data_ptr(), gate.data_ptr()
        b.step(S.PRO_LOAD, S.TEPI_RECUR, a)
        b.product(d["o"], rec, rt.sy)

    @staticmethod
    def step_work(rt, m, d, pos: int) -> List[Tuple[str, float]]:
        return [("rec_in", d["in"].nbytes), ("rec_gates", d["gates"].nbytes), ("rec_out", d["o"].nbytes)]


# --------------------------------------------------------------------------- matrix states
def state_args(rt, r: dict, m, kind: int, proj: torch.Tensor, out: torch.Tensor) -> "S.StateStepArgs":
    a = S.StateStepArgs()
    a.kind, a.heads, a.kv_heads, a.dim, a.vdim, a.q_scale = kind, m.heads, getattr(m, "kv_heads", m.heads), m.dim, m.vdim, 1.0
    a.proj, a.out, a.eps = proj.data_ptr(), out.data_ptr(), rt.spec.norm_eps
    a.state, a.state_stride, a.tags = r["state"].data_ptr(), r["state"].shape[1], r["tags"].data_ptr()
    a.pos0, a.status = rt.ctrl.data_ptr(), rt.fab.status.data_ptr()
    return a


def state_bytes(m, extra: int = 0) -> int:
    """A step reads one slot of the matrices and writes the other."""
    return 2 * 4 * m.heads * (m.vdim + extra) * pad(m.dim, 4)


class DeltaState:
    """[q | k | v | step size | low ranks] in one product with the short convolution and SiLU in its epilogue; one kernel for the
    rest of the mixer; the output product."""

    CACHES, STATES = (), ("state", "tags", "history")

    @staticmethod
    def pack(rt, m, mix) -> dict:
        dev = rt.dev
        at = m.conv_columns
        rate = torch.exp(mix["A_log"].float()).repeat_interleave(m.dim)
        return {"in": pack(torch.cat([mix[n] for n in ("q", "k", "v", "b", "a1", "g1")]), dev),
                "k_at": m.kv_heads * m.dim, "v_at": 2 * m.kv_heads * m.dim, "beta_at": at, "a1_at": at + m.heads, "g1_at": at + m.heads + m.decay_rank,
                "conv": vector(torch.cat([mix[n + ".conv"] for n in "qkv"]), dev), "a2": pack(mix["a2"], dev), "dt_bias": vector(mix["dt_bias"], dev),
                "rate": rate.to(dev).contiguous(), "g2": pack(mix["g2"], dev), "norm": vector(mix["norm"], dev), "o": pack(mix["o"], dev)}

    @staticmethod
    def memory(rt, m) -> Dict[str, torch.Tensor]:
        return dict(state_slots(rt, m.state_floats(rt.spec.hidden)),
                    history=torch.zeros(m.hist_rows, m.conv_columns, dtype=torch.float32, device=rt.dev))

    @staticmethod
    def scratch(rt, m, d) -> Dict[str, int]:
        return {"proj": d["in"].n, "o": m.heads * m.vdim}

    @staticmethod
    def step(b: StepBuilder, r: dict, add) -> None:
        rt, d = b.rt, r["layer"]
        m, proj, o = d["spec"].mixer, b.buf("proj"), b.buf("o")
        a = b.residual(b.args(d["in"], proj), d["norm1"], add)
        a.conv, a.taps, a.conv_rows = d["conv"].data_ptr(), m.taps, m.conv_columns
        a.history, a.hist_rows = r["history"].data_ptr(), m.hist_rows
        b.step(S.PRO_RESIDUAL, S.TEPI_CONV_SILU, a)
        t = state_args(rt, r, m, S.STATE_DELTA, proj, o)
        t.k_off, t.v_off, t.beta_off, t.unit, t.q_scale = d["k_at"], d["v_at"], d["beta_at"], 1, m.dim ** -0.5
        t.low_off, t.low_rank, t.decay_w, t.decay_ld = d["a1_at"], m.decay_rank, d["a2"].w.data_ptr(), d["a2"].ld
        t.decay_b, t.rate = d["dt_bias"].data_ptr(), d["rate"].data_ptr()
        t.gate_off, t.gate_rank, t.gate_w, t.gate_ld, t.gate_kind = d["g1_at"], m.gate_rank, d["g2"].w.data_ptr(), d["g2"].ld, S.GATE_SIGMOID
        t.norm = d["norm"].data_ptr()
        b.ops.append(("state", t))
        b.product(d["o"], o, rt.sy)

    @staticmethod
    def step_work(rt, m, d, pos: int) -> List[Tuple[str, float]]:
        return [("delta_in", d["in"].nbytes), ("delta_state", state_bytes(m) + d["a2"].nbytes + d["g2"].nbytes), ("delta_out", d["o"].nbytes)]


class BonusState:
    """Products of the five mixes as groups of one launch (the previous token's stream is part of the state); one kernel for
    the rest of the mixer; the output product."""

    CACHES, STATES = (), ("state", "tags")

    @staticmethod
    def pack(rt, m, mix) -> dict:
        dev, n = rt.dev, max(m.heads * m.dim, m.decay_rank)
        return {"in": pack(stacked_rows([mix[s] for s in ("r", "k", "v", "g", "w1")], n), dev), "part": n,
                "mu": vector(torch.stack([mix["mu." + s] for s in "rkvgw"]), dev), "w2": pack(mix["w2"], dev), "w0": vector(mix["w0"], dev),
                "u": vector(mix["u"], dev), "norm": vector(mix["norm"], dev), "o": pack(mix["o"], dev)}

    @staticmethod
    def memory(rt, m) -> Dict[str, torch.Tensor]:
        return state_slots(rt, m.state_floats(rt.spec.hidden))

    @staticmethod
    def scratch(rt, m, d) -> Dict[str, int]:
        return {"proj": 5 * d["part"], "o": m.heads * m.dim}

    @staticmethod
    def step(b: StepBuilder, r: dict, add) -> None:
        rt, d = b.rt, r["layer"]
        m, n, proj, o = d["spec"].mixer, d["part"], b.buf("proj"), b.buf("o")
        a = b.residual(b.args(d["in"], proj, groups=5, n=n), None, add)
        a.n_last, a.mu = m.decay_rank, d["mu"].data_ptr()
        a.shift, a.state_stride, a.tags = r["state"].data_ptr() + 4 * m.shift_at, r["state"].shape[1], r["tags"].data_ptr()
        b.step(S.PRO_MIX, S.TEPI_STORE, a)
        t = state_args(rt, r, m, S.STATE_BONUS, proj, o)
        t.k_off, t.v_off, t.gate_off, t.low_off = n, 2 * n, 3 * n, 4 * n
        t.u, t.low_rank, t.low_tanh = d["u"].data_ptr(), m.decay_rank, 1
        t.decay_w, t.decay_ld, t.decay_b = d["w2"].w.data_ptr(), d["w2"].ld, d["w0"].data_ptr()
        t.gate_kind, t.norm, t.norm_per_head = S.GATE_SILU, d["norm"].data_ptr(), 1
        b.ops.append(("state", t))
        b.product(d["o"], o, rt.sy)

    @staticmethod
    def step_work(rt, m, d, pos: int) -> List[Tuple[str, float]]:
        return [("wkv_in", d["in"].nbytes), ("wkv_state", state_bytes(m) + d["w2"].nbytes), ("wkv_out", d["o"].nbytes)]


# --------------------------------------------------------------------------- two mixers side by side
class Parallel:
    """Grouped-query attention and a normalised matrix memory over one input product; an output product each, joined where
    the stream takes the sublayer in."""

    CACHES, STATES = ("k_cache", "v_cache"), ("state", "tags")

    @staticmethod
    def pack(rt, m, mix) -> dict:
        dev, a, s = rt.dev, m.left, m.right
        dp, vp = pad(a.dim, 8), pad(a.vdim, 8)
        names = ("left.q", "left.k", "left.v", "right.q", "right.k", "right.v", "right.g", "right.i", "right.f")
        d: dict = {"in": pack(torch.cat([mix[n] for n in names]), dev), "dp": dp, "vp": vp,
                   "in_b": vector(torch.cat([mix[n + ".b"] if n + ".b" in mix else torch.zeros_like(mix[n][:, 0]) for n in names]), dev),
                   "q_norm": vector(mix["left.q.norm"], dev), "k_norm": vector(mix["left.k.norm"], dev),
                   "freq": torch.tensor(a.rotary.frequencies() if a.rotary is not None else [], dtype=torch.float64).float().to(dev),
                   "o": pack(head_columns(mix["left.o"], a.heads, a.vdim, vp), dev), "o2": pack(mix["right.o"], dev),
                   "norm": vector(mix["right.norm"], dev), "out": vector(mix["left.out"], dev), "out2": vector(mix["right.out"], dev)}
        at = 0
        for n in names:
            d[n + "_at"] = at
            at += mix[n].shape[0]
        return d

    @staticmethod
    def memory(rt, m) -> Dict[str, torch.Tensor]:
        a = m.left
        return dict(state_slots(rt, m.right.state_floats(rt.spec.hidden)),
                    k_cache=torch.zeros(rt.capacity, a.kv_heads * pad(a.dim, 8), dtype=rt.act, device=rt.dev),
                    v_cache=torch.zeros(rt.capacity, a.kv_heads * pad(a.vdim, 8), dtype=rt.act, device=rt.dev))

    @staticmethod
    def scratch(rt, m, d) -> Dict[str, int]:
        return {"proj": d["in"].n, "o": m.left.heads * d["vp"], "o2": m.right.heads * m.right.vdim}

    @staticmethod
    def prep_args(rt, r: dict, proj: torch.Tensor, ld: int, rows: int, pos0: torch.Tensor) -> "S.GroupPrepArgs":
        d = r["layer"]
        m = d["spec"].mixer.left
        p = S.GroupPrepArgs()
        p.proj, p.ld, p.q_off, p.k_off, p.v_off = proj.data_ptr(), ld, d["left.q_at"], d["left.k_at"], d["left.v_at"]
        p.rows, p.heads, p.kv_heads, p.dim, p.vdim, p.dp, p.vp = rows, m.heads, m.kv_heads, m.dim, m.vdim, d["dp"], d["vp"]
        p.q_norm, p.k_norm, p.freq, p.rot_dims = d["q_norm"].data_ptr(), d["k_norm"].data_ptr(), d["freq"].data_ptr(), 2 * d["freq"].numel()
        p.eps, p.scale = rt.spec.norm_eps, m.scale
        p.k_cache, p.v_cache, p.f32, p.pos0, p.capacity = r["k_cache"].data_ptr(), r["v_cache"].data_ptr(), int(rt.f32), pos0.data_ptr(), rt.capacity
        return p

    @staticmethod
    def splits(rt, m) -> int:
        """Context splits of the step's attention: 256 keys each, at most a cluster."""
        keys, n = min(m.window or rt.capacity, rt.capacity), 1
        while n < S.MAX_SPLITS and n * 256 < keys:
            n *= 2
        return n

    @staticmethod
    def step(b: StepBuilder, r: dict, add) -> None:
        rt, d = b.rt, r["layer"]
        m, s, proj, o, o2 = d["spec"].mixer.left, d["spec"].mixer.right, b.buf("proj"), b.buf("o"), b.buf("o2")
        a = b.residual(b.args(d["in"], proj), d["norm1"], add)
        a.bias = d["in_b"].data_ptr()
        b.step(S.PRO_RESIDUAL, S.TEPI_STORE, a)
        t = state_args(rt, r, s, S.STATE_NORMALIZED, proj, o2)
        t.q_off, t.k_off, t.v_off, t.q_scale = d["right.q_at"], d["right.k_at"], d["right.v_at"], s.dim ** -0.5
        t.gi_off, t.gf_off, t.cap = d["right.i_at"], d["right.f_at"], s.cap
        t.gate_off, t.gate_kind, t.norm, t.norm_per_head = d["right.g_at"], S.GATE_SIGMOID, d["norm"].data_ptr(), 1
        b.ops.append(("state", t))
        g = S.GroupDecodeArgs()
        g.p = Parallel.prep_args(rt, r, proj, d["in"].n, 1, rt.ctrl)
        g.window, g.splits, g.out = m.window, Parallel.splits(rt, m), o.data_ptr()
        b.ops.append(("group", g))
        b.product(d["o2"], o2, rt.sy2)
        b.product(d["o"], o, rt.sy)

    @staticmethod
    def step_work(rt, m, d, pos: int) -> List[Tuple[str, float]]:
        a, es = m.left, 4 if rt.f32 else 2
        keys = pos + 1 - (pos // a.window * a.window if a.window else 0)
        return [("parallel_in", d["in"].nbytes), ("mlstm_state", state_bytes(m.right, 1)), ("attention", keys * a.kv_heads * (a.dim + a.vdim) * es),
                ("mlstm_out", d["o2"].nbytes), ("attn_out", d["o"].nbytes)]


MIXERS = {"latent_attention": LatentAttention, "rglru": GatedRecurrence, "channel_delta": DeltaState, "wkv": BonusState, "parallel": Parallel}
