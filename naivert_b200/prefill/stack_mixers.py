"""The token mixers of layer-stack models on the chunk path (the step side is ``runtime/stack_mixers.py``).

    latent attention   [dq | dkv | g] product -> norms, latent rows into the cache -> queries; keys and values of the cached
                       positions expanded block by block -> causal attention, gated -> output product
    recurrence         [y | x] product with biases and GELU -> short convolution -> block-diagonal gate products ->
                       chunked scan from the carried state -> output product
    channel_delta      [q | k | v | step | low ranks] product -> convolution, SiLU, unit vectors -> decay and gate products ->
                       recurrence -> read-out norm and gate -> output product
    wkv                mixes with the previous token -> four products as groups, decay products -> recurrence -> norm, gate -> output
    parallel           one product for both halves; norms, rotation, cache rows -> attention over the row's chunk -> output product;
                       recurrence -> norm, gate -> output product; joined by the next row kernel

One class per mechanism: ``scratch(pf, m, d)`` names the buffers it needs (name -> elements, dtype; shared by name, the largest size
wins), ``run(pf, r, R, pos0)`` executes one layer run over R rows and leaves the sublayer's output in ``y`` (and ``y2``).
``work(...)`` gives the FLOPs and bytes of its stages for the benchmark's tables.
"""
from __future__ import annotations

from typing import Dict, Tuple

import torch

from ..ops import stack_kernels as S
from ..runtime.packing import pad
from ..runtime.stack_mixers import Parallel as StepParallel

Scratch = Dict[str, Tuple[int, torch.dtype]]
F32 = torch.float32


class LatentAttention:
    @staticmethod
    def scratch(pf, m, d) -> Scratch:
        C, KB, hq, hv = pf.C, pf.kv_block, m.heads * d["dp"], m.heads * d["vp"]
        out: Scratch = {"proj": (C * d["in"].n, F32), "cq": (C * pad(m.q_rank, 8), pf.act), "q": (C * hq, pf.act), "kx": (KB * hq, pf.act),
                        "vx": (KB * hv, pf.act), "o": (C * hv, pf.act)}
        if pf.t.capacity > KB:
            out["carry"] = (C * m.heads * (d["vp"] + 2), F32)
        return out

    @staticmethod
    def maps(pf, heads: int, dp: int, vp: int):
        key = ("attn", heads, dp, vp)
        if key not in pf.maps:
            q, kx, vx = pf.buf["q"], pf.buf["kx"], pf.buf["vx"]
            pf.maps[key] = (S.token_map(q, dp, heads, dp, pf.C, heads * dp, 128), S.token_map(kx, dp, heads, dp, pf.kv_block, heads * dp, 64),
                            S.value_map(vx, pf.kv_block, heads * vp, pad(vp, 16)))
        return pf.maps[key]

    @staticmethod
    def run(pf, r: dict, R: int, pos0: int) -> None:
        d, t = r["layer"], pf.t
        m, dp, vp = d["spec"].mixer, d["dp"], d["vp"]
        n_in, qp = d["in"].n, pad(m.q_rank, 8)
        proj, cq, q, kx, vx, o = (pf.buf[n] for n in ("proj", "cq", "q", "kx", "vx", "o"))
        with pf.stage("attn_in"):
            pf.gemm(S.EPI_STORE, d["in"], pf.h, pf.h_ld, R, proj, n_in)
        p = S.LatentPrepArgs()
        p.proj, p.ld, p.rows, p.q_rank, p.kv_rank = proj.data_ptr(), n_in, R, m.q_rank, m.kv_rank
        p.q_w, p.kv_w, p.eps = d["dq_norm"].data_ptr(), d["dkv_norm"].data_ptr(), pf.spec.norm_eps
        cache = r["cache"]
        p.cq, p.cq_ld, p.cache, p.cache_ld = cq.data_ptr(), qp, cache.data_ptr(), cache.shape[1]
        p.f32, p.pos0, p.capacity = int(pf.f32), pf.pos.data_ptr(), t.capacity
        with pf.stage("latent_prep"):
            S.latent_prep(p)
        hq, hv = m.heads * dp, m.heads * vp
        with pf.stage("queries"):
            pf.gemm(S.EPI_STORE, d["uq"], cq, qp, R, q, hq)
        a = S.LatentAttnArgs()
        a.q, a.k, a.v, a.out, a.f32 = q.data_ptr(), kx.data_ptr(), vx.data_ptr(), o.data_ptr(), int(pf.f32)
        a.gate, a.gate_ld = proj.data_ptr() + 4 * (m.q_rank + m.kv_rank), n_in
        a.rows, a.heads, a.dim, a.vdim, a.scale, a.pos0, a.group = R, m.heads, dp, vp, m.scale, pf.pos.data_ptr(), 1
        a.state = pf.buf["carry"].data_ptr() if "carry" in pf.buf else None
        a.status = t.fab.status.data_ptr()
        total = pos0 + R
        for kv0 in range(0, total, pf.kv_block):
            n = min(pf.kv_block, total - kv0)
            off = kv0 * cache.shape[1]
            kw = dict(x_off=off, x_rows=t.capacity - kv0)
            with pf.stage("expand_k"):
                pf.gemm(S.EPI_STORE, d["uk"], cache, cache.shape[1], n, kx, hq, **kw)
            a.kv0, a.kv_rows, a.first, a.last = kv0, n, int(kv0 == 0), int(kv0 + n == total)
            if pf.tensor_cores and max(dp, vp) <= 256:
                a.v_ld = pf.kv_block                 # values feature-major: the K-major operand of P V
                with pf.stage("expand_v"):
                    pf.gemm(S.EPI_TRANSPOSE, d["uv"], cache, cache.shape[1], n, vx, pf.kv_block, **kw)
                with pf.stage("attention"):
                    S.latent_attn_tc(*LatentAttention.maps(pf, m.heads, dp, vp), a)
            else:
                a.v_ld = hv
                pf.gemm(S.EPI_STORE, d["uv"], cache, cache.shape[1], n, vx, hv, **kw)
                with pf.stage("attention_plain"):
                    S.latent_attn_rows(a)
        with pf.stage("attn_out"):
            pf.gemm(S.EPI_STORE, d["o"], o, hv, R, pf.y, pf.spec.hidden)

    @staticmethod
    def work(w, m, d, pos0: int, R: int) -> None:
        ctx, es, hq, hv = pos0 + R, w.es, m.heads * d["dp"], m.heads * d["vp"]
        w.gemm("attn_in", d["in"].n, w.W, R, 4)
        w.add("latent_prep", 0, R * (m.q_rank + m.kv_rank) * (4 + es))
        w.gemm("queries", hq, m.q_rank, R, es)
        w.gemm("expand_k", hq, m.kv_rank, ctx, es)
        w.gemm("expand_v", hv, m.kv_rank, ctx, es)
        pairs = R * pos0 + R * (R + 1) / 2
        w.add("attention", 2.0 * pairs * (hq + hv), R * (hq + 2 * hv) * es + ctx * (hq + hv) * es)
        w.gemm("attn_out", w.W, hv, R, 4)


class GatedRecurrence:
    @staticmethod
    def scratch(pf, m, d) -> Scratch:
        C = pf.C
        return {"xy": (C * 2 * m.width, pf.act), "u": (C * m.blocks * pad(m.block, 8), pf.act), "gates": (C * 2 * m.width, F32),
                "agg": (-(-C // S.scan_tokens()) * 2 * m.width, F32), "o": (C * pad(m.width, 8), pf.act)}

    @staticmethod
    def run(pf, r: dict, R: int, pos0: int) -> None:
        d = r["layer"]
        m = d["spec"].mixer
        bp, wp = pad(m.block, 8), pad(m.width, 8)
        xy, u, gates, agg, o = (pf.buf[n] for n in ("xy", "u", "gates", "agg", "o"))
        with pf.stage("rec_in"):
            pf.gemm(S.EPI_BIAS, d["in"], pf.h, pf.h_ld, R, xy, 2 * m.width, bias=d["in_b"], act_cols=m.width)
        a = S.RecurrenceArgs()
        a.xy, a.xy_ld, a.conv, a.conv_b, a.taps = xy.data_ptr(), 2 * m.width, d["conv"].data_ptr(), d["conv_b"].data_ptr(), m.taps
        a.history, a.hist_rows, a.u = r["history"].data_ptr(), m.hist_rows, u.data_ptr()
        a.gates, a.softplus_lam, a.decay = gates.data_ptr(), d["sp"].data_ptr(), m.decay
        a.state, a.tags, a.agg = r["state"].data_ptr(), r["tags"].data_ptr(), agg.data_ptr()
        a.out, a.out_ld, a.f32, a.rows = o.data_ptr(), wp, int(pf.f32), R
        a.width, a.blocks, a.block, a.block_pad = m.width, m.blocks, m.block, bp
        a.pos0, a.status = pf.pos.data_ptr(), pf.t.fab.status.data_ptr()
        with pf.stage("conv"):
            S.conv(a)
        with pf.stage("rec_gates"):
            pf.gemm(S.EPI_BIAS, d["gates"], u, m.blocks * bp, R, gates, 2 * m.width, z=m.blocks, x_z=bp, out_z=2 * m.block, bias=d["gates_b"])
        with pf.stage("scan"):
            S.scan(a)
        with pf.stage("rec_out"):
            pf.gemm(S.EPI_STORE, d["o"], o, wp, R, pf.y, pf.spec.hidden)

    @staticmethod
    def work(w, m, d, pos0: int, R: int) -> None:
        es = w.es
        w.gemm("rec_in", 2 * m.width, w.W, R, es)
        w.add("conv", 0, R * m.width * 2 * es)
        w.gemm("rec_gates", 2 * m.block, m.block, R, 4, z=m.blocks)
        w.add("scan", 0, R * m.width * (2 * 8 + 2 * es + es + es))
        w.gemm("rec_out", w.W, m.width, R, 4)


# --------------------------------------------------------------------------- matrix states
def state_scratch(pf, m, kind: int) -> Scratch:
    return {"blocks": (-(-pf.C // S.STATE_BLOCK) * m.heads * S.state_block_floats(kind, m.dim), F32),
            "sums": (S.state_sum_floats(kind, m.heads, m.dim, m.vdim), F32)}


def state_args(pf, r: dict, m, R: int, o: torch.Tensor) -> "S.StateChunkArgs":
    a = S.StateChunkArgs()
    a.blocks, a.sums = pf.buf["blocks"].data_ptr(), pf.buf["sums"].data_ptr()
    a.rows, a.heads, a.kv_heads, a.dim, a.vdim, a.q_scale = R, m.heads, getattr(m, "kv_heads", m.heads), m.dim, m.vdim, 1.0
    a.o, a.state, a.state_stride, a.tags = o.data_ptr(), r["state"].data_ptr(), r["state"].shape[1], r["tags"].data_ptr()
    a.pos0, a.status = pf.pos.data_ptr(), pf.t.fab.status.data_ptr()
    return a


def head_gate(pf, m, R: int, o: torch.Tensor, gate: int, gate_ld: int, kind: int, norm: torch.Tensor, per_head: bool, out: torch.Tensor, den=None) -> int:
    """Read-out norm and gate into the output product's operand; returns its row width."""
    a = S.HeadGateArgs()
    hv = m.heads * m.vdim
    a.o, a.gate, a.gate_ld, a.gate_kind, a.norm, a.norm_per_head = o.data_ptr(), gate, gate_ld, kind, norm.data_ptr(), int(per_head)
    a.den = None if den is None else den.data_ptr()
    a.out, a.out_ld, a.f32, a.rows, a.heads, a.vdim, a.eps = out.data_ptr(), pad(hv, 8), int(pf.f32), R, m.heads, m.vdim, pf.spec.norm_eps
    with pf.stage("head_gate"):
        S.head_gate(a)
    return a.out_ld


def state_work(w, stage: str, m, R: int, g: bool, flops: float, extra: int = 0) -> None:
    """Recurrence: fp32 FLOPs per state element and token, operands once; read-out norm and gate."""
    kv = getattr(m, "kv_heads", m.heads)
    w.add32(stage, flops * R * m.heads * m.dim * (m.vdim + extra),
            R * 4 * (2 * kv * m.dim + (m.heads * m.dim if g else 0) + 2 * m.heads * m.vdim) + 2 * 4 * m.heads * (m.vdim + extra) * m.dim)
    w.add("head_gate", 0, R * m.heads * m.vdim * (8 + w.es))


class DeltaState:
    @staticmethod
    def scratch(pf, m, d) -> Scratch:
        C, qk, hd, hv = pf.C, m.kv_heads * m.dim, m.heads * m.dim, m.heads * m.vdim
        return {"proj": (C * pad(d["in"].n, 4), F32), "sq": (C * qk, F32), "sk": (C * qk, F32), "sv": (C * hv, F32), "low": (C * DeltaState.low_ld(m), pf.act),
                "decay": (C * hd, F32), "sgate": (C * hv, F32), "so": (C * hv, F32), "o": (C * pad(hv, 8), pf.act),
                **state_scratch(pf, m, S.STATE_DELTA)}

    @staticmethod
    def low_ld(m) -> int:
        return pad(m.decay_rank, 8) + pad(m.gate_rank, 8)

    @staticmethod
    def run(pf, r: dict, R: int, pos0: int) -> None:
        d = r["layer"]
        m = d["spec"].mixer
        qk, hd, hv, ld, low_ld = m.kv_heads * m.dim, m.heads * m.dim, m.heads * m.vdim, pad(d["in"].n, 4), DeltaState.low_ld(m)
        proj, sq, sk, sv, low, decay, sgate, so, o = (pf.buf[n] for n in ("proj", "sq", "sk", "sv", "low", "decay", "sgate", "so", "o"))
        with pf.stage("delta_in"):
            pf.gemm(S.EPI_STORE, d["in"], pf.h, pf.h_ld, R, proj, ld)
        c = S.ShortConvArgs()
        c.proj, c.ld, c.rows, c.heads, c.kv_heads, c.dim, c.vdim, c.taps = proj.data_ptr(), ld, R, m.heads, m.kv_heads, m.dim, m.vdim, m.taps
        c.conv, c.history, c.hist_rows, c.q_scale = d["conv"].data_ptr(), r["history"].data_ptr(), m.hist_rows, m.dim ** -0.5
        c.q, c.k, c.v, c.low, c.low_ld = sq.data_ptr(), sk.data_ptr(), sv.data_ptr(), low.data_ptr(), low_ld
        c.low_off, c.low_cols, c.low2_off, c.low2_cols, c.low2_at = d["a1_at"], m.decay_rank, d["g1_at"], m.gate_rank, pad(m.decay_rank, 8)
        c.f32, c.pos0 = int(pf.f32), pf.pos.data_ptr()
        with pf.stage("short_conv"):
            S.short_conv(c)
        with pf.stage("delta_decay"):
            pf.gemm(S.EPI_DECAY_SOFT, d["a2"], low, low_ld, R, decay, hd, bias=d["dt_bias"], rate=d["rate"])
        with pf.stage("delta_gate"):
            pf.gemm(S.EPI_STORE, d["g2"], low, low_ld, R, sgate, hv, x_off=pad(m.decay_rank, 8))
        a = state_args(pf, r, m, R, so)
        a.q, a.k, a.v, a.g, a.q_ld, a.k_ld, a.v_ld, a.g_ld = sq.data_ptr(), sk.data_ptr(), sv.data_ptr(), decay.data_ptr(), qk, qk, hv, hd
        a.beta, a.beta_ld = proj.data_ptr() + 4 * d["beta_at"], ld
        a.hist_src, a.hist_ld, a.hist_cols, a.taps = proj.data_ptr(), ld, m.conv_columns, m.taps
        a.hist_rows, a.history = m.hist_rows, r["history"].data_ptr()
        with pf.stage("delta_state"):
            S.state_chunk(S.STATE_DELTA, a)
        o_ld = head_gate(pf, m, R, so, sgate.data_ptr(), hv, S.GATE_SIGMOID, d["norm"], False, o)
        with pf.stage("delta_out"):
            pf.gemm(S.EPI_STORE, d["o"], o, o_ld, R, pf.y, pf.spec.hidden)

    @staticmethod
    def work(w, m, d, pos0: int, R: int) -> None:
        cols, hd, hv = m.conv_columns, m.heads * m.dim, m.heads * m.vdim
        w.gemm("delta_in", d["in"].n, w.W, R, 4)
        w.add("short_conv", 0, R * (8 * cols + (m.decay_rank + m.gate_rank) * (4 + w.es)))
        w.gemm("delta_decay", hd, m.decay_rank, R, 4)
        w.gemm("delta_gate", hv, m.gate_rank, R, 4)
        state_work(w, "delta_state", m, R, True, 7.0)
        w.gemm("delta_out", w.W, hv, R, 4)


class BonusState:
    @staticmethod
    def scratch(pf, m, d) -> Scratch:
        C, n = pf.C, m.heads * m.dim
        return {"mixes": (C * 5 * pf.h_ld, pf.act), "proj": (C * 4 * pad(d["part"], 4), F32), "low": (C * pad(m.decay_rank, 8), pf.act),
                "decay": (C * n, F32), "so": (C * n, F32), "o": (C * pad(n, 8), pf.act), **state_scratch(pf, m, S.STATE_BONUS)}

    @staticmethod
    def run(pf, r: dict, R: int, pos0: int) -> None:
        d, hl, W = r["layer"], pf.h_ld, pf.spec.hidden
        m, part = d["spec"].mixer, d["part"]
        n, zs = m.heads * m.dim, pad(part, 4)
        mixes, proj, low, decay, so, o = (pf.buf[x] for x in ("mixes", "proj", "low", "decay", "so", "o"))
        t = S.TokenMixArgs()
        t.x, t.rows, t.width, t.mixes, t.mu = pf.x.data_ptr(), R, W, 5, d["mu"].data_ptr()
        t.out, t.out_ld, t.f32 = mixes.data_ptr(), hl, int(pf.f32)
        t.shift, t.state_stride, t.tags = r["state"].data_ptr() + 4 * m.shift_at, r["state"].shape[1], r["tags"].data_ptr()
        t.pos0, t.status = pf.pos.data_ptr(), pf.t.fab.status.data_ptr()
        with pf.stage("token_mix"):
            S.token_mix(t)
        with pf.stage("wkv_in"):
            pf.gemm(S.EPI_STORE, d["in"].rows(0, part, 4), mixes, 5 * hl, R, proj, 4 * zs, z=4, x_z=hl, out_z=zs)
        lp = pad(m.decay_rank, 8)
        with pf.stage("wkv_low"):
            pf.gemm(S.EPI_TANH, d["in"].rows(4 * part, m.decay_rank), mixes, 5 * hl, R, low, lp, x_off=4 * hl)
        with pf.stage("wkv_decay"):
            pf.gemm(S.EPI_DECAY_EXP, d["w2"], low, lp, R, decay, n, bias=d["w0"])
        a = state_args(pf, r, m, R, so)
        at = proj.data_ptr()
        a.q, a.k, a.v, a.g, a.q_ld, a.k_ld, a.v_ld, a.g_ld = at, at + 4 * zs, at + 8 * zs, decay.data_ptr(), 4 * zs, 4 * zs, 4 * zs, n
        a.u = d["u"].data_ptr()
        with pf.stage("wkv_state"):
            S.state_chunk(S.STATE_BONUS, a)
        o_ld = head_gate(pf, m, R, so, at + 12 * zs, 4 * zs, S.GATE_SILU, d["norm"], True, o)
        with pf.stage("wkv_out"):
            pf.gemm(S.EPI_STORE, d["o"], o, o_ld, R, pf.y, W)

    @staticmethod
    def work(w, m, d, pos0: int, R: int) -> None:
        n = m.heads * m.dim
        w.add("token_mix", 0, R * w.W * (4 + 5 * w.es))
        w.gemm("wkv_in", n, w.W, R, 4, z=4)
        w.gemm("wkv_low", m.decay_rank, w.W, R, w.es)
        w.gemm("wkv_decay", n, m.decay_rank, R, 4)
        state_work(w, "wkv_state", m, R, True, 5.0)
        w.gemm("wkv_out", w.W, n, R, 4)


# --------------------------------------------------------------------------- two mixers side by side
class Parallel:
    @staticmethod
    def keys(pf, m) -> int:
        """Most positions the attention of one chunk looks at (the start of its mask chunk up to its last row)."""
        cap = pf.t.capacity
        return pad(min(cap, m.window - 1 + pf.C) if m.window else cap, 64)

    @staticmethod
    def scratch(pf, m, d) -> Scratch:
        C, a, s = pf.C, m.left, m.right
        hv = s.heads * s.vdim
        return {"proj": (C * pad(d["in"].n, 4), F32), "q": (C * a.heads * d["dp"], pf.act), "vx": (Parallel.keys(pf, a) * a.kv_heads * d["vp"], pf.act),
                "o": (C * max(a.heads * d["vp"], pad(hv, 8)), pf.act), "so": (C * hv, F32), "den": (C * s.heads * 2, F32), "keep": (C * s.heads * 2, F32), **state_scratch(pf, s, S.STATE_NORMALIZED)}

    @staticmethod
    def maps(pf, r: dict):
        d = r["layer"]
        m, dp, vp, keys = d["spec"].mixer.left, d["dp"], d["vp"], Parallel.keys(pf, d["spec"].mixer.left)
        key = ("grouped", r["run"].run)
        if key not in pf.maps:
            pf.maps[key] = (S.token_map(pf.buf["q"], dp, m.heads, dp, pf.C, m.heads * dp, 128),
                            S.token_map(r["k_cache"], dp, m.kv_heads, dp, pf.t.capacity, m.kv_heads * dp, 64),
                            S.value_map(pf.buf["vx"], keys, m.kv_heads * vp, pad(vp, 16)))
        return pf.maps[key]

    @staticmethod
    def attention(pf, r: dict, R: int, pos0: int, proj: torch.Tensor, ld: int) -> None:
        d, t = r["layer"], pf.t
        m, dp, vp, q, vx, o = d["spec"].mixer.left, d["dp"], d["vp"], pf.buf["q"], pf.buf["vx"], pf.buf["o"]
        p = StepParallel.prep_args(t, r, proj, ld, R, pf.pos)
        p.q = q.data_ptr()
        with pf.stage("group_prep"):
            S.group_prep(p)
        start = pos0 // m.window * m.window if m.window else 0           # keys before it belong to other mask chunks
        n, es = pos0 + R - start, q.element_size()
        a = S.LatentAttnArgs()
        a.q, a.out, a.f32, a.rows, a.heads, a.dim, a.vdim, a.scale = q.data_ptr(), o.data_ptr(), int(pf.f32), R, m.heads, dp, vp, 1.0
        a.group, a.window, a.k_row0 = m.heads // m.kv_heads, m.window, start
        a.k, a.v = r["k_cache"].data_ptr() + es * start * m.kv_heads * dp, r["v_cache"].data_ptr() + es * start * m.kv_heads * vp
        a.pos0, a.kv0, a.kv_rows, a.first, a.last, a.status = pf.pos.data_ptr(), start, n, 1, 1, t.fab.status.data_ptr()
        if pf.tensor_cores and max(dp, vp) <= 256:
            x = S.TransposeArgs()
            x.src, x.dst, x.dst_ld, x.rows, x.cols = a.v, vx.data_ptr(), Parallel.keys(pf, m), n, m.kv_heads * vp
            with pf.stage("values_t"):
                S.transpose(x)
            with pf.stage("attention"):
                S.latent_attn_tc(*Parallel.maps(pf, r), a)
        else:
            with pf.stage("attention_plain"):
                S.latent_attn_rows(a)
        with pf.stage("attn_out"):
            pf.gemm(S.EPI_STORE, d["o"], o, m.heads * vp, R, pf.y, pf.spec.hidden)

    @staticmethod
    def run(pf, r: dict, R: int, pos0: int) -> None:
        d = r["layer"]
        s, ld = d["spec"].mixer.right, pad(d["in"].n, 4)
        proj, so, den, o = (pf.buf[n] for n in ("proj", "so", "den", "o"))
        with pf.stage("parallel_in"):
            pf.gemm(S.EPI_BIAS, d["in"], pf.h, pf.h_ld, R, proj, ld, bias=d["in_b"])
        Parallel.attention(pf, r, R, pos0, proj, ld)

        def at(name: str) -> int:
            return proj.data_ptr() + 4 * d[f"right.{name}_at"]

        a = state_args(pf, r, s, R, so)
        a.q, a.k, a.v, a.q_ld, a.k_ld, a.v_ld, a.q_scale = at("q"), at("k"), at("v"), ld, ld, ld, s.dim ** -0.5
        a.gi, a.gf, a.gate_ld, a.cap, a.den = at("i"), at("f"), ld, s.cap, den.data_ptr()
        a.keep = pf.buf["keep"].data_ptr()
        with pf.stage("mlstm_state"):
            S.state_chunk(S.STATE_NORMALIZED, a)
        o_ld = head_gate(pf, s, R, so, at("g"), ld, S.GATE_SIGMOID, d["norm"], True, o, den)
        with pf.stage("mlstm_out"):
            pf.gemm(S.EPI_STORE, d["o2"], o, o_ld, R, pf.y2, pf.spec.hidden)

    @staticmethod
    def work(w, m, d, pos0: int, R: int) -> None:
        a, s, es = m.left, m.right, w.es
        hq, hv, kd, vd = a.heads * a.dim, a.heads * a.vdim, a.kv_heads * a.dim, a.kv_heads * a.vdim
        pairs = sum(p % a.window + 1 if a.window else p + 1 for p in range(pos0, pos0 + R))
        keys = pos0 + R - (pos0 // a.window * a.window if a.window else 0)
        w.gemm("parallel_in", d["in"].n, w.W, R, 4)
        w.add("group_prep", 0, R * (hq + kd + vd) * (4 + es))
        w.add("values_t", 0, 2 * keys * vd * es)
        w.add("attention", 2.0 * pairs * (hq + hv), R * (hq + hv) * es + keys * (kd + vd) * es)
        w.gemm("attn_out", w.W, hv, R, 4)
        state_work(w, "mlstm_state", s, R, False, 5.0, 1)
        w.gemm("mlstm_out", w.W, s.heads * s.vdim, R, 4)


MIXERS = {"latent_attention": LatentAttention, "rglru": GatedRecurrence, "channel_delta": DeltaState, "wkv": BonusState, "parallel": Parallel}
