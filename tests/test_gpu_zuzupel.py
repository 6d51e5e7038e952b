"""The Zuzupel design on the GPU against its plain implementation (``zuzupel_oracle``): every mechanism alone and together, prompts
against token-by-token decoding, portions, edges of mask chunks and tiles, carried and reused states, long decoding, kernels of the
matrix states by themselves, greedy generation through the engine and the session engine.

Configurations and weights are made here.  The float form is compared tightly, row by row; the bf16 form within the rounding of
its matrix operands, where a few rows may differ more: a head's read-out that happens to be nearly zero is blown up by its norm,
rounding errors with it (the plain implementation shows the same rows when its operands are rounded).
"""
import json
import math
import os
import subprocess

import pytest
import torch

import zuzupel_oracle as oracle
from stack_testing import TOL, error, feed, tokens

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


# --------------------------------------------------------------------------- cases
def delta(heads=4, kv_heads=2, dim=24, vdim=40, conv=3, ranks=(10, 14)):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, "ranks": ranks}


def wkv(heads=3, dim=20, rank=12):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim}, "ranks": (rank,)}


def both(heads=4, kv_heads=2, dim=24, vdim=32, size=40, rot=16, base=1000.0, factor=4.0, scale=None, rheads=3, rdim=28, rvdim=20, cap=9.0):
    return {"type": "parallel", "mixer": {
        "left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale,
                 "mask": {"size": size}, "rot": {"dims": rot, "base": base, "scaling": {"factor": factor}}},
        "right": {"heads": rheads, "dim": rdim, "vdim": rvdim, "gate_cap": cap}}}


def ff(n=104):
    return {"kind": "dense", "ff": n}


def shared(j, layer):
    return dict(layer, weights_of=j)


def model(layers, width=88, vocab=203, eps=1e-5):
    return {"architecture": "Zuzupel", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": [dict(m, mlp=f) for m, f in layers]}


def config_json(cfg):
    return dict(cfg, layers=[{k: v for k, v in x.items() if k != "ranks"} for x in cfg["layers"]])


def weights(cfg, seed=0):
    g = torch.Generator().manual_seed(seed)

    def r(*shape, s=None, mean=0.0):
        s = shape[-1] ** -0.5 if s is None else s
        return (mean + torch.randn(*shape, generator=g) * s).to(torch.bfloat16)

    def norm(n):
        return r(n, s=0.2, mean=1.0)

    W = cfg["width"]
    out = {"embed": r(cfg["vocab"], W, s=0.6), "final.norm": norm(W), "head": r(cfg["vocab"], W)}
    for i, layer in enumerate(cfg["layers"]):
        if layer.get("weights_of") is not None:
            continue
        p, m, f = f"l{i}.", layer["mixer"], layer.get("mlp")
        out[p + "norm1"] = norm(W)
        x = p + "mix."
        if layer["type"] == "channel_delta":
            H, G, D, V, t, (ra, rg) = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"], layer["ranks"]
            for n, rows in (("q", G * D), ("k", G * D), ("v", H * V)):
                out.update({x + n: r(rows, W), x + n + ".conv": r(rows, t)})
            out.update({x + "b": r(H, W), x + "A_log": r(H, s=0.7), x + "norm": norm(V), x + "a1": r(ra, W), x + "a2": r(H * D, ra), x + "dt_bias": r(H * D, s=1.0, mean=-1.0),
                        x + "g1": r(rg, W), x + "g2": r(H * V, rg), x + "o": r(W, H * V)})
        elif layer["type"] == "wkv":
            n = m["heads"] * m["dim"]
            rw = layer["ranks"][0]
            for s in "rkvgw":
                out[x + "mu." + s] = r(W, s=0.3, mean=0.5)
            for s in "rkvg":
                out[x + s] = r(n, W)
            out.update({x + "w1": r(rw, W), x + "w2": r(n, rw), x + "w0": r(n, s=1.0, mean=-1.0), x + "u": r(m["heads"], m["dim"], s=0.6), x + "norm": norm(n), x + "o": r(W, n)})
        else:
            a, b = m["left"], m["right"]
            for n, rows in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"])):
                out.update({x + "left." + n: r(rows, W), x + "left." + n + ".b": r(rows, s=0.3)})
            rk, rv = b["heads"] * b["dim"], b["heads"] * b["vdim"]
            out.update({x + "left.q.norm": r(a["dim"], s=0.5, mean=2.0), x + "left.k.norm": norm(a["dim"]), x + "left.o": r(W, a["heads"] * a["vdim"]), x + "left.out": norm(W),
                        x + "right.q": r(rk, W), x + "right.k": r(rk, W), x + "right.v": r(rv, W), x + "right.g": r(rv, W), x + "right.o": r(W, rv),
                        x + "right.norm": norm(rv), x + "right.i": r(b["heads"], W), x + "right.i.b": r(b["heads"], s=0.5, mean=-1.0),
                        x + "right.f": r(b["heads"], W), x + "right.f.b": r(b["heads"], s=1.0, mean=2.0), x + "right.out": norm(W)})
        if f:
            out.update({p + "norm2": norm(W), p + "mlp.up": r(f["ff"], W), p + "mlp.down": r(W, f["ff"])})
    return out


CASES = {
    "delta": model([(delta(), None)]),
    "delta_equal_heads": model([(delta(heads=3, kv_heads=3, dim=64, vdim=32, conv=4), None)]),
    "delta_odd": model([(delta(heads=3, kv_heads=1, dim=13, vdim=21, conv=1, ranks=(5, 3)), None)], width=51, vocab=97),
    "delta_wide": model([(delta(heads=2, kv_heads=1, dim=136, vdim=72, conv=6, ranks=(33, 8)), None)]),
    "delta_very_wide": model([(delta(heads=1, kv_heads=1, dim=300, vdim=260, conv=2, ranks=(16, 40)), None)]),
    "delta_128": model([(delta(heads=2, kv_heads=2, dim=128, vdim=130, conv=4, ranks=(130, 7)), None)]),
    "wkv": model([(wkv(), None)]),
    "wkv_64": model([(wkv(heads=2, dim=64, rank=16), None)]),
    "wkv_odd": model([(wkv(heads=5, dim=7, rank=3), None)], width=45, vocab=101),
    "wkv_rank_above_width": model([(wkv(heads=1, dim=16, rank=50), None)]),
    "wkv_wide": model([(wkv(heads=1, dim=140, rank=9), None)]),
    "parallel": model([(both(), None)]),
    "parallel_one_head": model([(both(heads=1, kv_heads=1, dim=10, vdim=6, size=16, rot=2, rheads=1, rdim=5, rvdim=3), None)], width=45, vocab=97),
    "parallel_many_heads": model([(both(heads=36, kv_heads=1, dim=16, vdim=24, size=64, rot=16, rheads=2, rdim=100, rvdim=70), None)]),
    "parallel_tile_of_32": model([(both(heads=40, kv_heads=2, dim=40, vdim=16, size=100, rot=40, scale=0.3), None)]),
    "parallel_beyond_tensor_cores": model([(both(heads=2, kv_heads=1, dim=264, vdim=272, size=33, rot=100), None)]),
    "parallel_chunks_of_one": model([(both(size=1), None)]),
    "parallel_one_chunk": model([(both(size=4096, factor=1.0, base=20.0, rdim=64, rvdim=256, rheads=1), None)]),
    "relu2": model([(wkv(), ff(130))], width=91),
    "shared": model([(delta(), ff()), (wkv(), None), (shared(0, delta()), ff()), (shared(2, delta()), ff()), (shared(1, wkv()), None)]),
    "shared_ahead": model([(shared(2, both()), ff()), (wkv(), None), (both(), ff())]),
    "mixed": model([(delta(conv=4), ff()), (wkv(heads=2, dim=48), ff(72)), (both(size=48), ff()), (shared(0, delta(conv=4)), ff()), (both(kv_heads=4, size=24), None)], width=136),
}


def shapes_of(w):
    return {n: tuple(t.shape) for n, t in w.items()}


def engine(cfg, w, dtype="fp32", capacity=512, chunk=96):
    from naivert_b200.models import zuzupel
    from naivert_b200.runtime.stack_engine import build_stack_engine
    spec = zuzupel.spec_from_config(config_json(cfg), "case", shapes_of(w))
    assert zuzupel.tensor_shapes(spec) == shapes_of(w)
    return build_stack_engine(spec, capacity=capacity, device=torch.device("cuda", 0), weights=zuzupel.gather_weights(spec, lambda n: w[n].cuda()),
                              prefill_chunk=chunk, dtype=dtype)


def check(got, want, dtype, what, tol=None):
    e = error(got, want)
    over = int((e > (tol or TOL[dtype])).sum())
    allowed = 0 if dtype == "fp32" else max(1, len(e) // 40)
    assert torch.isfinite(e).all() and over <= allowed, (what, dtype, over, int(e.argmax()), float(e.max()))
    assert dtype == "fp32" or e.median() < TOL["bf16"] / 2, (what, float(e.median()))


# --------------------------------------------------------------------------- mechanisms, prompts, decoding, portions
@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("name", sorted(CASES))
def test_mechanism_prompt_decode_and_portions(name, dtype):
    cfg = CASES[name]
    w = weights(cfg, seed=len(name))
    toks = tokens(cfg, 150)
    ref = oracle.forward(cfg, w, toks)
    eng = engine(cfg, w, dtype, chunk=160)
    try:
        for sizes in ([150], [1], [70, 2, 3, 2, 64, 1], [2], [96, 1]):
            check(feed(eng, toks, sizes), ref, dtype, (name, sizes))
    finally:
        eng.close()


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("name", ["delta", "wkv_64", "parallel_one_chunk"])
def test_long_chunks(name, dtype):
    """Chunks of many blocks and pieces, and of more rows than one scan of the gates takes."""
    cfg = CASES[name]
    w = weights(cfg, seed=3)
    toks = tokens(cfg, 1100)
    ref = oracle.forward(cfg, w, toks)
    eng = engine(cfg, w, dtype, capacity=1152, chunk=1100)
    try:
        for sizes in ([1100], [517, 583], [256, 64, 780]):
            check(feed(eng, toks, sizes), ref, dtype, (name, sizes))
    finally:
        eng.close()


def test_stream_after_every_layer_run():
    cfg = CASES["mixed"]
    w = weights(cfg, 3)
    toks, trace, got = tokens(cfg, 70), [], []
    oracle.forward(cfg, w, toks, trace=trace)
    eng = engine(cfg, w)
    try:
        eng.prefill.extend(torch.tensor(toks), 0, (), got)
        assert len(got) == len(trace) == 5
        for a, b in zip(got, trace):
            assert float((a.double().cpu() - b).norm() / b.norm()) < 1e-5
    finally:
        eng.close()


# --------------------------------------------------------------------------- keys at the edges of chunks and tiles
def needle_model(size, width=64):
    """One layer in which token 58 looks up token 59: that one key carries nearly the whole weight wherever it is visible.  The matrix
    memory beside the attention is silenced, the rotation slowed to nothing."""
    cfg = model([(both(heads=2, kv_heads=1, dim=width, vdim=32, size=size, rot=2, factor=1e7, scale=12.0 / width), None)], width=width, vocab=60)
    w = weights(cfg, 11)
    g = torch.Generator().manual_seed(1)
    basis = torch.linalg.qr(torch.randn(width, width, generator=g))[0] * math.sqrt(width)
    w["embed"] = basis[:60].to(torch.bfloat16)
    eye = torch.eye(width, dtype=torch.bfloat16)
    ask = torch.outer(basis[59], basis[58]) / width           # token 58 asks for token 59, the others for nothing in particular
    p = "l0.mix.left."
    w[p + "k"], w[p + "q"] = eye, torch.cat([ask, ask]).to(torch.bfloat16)
    for n in ("q.b", "k.b", "v.b"):
        w[p + n] = torch.zeros_like(w[p + n])
    w[p + "q.norm"] = w[p + "k.norm"] = torch.ones(width, dtype=torch.bfloat16)
    w["l0.mix.right.o"] = torch.zeros_like(w["l0.mix.right.o"])
    return cfg, w


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("size,n", [(64, 192), (64, 193), (64, 230), (100, 300), (100, 201), (48, 97), (500, 330), (130, 260)])
def test_one_key_stands_out_where_it_is_visible(size, n, dtype):
    """The last token asks for one key: inside its chunk the answer is the key's value, one position outside it the key is
    not there, in prompts, short portions and decoding."""
    cfg, w = needle_model(size)
    base = [2 + (i * 7) % 50 for i in range(n)]
    edge = (n - 1) // size * size                              # first position that the last token sees
    spots = sorted({p for p in (0, 1, edge - 65, edge - 64, edge - 2, edge - 1, edge, edge + 1, edge + 2, edge + 62, edge + 63, edge + 64, edge + 65, n - 3, n - 2)
                    if 0 <= p < n - 1})
    eng = engine(cfg, w, dtype, capacity=n + 8, chunk=128)
    try:
        for where in spots:
            toks = list(base)
            toks[where], toks[-1] = 59, 58
            ref = oracle.forward(cfg, w, toks)[-1:]
            gone = list(toks)
            gone[where] = 3
            shows = float(error(oracle.forward(cfg, w, gone)[-1:], ref))
            assert shows > 0.1 if where >= edge else shows < 1e-9
            for sizes in ([n], [n - 1, 1], [max(1, edge), n]) + (([n - 2, 2], [max(1, edge - 1), 2, n]) if dtype == "fp32" else ()):
                e = error(feed(eng, toks, sizes)[-1:], ref)
                assert e < TOL[dtype], (where, sizes, float(e))
    finally:
        eng.close()


# --------------------------------------------------------------------------- state
@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
def test_long_decoding_and_reused_state(dtype):
    """Hundreds of decoded tokens; then shorter and longer sequences over the same caches and state slots."""
    cfg = CASES["mixed"]
    w = weights(cfg, 2)
    eng = engine(cfg, w, dtype)
    try:
        first = {}
        for n in (320, 5, 130, 1, 2, 320):
            toks = tokens(cfg, n, 40 + n)
            got = feed(eng, toks, [9, 1] if n > 9 else [1])
            check(got, oracle.forward(cfg, w, toks), dtype, n)
            if n in first:
                assert torch.equal(got, first[n])           # nothing of what ran in between is left
            first[n] = got
    finally:
        eng.close()


@pytest.mark.parametrize("name", ["delta", "wkv", "parallel", "shared"])
def test_repeated_step_and_broken_hand_over(name):
    """A step may be repeated at its position; a step from a position no state was left for is reported, not computed."""
    cfg = CASES[name]
    w = weights(cfg, 4)
    toks = tokens(cfg, 40)
    ref = oracle.forward(cfg, w, toks)
    eng = engine(cfg, w)
    try:
        eng.extend(toks[:39])
        t = eng.target
        for _ in range(3):
            t.set_inputs([toks[39]], 39)
            t.step()
            torch.cuda.synchronize()
            assert error(t.logits, ref[39:]) < TOL["fp32"]
        t.set_inputs([toks[39]], 12)
        t.step()
        torch.cuda.synchronize()
        with pytest.raises(RuntimeError, match="no state for the position"):
            eng.fabric.check()
        eng.fabric.status.zero_()
        assert error(feed(eng, toks, [40])[-1:], ref[39:]) < TOL["fp32"]
    finally:
        eng.close()


@pytest.mark.parametrize("name", ["delta", "wkv", "parallel"])
def test_slow_decay_keeps_the_first_token(name):
    """With decays near one a state must still carry the first token after hundreds of steps, blocks and pieces."""
    layer = {"delta": delta(heads=2, kv_heads=1, dim=32, vdim=24, conv=2), "wkv": wkv(heads=2, dim=32), "parallel": both(size=8, rdim=32, rvdim=24)}[name]
    cfg = model([(layer, None)], vocab=50)
    w = weights(cfg, 6)
    if name == "delta":
        w["l0.mix.A_log"] = torch.full_like(w["l0.mix.A_log"], -9.0)
        w["l0.mix.b"] = w["l0.mix.b"] * 0.1
    elif name == "wkv":
        w["l0.mix.w0"] = torch.full_like(w["l0.mix.w0"], -11.0)
        w["l0.mix.w2"] = w["l0.mix.w2"] * 0.1
    else:
        w["l0.mix.right.f.b"] = torch.full_like(w["l0.mix.right.f.b"], 30.0)
        w["l0.mix.right.f"] = w["l0.mix.right.f"] * 0.1
    toks = tokens(cfg, 300)
    other = [(toks[0] + 1) % 50] + toks[1:]
    ref = oracle.forward(cfg, w, toks)
    assert error(oracle.forward(cfg, w, other)[-1:], ref[-1:]) > 1e-3
    eng = engine(cfg, w, capacity=320, chunk=300)
    try:
        for sizes in ([300], [65, 64, 63, 1], [200, 1]):
            assert error(feed(eng, toks, sizes), ref).max() < TOL["fp32"]
    finally:
        eng.close()


def test_gates_at_their_limits():
    """Input gates far above and below the running maximum, the denominator's floor and decays that wipe the state."""
    cfg = model([(both(size=8, cap=40.0), None), (wkv(), None), (delta(), None)])
    w = weights(cfg, 9)
    for n in ("right.i", "right.f"):
        w["l0.mix." + n] = w["l0.mix." + n] * 30
    w["l1.mix.w2"], w["l2.mix.a2"] = w["l1.mix.w2"] * 6, w["l2.mix.a2"] * 30
    toks = tokens(cfg, 200)
    ref = oracle.forward(cfg, w, toks)
    assert torch.isfinite(ref).all()
    eng = engine(cfg, w, chunk=200)
    try:
        for sizes in ([200], [1], [33, 2, 140, 1]):
            check(feed(eng, toks, sizes), ref, "fp32", sizes, 1e-3)
    finally:
        eng.close()


# --------------------------------------------------------------------------- kernels by themselves
@pytest.mark.parametrize("rows", [1, 8, 57, 300])
@pytest.mark.parametrize("kind,heads,kv,dim,vdim", [(0, 3, 1, 20, 36), (0, 2, 2, 128, 33), (0, 1, 1, 200, 16), (1, 2, 2, 48, 48), (1, 1, 1, 130, 130), (2, 3, 3, 24, 50), (2, 1, 1, 128, 7),
                                                    (2, 1, 1, 400, 20)])
def test_matrix_state_kernels(kind, heads, kv, dim, vdim, rows):
    """The recurrence over a chunk, entered with a state, against the plain rule; decays from nearly zero to one."""
    from naivert_b200.ops import stack_kernels as S
    g = torch.Generator().manual_seed(rows + dim)
    n = rows + 11                                            # the first 11 tokens leave the state that the chunk starts from

    def r(*shape):
        return torch.randn(*shape, generator=g)

    q, k, v = r(n, kv, dim) * dim ** -0.5, r(n, kv, dim) * dim ** -0.5, r(n, heads, vdim)
    decay = torch.rand(n, heads, dim, generator=g) ** 0.2
    decay[:: 5, :, ::3], decay[2:: 7] = 1e-7, 1.0
    beta, u, gi, gf = r(n, heads), r(heads, dim).to(torch.bfloat16), 3 * r(n, heads), 3 * r(n, heads) + 2
    cap, scale = 6.0, 0.7
    C = vdim + (kind == 2)
    d4 = (dim + 3) // 4 * 4
    stride = (heads * C * d4 + heads + 3) // 4 * 4
    state, tags = torch.full((2, stride), float("nan"), device="cuda"), torch.full((2,), -1, dtype=torch.int32, device="cuda")
    status = torch.zeros(16, dtype=torch.int32, device="cuda")
    out = []
    for lo, hi in ((0, 11), (11, n)):
        R = hi - lo
        t = {name: x[lo:hi].contiguous().cuda() for name, x in (("q", q), ("k", k), ("v", v), ("g", decay), ("beta", beta), ("gi", gi), ("gf", gf))}
        t.update(u=u.cuda(), o=torch.zeros(R, heads, vdim, device="cuda"), den=torch.zeros(R, heads, 2, device="cuda"), keep=torch.zeros(R, heads, 2, device="cuda"),
                 blocks=torch.full((-(-R // S.STATE_BLOCK) * heads * S.state_block_floats(kind, dim),), float("nan"), device="cuda"),
                 sums=torch.full((max(1, S.state_sum_floats(kind, heads, dim, vdim)),), float("nan"), device="cuda"),
                 pos=torch.tensor([lo], dtype=torch.int32, device="cuda"))
        a = S.StateChunkArgs()
        for f in ("q", "k", "v", "g", "beta", "u", "gi", "gf", "o", "den", "keep", "blocks", "sums"):
            setattr(a, f, t[f].data_ptr())
        a.q_ld = a.k_ld = kv * dim
        a.v_ld, a.g_ld, a.beta_ld, a.gate_ld = heads * vdim, heads * dim, heads, heads
        a.rows, a.heads, a.kv_heads, a.dim, a.vdim, a.q_scale, a.cap = R, heads, kv, dim, vdim, scale, cap
        a.state, a.state_stride, a.tags, a.pos0, a.status = state.data_ptr(), stride, tags.data_ptr(), t["pos"].data_ptr(), status.data_ptr()
        S.state_chunk(kind, a)
        torch.cuda.synchronize()
        o = t["o"].double().cpu()
        if kind == 2:
            d = t["den"].double().cpu()
            o = o / (torch.maximum(d[..., 0].abs(), d[..., 1])[..., None] + 1e-6)
        out.append(o)
    assert int(status[0]) == 0 and n in tags.tolist()
    got = torch.cat(out)
    q, k, v, decay, beta, u, gi, gf = (x.double() for x in (q, k, v, decay, beta, u, gi, gf))
    for h in range(heads):
        x = h * kv // heads
        if kind == 0:
            ref = oracle.delta_rule(q[:, x] * scale, k[:, x], v[:, h], oracle.sigmoid(beta[:, h]), decay[:, h])
        elif kind == 1:
            ref = oracle.wkv_rule(q[:, x] * scale, k[:, x], v[:, h], decay[:, h], u[h])
        else:
            ref = oracle.mlstm_rule(q[:, x] * scale, k[:, x], v[:, h], cap * torch.tanh(gi[:, h] / cap), oracle.log_sigmoid(cap * torch.tanh(gf[:, h] / cap)))
        e = (got[:, h] - ref).norm(dim=-1) / ref.norm(dim=-1).clamp(min=1e-2)
        assert e.max() < 1e-4, (h, int(e.argmax()), float(e.max()))


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
def test_map_products_against_torch(dtype):
    """Epilogues of the chunk products that map one value, and row slices of a stacked matrix."""
    from naivert_b200.ops import stack_kernels as S
    from naivert_b200.runtime.packing import pack, pad
    eng = engine(CASES["mixed"], weights(CASES["mixed"]), dtype, capacity=1024, chunk=1024)
    pf = eng.prefill
    g = torch.Generator(device="cuda").manual_seed(1)
    try:
        for rows, n, k in ((1, 37, 20), (63, 300, 136), (700, 129, 50), (300, 4000, 24)):
            kp = pad(k, 8)
            x = torch.zeros(rows, kp, dtype=pf.act, device="cuda")
            x[:, :k] = torch.randn(rows, k, generator=g, device="cuda")
            w = (torch.randn(n + 9, k, generator=g, device="cuda") * k ** -0.5).to(torch.bfloat16)
            bias, rate = torch.randn(n, generator=g, device="cuda").to(torch.bfloat16), torch.rand(n, generator=g, device="cuda") * 2
            p = pack(w, "cuda").rows(9, n)
            y = x[:, :k].double() @ w[9:].double().T

            def run(epi, **more):
                out = torch.full((rows, n), float("nan"), device="cuda")
                pf.gemm(epi, p, x, kp, rows, out, n, x_rows=rows, **more)
                torch.cuda.synchronize()
                return out.double()

            z = y + bias.double()
            for got, want in ((run(S.EPI_RELU2), y.clamp(min=0) ** 2), (run(S.EPI_TANH), torch.tanh(y)),
                              (run(S.EPI_DECAY_SOFT, bias=bias, rate=rate), torch.exp(-rate.double() * oracle.softplus(z))),
                              (run(S.EPI_DECAY_EXP, bias=bias), torch.exp(-torch.exp(z)))):
                assert torch.isfinite(got).all() and float((got - want).abs().max()) < 2e-5 * max(1.0, float(want.abs().max()))
        eng.fabric.check()
    finally:
        eng.close()


# --------------------------------------------------------------------------- generation
def greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(oracle.forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]


def test_greedy_generation_through_engine_and_sessions():
    from naivert_b200.models.spec import SamplingParams
    from naivert_b200.runtime.session_engine import SessionEngine
    cfg = CASES["mixed"]
    w = weights(cfg, 8)
    sp = SamplingParams(temperature=1.0, top_p=1e-6, seed=3)
    eng = engine(cfg, w, capacity=256)
    try:
        prompt = tokens(cfg, 40, 77)
        want = greedy(cfg, w, prompt, 20)                                    # passes the edges of both kinds of mask chunk
        for graphs in (False, True):
            out = eng.generate(torch.tensor(prompt, dtype=torch.int32), 20, sp, use_graphs=graphs)
            assert out.tokens == want and out.stop_reason == "output_limit" and out.rounds == 20
        short = tokens(cfg, 1, 78)                                           # a prompt of one token has no context rows
        assert eng.generate(torch.tensor(short, dtype=torch.int32), 6, sp).tokens == greedy(cfg, w, short, 6)
        assert feed(eng, prompt, [40]).argmax(-1)[-1] == want[0]             # step by step, between requests
        eng.native_min_rows = 10 ** 9                                        # the round's own token-by-token prompt replay
        out = eng.generate(torch.tensor(prompt, dtype=torch.int32), 8, sp)
        assert out.tokens == want[:8] and eng.last_prefill["path"] == "replay"
        eng.native_min_rows = 1

        se = SessionEngine(eng, store_gb=0.5, max_output_tokens=64)

        def turn(toks, n, key):
            s = se.open_session(toks, n, key, sp)
            while not s.done:
                s.step()
            stats = s.finish()
            return s, stats

        a, stats = turn(prompt, 12, "a")
        assert a.out == want[:12] and a.cached_tokens == 0 and stats["prefill_path"] == "native"
        turn(tokens(cfg, 33, 99), 9, "b")                                    # another sequence over the same memory
        follow = prompt + want[:12] + tokens(cfg, 7, 100)
        c, _ = turn(follow, 10, "a")
        assert c.cached_tokens > 40 and c.out == greedy(cfg, w, follow, 10)  # resumed from the parked caches and states
        branch = prompt + tokens(cfg, 5, 101)
        d, _ = turn(branch, 8, "a")
        assert d.cached_tokens == 39 and d.out == greedy(cfg, w, branch, 8)  # rewound to the state kept at the prompt's end
        eng.fabric.check()
    finally:
        eng.close()


def test_checkpoint_and_trace_program(tmp_path):
    """A written checkpoint, replayed by the command line program in both numeric forms."""
    from naivert_b200.models import zuzupel
    from naivert_b200.models.checkpoint import write_stack_checkpoint
    cfg = CASES["mixed"]
    w = weights(cfg, 12)
    spec = zuzupel.spec_from_config(config_json(cfg), "case", shapes_of(w))
    write_stack_checkpoint(str(tmp_path / "m"), spec, state_dict=w)
    reqs = {"p": tokens(cfg, 60, 1), "q": tokens(cfg, 25, 2)}
    steps = [("p", 40, [39, 0]), ("p", 2, [1]), ("p", 17, []), ("p", 1, [0]), ("q", 25, [24, 3])]
    lines, at, want = [], {"p": 0, "q": 0}, {}
    for i, (rid, n, ask) in enumerate(steps):
        lo = at[rid]
        at[rid] += n
        want[i] = [(rid, lo + a) for a in ask]
        lines.append(json.dumps({"step": i, "entries": [{"id": rid, "tokens": reqs[rid][lo:lo + n], "want": ask}],
                                 "end": [rid] if at[rid] == len(reqs[rid]) else []}))
    ref = {k: oracle.forward(cfg, w, v) for k, v in reqs.items()}
    for dtype, short in (("float32", "fp32"), ("bfloat16", "bf16")):
        out = tmp_path / dtype
        r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(out),
                            "--max-tokens", "60"], input="\n".join(lines) + "\n", capture_output=True, text=True, timeout=300)
        assert r.returncode == 0, r.stderr[-2000:]
        assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(len(steps))]
        for i, rows in want.items():
            path = out / f"{i}.f32"
            assert path.exists() == bool(rows)
            if rows:
                got = torch.frombuffer(bytearray(path.read_bytes()), dtype=torch.float32).view(len(rows), cfg["vocab"])
                check(got, torch.stack([ref[rid][p] for rid, p in rows]), short, i)
