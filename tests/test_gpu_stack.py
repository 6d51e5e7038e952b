"""Layer-stack models on the GPU against the plain implementation (``tumatar_oracle``): every mechanism alone, prompts
against token-by-token decoding, portions, borders of tiles, key blocks and chunks, reused state, long decoding, greedy
generation through the engine and the session engine.

Configurations and weights are made here.  The float form is compared tightly, row by row; the bf16 form within the
rounding of its matrix operands, where a few rows of a model with experts may differ more: two experts whose choice scores
agree to within a rounding can swap (in the mixed model, whose later layers would spread a swap over the sequence, the
router is weak against the spread of its biases).
"""
import json
import math
import os
import subprocess
import sys

import pytest
import torch

import tumatar_oracle as oracle
from stack_testing import TOL, error, feed, tokens

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


# --------------------------------------------------------------------------- cases
def attn(heads=3, dim=24, vdim=40, kv_rank=56, q_rank=36, scale=None):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
                                                  "scale": scale if scale is not None else dim ** -0.5}}


def rec(width=120, blocks=3, conv=4):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}}


def dense(ff=104, limit=0.75):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(experts=12, top=3, ff=40, count=4, keep=2):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}}}


def model(layers, width=88, vocab=203, loop=None, eps=1e-5, embed=7.0, logit=0.6, router=1.0):
    cfg = {"architecture": "Tumatar", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": embed},
           "logit_scale": logit, "router": router, "layers": [dict(m, mlp=f) for m, f in layers]}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


def weights(cfg, seed=0):
    g = torch.Generator().manual_seed(seed)

    def r(*shape, s=None):
        s = shape[-1] ** -0.5 if s is None else s
        return (torch.randn(*shape, generator=g) * s).to(torch.bfloat16)

    def norm(n):
        return (1 + 0.2 * torch.randn(n, generator=g)).to(torch.bfloat16)

    W = cfg["width"]
    out = {"embed": r(cfg["vocab"], W, s=0.15), "final.norm": norm(W)}
    if cfg.get("loop"):
        out["loop.step"] = r(cfg["loop"]["times"], W, s=0.5)
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer.get("mlp")
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if f else ()):
            out[p + n] = norm(W)
        if layer["type"] == "latent_attention":
            H, D, V = m["heads"], m["dim"], m["vdim"]
            out.update({p + "mix.dq": r(m["q_rank"], W), p + "mix.dq.norm": norm(m["q_rank"]), p + "mix.uq": r(H * D, m["q_rank"], s=1.0),
                        p + "mix.dkv": r(m["kv_rank"], W), p + "mix.dkv.norm": norm(m["kv_rank"]), p + "mix.uk": r(H * D, m["kv_rank"]),
                        p + "mix.uv": r(H * V, m["kv_rank"]), p + "mix.g": r(H * V, W), p + "mix.o": r(W, H * V)})
        else:
            w, b, t = m["width"], m["blocks"], m["conv"]
            n = w // b
            out.update({p + "mix.y": r(w, W), p + "mix.y.b": r(w, s=0.3), p + "mix.x": r(w, W), p + "mix.x.b": r(w, s=0.3),
                        p + "mix.conv": r(w, t), p + "mix.conv.b": r(w, s=0.3), p + "mix.ra": r(b, n, n), p + "mix.ra.b": r(b, n, s=0.5),
                        p + "mix.ri": r(b, n, n), p + "mix.ri.b": r(b, n, s=0.5), p + "mix.lam": r(w, s=1.5), p + "mix.o": r(W, w)})
        if f and f["kind"] == "dense":
            out.update({p + "mlp.gate": r(f["ff"], W), p + "mlp.up": r(f["ff"], W), p + "mlp.down": r(W, f["ff"])})
        elif f:
            E, F = f["router"]["experts"], f["expert"]["ff"]
            out.update({p + "mlp.router": r(E, W, s=cfg["router"] * W ** -0.5), p + "mlp.correction": r(E, s=0.6)})
            for e in range(E):
                out.update({f"{p}mlp.e{e}.gate": r(F, W), f"{p}mlp.e{e}.up": r(F, W), f"{p}mlp.e{e}.down": r(W, F)})
    return out


CASES = {
    "attention": model([(attn(), None)]),
    "attention_wide": model([(attn(heads=5, dim=136, vdim=72, kv_rank=200, q_rank=100), None)]),
    "attention_odd": model([(attn(heads=1, dim=13, vdim=21, kv_rank=37, q_rank=19), None)], width=51, vocab=97),
    "attention_large": model([(attn(heads=2, dim=264, vdim=24, kv_rank=520, q_rank=40), None)]),     # beyond the tensor-core forms
    "attention_many_heads": model([(attn(heads=36, dim=16, vdim=16, kv_rank=64, q_rank=48), None)]),
    "recurrence": model([(rec(), None)]),
    "recurrence_odd": model([(rec(width=115, blocks=5, conv=2), None)], width=45, vocab=101),
    "recurrence_one_block": model([(rec(width=64, blocks=1, conv=1), None)]),
    "recurrence_long_kernel": model([(rec(width=96, blocks=4, conv=7), None)]),
    "dense": model([(rec(), dense())]),
    "experts": model([(rec(), moe())]),
    "experts_one_group": model([(rec(), moe(experts=7, top=2, count=1, keep=1))]),
    "experts_pairs": model([(attn(), moe(experts=16, top=4, ff=24, count=8, keep=3))]),
    "experts_single": model([(attn(), moe(experts=6, top=1, ff=24, count=6, keep=1))]),
    "loop": model([(rec(), dense()), (attn(), None), (rec(), None)], loop=(1, 3, 3)),
    "loop_once": model([(attn(), dense())], loop=(0, 1, 1)),
    "mixed": model([(attn(), dense(limit=1.5)), (rec(width=104, blocks=2, conv=3), moe()), (attn(heads=2), moe(experts=10, count=2, keep=1)),
                    (rec(conv=5), None)], loop=(0, 3, 2), width=136, router=0.05),
}


def engine(cfg, w, dtype="fp32", capacity=512, chunk=96, kv_block=16384):
    from naivert_b200.models import tumatar
    from naivert_b200.runtime.stack_engine import build_stack_engine
    spec = tumatar.spec_from_config(cfg, "case")
    return build_stack_engine(spec, capacity=capacity, device=torch.device("cuda", 0),
                              weights=tumatar.gather_weights(spec, lambda n: w[n].cuda()), prefill_chunk=chunk, dtype=dtype, kv_block=kv_block)


def check(got, want, cfg, dtype, what, tol=None):
    e = error(got, want)
    over = int((e > (tol or TOL[dtype])).sum())
    allowed = 0
    if dtype == "bf16" and any((x.get("mlp") or {}).get("kind") == "moe" for x in cfg["layers"]):
        allowed = max(1, len(e) // 25)
    assert torch.isfinite(e).all() and over <= allowed, (what, dtype, over, int(e.argmax()), float(e.max()))


# --------------------------------------------------------------------------- mechanisms, prompts, decoding, portions
@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("name", sorted(CASES))
def test_mechanism_prompt_decode_and_portions(name, dtype):
    cfg = CASES[name]
    w = weights(cfg, seed=len(name))
    toks = tokens(cfg, 150)
    ref = oracle.forward(cfg, w, toks)
    eng = engine(cfg, w, dtype)
    try:
        for sizes in ([150], [1], [70, 2, 3, 2, 64, 1], [2], [96, 1]):
            check(feed(eng, toks, sizes), ref, cfg, dtype, (name, sizes))
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
        assert len(got) == len(trace) == 7
        for a, b in zip(got, trace):
            assert float((a.double().cpu() - b).norm() / b.norm()) < 1e-5
    finally:
        eng.close()


# --------------------------------------------------------------------------- keys far away and at borders
def needle_model(width=64):
    """One attention layer in which token 58 looks up token 59: that one key carries nearly the whole weight wherever it
    stands."""
    cfg = model([(attn(heads=2, dim=width, vdim=32, kv_rank=width, q_rank=width, scale=9.0 / width), None)], width=width, vocab=60, embed=1.0)
    w = weights(cfg, 11)
    g = torch.Generator().manual_seed(1)
    basis = torch.linalg.qr(torch.randn(width, width, generator=g))[0] * math.sqrt(width)
    w["embed"] = basis[:60].to(torch.bfloat16)
    w["l0.norm1"] = w["l0.mix.dq.norm"] = w["l0.mix.dkv.norm"] = torch.ones(width, dtype=torch.bfloat16)
    eye = torch.eye(width, dtype=torch.bfloat16)
    w["l0.mix.dq"] = w["l0.mix.dkv"] = eye
    w["l0.mix.uk"] = torch.cat([eye, eye])
    ask = torch.outer(basis[59], basis[58]) / width           # token 58 asks for token 59, the others for nothing in particular
    w["l0.mix.uq"] = torch.cat([ask, ask]).to(torch.bfloat16)
    return cfg, w


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
def test_one_key_stands_out_wherever_it_is(dtype):
    cfg, w = needle_model()
    n = 330
    base = [2 + (i * 7) % 50 for i in range(n)]
    eng = engine(cfg, w, dtype, capacity=n + 8, chunk=128, kv_block=128)
    try:
        for where in (0, 1, 62, 63, 64, 65, 126, 127, 128, 129, 191, 192, 255, 256, 257, 319, 327, 328):
            toks = list(base)
            toks[where], toks[-1] = 59, 58
            ref = oracle.forward(cfg, w, toks)[-1:]
            gone = list(toks)
            gone[where] = 3
            assert error(oracle.forward(cfg, w, gone)[-1:], ref) > 0.1                  # leaving the key out would show
            for sizes in ([n], [n - 1, 1], [200, 2]):
                e = error(feed(eng, toks, sizes)[-1:], ref)
                assert e < TOL[dtype], (where, sizes, float(e))
    finally:
        eng.close()


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("kv_block", [64, 128, 192])
def test_context_in_blocks_of_keys(dtype, kv_block):
    """Attention carried over several blocks of expanded keys equals one pass (maxima that grow late included)."""
    cfg = model([(attn(heads=3, dim=24, vdim=40, scale=0.4), None)])
    w = weights(cfg, 21)
    toks = tokens(cfg, 400, 9)
    ref = oracle.forward(cfg, w, toks)
    eng = engine(cfg, w, dtype, capacity=416, chunk=160, kv_block=kv_block)
    try:
        for sizes in ([400], [130, 3, 61, 160]):
            check(feed(eng, toks, sizes), ref, cfg, dtype, sizes)
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
        for k, n in enumerate((320, 5, 130, 1, 2, 320)):
            toks = tokens(cfg, n, 40 + n)
            got = feed(eng, toks, [9, 1] if n > 9 else [1])
            check(got, oracle.forward(cfg, w, toks), cfg, dtype, n)
            if n in first:
                assert torch.equal(got, first[n])           # nothing of what ran in between is left
            first[n] = got
    finally:
        eng.close()


def test_repeated_step_and_broken_hand_over():
    """A step may be repeated at its position; a step from a position no state was left for is reported, not computed."""
    cfg = CASES["recurrence"]
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


def test_slow_decay_keeps_the_first_token():
    """With decays near one the recurrence must still carry the first token after hundreds of steps and pieces."""
    cfg = model([(rec(width=64, blocks=2, conv=2), None)], vocab=50)
    w = weights(cfg, 6)
    w["l0.mix.lam"] = torch.full((64,), -9.0, dtype=torch.bfloat16)
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


# --------------------------------------------------------------------------- products
@pytest.mark.parametrize("rows", [1, 63, 200, 700])
def test_products_against_torch(rows):
    """Every epilogue and tile width of the chunk product, sizes off every multiple."""
    from naivert_b200.ops import stack_kernels as S
    from naivert_b200.runtime.packing import pack, pad
    cfg = CASES["mixed"]
    eng = engine(cfg, weights(cfg), "bf16", capacity=1024, chunk=1024)
    pf = eng.prefill
    g = torch.Generator(device="cuda").manual_seed(rows)
    try:
        for n, k, z in ((37, 20, 1), (300, 136, 1), (129, 520, 1), (40, 24, 5)):
            kp = pad(k, 8)
            x = torch.zeros(rows, z, kp, dtype=torch.bfloat16, device="cuda")
            x[:, :, :k] = torch.randn(rows, z, k, generator=g, device="cuda")
            w, w2 = (torch.randn(z, n, k, generator=g, device="cuda").to(torch.bfloat16) for _ in range(2))
            bias = torch.randn(z, n, generator=g, device="cuda").to(torch.bfloat16)
            a = torch.einsum("rzk,znk->rzn", x[:, :, :k].double(), w.double())
            b = torch.einsum("rzk,znk->rzn", x[:, :, :k].double(), w2.double())
            p, p2 = pack(w, "cuda"), pack(w2, "cuda")
            kw = dict(z=z, x_z=kp, out_z=n, x_rows=rows)

            def run(epi, dtype=torch.float32, **more):
                out = torch.full((rows, z, n), float("nan"), dtype=dtype, device="cuda")
                pf.gemm(epi, p, x, z * kp, rows, out, z * n, **kw, **more)
                torch.cuda.synchronize()
                return out.double()

            def close(got, want, tol=2e-3):
                assert torch.isfinite(got).all() and float((got - want).abs().max() / want.abs().max()) < tol

            close(run(S.EPI_STORE, scale=0.5), 0.5 * a, 1e-5)
            close(run(S.EPI_STORE, torch.bfloat16), a, 1e-2)
            y = a + bias.double()
            y[:, :, : n // 2] = oracle.gelu_tanh(y[:, :, : n // 2])
            close(run(S.EPI_BIAS, bias=bias, act_cols=n // 2), y, 1e-5)
            gl, u = a.clamp(max=1.2), b.clamp(-1.2, 1.2)
            close(run(S.EPI_CLAMPED_GLU, w2=p2, limit=1.2, alpha=1.702), gl * torch.sigmoid(1.702 * gl) * (u + 1), 1e-4)
            close(run(S.EPI_SILU_GLU, w2=p2), a * torch.sigmoid(a) * b, 1e-4)
            if z == 1:
                ld = pad(rows, 64)
                out = torch.zeros(n, ld, dtype=torch.bfloat16, device="cuda")
                pf.gemm(S.EPI_TRANSPOSE, p, x, kp, rows, out, ld, x_rows=rows)
                close(out[:, :rows].t().double(), a[:, 0], 1e-2)
        eng.fabric.check()
    finally:
        eng.close()


@pytest.mark.parametrize("experts,top,count,keep", [(24, 3, 4, 2), (256, 8, 8, 4), (30, 5, 10, 4), (9, 2, 1, 1), (32, 1, 32, 1)])
def test_group_limited_choice(experts, top, count, keep):
    """Choices and weights of the routing kernel, with negative choice scores and exact ties."""
    from naivert_b200.ops import kernels as K
    from naivert_b200.ops import stack_kernels as S
    g = torch.Generator().manual_seed(experts)
    rows = 70
    logits = torch.randn(rows, experts, generator=g) * 1.5
    corr = torch.randn(experts, generator=g) * 0.8 - 0.6
    logits[3], corr_t = 0.25, corr.clone()                                  # a row of equal scores: the correction decides
    cfg = {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}}
    ids_ref, ws_ref = oracle.route(logits.double(), {"router": torch.eye(experts).double(), "correction": corr.double()}, "", cfg)
    dl, dc = logits.cuda(), corr_t.cuda()
    ids = torch.zeros(rows, top, dtype=torch.int32, device="cuda")
    ps = torch.zeros(rows, top, device="cuda")
    q = K.RouterArgs()
    q.bias, q.hidden, q.experts, q.rows, q.top_k = dc.data_ptr(), 64, experts, rows, top
    q.sigmoid, q.normalize, q.route_scale = 1, 0, 1.0
    q.scores, q.topk_ids, q.topk_p = dl.data_ptr(), ids.data_ptr(), ps.data_ptr()
    S.route(q, count, keep)
    torch.cuda.synchronize()
    for t in range(rows):
        assert sorted(ids[t].tolist()) == sorted(ids_ref[t]), t
        want = dict(zip(ids_ref[t], (float(x) for x in ws_ref[t])))
        for e, p in zip(ids[t].tolist(), ps[t].tolist()):
            assert abs(p - want[e]) < 2e-6


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
        want = greedy(cfg, w, prompt, 20)
        for graphs in (False, True):
            out = eng.generate(torch.tensor(prompt, dtype=torch.int32), 20, sp, use_graphs=graphs)
            assert out.tokens == want and out.stop_reason == "output_limit" and out.rounds == 20
        short = tokens(cfg, 1, 78)                                           # a prompt of one token has no context rows
        assert eng.generate(torch.tensor(short, dtype=torch.int32), 6, sp).tokens == greedy(cfg, w, short, 6)
        assert feed(eng, prompt, [40]).argmax(-1)[-1] == want[0]             # step by step, between requests

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


def test_replayed_prompt_equals_chunks():
    """The round's own token-by-token prompt replay leaves the same context as the chunk path."""
    from naivert_b200.models.spec import SamplingParams
    cfg = CASES["mixed"]
    w = weights(cfg, 8)
    sp = SamplingParams(temperature=1.0, top_p=1e-6, seed=3)
    eng = engine(cfg, w, capacity=256)
    try:
        prompt = torch.tensor(tokens(cfg, 30, 5), dtype=torch.int32)
        want = eng.generate(prompt, 10, sp).tokens
        eng.native_min_rows = 10 ** 9
        assert eng.generate(prompt, 10, sp).tokens == want and eng.last_prefill["path"] == "replay"
    finally:
        eng.close()


def test_stepwise_use_loads_only_the_stack_library():
    """A process that feeds tokens step by step never builds or loads the speculative target's library."""
    code = ("import torch; from naivert_b200.models import tumatar; from naivert_b200.ops import build; from naivert_b200.runtime.engine import Engine\n"
            "e = Engine.build(tumatar.small_spec(), capacity=64, device=torch.device('cuda', 0))\n"
            "e.extend([1, 2, 3], [2]); e.extend([4], [0]); e.close(); print(sorted(build._LIBS))")
    r = subprocess.run([sys.executable, "-c", code], cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0 and r.stdout.split("\n")[-2] == "['stack']", r.stdout + r.stderr[-2000:]


def test_checkpoint_and_trace_program(tmp_path):
    """A written checkpoint, replayed by the command line program in both numeric forms."""
    from naivert_b200.models import tumatar
    from naivert_b200.models.checkpoint import write_stack_checkpoint
    cfg = CASES["mixed"]
    w = weights(cfg, 12)
    spec = tumatar.spec_from_config(cfg)
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
    for dtype, tol in (("float32", TOL["fp32"]), ("bfloat16", TOL["bf16"])):
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
                exp = torch.stack([ref[rid][p] for rid, p in rows])
                check(got, exp, cfg, "fp32" if dtype == "float32" else "bf16", i, tol)
