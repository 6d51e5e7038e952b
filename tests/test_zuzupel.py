"""The Zuzupel design without a GPU: configuration, sizes read from tensors, tensor lists, layers that borrow weights, refusals,
checkpoint files, weight layout, and the plain implementation's own invariants."""
import json
import math

import pytest
import torch

import zuzupel_oracle as oracle
from naivert_b200.models import zuzupel
from naivert_b200.models.blocks import RotarySpec
from naivert_b200.models.registry import MODELS, design_of, resolve_checkpoint_model, resolve_model, spec_from_config


def small():
    spec = zuzupel.small_spec()
    return spec, zuzupel.config_from_spec(spec), zuzupel.tensor_shapes(spec)


def test_configuration_round_trip_and_registry():
    spec, cfg, shapes = small()
    again = spec_from_config(json.loads(json.dumps(cfg)), spec.name, shapes)
    assert again == spec and resolve_model("zuzupel-small") == spec and design_of(spec) is zuzupel
    assert {"zuzupel-small", "zuzupel-bench"} <= set(MODELS)
    assert again.norm == "layer" and not again.pre_norm and not again.tied_head
    with_stop = spec_from_config(dict(cfg, eos_token_id=7), spec.name, shapes)
    assert with_stop.stop_token_ids == (7,) and zuzupel.config_from_spec(with_stop)["eos_token_id"] == [7]


def test_low_rank_widths_come_from_the_tensors():
    spec, cfg, shapes = small()
    with pytest.raises(ValueError, match="l0.mix.a1"):
        spec_from_config(cfg)
    shapes = dict(shapes)
    shapes["l0.mix.a1"], shapes["l0.mix.g1"], shapes["l1.mix.w1"] = (9, spec.hidden), (11, spec.hidden), (13, spec.hidden)
    got = spec_from_config(cfg, "x", shapes)
    assert (got.layers[0].mixer.decay_rank, got.layers[0].mixer.gate_rank, got.layers[1].mixer.decay_rank) == (9, 11, 13)
    assert got.layers[3].mixer == got.layers[0].mixer                       # the borrower's widths are the owner's


def test_rotation_scaling_defaults():
    spec, cfg, shapes = small()
    rot = cfg["layers"][2]["mixer"]["left"]["rot"]
    del rot["scaling"]
    assert spec_from_config(cfg, "x", shapes).layers[2].mixer.left.rotary.factor == 1.0
    f = RotarySpec(8, 10000.0, 4.0).frequencies()
    assert [round(x, 9) for x in f] == [0.25, 0.025, 0.0025, 0.00025]


def test_layers_that_borrow_weights():
    spec, cfg, shapes = small()
    assert [spec.owner(i) for i in range(5)] == [0, 1, 2, 0, 4] and [oracle.owner(cfg, i) for i in range(5)] == [0, 1, 2, 0, 4]
    assert [r.layer for r in spec.runs()] == list(range(5))                 # every layer is a run with a state of its own
    assert not any(n.startswith("l3.") for n in shapes)
    chain = dict(cfg, layers=cfg["layers"] + [dict(cfg["layers"][0], weights_of=3)])
    assert spec_from_config(chain, "x", shapes).layers[5].weights_of == 0
    ahead = dict(cfg, layers=[dict(cfg["layers"][0], weights_of=1)] + [cfg["layers"][0]])
    moved = {("l1." + n[3:] if n.startswith("l0.") else n): s for n, s in shapes.items()}
    cut = spec_from_config(ahead, "x", moved).with_layers(1)
    assert cut.layers[0].weights_of is None and "l0.mix.q" in zuzupel.tensor_shapes(cut)
    w = zuzupel.gather_weights(spec, lambda n: torch.zeros(shapes[n]))
    assert w["layers"][3] is None and w["layers"][4]["mlp"] is None and "norm2b" not in w["layers"][4]


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0].update(type="other"), "unknown layer type"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "unknown feed-forward"),
    (lambda c: [c["layers"][i]["mixer"].update(kv_heads=3) for i in (0, 3)], "4 heads over 3 key heads"),
    (lambda c: c["layers"][2]["mixer"]["left"].update(kv_heads=3), "4 heads over 3 key heads"),
    (lambda c: c["layers"][1]["mixer"].update(dim=600), "head width"),
    (lambda c: c["layers"][2]["mixer"]["left"].update(dim=600), "head width"),
    (lambda c: c["layers"][2]["mixer"]["left"]["rot"].update(dims=33), "rotated columns"),
    (lambda c: c["layers"][2]["mixer"]["right"].update(gate_cap=0.0), "gate cap"),
    (lambda c: c["layers"][3].update(weights_of=9), "no layer 9"),
    (lambda c: c["layers"][3].update(weights_of=3), "in a circle"),
    (lambda c: c["layers"][3]["mixer"].update(vdim=8), "differs from layer 0"),
])
def test_what_the_kernels_cannot_run_is_refused_by_name(change, message):
    _, cfg, shapes = small()
    cfg = json.loads(json.dumps(cfg))
    change(cfg)
    with pytest.raises(ValueError, match=message):
        spec_from_config(cfg, "x", shapes)


def test_checkpoint_files(tmp_path):
    from naivert_b200.models.checkpoint import CheckpointError, load_stack_weights, write_stack_checkpoint
    spec, cfg, shapes = small()
    sd = zuzupel.init_state_dict(spec, seed=3)
    assert {n: tuple(t.shape) for n, t in sd.items()} == shapes and all(t.dtype == torch.bfloat16 for t in sd.values())
    write_stack_checkpoint(str(tmp_path), spec, state_dict=sd)
    found = resolve_checkpoint_model(str(tmp_path))                         # sizes from config.json and the tensors' shapes
    assert found.layers == spec.layers
    w = load_stack_weights(found, str(tmp_path))
    assert torch.equal(w["head"], sd["head"]) and torch.equal(w["layers"][2]["mix"]["right.i.b"], sd["l2.mix.right.i.b"]) and w["layers"][3] is None
    cfg["layers"][0]["mixer"]["conv"] = cfg["layers"][3]["mixer"]["conv"] = 5
    with pytest.raises(CheckpointError, match="the configuration needs"):
        load_stack_weights(spec_from_config(cfg, "x", shapes), str(tmp_path))


def test_cache_bytes_and_single_gpu():
    from naivert_b200.runtime.engine import Engine, RuntimeContractError
    spec, _, _ = small()
    assert spec.kv_bytes_per_token() == 2 * (56 + 48) * 2                   # keys and values of the one attention layer
    with pytest.raises(RuntimeContractError, match="one GPU"):
        Engine.build(spec, tp=2)


def test_weight_layout():
    from naivert_b200.runtime.packing import head_columns, pack, stacked_rows
    w = torch.randn(4, 3 * 5)
    p = head_columns(w, 3, 5, 8).view(4, 3, 8)
    assert torch.equal(p[:, :, :5], w.view(4, 3, 5)) and not p[:, :, 5:].any()
    a, b, c = torch.randn(2, 6), torch.randn(3, 6), torch.randn(1, 6)
    s = stacked_rows([a, b, c], 3)
    assert s.shape == (7, 6) and torch.equal(s[:2], a) and not s[2].any() and torch.equal(s[3:6], b) and torch.equal(s[6:], c)
    packed = pack(s, "cpu")
    assert torch.equal(packed.rows(0, 3, 2).w[1, :, :6], b.to(torch.bfloat16)) and packed.rows(6, 1).n == 1 and packed.rows(0, 3, 2).k == 6


def test_blocks_of_tokens_equal_the_rules_token_by_token():
    """The algebra of the chunk kernels: what a block of tokens needs from the state at its start are products with decayed keys
    and queries; the tokens' influence on one another is a number per pair (``csrc/stack.cuh``)."""
    g = torch.Generator().manual_seed(0)
    B, D, V = 8, 5, 3
    q, k, v = (torch.randn(B, n, generator=g, dtype=torch.float64) for n in (D, D, V))
    d, u = torch.rand(B, D, generator=g, dtype=torch.float64), torch.randn(D, generator=g, dtype=torch.float64)
    beta = torch.rand(B, generator=g, dtype=torch.float64)
    S0 = torch.randn(D, V, generator=g, dtype=torch.float64)

    def through(lo, hi):                                                    # decays of tokens lo .. hi - 1
        return d[lo:hi].prod(0)

    def sequential(kind):
        S, out = S0.clone(), []
        for t in range(B):
            if kind == "delta":
                S = d[t][:, None] * S
                S = S + torch.outer(k[t], beta[t] * (v[t] - k[t] @ S))
                out.append(q[t] @ S)
            else:
                kv = torch.outer(k[t], v[t])
                out.append(q[t] @ (S + u[:, None] * kv))
                S = d[t][:, None] * S + kv
        return torch.stack(out), S

    for kind in ("delta", "bonus"):
        shift = 0 if kind == "bonus" else 1                                 # the bonus form reads out ahead of the token's decay
        upd = torch.zeros(B, V, dtype=torch.float64)
        out = []
        for t in range(B):
            upd[t] = v[t]
            if kind == "delta":
                seen = (through(0, t + 1) * k[t]) @ S0 + sum((k[t] * through(s + 1, t + 1)) @ k[s] * upd[s] for s in range(t))
                upd[t] = beta[t] * (v[t] - seen)
            o = (through(0, t + shift) * q[t]) @ S0 + sum((q[t] * through(s + 1, t + shift)) @ k[s] * upd[s] for s in range(t))
            out.append(o + (q[t] * (u if kind == "bonus" else 1)) @ k[t] * upd[t])
        S = through(0, B)[:, None] * S0 + sum(torch.outer(through(s + 1, B) * k[s], upd[s]) for s in range(B))
        want, end = sequential(kind)
        assert torch.allclose(torch.stack(out), want) and torch.allclose(S, end)


# --------------------------------------------------------------------------- the plain implementation
def t64(*v):
    return torch.tensor(v, dtype=torch.float64)


def test_plain_recurrences_by_hand():
    one = t64([1.0], [1.0])
    got = oracle.delta_rule(t64([2.0], [2.0]), one, t64([3.0], [5.0]), t64(0.5, 1.0), t64([0.5], [0.5]))
    assert got.flatten().tolist() == [3.0, 10.0]                            # S = 1.5; then 0.75 corrected fully to 5
    got = oracle.wkv_rule(one, one, t64([3.0], [5.0]), t64([0.5], [0.5]), t64(10.0))
    assert got.flatten().tolist() == [30.0, 53.0]                           # the bonus alone; then the undecayed first term
    got = oracle.mlstm_rule(one, one, t64([3.0], [5.0]), t64(math.log(2.0), 0.0), t64(-1e9, 0.0))
    m = math.log(2.0)
    want = [3.0 / (1 + 1e-6), (3.0 + 0.5 * 5) / (1.5 + 1e-6)]               # m = log 2 in both steps
    assert torch.allclose(got.flatten(), t64(*want)) and m > 0
    low = oracle.mlstm_rule(one[:1], one[:1], t64([3.0]), t64(-5.0), t64(0.0))
    assert torch.allclose(low.flatten(), t64(3 * math.exp(-5.0) / (1 + 1e-6)))              # the maximum starts at 0: floor exp(0)


def test_plain_convolution_rotation_and_visibility():
    x = t64([1.0], [2.0], [3.0])
    assert oracle.causal_conv(x, t64([10.0, 1.0])).flatten().tolist() == [1.0, 12.0, 23.0]
    assert oracle.causal_conv(x, t64([7.0, 10.0, 1.0])).flatten().tolist() == [1.0, 12.0, 30.0]
    r = oracle.rotate(torch.ones(3, 1, 5, dtype=torch.float64), {"dims": 4, "base": 100.0, "scaling": {"factor": 2.0}})
    a, b = 2 * 0.5, 2 * 0.05
    want = [math.cos(a) - math.sin(a), math.cos(b) - math.sin(b), math.cos(a) + math.sin(a), math.cos(b) + math.sin(b), 1.0]
    assert torch.allclose(r[2, 0], t64(*want)) and torch.allclose(r[0, 0], torch.ones(5, dtype=torch.float64))
    assert [list(oracle.visible(i, 3)) for i in (0, 2, 3, 7)] == [[0], [0, 1, 2], [3], [6, 7]]


def test_plain_norms():
    x = t64([1.0, 2.0, 6.0])
    d = t64([-2.0, -1.0, 3.0])
    assert torch.allclose(oracle.layer_norm(x, t64(1.0, 2.0, 1.0), 0.5), d / math.sqrt(14 / 3 + 0.5) * t64(1.0, 2.0, 1.0))
    assert torch.allclose(oracle.unit(t64([3.0, 4.0])), t64([0.6, 0.8]), atol=1e-6)


def test_plain_model_is_causal():
    spec, cfg, _ = small()
    sd = zuzupel.init_state_dict(spec, seed=1)
    toks = torch.randint(0, spec.vocab, (9,), generator=torch.Generator().manual_seed(2)).tolist()
    full = oracle.forward(cfg, sd, toks)
    assert torch.allclose(full[:6], oracle.forward(cfg, sd, toks[:6]))
    assert torch.isfinite(full).all() and full.std() > 1e-3
