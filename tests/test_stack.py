"""Layer-stack models without a GPU: configuration, tensor lists, order of runs, refusals, the plain implementation's own
invariants, the trace replay logic."""
import io
import json
import math
import os
import struct

import pytest
import torch

import tumatar_oracle as oracle
from naivert_b200.models import tumatar
from naivert_b200.models.blocks import LoopSpec, StackSpec
from naivert_b200.models.registry import MODELS, design_of, resolve_checkpoint_model, resolve_model, spec_from_config


def small():
    spec = tumatar.small_spec()
    return spec, tumatar.config_from_spec(spec)


def test_configuration_round_trip_and_registry():
    spec, cfg = small()
    again = spec_from_config(json.loads(json.dumps(cfg)), spec.name)
    assert again == spec and resolve_model("tumatar-small") == spec and design_of(spec) is tumatar
    assert {"tumatar-small", "tumatar-bench", "tumatar-bench-dense"} <= set(MODELS)
    with pytest.raises(KeyError, match="no registered model"):
        spec_from_config({"architecture": "Nobody"})
    for name in ("naive-n0.5", "small-w8a8"):
        assert not isinstance(resolve_model(name), StackSpec)


def test_speculative_target_is_found_by_its_config():
    from naivert_b200.models.checkpoint import target_config
    spec = resolve_model("naive-n0.5")
    assert spec_from_config(target_config(spec)) is spec


def test_order_of_layer_runs():
    spec, cfg = small()
    got = [(r.layer, r.pass_start) for r in spec.runs()]
    assert got == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)] == oracle.layer_order(cfg)
    assert [r.run for r in spec.runs()] == list(range(6))
    assert [r.layer for r in spec.with_layers(2).runs()] == [0, 1]            # a loop that would be cut is dropped
    no_loop = dict(cfg, loop=None)
    assert [r.layer for r in spec_from_config(no_loop).runs()] == [0, 1, 2, 3]


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0]["mixer"].update(blocks=7), "does not split into blocks"),
    (lambda c: c["layers"][0].update(type="other"), "unknown layer type"),
    (lambda c: c["layers"][0]["mlp"].update(kind="other"), "unknown feed-forward"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(experts=300), "router of 300 experts"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(groups={"count": 5, "keep": 1}), "expert groups"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=13, groups={"count": 4, "keep": 2}), "fewer eligible experts"),
    (lambda c: c["layers"][1]["mixer"].update(dim=600), "head width"),
    (lambda c: c.update(loop={"start": 2, "stop": 2, "times": 1}), "loop bounds"),
])
def test_what_the_kernels_cannot_run_is_refused_by_name(change, message):
    _, cfg = small()
    change(cfg)
    with pytest.raises(ValueError, match=message):
        spec_from_config(cfg)


def test_checkpoint_files(tmp_path):
    from naivert_b200.models.checkpoint import CheckpointError, load_stack_weights, write_stack_checkpoint
    spec, cfg = small()
    sd = tumatar.init_state_dict(spec, seed=3)
    write_stack_checkpoint(str(tmp_path), spec, state_dict=sd)
    found = resolve_checkpoint_model(str(tmp_path))
    assert found.layers == spec.layers and found.loop == spec.loop
    w = load_stack_weights(found, str(tmp_path))
    assert torch.equal(w["layers"][0]["mlp"]["gate"][5], sd["l0.mlp.e5.gate"]) and torch.equal(w["loop"], sd["loop.step"])
    assert torch.equal(w["layers"][3]["mix"]["dkv.norm"], sd["l3.mix.dkv.norm"]) and w["layers"][2]["mlp"] is None
    cfg["layers"][1]["mixer"]["kv_rank"] += 8
    with pytest.raises(CheckpointError, match="the configuration needs"):
        load_stack_weights(spec_from_config(cfg), str(tmp_path))
    cfg2 = tumatar.config_from_spec(spec)
    cfg2["layers"].append(cfg2["layers"][0])
    with pytest.raises(CheckpointError, match="lacks"):
        load_stack_weights(spec_from_config(cfg2), str(tmp_path))


def test_engine_refuses_what_the_family_has_not():
    from naivert_b200.runtime.engine import Engine, RuntimeContractError
    spec, _ = small()
    with pytest.raises(RuntimeContractError, match="one GPU"):
        Engine.build(spec, tp=2)
    with pytest.raises(RuntimeContractError, match="no draft"):
        Engine.build(spec, draft_ckpt="somewhere")
    with pytest.raises(RuntimeContractError, match="32-bit"):
        Engine.build(resolve_model("small-w8a8"), dtype="fp32")
    assert spec.kv_bytes_per_token() == 3 * 112 * 2                          # three attention runs


def test_head_padding_keeps_the_products():
    from naivert_b200.runtime.packing import head_rows, pack
    w = torch.randn(3 * 5, 7)
    p = head_rows(w, 3, 5, 8)
    assert p.shape == (24, 7) and torch.equal(p.view(3, 8, 7)[:, :5], w.view(3, 5, 7)) and not p.view(3, 8, 7)[:, 5:].any()
    k = pack(w, "cpu")
    assert (k.z, k.n, k.ld, k.k) == (1, 15, 8, 7) and not k.w[:, :, 7].any()


def test_segment_bound_covers_every_distribution():
    """Segments needed by any split of the choices over the experts stay inside the list the chunk path allocates."""
    from naivert_b200.prefill.stack import StackPrefill
    rt = tumatar.small_spec().layers[0].mlp.routing
    g = torch.Generator().manual_seed(0)
    for rows in (1, 2, 7, 64, 300):
        for ir in (64, 128):
            bound = StackPrefill._items(None, rows, rt, ir)
            worst = 0
            for trial in range(40):
                p = torch.rand(rt.expert_count, generator=g) ** (trial % 9)
                ids = torch.multinomial(p.expand(rows, -1), rt.top_k, generator=g).flatten()
                n = torch.bincount(ids, minlength=rt.expert_count)
                worst = max(worst, int((-(-n // ir)).sum()))
            assert worst <= bound


def test_server_chooses_the_model_by_the_checkpoint(tmp_path):
    import sys
    sys.path.insert(0, os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "examples"))
    import serve_sessions
    spec, cfg = small()
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    assert serve_sessions.choose_model(None, str(tmp_path)).layers == spec.layers
    assert serve_sessions.choose_model("tumatar-small", None) is resolve_model("tumatar-small")
    assert serve_sessions.choose_model(None, None).name == "naive-n0.5"
    assert serve_sessions.parse_args(["--dtype", "fp32"]).dtype == "fp32"
    with pytest.raises(SystemExit):
        serve_sessions.main(["--model", "tumatar-small", "--log-level", "error"])          # neither a checkpoint nor --random-init


# --------------------------------------------------------------------------- the plain implementation
def test_plain_convolution_and_recurrence_by_hand():
    x = torch.tensor([[1.0], [2.0], [3.0]], dtype=torch.float64)
    k, b = torch.tensor([[10.0, 1.0]], dtype=torch.float64), torch.tensor([0.5], dtype=torch.float64)
    assert oracle.causal_conv(x, k, b).flatten().tolist() == [1.5, 12.5, 23.5]
    w = {"y": torch.zeros(1, 1), "y.b": torch.tensor([1.0]), "x": torch.ones(1, 1), "x.b": torch.zeros(1), "conv": torch.ones(1, 1),
         "conv.b": torch.zeros(1), "ra": torch.zeros(1, 1, 1), "ra.b": torch.zeros(1, 1), "ri": torch.zeros(1, 1, 1), "ri.b": torch.zeros(1, 1),
         "lam": torch.zeros(1), "o": torch.ones(1, 1)}
    w = {n: t.double() for n, t in w.items()}
    out = oracle.rglru(torch.tensor([[1.0], [2.0]]).double(), w, "", {"width": 1, "blocks": 1})
    a = math.exp(-8 * 0.5 * math.log(2.0))
    y = float(oracle.gelu_tanh(torch.tensor(1.0, dtype=torch.float64)))
    drive = math.sqrt(1 - a * a) * 0.5
    assert torch.allclose(out.flatten(), torch.tensor([drive * y, (a * drive + 2 * drive) * y], dtype=torch.float64))


def test_plain_choice_by_hand():
    eye = torch.eye(6).double()
    w = {"router": eye, "correction": torch.tensor([0.0, 0.0, -3.0, -3.0, 0.4, -2.0]).double()}
    z = torch.tensor([[0.0, 0.1, 5.0, 4.0, 0.0, 0.2]]).double()
    r = {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 1}}
    ids, ws = oracle.route(z, w, "", r)
    assert ids == [[1, 0]]                                                   # pair scores: 1.02, about -4, about -0.5
    assert [round(float(v), 6) for v in ws[0]] == [round(1 / (1 + math.exp(-0.1)), 6), 0.5]      # weights without the correction
    ids, _ = oracle.route(z, w, "", dict(r, groups={"count": 3, "keep": 3}))
    assert ids == [[4, 1]]


def test_plain_model_is_causal():
    spec, cfg = small()
    sd = tumatar.init_state_dict(spec, seed=1)
    g = torch.Generator().manual_seed(2)
    toks = torch.randint(0, spec.vocab, (9,), generator=g).tolist()
    full = oracle.forward(cfg, sd, toks)
    assert torch.allclose(full[:6], oracle.forward(cfg, sd, toks[:6]))
    assert torch.isfinite(full).all() and full.std() > 1e-3


# --------------------------------------------------------------------------- trace replay
class FakeEngine:
    def __init__(self):
        self.log, self.seq = [], []

    def reset(self):
        self.log.append("reset")
        self.seq = []

    def extend(self, tokens, want=()):
        base = len(self.seq)
        self.seq += list(tokens)
        self.log.append((tuple(tokens), tuple(want)))
        return torch.tensor([[float(base + w), float(self.seq[base + w])] for w in want]).view(len(want), 2)

    def close(self):
        self.log.append("close")


def test_trace_steps_map_to_engine_calls(tmp_path, monkeypatch, capsys):
    from naivert_b200.runtime import trace_run
    fake = FakeEngine()
    monkeypatch.setattr(trace_run, "build_engine", lambda model, dtype, n: fake)
    lines = [{"step": 0, "entries": [{"id": "a", "tokens": [4, 5, 6], "want": [2, 0]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [7], "want": []}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "b", "tokens": [8, 9], "want": [1]}], "end": ["b"]}]
    monkeypatch.setattr("sys.stdin", io.StringIO("\n".join(json.dumps(x) for x in lines) + "\n"))
    assert trace_run.main(["--model", "m", "--out", str(tmp_path / "o"), "--max-tokens", "8"]) == 0
    assert capsys.readouterr().out.splitlines() == ["done 0", "done 1", "done 2"]
    assert fake.log[-1] == "close" and [x for x in fake.log if isinstance(x, tuple)] == [((4, 5, 6), (0, 2)), ((7,), ()), ((8, 9), (1,))]
    assert struct.unpack("<4f", (tmp_path / "o" / "0.f32").read_bytes()) == (2.0, 6.0, 0.0, 4.0)
    assert struct.unpack("<2f", (tmp_path / "o" / "2.f32").read_bytes()) == (1.0, 9.0)
    assert sorted(os.listdir(tmp_path / "o")) == ["0.f32", "2.f32"]


def test_trace_refuses_a_second_live_request(tmp_path):
    from naivert_b200.runtime.trace_run import TraceError, TraceRunner
    r = TraceRunner(FakeEngine(), str(tmp_path))
    r.step({"step": 0, "entries": [{"id": "a", "tokens": [1], "want": []}], "end": []})
    with pytest.raises(TraceError, match="one sequence"):
        r.step({"step": 1, "entries": [{"id": "b", "tokens": [1], "want": []}], "end": []})
