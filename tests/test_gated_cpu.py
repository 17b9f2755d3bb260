"""Gated-residual decoders on the CPU path (fp32): schedules, pages, slots, generation, loader and registry against the oracle."""
import json

import pytest
import torch

from disagmoe_b200.config import (AttentionSpec, GatedUnitSpec, HeadDecaySpec, LayerListConfig, LayerSpec, MatrixMemorySpec,
                                  QueryTemperature, RoutedSpec, SideBySideSpec, get_preset)
from disagmoe_b200.models import weights as W
from disagmoe_b200.models.registry import load_model, panarax_config_from_json
from gated_util import MODELS, both, dense, left, lightning, make_engine, model, right, unit
from layer_list_util import error, feed, tokens
from oracles import gated_stack as oracle

TOL = 2e-5


@pytest.fixture(scope="module", params=sorted(MODELS))
def case(request):
    raw = MODELS[request.param]
    w = oracle.random_weights(raw, seed=3)
    toks = tokens(90, raw["vocab"], 1)
    return raw, w, toks, oracle.run(raw, w, toks)[0]


def test_reader_agrees_with_the_checkpoint_layout(case):
    raw, w, _, _ = case
    cfg = panarax_config_from_json(raw, {n: tuple(t.shape) for n, t in w.items()})
    assert W.param_shapes(cfg) == oracle.shapes(raw) and W.check_state_dict(cfg, w) == []


@pytest.mark.parametrize("cuts", [[90], [1], [17, 2, 16, 1, 31], [2]])
def test_any_cut_gives_the_same_logits(case, cuts):
    raw, w, toks, want = case
    eng = make_engine(raw, w)
    assert error(feed(eng, 0, toks, cuts), want) < TOL
    assert eng.block_mgr.num_free_blocks() == 40


def test_mixed_batches_and_reused_pages(case):
    raw, w, toks, want = case
    eng = make_engine(raw, w, max_seqs=2, pool=144)
    other = tokens(33, raw["vocab"], 4)
    want_o = oracle.run(raw, w, other)[0]
    for _ in range(2):
        rows, lens = {0: [], 1: []}, {0: 0, 1: 0}
        for a, b in [(3, 2), (16, 1), (2, 1), (30, 5), (1, 16), (0, 7), (1, 1), (37, 0)]:
            ent = [(s, seq[lens[s]:lens[s] + n], list(range(n))) for s, seq, n in ((1, other, b), (0, toks, a)) if n]
            out = eng.feed(ent).clone()
            for s, part, _ in ent:
                rows[s].append(out[:len(part)])
                out = out[len(part):]
                lens[s] += len(part)
        assert error(torch.cat(rows[0]), want) < TOL and error(torch.cat(rows[1]), want_o) < TOL
        eng.end_fed([1])
        assert error(feed(eng, 7, other, [10, 1]), want_o) < TOL      # pages and slot of the finished one, beside one that is live
        eng.end_fed([0])
    assert eng.block_mgr.num_free_blocks() == 9


def greedy(raw, w, prompt, n):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(oracle.run(raw, w, seq)[0][-1].argmax()))
    return seq[len(prompt):]


@pytest.mark.parametrize("mixed", [False, True])
def test_greedy_generation_through_the_scheduler(mixed):
    raw = MODELS["odd"]
    w = oracle.random_weights(raw, seed=5)
    eng = make_engine(raw, w, max_seqs=3, pool=192, mixed=mixed, **(dict(prefill_budget=24) if mixed else {}))
    prompts = {i: tokens(n, raw["vocab"], 10 + i) for i, n in enumerate((1, 45, 7, 30, 18))}
    for i, p in prompts.items():
        eng.add_request(i, p, 5)
    out = eng.run_until_done(200)
    for i, p in prompts.items():
        assert out[i] == greedy(raw, w, p, 5), f"request {i}"
    assert eng.block_mgr.num_free_blocks() == 12


@pytest.mark.parametrize("mixed", [False, True])
def test_snapshot_continues_with_the_same_tokens(tmp_path, mixed):
    raw = MODELS["odd"]
    w = oracle.random_weights(raw, seed=6)
    kw = dict(max_seqs=3, pool=192, mixed=mixed, **(dict(prefill_budget=16) if mixed else {}))

    def start():
        e = make_engine(raw, w, **kw)
        for i, n in enumerate((28, 9, 14)):
            e.add_request(i, tokens(n, raw["vocab"], 20 + i), 8)
        return e
    want = start().run_until_done(100)
    a = start()
    for _ in range(4):
        a.step()
    a.save_state(str(tmp_path / "s.pt"))
    b = make_engine(raw, w, **{**kw, "max_seqs": 4})
    b.block_mgr.allocate(99, 30)          # other pages and rows than before
    b.load_state(str(tmp_path / "s.pt"))
    assert b.run_until_done(100) == want


def test_every_layer_has_its_own_memory():
    raw = MODELS["even"]
    ex = make_engine(raw, oracle.random_weights(raw, seed=3)).executor
    memory = [t for kv in ex.kv.values() for t in kv] + ex._slot_tensors()
    # two layers with pages; 2 x (S, n, m), 2 x (S, ring), 3 x S; one ring of inputs per layer
    assert len(memory) == len({t.data_ptr() for t in memory}) == 2 * 2 + 2 * 3 + 2 * 2 + 3 + 7
    assert all(t.dtype == torch.float32 for s in ex.states.values() for t in (s.S, s.n, s.m) if t is not None)


def test_a_sequence_ends_at_the_last_position():
    raw = model(32, 50, [unit(16, 2)], positions=40)
    w = oracle.random_weights(raw, seed=1)
    eng = make_engine(raw, w, pool=160)
    toks = tokens(40, 50, 1)
    assert eng.cfg.max_seq_len == 40 and error(feed(eng, 0, toks, [23, 1, 16]), oracle.run(raw, w, toks)[0]) < TOL
    eng.feed([(1, toks, [0])])
    with pytest.raises(ValueError, match="beyond 40"):
        eng.feed([(1, [3], [0])])
    eng.end_fed([1])
    assert eng.block_mgr.num_free_blocks() == 10


def test_checkpoint_folder_and_command_line(tmp_path):
    raw = MODELS["even"]
    w = {n: t.bfloat16() for n, t in oracle.random_weights(raw, seed=7).items()}
    W.save_safetensors(w, str(tmp_path / "model.safetensors"))
    (tmp_path / "config.json").write_text(json.dumps(raw))
    cfg, sd = load_model(str(tmp_path), torch.float32, max_seq_len=64)
    assert isinstance(cfg, LayerListConfig) and cfg.block == "prenorm" and all(torch.equal(sd[n], w[n]) for n in w)
    assert cfg.layer_norm and cfg.residual_gate and cfg.tied_head and cfg.input_conv == 4 and cfg.positions == 1200
    assert cfg.layers[1].mixer == GatedUnitSpec(96, 3, 4) and cfg.layers[2].mixer == HeadDecaySpec(3, 32, 48, (0.3, 0.95, 0.998))
    assert cfg.layers[4].mixer == SideBySideSpec(
        AttentionSpec(6, 1, 40, 72, 0.2, qk_norm=False, value_norm=True, gate=True, q_temp=QueryTemperature(1.3, 7)),
        MatrixMemorySpec(2, 64, 128, 3.0))
    assert cfg.layers[1].routed == RoutedSpec(8, 2, 40, act="clamped", scoring="sigmoid", limit=1.5, weigh_input=True)
    from benchmark.benchmark_serving import main
    argv = ["--device", "cpu", "--model", str(tmp_path), "-n", "4", "-r", "0", "--min-input-len", "4", "-i", "30",
            "--min-output-len", "2", "-o", "5", "-f", str(tmp_path / "b.csv"), "--num-blocks", "32",
            "--max-batch-size-attn", "3", "--backend", "colocated"]
    for budget in ("0", "16"):
        assert main(argv + ["--prefill-budget", budget]).token_throughput > 0
    for n in ("l0.mix.right.i.b", "l3.rg1.b", "pos"):
        W.save_safetensors({k: t for k, t in sd.items() if k != n}, str(tmp_path / "model.safetensors"))
        with pytest.raises(ValueError, match=n):
            load_model(str(tmp_path))
    bad = json.loads(json.dumps(raw))
    bad["layers"][1]["type"] = "attention"
    (tmp_path / "config.json").write_text(json.dumps(bad))
    with pytest.raises(ValueError, match="unknown mixer"):
        load_model(str(tmp_path))


def test_mechanisms_show_in_the_logits():
    """What a fault in one mechanism would look like: the oracle with that mechanism changed differs by far more than the
    tolerance, so the comparisons above would catch it."""
    raw = MODELS["even"]
    w = oracle.random_weights(raw, seed=3)
    toks = tokens(90, raw["vocab"], 1)
    want = oracle.run(raw, w, toks)[0]

    def differs(change, weights=w):
        other = json.loads(json.dumps(raw))
        change(other)
        return error(oracle.run(other, weights, toks)[0], want) > 100 * TOL
    side = lambda c, i, s: c["layers"][i]["mixer"][s]
    assert differs(lambda c: side(c, 0, "left")["q_temp"].update(every=17))
    assert differs(lambda c: side(c, 4, "left")["q_temp"].update(coef=1.25))
    assert differs(lambda c: side(c, 0, "left").update(scale=0.13))
    assert differs(lambda c: side(c, 0, "right").update(gate_cap=7.0))
    assert differs(lambda c: c["layers"][2]["mixer"].update(decay=[0.3, 0.95, 0.99]))
    assert differs(lambda c: c["layers"][6]["mixer"].update(decay=[1.0, 0.05, 0.9]))
    assert differs(lambda c: c["layers"][1]["mlp"]["router"].update(top=1))
    assert differs(lambda c: c["layers"][2]["mlp"]["expert"].update(limit=0.9))
    assert differs(lambda c: c["norm"].update(eps=1e-2))
    for n in w:
        leaf = n.split(".", 1)[-1]
        if len(w[n].shape) == 1 or leaf in ("canon1", "rg1", "rg2", "mix.conv", "mix.ra", "mix.ri", "mix.g", "mix.left.g", "mix.right.g",
                                            "mix.right.i", "mix.right.f", "mix.right.k") or n == "pos":
            assert differs(lambda c: None, {**w, n: torch.zeros_like(w[n])}), n
    taps = {**w, "l3.canon1": w["l3.canon1"].roll(1, 1)}
    assert differs(lambda c: None, taps)


def test_the_normaliser_floor_and_the_running_maximum_count():
    """A memory whose gates hardly open: the floor exp(-m) of the divisor, m from 0 on, decides; gates wide open: the small number
    beside it does."""
    q, k, v = (torch.randn(30, 2, 8, generator=torch.Generator().manual_seed(i), dtype=torch.float64) for i in range(3))
    small = torch.full((30, 2), -9.0, dtype=torch.float64)
    f = torch.full((30, 2), -0.01, dtype=torch.float64)
    o, (_, _, m) = oracle.memory_recurrence(q, k, v, small, f, with_state=True)
    plain = oracle.decay_recurrence(q, k * torch.exp(small)[..., None], v, torch.exp(f))
    assert float((o * (1 + 1e-6 * torch.exp(m[0])) - plain).abs().max()) < 1e-6 * float(plain.abs().max())
    big = oracle.memory_recurrence(q, k, v, -small * 2, f)
    ratio = (big / oracle.memory_recurrence(q, k, v, 0 * small, f)).abs()
    assert float((ratio - 1).abs().max()) > 0.1


def test_bad_configurations_are_refused():
    mk = lambda *layers, **kw: LayerListConfig.make(16, 10, list(layers), **{"block": "prenorm", **kw})
    attn = AttentionSpec(2, 2, 8, 8, 1.0, qk_norm=False, value_norm=True, gate=True, q_temp=QueryTemperature(0.1, 4))
    ok = RoutedSpec(4, 2, 8, act="clamped", scoring="sigmoid", limit=2.0, weigh_input=True)
    mk(LayerSpec(SideBySideSpec(attn, MatrixMemorySpec(2, 8, 8, 5.0)), routed=ok), LayerSpec(attn), LayerSpec(HeadDecaySpec(2, 8, 8, (0.0, 1.0))))
    for bad in (LayerSpec(HeadDecaySpec(2, 8, 8, (0.5,))), LayerSpec(HeadDecaySpec(1, 8, 8, (1.5,))), LayerSpec(GatedUnitSpec(10, 4, 4)),
                LayerSpec(attn, routed=RoutedSpec(4, 2, 8, act="clamped")), LayerSpec(attn, 8, "clamped"),
                LayerSpec(AttentionSpec(2, 2, 8, 8, 1.0, qk_norm=False, q_temp=QueryTemperature(0.1, 0))),
                LayerSpec(AttentionSpec(2, 2, 8, 8, 1.0, qk_norm=False, value_norm=True, tied_values=True)),
                LayerSpec(SideBySideSpec(AttentionSpec(2, 2, 8, 8, 1.0, v_mix=True), MatrixMemorySpec(2, 8, 8, 5.0)))):
        with pytest.raises(ValueError):
            mk(bad)
    for kw in (dict(residual_gate=True), dict(input_conv=3), dict(layer_norm=True)):
        with pytest.raises(ValueError):
            mk(LayerSpec(HeadDecaySpec(1, 8, 8, (0.5,))), block="parallel", **kw)
    raw = model(32, 50, [lightning(8, 8, (0.5,))], taps=9)
    with pytest.raises(ValueError, match="taps"):
        make_engine(raw, oracle.random_weights(raw))


def test_preset_and_seeded_weights():
    cfg = get_preset("panarax")
    shapes = W.param_shapes(cfg)
    assert cfg.tied_head and "head" not in shapes and shapes["pos"] == (cfg.positions, cfg.hidden_size)
    for name in ("l0.mix.right.f.b", "l1.mix.lam", "l1.canon1"):
        assert torch.equal(W.init_tensor(cfg, name, shapes[name]), W.init_tensor(cfg, name, shapes[name]))


def test_disaggregated_paths_refuse_the_design():
    from disagmoe_b200.frontend.controller import init_controller
    with pytest.raises(ValueError, match="beside the attention"):
        init_controller(1, 2, device="cpu").init_engine(None, get_preset("panarax"))


def test_a_layer_without_a_feed_forward_in_every_place():
    raw = model(48, 60, [both(left(2, 1, 12, 8), right(2, 4, 6)), lightning(6, 10, (0.9, 0.4)), unit(24, 3, 5), unit(18, 1, 4, dense(10))],
                taps=3)
    w = oracle.random_weights(raw, seed=2)
    assert "l0.norm2" not in w and "l0.rg2" not in w
    toks = tokens(40, 60, 2)
    assert error(feed(make_engine(raw, w), 0, toks, [5, 1, 2, 9]), oracle.run(raw, w, toks)[0]) < TOL
