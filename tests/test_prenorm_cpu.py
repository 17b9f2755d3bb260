"""Pre-norm decoders on the CPU path (fp32): schedules, pages, slots, generation, loader and registry against the oracle."""
import json

import pytest
import torch

from disagmoe_b200.config import AttentionSpec, LayerListConfig, LayerSpec, RoutedSpec, WkvSpec, get_preset
from disagmoe_b200.models import weights as W
from disagmoe_b200.models.registry import load_model, vufinex_config_from_json
from layer_list_util import error, feed, tokens
from oracles import prenorm_stack as oracle
from prenorm_util import MODELS, attn, make_engine, model, wkv

TOL = 2e-5


@pytest.fixture(scope="module", params=sorted(MODELS))
def case(request):
    raw = MODELS[request.param]
    w = oracle.random_weights(raw, seed=3)
    toks = tokens(90, raw["vocab"], 1)
    return raw, w, toks, oracle.run(raw, w, toks)[0]


def test_reader_agrees_with_the_checkpoint_layout(case):
    raw, w, _, _ = case
    cfg = vufinex_config_from_json(raw, {n: tuple(t.shape) for n, t in w.items()})
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


def test_shared_weights_have_their_own_memory():
    raw = MODELS["even"]
    w = oracle.random_weights(raw, seed=3)
    ex = make_engine(raw, w).executor
    assert [ex.cfg.weight_layer(i) for i in range(8)] == [0, 1, 2, 3, 4, 2, 0, 1]
    assert ex.mixers[5] is ex.mixers[2] and ex.ffs[6] is ex.ffs[0] and ex.norms[7] is ex.norms[1]
    memory = [t.data_ptr() for kv in ex.kv.values() for t in kv] + [t.data_ptr() for s in ex.states.values() for t in s.tensors()]
    assert len(memory) == len(set(memory)) == 2 * 3 + 2 + 2 * 3
    assert all(t.dtype == torch.float32 for s in ex.states.values() for t in s.tensors())
    # chains of references and a reference forwards
    layers = [attn(2, 2, 8, 5), wkv(2, 8), wkv(2, 8)]
    layers[1] = {**layers[1], "weights_of": 2}
    layers.append({**wkv(2, 8), "weights_of": 1})
    raw = model(32, 50, layers)
    w = oracle.random_weights(raw, seed=1)
    assert "l1.mix.r" not in w and "l2.mix.r" in w
    w1 = {**w, **{n.replace("l2.", f"l{i}."): t for n, t in w.items() if n.startswith("l2.") for i in (1, 3)}}
    flat = model(32, 50, [{k: v for k, v in l.items() if k != "weights_of"} for l in layers])
    toks = tokens(30, 50, 1)
    assert error(feed(make_engine(raw, w), 0, toks, [7, 1]), oracle.run(flat, w1, toks)[0]) < TOL


def test_checkpoint_folder_and_command_line(tmp_path):
    raw = MODELS["even"]
    w = {n: t.bfloat16() for n, t in oracle.random_weights(raw, seed=7).items()}
    W.save_safetensors(w, str(tmp_path / "model.safetensors"))
    (tmp_path / "config.json").write_text(json.dumps(raw))
    cfg, sd = load_model(str(tmp_path), torch.float32, max_seq_len=64)
    assert isinstance(cfg, LayerListConfig) and cfg.block == "prenorm" and all(torch.equal(sd[n], w[n]) for n in w)
    assert cfg.residual_mult == 0.4 and cfg.embed_scale == 6.0 and cfg.layers[2].mixer.chunk == 37 and cfg.layers[0].mixer.rank == 8
    assert cfg.layers[0].routed == RoutedSpec(8, 2, 40, renormalize=True, scoring="sigmoid", correction=True, groups=4, keep=2, scale=1.7)
    from benchmark.benchmark_serving import main
    argv = ["--device", "cpu", "--model", str(tmp_path), "-n", "4", "-r", "0", "--min-input-len", "4", "-i", "30",
            "--min-output-len", "2", "-o", "5", "-f", str(tmp_path / "b.csv"), "--num-blocks", "32",
            "--max-batch-size-attn", "3", "--backend", "colocated"]
    for budget in ("0", "16"):
        assert main(argv + ["--prefill-budget", budget]).token_throughput > 0
    del sd["l1.mlp.correction"]
    W.save_safetensors(sd, str(tmp_path / "model.safetensors"))
    with pytest.raises(ValueError, match="l1.mlp.correction"):
        load_model(str(tmp_path))
    bad = json.loads(json.dumps(raw))
    bad["layers"][1]["mlp"] = {"kind": "dense", "ff": 8}
    (tmp_path / "config.json").write_text(json.dumps(bad))
    with pytest.raises(ValueError, match="unknown feed-forward"):
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
    assert differs(lambda c: c["layers"][2]["mixer"]["mask"].update(size=38))
    assert differs(lambda c: c["layers"][5]["mixer"]["mask"].update(size=36))
    assert differs(lambda c: c["layers"][2]["mixer"]["rot"].update(base=2000.0))
    assert differs(lambda c: c["layers"][0]["mlp"]["router"].update(groups={"count": 4, "keep": 3}))
    assert differs(lambda c: c["layers"][0]["mlp"]["router"].update(scale=1.71))
    assert differs(lambda c: c["layers"][1]["mlp"]["router"].update(top=2))
    assert differs(lambda c: c.update(residual_mult=0.41))
    for n in w:
        leaf = n.split(".", 1)[-1]
        if leaf.startswith("mix.mu") or leaf in ("mix.u", "mix.w0", "mix.g", "mix.norm", "mlp.correction", "norm2", "mix.dkv.norm"):
            assert differs(lambda c: None, {**w, n: torch.zeros_like(w[n])}), n


def test_bad_configurations_are_refused():
    mk = lambda *layers, **kw: LayerListConfig.make(16, 10, list(layers), **{"block": "prenorm", **kw})
    ok = RoutedSpec(6, 2, 8, scoring="sigmoid", groups=3, keep=1)
    mk(LayerSpec(WkvSpec(2, 8), routed=ok), LayerSpec(WkvSpec(2, 8), routed=ok, weights_of=0))
    tied = AttentionSpec(2, 2, 8, 8, 1.0, qk_norm=False, tied_values=True)
    mk(LayerSpec(tied))
    for bad in ([LayerSpec(tied, routed=RoutedSpec(6, 3, 8, scoring="sigmoid", groups=3, keep=1))],
                [LayerSpec(tied, routed=RoutedSpec(6, 2, 8, scoring="sigmoid", groups=4, keep=2))],
                [LayerSpec(tied, routed=RoutedSpec(6, 2, 8, groups=2, keep=1))],
                [LayerSpec(tied, routed=RoutedSpec(6, 2, 8, scoring="tanh"))],
                [LayerSpec(WkvSpec(2, 8)), LayerSpec(WkvSpec(2, 4), weights_of=0)],
                [LayerSpec(WkvSpec(2, 8), weights_of=0)], [LayerSpec(WkvSpec(2, 8), weights_of=3)],
                [LayerSpec(AttentionSpec(2, 2, 8, 4, 1.0, qk_norm=False, tied_values=True))]):
        with pytest.raises(ValueError):
            mk(*bad)


def test_preset_and_seeded_weights():
    cfg = get_preset("vufinex")
    shapes = W.param_shapes(cfg)
    assert cfg.block == "prenorm" and any(l.weights_of is not None for l in cfg.layers)
    for i, l in enumerate(cfg.layers):
        assert (f"l{i}.norm1" in shapes) == (l.weights_of is None)
    name = "l0.mix.w0"
    assert torch.equal(W.init_tensor(cfg, name, shapes[name]), W.init_tensor(cfg, name, shapes[name]))


def test_disaggregated_paths_refuse_the_design():
    from disagmoe_b200.frontend.controller import init_controller
    with pytest.raises(ValueError, match="beside the attention"):
        init_controller(1, 2, device="cpu").init_engine(None, get_preset("vufinex"))
