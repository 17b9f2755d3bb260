"""Parallel-block decoders on the CPU path (fp32): schedules, pages, generation, loader and registry against the oracle."""
import json

import pytest
import torch

from disagmoe_b200.config import AttentionSpec, LatentAttentionSpec, LayerListConfig, LayerSpec, RotarySpec, RoutedSpec, get_preset
from disagmoe_b200.models import weights as W
from disagmoe_b200.models.mixers import LatentTables
from disagmoe_b200.models.registry import load_model, supinex_config_from_json
from layer_list_util import error, feed, tokens
from oracles import parallel_stack as oracle
from parallel_block_util import MODELS, attn, dense, latent, make_engine, model, moe

TOL = 2e-5


@pytest.fixture(scope="module", params=sorted(MODELS))
def case(request):
    raw = MODELS[request.param]
    w = oracle.random_weights(raw, seed=3)
    toks = tokens(90, raw["vocab"], 1)
    return raw, w, toks, oracle.run(raw, w, toks)[0]


def test_reader_agrees_with_the_checkpoint_layout(case):
    raw, w, _, _ = case
    cfg = supinex_config_from_json(raw, {})
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
        assert error(feed(eng, 7, other, [10, 1]), want_o) < TOL      # pages of the finished one, beside one that is live
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


def test_checkpoint_folder_and_command_line(tmp_path):
    raw = MODELS["even"]
    w = {n: t.bfloat16() for n, t in oracle.random_weights(raw, seed=7).items()}
    W.save_safetensors(w, str(tmp_path / "model.safetensors"))
    (tmp_path / "config.json").write_text(json.dumps(raw))
    cfg, sd = load_model(str(tmp_path), torch.float32, max_seq_len=64)
    assert isinstance(cfg, LayerListConfig) and cfg.block == "parallel" and all(torch.equal(sd[n], w[n]) for n in w)
    assert sd["l1.mix.vmix"].shape == () and cfg.layers[0].mixer.window == 37 and cfg.layers[4].mixer.rot.dims == 32
    from benchmark.benchmark_serving import main
    argv = ["--device", "cpu", "--model", str(tmp_path), "-n", "4", "-r", "0", "--min-input-len", "4", "-i", "30",
            "--min-output-len", "2", "-o", "5", "-f", str(tmp_path / "b.csv"), "--num-blocks", "32",
            "--max-batch-size-attn", "3", "--backend", "colocated"]
    for budget in ("0", "16"):
        assert main(argv + ["--prefill-budget", budget]).token_throughput > 0
    del sd["l3.mlp.e2.up"]
    W.save_safetensors(sd, str(tmp_path / "model.safetensors"))
    with pytest.raises(ValueError, match="l3.mlp.e2.up"):
        load_model(str(tmp_path))
    raw["layers"][1]["mlp"] = {"kind": "sparse"}
    (tmp_path / "config.json").write_text(json.dumps(raw))
    with pytest.raises(ValueError, match="unknown feed-forward"):
        load_model(str(tmp_path))
    raw["layers"][1]["mlp"] = dense(96)


def test_mechanisms_show_in_the_logits():
    """What a fault in one mechanism would look like: the oracle with that mechanism changed differs by far more than the
    tolerance, so the comparisons above would catch it."""
    raw = MODELS["even"]
    w = oracle.random_weights(raw, seed=3)
    toks = tokens(90, raw["vocab"], 1)
    want = oracle.run(raw, w, toks)[0]
    other = json.loads(json.dumps(raw))
    other["layers"][0]["mixer"]["mask"]["size"] += 1
    assert error(oracle.run(other, w, toks)[0], want) > 100 * TOL
    other = json.loads(json.dumps(raw))
    other["layers"][3]["mlp"]["router"]["top"] -= 1
    assert error(oracle.run(other, w, toks)[0], want) > 100 * TOL
    for name, t in (("l0.mix.sink", -100.0), ("l1.mix.sink", -100.0), ("l3.mix.vmix", 0.0)):
        assert error(oracle.run(raw, {**w, name: torch.full_like(w[name], t)}, toks)[0], want) > 100 * TOL, name
    assert error(oracle.run(raw, {**w, "l1.mix.vmix": torch.tensor(0.9)}, toks)[0], want) < 1e-12      # the first one's is unused


def test_bad_configurations_are_refused():
    a = AttentionSpec(2, 1, 8, 8, 1.0, qk_norm=False, v_mix=True)
    mk = lambda *layers, **kw: LayerListConfig.make(16, 10, list(layers), **{"block": "parallel", **kw})
    mk(LayerSpec(a), LayerSpec(a))
    for bad in ([LayerSpec(a), LayerSpec(AttentionSpec(2, 2, 8, 8, 1.0, qk_norm=False, v_mix=True))],
                [LayerSpec(a, routed=RoutedSpec(4, 5, 8))], [LayerSpec(a, 8, "tanh")],
                [LayerSpec(LatentAttentionSpec(2, 8, 4, 8, 8, 1.0, RotarySpec(6, 100.0)))]):
        with pytest.raises(ValueError):
            mk(*bad)
    with pytest.raises(ValueError):
        mk(LayerSpec(a, routed=RoutedSpec(4, 2, 8)), block="sandwich")


def test_prompt_tables_of_latent_layers():
    """Runs, workspace rows and loose rows of a batch, checked against their definition."""
    class FakeCuda:
        type = "cuda"
    m = LatentAttentionSpec(3, 64, 32, 64, 64, 1.0, None, 50)
    runs = [(4, 30, 1), (2, 500, 140), (0, 0, 129), (1, 7, 5)]           # (block-table row, first position, tokens)
    rows = [r for r, _, n in runs for _ in range(n)]
    pos = [p + i for _, p, n in runs for i in range(n)]
    moved = torch.Tensor.to
    try:
        torch.Tensor.to = lambda t, *a, **k: t if a and isinstance(a[0], FakeCuda) else moved(t, *a, **k)
        t = LatentTables.prefill(m, rows, pos, FakeCuda(), torch.bfloat16)
    finally:
        torch.Tensor.to = moved
    assert t.rows.tolist() == [0] + list(range(270, 275)) and t.n_loose == 6
    assert [int(t.loose[r]) for r in t.rows] == list(range(6)) and int((t.loose < 0).sum()) == 269
    assert t.offs.tolist() == [0, 6, 12, 18] and t.recs[7].tolist()[:2] == [0, 270 * 3 + 1]
    for i in range(t.n_tiles):
        r0, n, row, p0 = t.tiles[i].tolist()
        for p in range(max(0, p0 - 49), p0 + n):
            assert t.keys[t.base[i] + p].tolist() == [row, p]
    assert t.n_keys == 140 + 49 + 129


def test_preset_and_seeded_weights():
    cfg = get_preset("supinex")
    shapes = W.param_shapes(cfg)
    assert "l1.mlp.gate" not in shapes and shapes["l1.mlp.e63.up"] == (1408, 2048) and shapes["l1.mix.uk"] == (2048, 512)
    one = W.init_tensor(cfg, "l3.mix.sink", shapes["l3.mix.sink"])
    assert torch.equal(one, W.init_tensor(cfg, "l3.mix.sink", shapes["l3.mix.sink"]))


def test_disaggregated_paths_refuse_the_design():
    from disagmoe_b200.frontend.controller import init_controller
    with pytest.raises(ValueError, match="beside the attention"):
        init_controller(1, 2, device="cpu").init_engine(None, get_preset("supinex"))
