"""Layer-list decoders on the CPU path (fp32): schedules, slots, generation, loader and registry against the oracle."""
import json

import pytest
import torch

from disagmoe_b200.config import AttentionSpec, LayerListConfig, LayerSpec, get_preset
from disagmoe_b200.models import weights as W
from disagmoe_b200.models.registry import load_model, resolve_model
from disagmoe_b200.ops import functional as F
from disagmoe_b200.ops.recurrent import build_segments
from layer_list_util import MODELS, error, feed, make_engine, model, tokens, attn, gla
from oracles import layer_stack as oracle

TOL = 2e-5


@pytest.fixture(scope="module", params=sorted(MODELS))
def case(request):
    raw = MODELS[request.param]
    w = oracle.random_weights(raw, seed=3)
    toks = tokens(90, raw["vocab"], 1)
    return raw, w, toks, oracle.run(raw, w, toks)[0]


@pytest.mark.parametrize("cuts", [[90], [1], [17, 2, 16, 1, 31], [2]])
def test_any_cut_gives_the_same_logits(case, cuts):
    raw, w, toks, want = case
    eng = make_engine(raw, w)
    assert error(feed(eng, 0, toks, cuts), want) < TOL
    assert eng.block_mgr.num_free_blocks() == 40


def test_mixed_batches_and_reused_slots(case):
    """Portions of one sequence beside single tokens of others; freed pages and slots are taken by later sequences."""
    raw, w, toks, want = case
    eng = make_engine(raw, w, max_seqs=2, pool=144)
    other = tokens(33, raw["vocab"], 4)
    want_o = oracle.run(raw, w, other)[0]
    for _ in range(2):
        rows = {0: [], 1: []}
        lens = {0: 0, 1: 0}
        for a, b in [(3, 2), (16, 1), (2, 1), (30, 5), (1, 16), (0, 7), (1, 1), (37, 0)]:
            ent = [(s, seq[lens[s]:lens[s] + n], list(range(n))) for s, seq, n in ((1, other, b), (0, toks, a)) if n]
            out = eng.feed(ent).clone()
            for s, part, _ in ent:
                rows[s].append(out[:len(part)])
                out = out[len(part):]
                lens[s] += len(part)
        assert error(torch.cat(rows[0]), want) < TOL and error(torch.cat(rows[1]), want_o) < TOL
        eng.end_fed([1])
        # a third sequence takes the freed slot while sequence 0 still holds its own
        assert error(feed(eng, 7, other, [10, 1]), want_o) < TOL
        eng.end_fed([0])
    assert eng.block_mgr.num_free_blocks() == 9


def test_wanted_rows_only(case):
    raw, w, toks, want = case
    eng = make_engine(raw, w)
    got = eng.feed([(0, toks[:40], [39, 0, 7])])
    assert error(got, want[[39, 0, 7]]) < TOL
    assert eng.feed([(0, toks[40:60], [])]).shape[0] == 0
    assert error(eng.feed([(0, toks[60:61], [0])]), want[60:61]) < TOL


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
    prompts = {i: tokens(n, raw["vocab"], 20 + i) for i, n in enumerate((28, 9, 14))}

    def start():
        e = make_engine(raw, w, **kw)
        for i, p in prompts.items():
            e.add_request(i, p, 8)
        return e
    want = start().run_until_done(100)
    a = start()
    for _ in range(4):
        a.step()
    a.save_state(str(tmp_path / "s.pt"))
    b = make_engine(raw, w, **{**kw, "max_seqs": 4})
    b.block_mgr.allocate(99, 30)          # other pages and slots than before
    b.load_state(str(tmp_path / "s.pt"))
    assert b.run_until_done(100) == want


def test_checkpoint_folder_round_trip(tmp_path):
    raw = MODELS["odd"]
    w = {n: t.bfloat16() for n, t in oracle.random_weights(raw, seed=7).items()}
    W.save_safetensors(w, str(tmp_path / "model.safetensors"))
    (tmp_path / "config.json").write_text(json.dumps(raw))
    cfg, sd = load_model(str(tmp_path), torch.float32, max_seq_len=64)
    assert isinstance(cfg, LayerListConfig) and cfg.max_seq_len == 64 and cfg.rms_norm_eps == raw["norm"]["eps"]
    assert all(torch.equal(sd[n], w[n]) for n in w) and cfg.layers[4].mixer.kv_from == 1
    assert resolve_model(str(tmp_path))[0].layers == cfg.layers
    eng = make_engine(raw, w)
    toks = tokens(20, raw["vocab"], 1)
    assert error(feed(eng, 0, toks, [20]), oracle.run(raw, w, toks)[0]) < TOL
    del sd["l2.mix.a1"]
    W.save_safetensors(sd, str(tmp_path / "model.safetensors"))
    with pytest.raises(ValueError, match="l2.mix.a1"):
        load_model(str(tmp_path))
    (tmp_path / "config.json").write_text(json.dumps({**raw, "architecture": "nothing"}))
    with pytest.raises(ValueError, match="unknown architecture"):
        load_model(str(tmp_path))
    with pytest.raises(ValueError, match="neither a preset"):
        resolve_model(str(tmp_path / "absent"))


def test_bad_key_sources_are_refused():
    a = AttentionSpec(2, 1, 8, 8, 1.0)
    bad = AttentionSpec(2, 2, 8, 8, 1.0, kv_from=0)
    for layers in ([LayerSpec(a), LayerSpec(bad)], [LayerSpec(AttentionSpec(2, 1, 8, 8, 1.0, kv_from=0))]):
        with pytest.raises(ValueError):
            LayerListConfig.make(16, 10, layers)
    with pytest.raises(ValueError):
        LayerListConfig.make(16, 10, [LayerSpec(AttentionSpec(3, 2, 8, 8, 1.0))])


def test_yarn_frequencies_match_the_oracle():
    for dims, base, sc in [(64, 1e4, dict(factor=8.0, original=512, fast=32.0, slow=1.0)), (12, 500.0, None),
                           (20, 3e5, dict(factor=2.5, original=4096, fast=4.0, slow=4.0)),
                           (128, 1e6, dict(factor=32.0, original=100, fast=32.0, slow=0.5))]:
        f, m = F.rope_frequencies(dims, base, **(sc or {}))
        of, om = oracle.inverse_frequencies({"dims": dims, "base": base, "scaling": sc})
        assert torch.allclose(torch.tensor(f, dtype=torch.float64), of, rtol=1e-13) and abs(m - om) < 1e-13


def test_segment_tables():
    rows = [4] * 70 + [1] + [2] * 2 + [0]
    pos = list(range(5, 75)) + [9] + [0, 1] + [3]
    t = build_segments(rows, pos, "cpu")
    assert t.singles.tolist() == [[70, 1, 1, 9], [73, 1, 0, 3]] and t.max_multi == 70
    assert t.multi.tolist() == [[0, 70, 4, 5], [71, 2, 2, 0]]
    assert t.chunks.tolist() == [[0, 64, 0, 0], [64, 6, 0, 1], [71, 2, 1, 0]]


def test_too_many_live_sequences():
    raw = model(16, 20, [gla(1, 4, 4), attn(1, 1, 4, 4, 5)])
    eng = make_engine(raw, oracle.random_weights(raw), max_seqs=2)
    eng.feed([(0, [1], []), (1, [2, 3], [])])
    with pytest.raises(ValueError, match="live"):
        eng.feed([(2, [1], [])])
    eng.end_fed([0])
    eng.feed([(2, [1], [])])


def test_preset_shapes_and_seeded_weights():
    cfg = get_preset("rurunex")
    shapes = W.param_shapes(cfg)
    assert "l5.mix.k" not in shapes and shapes["l2.mix.k"] == (512, 2048)
    one = W.init_tensor(cfg, "l0.mix.a2", shapes["l0.mix.a2"])
    assert torch.equal(one, W.init_tensor(cfg, "l0.mix.a2", shapes["l0.mix.a2"])) and one.dtype == torch.bfloat16


@pytest.mark.parametrize("budget", [0, 16])
def test_serving_command_line_from_a_checkpoint_folder(tmp_path, budget):
    from benchmark.benchmark_serving import main
    raw = MODELS["odd"]
    W.save_safetensors({n: t.bfloat16() for n, t in oracle.random_weights(raw).items()}, str(tmp_path / "model.safetensors"))
    (tmp_path / "config.json").write_text(json.dumps(raw))
    argv = ["--device", "cpu", "--model", str(tmp_path), "-n", "4", "-r", "0", "--min-input-len", "4", "-i", "30",
            "--min-output-len", "2", "-o", "5", "-f", str(tmp_path / "b.csv"), "--num-blocks", "32",
            "--max-batch-size-attn", "3", "--prefill-budget", str(budget)]
    assert main(argv + ["--backend", "colocated"]).token_throughput > 0
    with pytest.raises(SystemExit, match="colocated"):
        from benchmark.benchmark_serving import model_from_args
        from benchmark.utils import get_parser_base
        model_from_args(get_parser_base().parse_args(argv + ["--backend", "controller"]))


def test_disaggregated_paths_refuse_models_without_experts():
    from disagmoe_b200.frontend.controller import init_controller
    from disagmoe_b200.parallel.serving import FusedServingRank
    cfg = get_preset("rurunex")
    with pytest.raises(ValueError, match="no routed experts"):
        FusedServingRank(cfg, 2, 0, 0, 1)
    with pytest.raises(ValueError, match="no routed experts"):
        init_controller(1, 2, device="cpu").init_engine(None, cfg)
