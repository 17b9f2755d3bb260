"""Gated-residual decoders end to end on the GPU: every schedule against the oracle, in fp32 and as served (bf16)."""
import io
import json

import pytest
import torch

from disagmoe_b200.frontend.trace import TraceReplay
from disagmoe_b200.models import weights as W
from disagmoe_b200.ops import gemm
from gated_util import MODELS, both, dense, left, lightning, make_engine, model, moe, right, unit
from layer_list_util import error, feed, tokens
from oracles import gated_stack as oracle

pytestmark = pytest.mark.gpu
DEV = "cuda"
DTYPES = [torch.float32, torch.bfloat16]
N = 200
_cases = {}


def case(name):
    if name not in _cases:
        raw = MODELS[name]
        w = oracle.random_weights(raw, seed=3)
        toks = tokens(N, raw["vocab"], 1)
        _cases[name] = raw, w, toks, oracle.run(raw, w, toks)[0]
    return _cases[name]


def check(got, want, dtype):
    """fp32: every row. bf16: a router's close call may go the other way, so a few rows may be far off; the others are not."""
    if dtype == torch.float32:
        assert error(got, want) < 2e-4
        return
    d = got.double() - want
    d = (d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / (want - want.mean(-1, keepdim=True)).pow(2).mean().sqrt()
    assert float(d.median()) < 0.03 and float(torch.quantile(d, 0.9)) < 0.12, (float(d.median()), float(d.max()))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(MODELS))
def test_cuts(name, dtype):
    raw, w, toks, want = case(name)
    eng = make_engine(raw, w, DEV, dtype, graph=True)
    for cuts in ([N], [2], [64], [150, 50], [17, 2, 16, 1, 1, 31, 40], [130] + [1] * 70, [3, 65, 7, 1]):
        check(feed(eng, 0, toks, cuts), want, dtype)
    assert eng.block_mgr.num_free_blocks() == 40 and gemm.check_status(DEV) == 0


@pytest.mark.parametrize("name", sorted(MODELS))
def test_cuts_agree_with_each_other(name):
    """bf16: prompts (chunked and tiled kernels) against portions and single tokens."""
    raw, w, toks, _ = case(name)
    eng = make_engine(raw, w, DEV, torch.bfloat16, graph=True)
    whole = feed(eng, 0, toks, [N]).double()
    for cuts in ([1], [2], [150, 1, 49]):
        check(feed(eng, 0, toks, cuts), whole, torch.bfloat16)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(MODELS))
def test_mixed_batches_reuse_pages(name, dtype):
    raw, w, toks, want = case(name)
    eng = make_engine(raw, w, DEV, dtype, max_seqs=3, pool=352, graph=True)
    short = tokens(40, raw["vocab"], 9)
    want_s = oracle.run(raw, w, short)[0]
    long_cuts = [5, 1, 64, 1, 1, 2, 80, 1, 16, 1, 1, 27]
    assert sum(long_cuts) == N
    at, sid, rows, done = 0, 100, [], 0
    live = {}                                     # short sequences that come and go beside the long one
    for n in long_cuts:
        if len(live) < 2:
            live[sid] = [0, []]
            sid += 1
        ent = [(s, short[a:a + (7 if a % 2 == 0 else 1)]) for s, (a, _) in live.items() if a < 40]
        ent.insert(len(ent) // 2, (0, toks[at:at + n]))
        out = eng.feed([(s, p, list(range(len(p)))) for s, p in ent]).float().cpu()
        for s, p in ent:
            part, out = out[:len(p)], out[len(p):]
            if s == 0:
                rows.append(part)
            else:
                live[s][0] += len(p)
                live[s][1].append(part)
        at += n
        for s in [s for s, (a, _) in live.items() if a >= 40 or (s % 3 == 0 and a > 20)]:
            got = torch.cat(live.pop(s)[1])
            check(got, want_s[:len(got)], dtype)
            eng.end_fed([s])
            done += 1
    check(torch.cat(rows), want, dtype)
    assert done >= 2


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_over_pages_and_temperatures(dtype):
    raw = model(128, 200, [both(left(4, 2, 64, 64, None, (0.5, 32)), right(2, 40, 64), moe(8, 2, 48)), unit(128, 2, 4, dense(96)),
                           lightning(64, 32, (0.5, 0.99, 0.9999), moe(8, 2, 48)), both(left(4, 1, 48, 80), right(3, 64, 32), None)], taps=3)
    w = oracle.random_weights(raw, seed=8)
    toks = tokens(400, raw["vocab"], 2)
    want = oracle.run(raw, w, toks)[0]
    eng = make_engine(raw, w, DEV, dtype, graph=True)
    check(feed(eng, 0, toks, [3] + [1] * 397), want, dtype)
    check(feed(eng, 1, toks, [200] + [1] * 200), want, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_prompt_in_portions(dtype):
    """Over a thousand tokens: many chunks and passes of every recurrence, tiles of the prompt attention."""
    raw = model(128, 150, [lightning(64, 64, (0.7, 0.999)), both(left(4, 4, 64, 128), right(2, 64, 64), dense(64)), unit(96, 3, 4, moe(8, 2, 32)),
                           both(left(6, 2, 64, 32), right(1, 128, 48))])
    w = oracle.random_weights(raw, seed=4)
    toks = tokens(1100, raw["vocab"], 3)
    want = oracle.run(raw, w, toks)[0]
    eng = make_engine(raw, w, DEV, dtype, pool=1120, graph=True)
    for cuts in ([1100], [700, 300, 2, 1, 64], [257, 2, 511, 3, 1]):
        check(feed(eng, 0, toks, cuts), want, dtype)


@pytest.mark.parametrize("mixed", [False, True])
@pytest.mark.parametrize("name", sorted(MODELS))
def test_greedy_generation(name, mixed):
    """fp32: the oracle's tokens. bf16: nearly every token is the engine's own best one for its prefix, fed as a prompt."""
    raw, w, _, _ = case(name)
    kw = dict(prefill_budget=20) if mixed else {}
    prompts = {i: tokens(n, raw["vocab"], 30 + i) for i, n in enumerate((1, 45, 3, 66, 18, 30))}
    for dtype in DTYPES:
        eng = make_engine(raw, w, DEV, dtype, max_seqs=4, pool=320, mixed=mixed, graph=True, **kw)
        for i, p in prompts.items():
            eng.add_request(i, p, 12)
        out = eng.run_until_done(400)
        assert eng.block_mgr.num_free_blocks() == 20
        again = make_engine(raw, w, DEV, dtype)
        gaps = []
        for i, p in prompts.items():
            seq = p + out[i]
            ref = oracle.run(raw, w, seq[:-1])[0] if dtype == torch.float32 else feed(again, i, seq[:-1], [len(seq) - 1])
            ref = ref[len(p) - 1:]
            gaps.append((ref.max(-1).values - ref.gather(1, torch.tensor(out[i])[:, None])[:, 0]) / ref.std())
        gaps = torch.cat(gaps)
        assert float(gaps.max() if dtype == torch.float32 else torch.quantile(gaps.float(), 0.9)) < (1e-3 if dtype == torch.float32 else 0.1)


def test_snapshot_on_the_gpu(tmp_path):
    raw, w, _, _ = case("even")
    def start():
        e = make_engine(raw, w, DEV, torch.float32, max_seqs=3, pool=192, graph=True)
        for i, n in enumerate((28, 9, 14)):
            e.add_request(i, tokens(n, raw["vocab"], 20 + i), 8)
        return e
    want = start().run_until_done(100)
    a = start()
    for _ in range(4):
        a.step()
    a.save_state(str(tmp_path / "s.pt"))
    b = make_engine(raw, w, DEV, torch.float32, max_seqs=4, pool=192, graph=True)
    b.block_mgr.allocate(99, 30)
    b.load_state(str(tmp_path / "s.pt"))
    assert b.run_until_done(100) == want


def test_trace_replay_from_a_folder(tmp_path):
    raw, w, toks, want = case("odd")
    W.save_safetensors({n: t.bfloat16() for n, t in w.items()}, str(tmp_path / "model.safetensors"))
    (tmp_path / "config.json").write_text(json.dumps(raw))
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:40], "want": [0, 39]}], "end": []},
             {"step": 1, "entries": [{"id": "y", "tokens": toks[:2], "want": []}, {"id": "x", "tokens": toks[40:41], "want": [0]}],
              "end": ["y"]},
             {"step": 2, "entries": [{"id": "y", "tokens": toks[:5], "want": [4]}], "end": ["x", "y"]}]
    for name in ("float32", "bfloat16"):
        replay = TraceReplay(str(tmp_path), getattr(torch, name), 64 + 16)
        out = io.StringIO()
        replay.replay([json.dumps(s) for s in steps], str(tmp_path), out)
        assert out.getvalue() == "done 0\ndone 1\ndone 2\n"
        read = lambda n: torch.frombuffer(bytearray((tmp_path / f"{n}.f32").read_bytes()), dtype=torch.float32).view(-1, raw["vocab"])
        check(torch.cat([read(0), read(1), read(2)]), want[[0, 39, 40, 4]], getattr(torch, name))
        assert replay.engine.block_mgr.num_free_blocks() == 5
