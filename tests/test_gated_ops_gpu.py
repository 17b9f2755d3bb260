"""Kernels of the gated-residual decoders, one mechanism at a time, against the oracle's functions."""
import pytest
import torch

from disagmoe_b200.config import QueryTemperature, RoutedSpec
from disagmoe_b200.models.mixers import RoutedBuffers, RoutedFeedForward
from disagmoe_b200.ops import functional as F
from disagmoe_b200.ops import gemm
from disagmoe_b200.ops.recurrent import (GatedUnit, Recurrence, build_segments, decode_segments, recurrent_attention,
                                         unit_recurrence)
from oracles import gated_stack as oracle
from oracles import prenorm_stack

pytestmark = pytest.mark.gpu
DEV = "cuda"
BOTH = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])


def rnd(*shape, seed=0, scale=1.0, dtype=torch.float32):
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale).to(dtype)


def close(got, want, tol):
    want = want.double().cpu()
    err = (got.double().cpu() - want).abs().max() / want.pow(2).mean().sqrt()
    assert float(err) < tol, f"max error {float(err):.3g} of the rms"


def near(got, want, tol):
    """Error of every number relative to its own size, or the rms of all where that is larger (products of two heavy tails)."""
    want = want.double().cpu()
    err = (got.double().cpu() - want).abs() / want.abs().clamp(min=want.pow(2).mean().sqrt())
    assert float(err.max()) < tol, f"max error {float(err.max()):.3g}"


def heads_close(got, want, tol):
    """Root mean square error of every (row, head) vector; a key seen or missed by mistake changes the whole vector."""
    want = want.double().cpu()
    err = ((got.double().cpu() - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()).max()
    assert float(err) < tol, f"worst vector is off by {float(err):.3g} of the rms"


def tol(dtype, f32=2e-5, bf16=3e-2):
    return f32 if dtype == torch.float32 else bf16


# sequences of 150, 40 and 7 tokens in slots 4, 0 and 2 of five: steps of (sequence, tokens)
LENS, SLOTS = (150, 40, 7), (4, 0, 2)
STEPS = [[(0, 30), (1, 1)], [(1, 2), (2, 1), (0, 1)], [(0, 1), (1, 30), (2, 1)], [(0, 66), (2, 5)], [(1, 1)], [(0, 2)],
         [(0, 1), (1, 6)], [(0, 49)]]


def step_tables(step, at, slots=SLOTS):
    """Segment tables of a step (also as a decode step with padding rows, where all have one token)."""
    pos = torch.cat([torch.arange(at[i], at[i] + n) for i, n in step]).int()
    row = torch.cat([torch.full((n,), slots[i]) for i, n in step]).int()
    out = [build_segments(row, pos, DEV)]
    if all(n == 1 for _, n in step):
        kv = torch.tensor([0] * len(step) + [-1] * len(step), dtype=torch.int64, device=DEV)
        out.append(decode_segments(torch.cat([pos, pos]).to(DEV), torch.cat([row, row]).to(DEV), kv))
    return out


# ---- residual, norms, gates, convolutions ------------------------------------------------------------------------------
@BOTH
@pytest.mark.parametrize("n,W,P,mult", [(7, 96, 3, 1.0), (300, 44, 2, 0.3), (700, 2048, 6, 1.0), (5, 2056, 1, 1.0)])
def test_gated_sum_and_layer_norm(n, W, P, mult, dtype):
    x, y, parts, z = rnd(n, W, seed=1, scale=3.0), rnd(n, W, seed=2, dtype=dtype), rnd(n, P, W, seed=3, dtype=dtype), \
        rnd(n, W, seed=4, scale=2.0, dtype=dtype)
    w, b, zb = 1 + 0.3 * rnd(W, seed=5), rnd(W, seed=6), rnd(W, seed=7)
    d = lambda t: t.double()
    new = d(x) + mult * oracle.sigmoid(d(z) + d(zb)) * (d(y) + d(parts).sum(1))
    gate, kw = F.ResidualGate(z.to(DEV), zb.to(DEV)), dict(bias=b.to(DEV), mult=mult)
    rows = torch.tensor([n - 1, 0, n // 2, 3], dtype=torch.int32)
    g = x.to(DEV)
    got, _, _ = F.sum_norm(g, y.to(DEV), parts.to(DEV), w.to(DEV), 1e-5, dtype, True, rows=rows.to(DEV), gate=gate, **kw)
    close(got, oracle.layer_norm(new[rows.long()], d(w), d(b), 1e-5), tol(dtype))
    assert torch.equal(g.cpu(), x)               # chosen rows leave the residual as it is
    got, _, _ = F.sum_norm(g, y.to(DEV), parts.to(DEV), w.to(DEV), 1e-5, dtype, True, gate=gate, **kw)
    close(got, oracle.layer_norm(new, d(w), d(b), 1e-5), tol(dtype))
    close(g, new, 1e-5)
    router = F.Router(rnd(5, W, seed=8, scale=W ** -0.5, dtype=dtype).to(DEV), 2, sigmoid=True)
    h, ids, wts = F.sum_norm(x.to(DEV), y.to(DEV), None, w.to(DEV), 1e-5, dtype, True, gate=gate, router=router, **kw)
    s = oracle.sigmoid(d(h.cpu()) @ d(router.weight.cpu()).T)
    close(wts, s.sort(-1, descending=True).values[:, :2], 1e-5)
    close(s.gather(1, ids.cpu().long()), s.sort(-1, descending=True).values[:, :2], 1e-5)


@BOTH
@pytest.mark.parametrize("n,W", [(7, 96), (300, 44), (500, 2048)])
@pytest.mark.parametrize("gated", [False, True])
def test_two_sides(gated, n, W, dtype):
    x, s, z = rnd(n, W, seed=1), rnd(2, n, W, seed=2, dtype=dtype), rnd(n, W, seed=3, dtype=dtype)
    s[1] *= 50.0                                  # sizes of the sides do not count
    sw, w, zb = 1 + 0.3 * rnd(2, W, seed=4), 1 + 0.3 * rnd(W, seed=5), rnd(W, seed=6)
    d = lambda t: t.double()
    y = oracle.side_by_side(d(s[0]), d(s[1]), {"left.out": d(sw[0]), "right.out": d(sw[1])}, "", 1e-5)
    new = d(x) + y * (oracle.sigmoid(d(z) + d(zb)) if gated else 1.0)
    g = x.to(DEV)
    got, _, _ = F.sum_norm(g, F.Sides(s.to(DEV), sw.to(DEV)), None, w.to(DEV), 1e-5, dtype, True,
                           gate=F.ResidualGate(z.to(DEV), zb.to(DEV)) if gated else None)
    close(got, oracle.layer_norm(new, d(w), 0.0, 1e-5), tol(dtype))
    close(g, new, 1e-5)


@BOTH
@pytest.mark.parametrize("W,taps", [(128, 4), (44, 2), (2056, 3), (9, 8), (64, 1), (256, 5)])
def test_input_convolution(W, taps, dtype):
    """Sequences in portions (down to two tokens and one) and single tokens, mixed in one batch, in slots that were used before;
    padding rows; every tap stands out at some token."""
    seqs = [rnd(n, W, seed=i, scale=2.0) for i, n in enumerate(LENS)]
    w, b, cw = 1 + 0.3 * rnd(W, seed=10), rnd(W, seed=11), rnd(W, taps, seed=12)
    normed = [oracle.layer_norm(s.double(), w.double(), b.double(), 1e-5).to(dtype) for s in seqs]
    want = [oracle.input_convolution(h.double(), cw.double()) for h in normed]
    ring = torch.full((5, taps, W), 7.0, dtype=dtype, device=DEV)
    at = [0, 0, 0]
    for step in STEPS:
        x = torch.cat([seqs[i][at[i]:at[i] + n] for i, n in step])
        kept = ring.clone()
        for segs in step_tables(step, at):
            ring.copy_(kept)
            rows = torch.cat([x, x + 100.0]) if segs.singles is None else x
            conv = F.InputConv(cw.T.contiguous().to(DEV), ring, segs)
            got, _, _ = F.sum_norm(rows.to(DEV), None, None, w.to(DEV), 1e-5, dtype, True, bias=b.to(DEV), conv=conv)
            cat = lambda seq: torch.cat([seq[i][at[i]:at[i] + n] for i, n in step])
            close(got[0, :len(x)], cat(normed), tol(dtype, 1e-5))
            close(got[1, :len(x)], cat(want), tol(dtype, 1e-5))
        for i, n in step:
            at[i] += n
    assert tuple(at) == LENS and bool((ring[[1, 3]] == 7.0).all())


@BOTH
@pytest.mark.parametrize("C,taps,blocks", [(128, 4, 2), (45, 3, 3), (2048, 4, 16), (26, 1, 2), (96, 8, 1), (21, 2, 1), (64, 4, 64)])
def test_biased_convolution_in_blocks(C, taps, blocks, dtype):
    """The input's bias counts from the sequence's first token on, not before it."""
    seqs = [rnd(n, C, seed=i, dtype=dtype) for i, n in enumerate(LENS)]
    cw, ib, ob = rnd(C, taps, seed=5), rnd(C, seed=6, scale=3.0), rnd(C, seed=7)
    want = [oracle.convolve(s.double() + ib.double(), cw.double()) + ob.double() for s in seqs]
    ring = torch.full((5, taps, C), 7.0, dtype=dtype, device=DEV)
    at, per = [0, 0, 0], C // blocks
    for step in STEPS:
        x = torch.cat([torch.nn.functional.pad(seqs[i][at[i]:at[i] + n], (0, 8)) for i, n in step]).to(DEV)
        y = F.seq_conv(x[:, :C], cw.T.contiguous().to(DEV), ring, step_tables(step, at)[0], ib.to(DEV), ob.to(DEV), blocks=blocks)
        assert y.shape == (blocks, len(x), (per + 7) // 8 * 8) and bool((y[..., per:] == 0).all())
        close(y[..., :per].transpose(0, 1).reshape(len(x), C), torch.cat([want[i][at[i]:at[i] + n] for i, n in step]), tol(dtype, 1e-5))
        for i, n in step:
            at[i] += n
    assert bool((ring[[1, 3]] == 7.0).all())


def test_embedding_with_positions():
    for dtype in (torch.float32, torch.bfloat16):
        t, p = rnd(50, 44, seed=1, dtype=dtype), rnd(30, 44, seed=2, dtype=dtype)
        ids, pos = torch.tensor([3, 49, 0, 3], dtype=torch.int32), torch.tensor([0, 29, 7, 7], dtype=torch.int32)
        out = torch.empty(4, 44, device=DEV)
        F.embed_f32(ids.to(DEV), t.to(DEV), 1.5, out, pos.to(DEV), p.to(DEV))
        close(out, t[ids.long()].double() * 1.5 + p[pos.long()].double(), 1e-6)


# ---- feed-forwards, GEMM epilogues ----------------------------------------------------------------------------------------
@BOTH
@pytest.mark.parametrize("T,K,F_,cols", [(3, 128, 64, 40), (200, 2048, 512, 384), (700, 256, 136, 136), (33, 44, 13, 7)])
def test_linear_with_silu_of_some_columns(T, K, F_, cols, dtype):
    x, w = rnd(T, K, seed=1, scale=2.0, dtype=dtype), rnd(F_, K, seed=2, scale=K ** -0.5, dtype=dtype)
    want = x.double() @ w.double().T
    want[:, :cols] = oracle.silu(want[:, :cols])
    close(gemm.linear(x.to(DEV), w.to(DEV), silu_cols=cols), want, tol(dtype))
    close(gemm.linear(x.to(DEV), w.to(DEV), silu_cols=cols, out_dtype=torch.float32), want, 2e-5)


@BOTH
@pytest.mark.parametrize("T,B,K,F_", [(5, 3, 32, 64), (300, 16, 128, 256), (40, 4, 20, 24), (700, 2, 64, 16)])
def test_grouped_linear_with_fp32_output(T, B, K, F_, dtype):
    x, w = rnd(B * T, K, seed=1, dtype=dtype), rnd(B, F_, K, seed=2, scale=K ** -0.5, dtype=dtype)
    want = torch.einsum("btk,bfk->btf", x.double().view(B, T, K), w.double()).reshape(B * T, F_)
    offs = (torch.arange(B + 1, dtype=torch.int32) * T).to(DEV)
    got = gemm.grouped_linear(x.to(DEV), w.to(DEV), offs, out_dtype=torch.float32)
    assert got.dtype == torch.float32
    close(got, want, 2e-5)


@BOTH
@pytest.mark.parametrize("T,W,E,K,ff,limit", [(1, 64, 4, 1, 48, 0.5), (40, 128, 8, 2, 128, 1.0), (300, 44, 6, 3, 13, 2.0),
                                              (600, 256, 16, 16, 72, 0.7), (130, 128, 1, 1, 64, 1e9)])
def test_clamped_experts_with_weighed_inputs(T, W, E, K, ff, limit, dtype):
    h = rnd(T, W, seed=1, scale=1.5)
    w = {"router": rnd(E, W, seed=2, scale=1.5 * W ** -0.5)}
    for e in range(E):
        w.update({f"e{e}.gate": rnd(ff, W, seed=3 * e + 3, scale=2 * W ** -0.5), f"e{e}.up": rnd(ff, W, seed=3 * e + 4, scale=2 * W ** -0.5),
                  f"e{e}.down": rnd(W, ff, seed=3 * e + 5, scale=ff ** -0.5)})
    w = {n: t.to(dtype).float() for n, t in w.items()}
    ffn = RoutedFeedForward(w, "", RoutedSpec(E, K, ff, act="clamped", scoring="sigmoid", limit=limit, weigh_input=True), DEV, dtype)
    buf = RoutedBuffers(T + 3, W, E, K, DEV, dtype)
    rows, ids, wts = F.sum_norm(h.to(DEV), None, None, torch.ones(W, device=DEV), 1e-5, dtype, True, router=ffn.router(buf))
    # the oracle's experts on the rows, choices and weights that the router left (its close calls are its own)
    x, want = rows.double().cpu(), torch.zeros(T, W, dtype=torch.float64)
    s = oracle.sigmoid(x @ w["router"].double().T)
    close(wts, s.gather(1, ids.cpu().long()), 1e-5)
    wd = {n: t.double() for n, t in w.items()}
    for t in range(T):
        for e, f in zip(ids[t].tolist(), wts[t].double().tolist()):
            want[t] += oracle.clamped_expert(f * x[t:t + 1], wd, f"e{e}.", limit)[0]
    got = ffn(rows, ids, wts, buf).double().sum(1)
    close(got, want, tol(dtype, 2e-5, 4e-2))
    full = oracle.experts(x, wd, "", {"router": {"experts": E, "top": K}, "expert": {"limit": limit}})
    same = (s.sort(-1, descending=True).indices[:, :K].sort(-1).values == ids.cpu().long().sort(-1).values).all(-1)
    close(got[same.to(DEV)], full[same], tol(dtype, 2e-5, 4e-2))
    assert int(same.sum()) >= T - 2


# ---- attention -----------------------------------------------------------------------------------------------------------
def attend(q, k, v, scale, temp):
    """Vectorised form of the oracle's causal attention with temperatures [T]."""
    T, H, _ = q.shape
    g = H // k.shape[1]
    k, v = k.double().repeat_interleave(g, 1), v.double().repeat_interleave(g, 1)
    s = torch.einsum("ihd,jhd->hij", q.double() * temp[:, None, None], k) * scale
    p = torch.softmax(s.masked_fill(torch.arange(T)[None] > torch.arange(T)[:, None], float("-inf")), -1)
    return torch.einsum("hij,jhd->ihd", p, v)


def test_vectorised_oracle():
    q, k, v = rnd(20, 4, 8).double(), rnd(20, 2, 8, seed=1).double(), rnd(20, 2, 6, seed=2).double()
    t = oracle.query_temperature(range(20), {"coef": 0.7, "every": 3})
    assert float(t[1]) == 1.0 and float(t[2]) > 1.4 and float(t[4]) == float(t[2]) and float(t[5]) > float(t[4])
    close(attend(q, k, v, 0.3, t), prenorm_stack.attend(q * t[:, None, None], k, v, 0.3, lambda i: 0), 1e-10)


def pages(T, bs, seed=2):
    return torch.randperm((T + bs - 1) // bs + 2, generator=torch.Generator().manual_seed(seed))[:(T + bs - 1) // bs].to(torch.int32)


@BOTH
@pytest.mark.parametrize("n_kv,dk,dv,pad", [(3, 64, 128, 112), (2, 64, 64, 64), (1, 128, 128, 100), (5, 10, 14, 14), (4, 40, 72, 72),
                                            (2, 64, 256, 256), (2, 64, 512, 300)])
def test_value_norm_at_the_append(n_kv, dk, dv, pad, dtype):
    """Norm over the real part of a padded head; rows without a slot are left out; queries and keys stay as they are."""
    T, bs, blocks, n_q = 37, 16, 6, 2 * n_kv
    row = rnd(T, (n_q + n_kv) * dk + n_kv * dv + 8, seed=5, dtype=dtype)
    v = row[:, (n_q + n_kv) * dk:-8].reshape(T, n_kv, dv)
    v[..., pad:] = 0
    v[3] *= 1e-3                                  # eps counts
    row[:, (n_q + n_kv) * dk:-8] = v.reshape(T, -1)
    slots = torch.randperm(blocks * bs, generator=torch.Generator().manual_seed(1))[:T]
    slots[5] = -1
    kc, vc = torch.full((blocks, bs, n_kv, dk), 7.0, dtype=dtype, device=DEV), torch.full((blocks, bs, n_kv, dv), 7.0, dtype=dtype, device=DEV)
    g = row.to(DEV)
    F.qk_norm_rope(g[:, :-8], torch.arange(T, dtype=torch.int32, device=DEV), slots.to(DEV), kc, vc, n_q, n_kv, dk, dv, None, None, None,
                   1e-5, v_norm=pad)
    want = torch.zeros(T, n_kv, dv, dtype=torch.float64)
    want[..., :pad] = oracle.rms(v[..., :pad].double(), 1e-5)
    ok = slots >= 0
    close(vc.view(-1, n_kv, dv)[slots[ok].to(DEV)], want[ok], tol(dtype, 1e-5, 2e-2))
    assert torch.equal(g.cpu(), row)
    assert torch.equal(kc.view(-1, n_kv, dk)[slots[ok].to(DEV)].cpu(), row[ok][:, n_q * dk:(n_q + n_kv) * dk].reshape(-1, n_kv, dk))
    used = torch.zeros(blocks * bs, dtype=torch.bool)
    used[slots[ok]] = True
    assert bool((vc.view(-1, n_kv, dv)[~used.to(DEV)] == 7.0).all())


ATTN = [(8, 2, 64, 32), (10, 5, 64, 128), (12, 1, 128, 128), (4, 2, 128, 64), (3, 3, 20, 28), (5, 5, 64, 64)]


@BOTH
@pytest.mark.parametrize("H,G,D,V", ATTN)
@pytest.mark.parametrize("coef,every", [(0.8, 16), (2.5, 7), (0.3, 1), (1.0, 1000)])
def test_temperature_and_head_gates(coef, every, H, G, D, V, dtype):
    """Temperatures change from one query to the next at multiples of ``every``; gates far apart; single rows with and without
    splits, and prompt portions."""
    T, bs = 210, 16
    q, k, v = rnd(T, H, D, seed=1, dtype=dtype), rnd(T, G, D, seed=2, dtype=dtype), rnd(T, G, V, seed=3, dtype=dtype)
    gate = rnd(T, H, seed=4, scale=3.0, dtype=dtype)
    temp = oracle.query_temperature(range(T), {"coef": coef, "every": every})
    want = attend(q, k, v, D ** -0.5, temp) * oracle.sigmoid(gate.double())[..., None]
    blocks = pages(T, bs)
    kc, vc = torch.zeros(20, bs, G, D, dtype=dtype), torch.zeros(20, bs, G, V, dtype=dtype)
    t = torch.arange(T)
    kc[blocks[t // bs].long(), t % bs], vc[blocks[t // bs].long(), t % bs] = k, v
    kc, vc, qd, bt = kc.to(DEV), vc.to(DEV), q.reshape(T, H * D).to(DEV), blocks[None].to(DEV)
    wide = torch.nn.functional.pad(gate, (3, 5)).to(DEV)
    gd = wide[:, 3:3 + H]
    rows, ctx = torch.zeros(T, dtype=torch.int32), torch.arange(1, T + 1, dtype=torch.int32)
    opt = dict(fp32_weights=True, q_temp=QueryTemperature(coef, every))
    for splits in (1, 3):
        got = F.paged_attention(qd, kc, vc, bt, rows.to(DEV), ctx.to(DEV), H, G, D, splits=splits, gate=gd, **opt)
        heads_close(got.view(T, H, V), want, tol(dtype, 1e-4))
    if not F.attention_on_tensor_cores(dtype, H, G, D, V):
        return
    for start in (0, 1, 63, 101):                # whole prompt, and portions that continue one
        tiles, _ = F.build_prefill_tiles(rows[start:], ctx[start:] - 1, F.prefill_tile_tokens(H, G))
        out = torch.full((T - start + 1, H * V), 7.0, dtype=dtype, device=DEV)
        F.prefill_attention(qd[start:], kc, vc, bt, tiles.to(DEV), len(tiles), H, G, D, out, gate=gd[start:], **opt)
        heads_close(out[:-1].view(T - start, H, V), want[start:], tol(dtype, 1e-4))
        assert bool((out[-1] == 7.0).all())


@BOTH
@pytest.mark.parametrize("H,G,D,V", [(10, 5, 64, 128), (8, 2, 128, 64), (3, 3, 20, 28)])
def test_one_far_key_takes_the_weight(H, G, D, V, dtype):
    """Of 700 keys, one far back (first, at a page's first and last place) stands out for some late queries, but only at their
    temperature: without it the other keys would keep a visible share."""
    T, bs = 700, 16
    q, k, v = rnd(T, H, D, seed=1, dtype=dtype), rnd(T, G, D, seed=2, dtype=dtype), rnd(T, G, V, seed=3, dtype=dtype)
    pairs = [(699, 0), (650, 31), (500, 32), (497, 255), (300, 1)]
    size = 7.0 * D ** 0.5                         # score of the far key at temperature 1
    for i, j in pairs:
        t = q[i].view(G, -1, D)[:, 0].float()
        k[j] = (t * (size / t.pow(2).sum(-1, keepdim=True))).to(dtype)
    temp = oracle.query_temperature(range(T), {"coef": 0.6, "every": 50})
    want = attend(q, k, v, D ** -0.5, temp)
    cold = attend(q, k, v, D ** -0.5, torch.ones(T, dtype=torch.float64))
    for i, j in pairs:
        assert float((want[i, 0] - v[j, 0].double()).abs().max()) < 0.2 < float((cold[i, 0] - v[j, 0].double()).abs().max())
    blocks = pages(T, bs)
    kc, vc = torch.zeros(len(blocks) + 2, bs, G, D, dtype=dtype), torch.zeros(len(blocks) + 2, bs, G, V, dtype=dtype)
    t = torch.arange(T)
    kc[blocks[t // bs].long(), t % bs], vc[blocks[t // bs].long(), t % bs] = k, v
    kc, vc, bt = kc.to(DEV), vc.to(DEV), blocks[None].to(DEV)
    opt = dict(fp32_weights=True, q_temp=QueryTemperature(0.6, 50))
    late = torch.tensor([i for i, _ in pairs])
    for splits in (1, 5):
        got = F.paged_attention(q[late].reshape(len(late), -1).to(DEV), kc, vc, bt, torch.zeros(len(late), dtype=torch.int32, device=DEV),
                                (late + 1).int().to(DEV), H, G, D, splits=splits, **opt)
        heads_close(got.view(-1, H, V), want[late], tol(dtype, 1e-4))
    if F.attention_on_tensor_cores(dtype, H, G, D, V):
        tiles, _ = F.build_prefill_tiles([0] * 210, range(490, T), F.prefill_tile_tokens(H, G))
        out = torch.zeros(210, H * V, dtype=dtype, device=DEV)
        F.prefill_attention(q[490:].reshape(210, -1).to(DEV), kc, vc, bt, tiles.to(DEV), len(tiles), H, G, D, out, **opt)
        heads_close(out.view(-1, H, V), want[490:], tol(dtype, 1e-4))


# ---- matrix-state recurrences ------------------------------------------------------------------------------------------------
class Linear:
    """Random inputs of one sequence for lightning attention ("decay") or a matrix memory ("memory"), the oracle's output
    [T, H V] and state. ``pace``: of the decays, or of the forget gates' logits."""

    def __init__(self, kind, H, D, V, T, dtype, seed=0, pace=0.0, change=None):
        r = lambda *s, k=0, scale=1.0: rnd(*s, seed=seed * 100 + k, scale=scale)
        self.dtype = dtype
        self.q, self.k, self.v, self.gate = (r(T, H * n, k=i).to(dtype) for i, n in enumerate((D, D, V, V)))
        nw = 1 + 0.3 * r(H * V, k=8)
        dv = lambda t: t.to(DEV).contiguous()
        d = lambda t: t.double().view(T, H, -1)
        kw = dict(sigmoid_gate=True)
        self.z = torch.zeros(T, 0)
        if kind == "memory":
            self.z, b, cap = r(T, 2 * H, k=5, scale=2.0), r(2 * H, k=6), 6.0
            self.z[:, H:] += pace + 2.0
        if change is not None:
            change(self)
        if kind == "decay":
            self.log = -torch.exp(r(H, k=7) + pace - 2.0)
            self.r = Recurrence(H, H, D, V, False, None, dv(nw), 1e-5, qscale=1.0, head_decay=dv(self.log), joint_norm=True, **kw)
            o, self.state = oracle.decay_recurrence(d(self.q), d(self.k), d(self.v), torch.exp(self.log.double()), with_state=True)
            o = oracle.rms(o.reshape(T, -1), 1e-5)
        else:
            self.r = Recurrence(H, H, D, V, False, None, dv(nw), 1e-5, gate_bias=dv(b), gate_cap=cap, **kw)
            zz = cap * torch.tanh((self.z.double() + b.double()) / cap)
            o, (self.state, self.n, self.m) = oracle.memory_recurrence(d(self.q) * D ** -0.5, d(self.k), d(self.v), zz[:, :H],
                                                                       oracle.log_sigmoid(zz[:, H:]), with_state=True)
            o = oracle.rms(o, 1e-5).reshape(T, -1)
        self.want = o * nw.double() * oracle.sigmoid(self.gate.double())


def run_steps(seqs, schedule, n_slots, slots, implicit=False, state=None):
    """``schedule``: steps of (sequence, tokens); returns each sequence's outputs. Sequence i lives in slot slots[i]."""
    state = state or seqs[0].r.new_state(n_slots, seqs[0].dtype, DEV)
    for t in state.tensors():
        t.fill_(7.0)                            # slots that were used before
    at, out = [0] * len(seqs), [[] for _ in seqs]
    for step in schedule:
        cat = lambda name: torch.cat([getattr(seqs[i], name)[at[i]:at[i] + n] for i, n in step]).to(DEV)
        pos = torch.cat([torch.arange(at[i], at[i] + n) for i, n in step]).int()
        row = torch.cat([torch.full((n,), slots[i]) for i, n in step]).int()
        segs = decode_segments(pos.to(DEV), row.to(DEV), torch.zeros(len(pos), dtype=torch.int64, device=DEV)) if implicit else \
            build_segments(row, pos, DEV)
        z = cat("z") if seqs[0].r.gate_bias is not None else None
        y = recurrent_attention(seqs[0].r, cat("q"), cat("k"), cat("v"), cat("gate"), None, z, state, segs).cpu()
        o = 0
        for i, n in step:
            out[i].append(y[o:o + n])
            o, at[i] = o + n, at[i] + n
    return [torch.cat(x) if x else None for x in out]


KINDS = pytest.mark.parametrize("kind", ["decay", "memory"])
SHAPES = pytest.mark.parametrize("H,D,V", [(3, 64, 64), (2, 128, 128), (1, 32, 64), (5, 16, 40), (2, 48, 32), (3, 7, 9), (2, 64, 20),
                                           (1, 256, 64), (16, 32, 64)])


@BOTH
@KINDS
@SHAPES
def test_recurrence_cuts(kind, H, D, V, dtype):
    s = Linear(kind, H, D, V, 150, dtype)
    for cuts in ([150], [64, 64, 22], [2] * 20 + [3, 61, 1, 1, 44], [63, 1, 1, 65, 20], [1] * 12 + [2, 136]):
        assert sum(cuts) == 150
        got, = run_steps([s], [[(0, n)] for n in cuts], 3, [1])
        close(got, s.want, tol(dtype, 2e-4, 6e-2))


@BOTH
@KINDS
@SHAPES
@pytest.mark.parametrize("pace", [-8.0, 0.0, 4.0])
def test_recurrent_state_is_fp32(kind, H, D, V, pace, dtype):
    """Read-outs and everything in the slot after prompts, portions and single tokens, from decays that hardly fade anything to
    decays that wipe the state within a token: fp32 accuracy also where the activations are bf16."""
    s = Linear(kind, H, D, V, 300, dtype, seed=5, pace=pace)
    for cuts in ([300], [129, 1, 170], [1] * 30 + [100, 2, 168], [257, 43]):
        state = s.r.new_state(2, dtype, DEV)
        got, = run_steps([s], [[(0, n)] for n in cuts], 2, [1], state=state)
        assert torch.isfinite(got).all()
        close(got, s.want, tol(dtype, 1e-3, 6e-2))
        if kind == "decay":
            close(state.S[1], s.state, 3e-4)
            continue
        # the running maximum is a scale: compare what does not depend on it, and itself
        m = state.m[1, 299 % 2].double().cpu()
        close(m, s.m, 1e-4)
        close(state.S[1].double().cpu() * torch.exp(m)[:, None, None], s.state * torch.exp(s.m)[:, None, None], 1e-3)
        close(state.n[1].double().cpu() * torch.exp(m)[:, None], s.n * torch.exp(s.m)[:, None], 1e-3)


@KINDS
@SHAPES
def test_recurrence_mixed_batch(kind, H, D, V):
    seqs = [Linear(kind, H, D, V, n, torch.bfloat16, seed=2) for n in (100, 40, 7)]
    for s in seqs[1:]:
        s.r = seqs[0].r                         # same weights: same seed
    steps = [[(0, 30), (1, 1)], [(1, 2), (2, 1), (0, 1)], [(0, 1), (1, 30), (2, 1)], [(0, 66), (2, 5)], [(1, 1)],
             [(0, 1), (1, 6)], [(0, 1)]]
    for got, s in zip(run_steps(seqs, steps, 5, SLOTS), seqs):
        close(got, s.want, 6e-2)


@BOTH
@KINDS
@SHAPES
def test_recurrence_decode_only(kind, H, D, V, dtype):
    """Long decoding of several sequences through the path that CUDA graphs capture; one joins late in a used slot."""
    seqs = [Linear(kind, H, D, V, n, dtype, seed=3) for n in (70, 70, 30)]
    for s in seqs[1:]:
        s.r = seqs[0].r
    steps = [[(0, 1), (1, 1)]] * 40 + [[(1, 1), (2, 1), (0, 1)]] * 30
    for got, s in zip(run_steps(seqs, steps, 4, [2, 3, 0], implicit=True), seqs):
        close(got, s.want, tol(dtype, 2e-4, 6e-2))


@KINDS
@pytest.mark.parametrize("place", [0, 63, 64, 127, 140])
def test_one_far_token_is_remembered(kind, place):
    """One token's write stands out; without decay it dominates every later read-out, through the state and within its chunk."""
    def change(s):
        s.k[place] *= 64.0
    s = Linear(kind, 2, 64, 64, 200, torch.bfloat16, seed=6, pace=-12.0 if kind == "decay" else 20.0, change=change)
    for cuts in ([200], [place + 1, 199 - place], [150] + [1] * 50, [2] * 100):
        close(run_steps([s], [[(0, n)] for n in cuts if n], 1, [0])[0], s.want, 6e-2)


@BOTH
@pytest.mark.parametrize("place", [0, 1, 62, 63, 64, 130])
def test_memory_with_one_wide_open_gate(place, dtype):
    """One input gate near its cap, the others nearly shut: the running maximum jumps there and falls back only as the forget gates
    let it; the divisor's floor and the small number beside it count. Also at the first token, where m starts at 0."""
    def change(s):
        s.z[:, :3] = -20.0
        s.z[place, :3] = 20.0
    s = Linear("memory", 3, 32, 40, 160, dtype, seed=9, pace=0.0, change=change)
    for cuts in ([160], [place + 1, 159 - place], [1] * 160, [2] * 80, [100, 1, 59]):
        close(run_steps([s], [[(0, n)] for n in cuts if n], 1, [0])[0], s.want, tol(dtype, 5e-4, 6e-2))


def test_padding_rows_leave_the_slots_alone():
    for kind in ("decay", "memory"):
        s = Linear(kind, 2, 32, 32, 4, torch.bfloat16)
        state = s.r.new_state(3, s.dtype, DEV)
        for t in state.tensors():
            t.fill_(5.0)
        segs = decode_segments(torch.tensor([3, 3], dtype=torch.int32, device=DEV), torch.tensor([1, 2], dtype=torch.int32, device=DEV),
                               torch.tensor([8, -1], dtype=torch.int64, device=DEV))
        rows = lambda t: t[:2].to(DEV)
        recurrent_attention(s.r, rows(s.q), rows(s.k), rows(s.v), rows(s.gate), None, rows(s.z) if kind == "memory" else None, state, segs)
        assert all(bool((t[[0, 2]] == 5.0).all()) and not bool((t[1] == 5.0).all()) for t in state.tensors())


# ---- diagonal recurrence -------------------------------------------------------------------------------------------------------
class Unit:
    """Random inputs of one sequence for the gated diagonal recurrence after its convolution, the oracle's output and state."""

    def __init__(self, C, B, T, dtype, seed=0, lam=-2.0):
        r = lambda *s, k=0, scale=1.0: rnd(*s, seed=seed * 100 + k, scale=scale)
        n, p = C // B, (C // B + 7) // 8 * 8
        self.dtype, self.C, self.B, self.p = dtype, C, B, p
        self.u, self.y, z = r(T, C, k=1).to(dtype), r(T, C, k=2).to(dtype), r(T, 2, C, k=3, scale=2.0)
        gb, lam, yb = r(2, C, k=4), r(C, k=5) + lam, r(C, k=6)
        blocked = lambda t: torch.nn.functional.pad(t.reshape(*t.shape[:-1], B, n), (0, p - n))
        self.ub = blocked(self.u)                                # [T, B, p]
        self.zb = blocked(z).transpose(1, 2)                     # [T, B, 2, p]
        dv = lambda t: t.to(DEV).contiguous()
        decay = -8.0 * torch.nn.functional.softplus(lam.double())
        self.r = GatedUnit(C, B, torch.zeros(1, C, device=DEV), None, None, dv(blocked(gb).transpose(0, 1)), dv(decay.float()), dv(yb))
        d = lambda t: t.double()
        gates = oracle.sigmoid(d(z) + d(gb))
        S, self.state = oracle.unit_recurrence(d(self.u), gates[:, 0], gates[:, 1], d(lam), with_state=True)
        self.want = S * oracle.gelu_tanh(d(self.y) + d(yb))

    def run(self, state, parts, segs):
        """``parts``: (sequence, first token, end) of the step's rows."""
        cat = lambda name: torch.cat([getattr(s, name)[a:b] for s, a, b in parts]).to(DEV)
        u, z = cat("ub").transpose(0, 1).contiguous(), cat("zb").transpose(0, 1).contiguous()
        y = torch.nn.functional.pad(cat("y"), (0, 8))[:, :self.C]
        return unit_recurrence(self.r, u, z, y, state, segs).cpu()


UNITS = pytest.mark.parametrize("C,B", [(128, 2), (45, 3), (2048, 16), (26, 2), (21, 1), (64, 64), (320, 5)])


@BOTH
@UNITS
@pytest.mark.parametrize("lam", [-12.0, -2.0, 4.0])
def test_unit_recurrence_cuts(C, B, lam, dtype):
    """From gates that hardly fade anything to gates that wipe the state; portions across the scan's passes; fp32 state."""
    T = 700
    s = Unit(C, B, T, dtype, lam=lam)
    for cuts in ([T], [256, 257, 187], [2] * 20 + [3, 1, 1, 513, 142], [127, 1, 128, 444], [1] * 12 + [688]):
        assert sum(cuts) == T
        state = s.r.new_state(3, dtype, DEV)
        state.S.fill_(7.0)
        at, out = 0, []
        for n in cuts:
            segs = build_segments([1] * n, range(at, at + n), DEV)
            out.append(s.run(state, [(s, at, at + n)], segs))
            at += n
        near(torch.cat(out), s.want, tol(dtype, 1e-4, 1e-2))
        close(state.S[1], s.state, 1e-4)
        assert bool((state.S[[0, 2]] == 7.0).all())


@BOTH
@UNITS
def test_unit_recurrence_mixed_batch_and_decoding(C, B, dtype):
    seqs = [Unit(C, B, n, dtype, seed=2) for n in LENS]
    for s in seqs[1:]:
        s.r = seqs[0].r
    state = seqs[0].r.new_state(5, dtype, DEV)
    state.S.fill_(7.0)
    at = [0, 0, 0]
    for step in STEPS:
        kept = state.S.clone()
        for segs in step_tables(step, at):
            state.S.copy_(kept)
            parts = [(seqs[i], at[i], at[i] + n) for i, n in step] * (2 if segs.singles is None else 1)
            got = seqs[0].run(state, parts, segs)
            want = torch.cat([seqs[i].want[at[i]:at[i] + n] for i, n in step])
            near(got[:len(want)], want, tol(dtype, 1e-4, 1e-2))
        for i, n in step:
            at[i] += n
            if at[i] == LENS[i]:
                close(state.S[SLOTS[i]], seqs[i].state, 1e-4)
    assert bool((state.S[[1, 3]] == 7.0).all())
