"""Kernels of the parallel-block decoders, one mechanism at a time, against the oracle's functions."""
import pytest
import torch

from disagmoe_b200.config import RotarySpec
from disagmoe_b200.models.mixers import LatentTables, latent_layout
from disagmoe_b200.config import LatentAttentionSpec
from disagmoe_b200.ops import functional as F
from disagmoe_b200.ops import gemm
from oracles import parallel_stack as oracle

pytestmark = pytest.mark.gpu
DEV = "cuda"
BOTH = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])


def rnd(*shape, seed=0, scale=1.0, dtype=torch.float32):
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale).to(dtype)


def close(got, want, tol):
    want = want.double().cpu()
    err = (got.double().cpu() - want).abs().max() / want.pow(2).mean().sqrt()
    assert float(err) < tol, f"max error {float(err):.3g} of the rms"


def heads_close(got, want, tol):
    """Root mean square error of every (row, head) vector; a key seen or missed by mistake changes the whole vector."""
    want = want.double().cpu()
    err = ((got.double().cpu() - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()).max()
    assert float(err) < tol, f"worst vector is off by {float(err):.3g} of the rms"


def tol(dtype, f32=2e-5, bf16=3e-2):
    return f32 if dtype == torch.float32 else bf16


@BOTH
@pytest.mark.parametrize("n,W,P", [(7, 96, 3), (5, 44, 1), (300, 200, 2), (700, 2048, 6), (3, 5, 4), (2, 8192, 0)])
def test_sum_and_norm(n, W, P, dtype):
    x, y, parts = rnd(n, W, seed=1, scale=3.0) + 2.0, rnd(n, W, seed=2, dtype=dtype), rnd(n, max(P, 1), W, seed=3, dtype=dtype)
    w = 1 + 0.3 * rnd(W, seed=4)
    parts_d = parts.to(DEV) if P else None
    new = x.double() + y.double() + (parts.double().sum(1) if P else 0)
    rows = torch.tensor([n - 1, 0, 1], dtype=torch.int32)
    for centred, fn in ((True, lambda v: oracle.layer_norm(v, w, 1e-5)), (False, lambda v: oracle.rms(v, 1e-5) * w)):
        g = x.to(DEV)
        got, ids, wts = F.sum_norm(g, y.to(DEV), parts_d, w.to(DEV), 1e-5, dtype, centred, rows=rows.to(DEV))
        close(got, fn(new)[rows.long()], tol(dtype))
        assert torch.equal(g.cpu(), x) and ids is None and wts is None
        close(F.sum_norm(g, y.to(DEV), parts_d, w.to(DEV), 1e-5, dtype, centred)[0], fn(new), tol(dtype))
        close(g, new, 1e-5)
        close(F.sum_norm(g, None, None, w.to(DEV), 1e-5, dtype, centred)[0], fn(new), tol(dtype))


@BOTH
@pytest.mark.parametrize("n,W,E,K", [(1, 64, 8, 3), (33, 44, 5, 5), (200, 128, 64, 6), (700, 96, 256, 8), (900, 101, 40, 32), (9, 16, 1, 1)])
def test_router(n, W, E, K, dtype):
    x, w, gate = rnd(n, W, seed=1), 1 + 0.3 * rnd(W, seed=2), rnd(E, W, seed=3, scale=0.3, dtype=dtype)
    counts = torch.zeros(E, dtype=torch.int32, device=DEV)
    for renorm in (False, True):
        r = F.Router(gate.to(DEV), K, renorm, counts)
        h, ids, wts = F.sum_norm(x.to(DEV), None, None, w.to(DEV), 1e-6, dtype, True, router=r)
        want, s = oracle.route(h.double().cpu(), gate.double(), K)
        if renorm:
            s = s / s.sum(-1, keepdim=True)
        close(wts, s, 1e-4)
        full = torch.softmax(h.double().cpu() @ gate.double().T, -1)
        full = full / (full.gather(1, want).sum(-1, keepdim=True) if renorm else 1.0)
        close(full.gather(1, ids.long().cpu()), s, 1e-4)          # the chosen ones are the best, up to ties
        assert all(len(set(i)) == K for i in ids.tolist())
    assert torch.equal(counts.cpu(), 2 * torch.bincount(ids.reshape(-1).cpu(), minlength=E).int())


@BOTH
@pytest.mark.parametrize("T,W,E,K,ff", [(1, 64, 4, 2, 64), (70, 128, 8, 3, 40), (33, 44, 5, 5, 13), (300, 256, 16, 4, 128)])
def test_experts(T, W, E, K, ff, dtype):
    from disagmoe_b200.config import RoutedSpec
    from disagmoe_b200.models.mixers import RoutedBuffers, RoutedFeedForward
    sd = {f"m.e{e}.{n}": rnd(*s, seed=10 * e + i, scale=s[1] ** -0.5, dtype=dtype)
          for e in range(E) for i, (n, s) in enumerate((("gate", (ff, W)), ("up", (ff, W)), ("down", (W, ff))))}
    sd["m.router"] = rnd(E, W, seed=999, dtype=dtype)
    ffn, buf = RoutedFeedForward(sd, "m.", RoutedSpec(E, K, ff), torch.device(DEV), dtype), RoutedBuffers(T, W, E, K, DEV, dtype)
    x, w = rnd(T, W, seed=5), torch.ones(W)
    for _ in range(2):                            # the histogram is left clean
        h, ids, wts = F.sum_norm(x.to(DEV), None, None, w.to(DEV), 1e-5, dtype, True, router=ffn.router(buf))
        got = ffn(h, ids, wts, buf).float().sum(1)
        want = oracle.experts(h.double().cpu(), {n: t.double() for n, t in sd.items()}, "m.",
                              {"router": {"experts": E, "top": K}})
        close(got, want, tol(dtype, 2e-5, 0.1))
    assert gemm.check_status(DEV) == 0


@BOTH
@pytest.mark.parametrize("T,W,ff", [(3, 64, 64), (140, 128, 136), (9, 44, 40)])
def test_gelu_gate(T, W, ff, dtype):
    x, w = rnd(T, W, seed=1, scale=2.0, dtype=dtype), rnd(2 * ff, W, seed=2, scale=W ** -0.5, dtype=dtype)
    gu = x.double() @ w.double().T
    close(gemm.swiglu_linear(x.to(DEV), w.to(DEV), act="gelu_tanh"), oracle.gelu_tanh(gu[:, :ff]) * gu[:, ff:], tol(dtype, 1e-5, 0.08))


@BOTH
@pytest.mark.parametrize("n_q,n_kv,dk,dv,rot", [(6, 3, 64, 32, RotarySpec(64, 1e4, 4.0, 100, interleaved=True)),
                                               (3, 1, 10, 14, RotarySpec(6, 300.0, interleaved=True)), (5, 5, 128, 96, None)])
def test_interleaved_rotation_and_value_mixing(n_q, n_kv, dk, dv, rot, dtype):
    T, bs, blocks = 40, 16, 6
    row = rnd(T, n_q * dk + n_kv * (dk + dv), seed=5, dtype=dtype)
    first = rnd(T, n_kv, dv + 2, seed=6, dtype=dtype)
    slots = torch.randperm(bs * blocks, generator=torch.Generator().manual_seed(1))[:T]
    slots[11] = -1
    kc, vc = (torch.zeros(blocks, bs, n_kv, d, dtype=dtype, device=DEV) for d in (dk, dv))
    g = row.to(DEV)
    F.qk_norm_rope(g, torch.arange(T, dtype=torch.int32, device=DEV), slots.to(DEV), kc, vc, n_q, n_kv, dk, dv,
                   F.rope_freq_table(rot, 64, DEV), None, None, 1e-5, True, first.to(DEV), 0.3)
    spec = rot and {"dims": rot.dims, "base": rot.base, "scaling": rot.factor and
                    {"factor": rot.factor, "original": rot.original, "fast": rot.fast, "slow": rot.slow}}
    d, ok = row.double(), slots >= 0
    close(g[:, :n_q * dk], oracle.rotate_pairs(d[:, :n_q * dk].view(T, n_q, dk), spec).reshape(T, -1), tol(dtype))
    k = oracle.rotate_pairs(d[:, n_q * dk:(n_q + n_kv) * dk].view(T, n_kv, dk), spec)
    close(kc.view(-1, n_kv, dk)[slots[ok].to(DEV)], k[ok], tol(dtype))
    v = oracle.mix_values(d[:, (n_q + n_kv) * dk:].view(T, n_kv, dv), first[..., :dv].double(), 0.3)
    close(vc.view(-1, n_kv, dv)[slots[ok].to(DEV)], v[ok], tol(dtype))


def attend(q, k, v, scale, sink, window):
    """Vectorised form of oracle.attend."""
    T, H = q.shape[:2]
    g = H // k.shape[1]
    s = torch.einsum("ihd,jhd->hij", q.double(), k.double().repeat_interleave(g, 1)) * scale
    d = torch.arange(T)[:, None] - torch.arange(T)[None]
    s = s.masked_fill((d < 0) | (d >= (window or T + 1)), -1e30)
    return torch.einsum("hij,jhv->ihv", oracle.sink_softmax(s, sink.double()[:, None]), v.double().repeat_interleave(g, 1))


def planted(q, k, window):
    """Keys just inside and just outside the reach of some queries get nearly all the weight if they are seen."""
    T, G = k.shape[:2]
    for n, i in enumerate(range(window or 40, T, 5)):
        j = i - (window or 40) + (1 if n % 2 else 0)
        k[j] = (3 * q[i].view(G, -1, q.shape[-1])[:, 0].float()).to(k.dtype)


def pages(T, bs, seed=2):
    return torch.randperm((T + bs - 1) // bs, generator=torch.Generator().manual_seed(seed)).to(torch.int32)


def test_vectorised_oracle():
    q, k, v, s = rnd(20, 4, 8), rnd(20, 2, 8, seed=1), rnd(20, 2, 6, seed=2), rnd(4, seed=3)
    for window in (None, 5):
        close(attend(q, k, v, 0.3, s, window), oracle.attend(q.double(), k.double(), v.double(), 0.3, s.double(), window), 1e-10)


@BOTH
@pytest.mark.parametrize("H,G,D,V", [(8, 2, 64, 32), (6, 2, 64, 64), (12, 1, 64, 32), (5, 1, 128, 64), (20, 1, 128, 128), (3, 3, 20, 12)])
@pytest.mark.parametrize("window", [None, 1, 37, 64])
def test_attention_with_sinks(window, H, G, D, V, dtype):
    T, bs = 150, 16
    q, k, v = rnd(T, H, D, seed=1, dtype=dtype), rnd(T, G, D, seed=2, dtype=dtype), rnd(T, G, V, seed=3, dtype=dtype)
    planted(q, k, window)
    sink = rnd(H, seed=4, scale=3.0)
    sink[0] = 9.0
    want = attend(q, k, v, D ** -0.5, sink, window)
    blocks = pages(T, bs)
    kc, vc = torch.zeros(10, bs, G, D, dtype=dtype), torch.zeros(10, bs, G, V, dtype=dtype)
    for t in range(T):
        kc[blocks[t // bs], t % bs], vc[blocks[t // bs], t % bs] = k[t], v[t]
    kc, vc, qd, bt = kc.to(DEV), vc.to(DEV), q.reshape(T, H * D).to(DEV), blocks[None].to(DEV)
    rows, ctx = torch.zeros(T, dtype=torch.int32), torch.arange(1, T + 1, dtype=torch.int32)
    opt = dict(window=window, fp32_weights=True, sink=sink.to(DEV))
    for splits in (1, 3):
        got = F.paged_attention(qd, kc, vc, bt, rows.to(DEV), ctx.to(DEV), H, G, D, splits=splits, **opt)
        heads_close(got.view(T, H, V), want, tol(dtype, 1e-4))
    if not F.attention_on_tensor_cores(dtype, H, G, D, V):
        return
    for start in (0, 63, 70):
        tiles, _ = F.build_prefill_tiles(rows[start:], ctx[start:] - 1, F.prefill_tile_tokens(H, G))
        out = torch.full((T - start + 1, H * V), 7.0, dtype=dtype, device=DEV)
        F.prefill_attention(qd[start:], kc, vc, bt, tiles.to(DEV), len(tiles), H, G, D, out, **opt)
        heads_close(out[:-1].view(T - start, H, V), want[start:], tol(dtype, 1e-4))
        assert bool((out[-1] == 7.0).all())


@BOTH
@pytest.mark.parametrize("H,G,D,V", [(8, 2, 64, 32), (6, 2, 128, 64)])
def test_one_far_key_takes_the_weight(H, G, D, V, dtype):
    """Of 700 keys, one far back (first, at a page's first and last place) stands out for some late queries: single rows with
    and without splits, and prompt portions."""
    T, bs = 700, 16
    q, k, v = rnd(T, H, D, seed=1, dtype=dtype), rnd(T, G, D, seed=2, dtype=dtype), rnd(T, G, V, seed=3, dtype=dtype)
    pairs = [(699, 0), (650, 31), (500, 32), (497, 255), (300, 1)]
    for i, j in pairs:
        k[j] = (4 * q[i].view(G, -1, D)[:, 0].float()).to(dtype)
    sink = rnd(H, seed=4)
    want = attend(q, k, v, D ** -0.5, sink, None)
    for i, j in pairs:
        assert float((want[i, 0] - v[j, 0].double()).abs().max()) < 0.05      # what a missed key would change
    blocks = pages(T, bs)
    kc, vc = torch.zeros(len(blocks), bs, G, D, dtype=dtype), torch.zeros(len(blocks), bs, G, V, dtype=dtype)
    t = torch.arange(T)
    kc[blocks[t // bs].long(), t % bs], vc[blocks[t // bs].long(), t % bs] = k, v
    kc, vc, bt = kc.to(DEV), vc.to(DEV), blocks[None].to(DEV)
    opt = dict(fp32_weights=True, sink=sink.to(DEV))
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


LATENT = [(4, 32, 16, 48, 32), (5, 64, 32, 64, 96), (16, 128, 64, 128, 512), (35, 16, 8, 16, 264), (5, 9, 6, 11, 21), (2, 16, 2, 24, 130)]


@BOTH
@pytest.mark.parametrize("H,D,R,V,K", LATENT)
@pytest.mark.parametrize("window", [None, 1, 37, 64, 100])
def test_latent_attention(window, H, D, R, V, K, dtype):
    """Every path over one sequence: all rows on their own, prompt runs that start in the middle, and both in one batch."""
    T, bs, eps = 170, 16, 1e-5
    rot = RotarySpec(R, 5000.0, 3.0, 50, interleaved=True)
    m = LatentAttentionSpec(H, D, R, V, K, (D + R) ** -0.5, rot, window, True)
    lay = latent_layout(m)
    q, d = rnd(T, H, D + R, seed=1, dtype=dtype), rnd(T, K + R, seed=2, dtype=dtype)
    uk, uv = rnd(H * D, K, seed=3, scale=K ** -0.5, dtype=dtype), rnd(H * V, K, seed=4, scale=K ** -0.5, dtype=dtype)
    nw, sink = 1 + 0.3 * rnd(K, seed=5), rnd(H, seed=6, scale=2.0)
    spec = {"dims": R, "base": 5000.0, "scaling": {"factor": 3.0, "original": 50, "fast": 32.0, "slow": 1.0}}
    # the key just inside (outside) the window of some queries stands out through its rotated part
    for n, i in enumerate(range(window or 40, T, 5)):
        j = i - (window or 40) + (1 if n % 2 else 0)
        pad = torch.zeros(T, 1, R, dtype=torch.float64)
        pad[i] = q[i, :1, D:].double()
        turned = oracle.rotate_pairs(pad, spec)[i, 0]
        back = torch.zeros(T, 1, R, dtype=torch.float64)
        back[j] = turned                                           # rotate back by the key's own position: conjugate, rotate
        back[..., 1::2] *= -1
        back = oracle.rotate_pairs(back, spec)
        back[..., 1::2] *= -1
        d[j, K:] = (4 * back[j, 0]).to(dtype)
    # oracle, from the projections on
    dd = d.double()
    c = oracle.rms(dd[:, :K], eps) * nw
    key = torch.cat([(c @ uk.double().T).view(T, H, D), oracle.rotate_pairs(dd[:, None, K:], spec).expand(T, H, R)], -1)
    qq = torch.cat([q[..., :D].double(), oracle.rotate_pairs(q[..., D:].double(), spec)], -1)
    want = attend(qq, key, (c @ uv.double().T).view(T, H, V), m.scale, sink, window)
    # rows as the projection leaves them
    y = torch.zeros(T, H * lay.qd + lay.kd, dtype=dtype)
    yq = y[:, :H * lay.qd].view(T, H, lay.qd)
    yq[..., :D], yq[..., lay.dimp:lay.dimp + R] = q[..., :D], q[..., D:]
    y[:, H * lay.qd:H * lay.qd + K], y[:, H * lay.qd + lay.rankp:H * lay.qd + lay.rankp + R] = d[:, :K], d[:, K:]
    up = lambda w, n, p: torch.zeros(H, p, lay.rankp, dtype=dtype).index_put_((torch.arange(H)[:, None, None], torch.arange(n)[None, :, None], torch.arange(K)), w.view(H, n, K)).to(DEV)
    wk, wv = up(uk, D, lay.dimp), up(uv, V, lay.vdimp)
    blocks = pages(T, bs)
    cache = torch.zeros(len(blocks), bs, lay.row, dtype=dtype, device=DEV)
    bt, table = blocks[None].to(DEV), F.rope_freq_table(rot, 256, DEV)
    slot = lambda p: blocks[p // bs].long() * bs + p % bs
    for cuts in ([T], [1] * 3 + [T - 3], [130, 2, 38], [20, 150]):
        at = 0
        cache.zero_()
        for n in cuts:
            pos = torch.arange(at, at + n)
            rows, ctx = torch.zeros(n, dtype=torch.int32), (pos + 1).int()
            for t in ([LatentTables.prefill(m, rows, pos, torch.device(DEV), dtype)] + ([LatentTables.decode(m, n, DEV)] if n < 40 else [])):
                g = y[at:at + n].to(DEV)
                xq, qa = F.latent_prep(g, pos.int().to(DEV), slot(pos).to(DEV), cache, lay, table, nw.to(DEV), eps, t.loose, t.n_loose)
                out = torch.full((n + 1, H * lay.vdimp), 7.0, dtype=dtype, device=DEV)
                base = torch.tensor([out.data_ptr()], dtype=torch.int64, device=DEV)
                assert t.n_loose + (0 if t.loose is None else int((t.loose < 0).sum())) == n
                if t.n_loose:
                    gemm.grouped_linear(xq.view(-1, lay.dimp), wk.transpose(1, 2).contiguous(), t.offs, out=qa.view(-1, lay.row)[:, :lay.rankp])
                    o = F.latent_attention(qa, cache, bt, rows.to(DEV), ctx.to(DEV), t.rows, lay, m.scale, window, sink.to(DEV))
                    gemm.grouped_combine(o.view(-1, lay.rankp), wv, t.offs, t.recs, base, lay.vdimp)
                if t.n_tiles:
                    lat = F.latent_gather(cache, bt, t.keys, t.n_keys)
                    kv = gemm.linear(lat[:, :lay.rankp], torch.cat([wk, wv], 1).reshape(-1, lay.rankp))
                    F.latent_prefill(g, kv, lat, t.tiles, t.base, t.n_tiles, lay, m.scale, window, sink.to(DEV), out)
                assert bool((out[-1] == 7.0).all())
                full = want.clone()                                # the errors are relative to the whole sequence's size
                full[at:at + n] = out[:n].view(n, H, lay.vdimp)[..., :V].double().cpu()
                heads_close(full, want, tol(dtype, 1e-4, 6e-2))
            at += n
    assert gemm.check_status(DEV) == 0
