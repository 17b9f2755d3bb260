"""Kernels of the pre-norm decoders, one mechanism at a time, against the oracle's functions."""
import pytest
import torch

from disagmoe_b200.config import LatentAttentionSpec, RotarySpec, RoutedSpec
from disagmoe_b200.models.mixers import LatentTables, RoutedBuffers, RoutedFeedForward, latent_layout
from disagmoe_b200.ops import functional as F
from disagmoe_b200.ops import gemm
from disagmoe_b200.ops.recurrent import Recurrence, build_segments, decode_segments, recurrent_attention
from oracles import parallel_stack
from oracles import prenorm_stack as oracle

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


# ---- residual, norm, token shift --------------------------------------------------------------------------------------
@BOTH
@pytest.mark.parametrize("n,W,P", [(7, 96, 3), (300, 44, 2), (700, 2048, 6)])
def test_sum_and_norm_with_a_multiplier(n, W, P, dtype):
    x, y, parts = rnd(n, W, seed=1, scale=3.0), rnd(n, W, seed=2, dtype=dtype), rnd(n, P, W, seed=3, dtype=dtype)
    w = 1 + 0.3 * rnd(W, seed=4)
    new = x.double() + 0.37 * (y.double() + parts.double().sum(1))
    g = x.to(DEV)
    got, _, _ = F.sum_norm(g, y.to(DEV), parts.to(DEV), w.to(DEV), 1e-5, dtype, False, mult=0.37)
    close(got, oracle.centred_norm(new, w.double() - 1, 1e-5), tol(dtype))
    close(g, new, 1e-5)


@BOTH
@pytest.mark.parametrize("W,S", [(128, 5), (44, 5), (2056, 2), (9, 7)])
def test_token_shift(W, S, dtype):
    """Sequences in portions and single tokens, mixed in one batch, in slots that were used before; padding rows."""
    seqs = [rnd(n, W, seed=i, scale=2.0) for i, n in enumerate((150, 40, 7))]
    mu = torch.sigmoid(rnd(S, W, seed=9))
    w = 1 + 0.3 * rnd(W, seed=10)
    normed = [oracle.centred_norm(s.double(), w.double() - 1, 1e-5) for s in seqs]
    want = [torch.stack([oracle.token_shift(h, m.double()) for m in mu]) for h in normed]
    slots, last = [4, 0, 2], torch.full((5, W), 7.0, device=DEV)
    steps = [[(0, 30), (1, 1)], [(1, 2), (2, 1), (0, 1)], [(0, 1), (1, 30), (2, 1)], [(0, 66), (2, 5)], [(1, 1)], [(0, 2)],
             [(0, 1), (1, 6)], [(0, 49)]]
    at = [0, 0, 0]
    for step in steps:
        x = torch.cat([seqs[i][at[i]:at[i] + n] for i, n in step])
        pos = torch.cat([torch.arange(at[i], at[i] + n) for i, n in step]).int()
        row = torch.cat([torch.full((n,), slots[i]) for i, n in step]).int()
        tables = [build_segments(row, pos, DEV)]
        if all(n == 1 for _, n in step):
            pad = torch.cat([pos, pos]).to(DEV), torch.cat([row, row]).to(DEV)
            tables.append(decode_segments(*pad, torch.tensor([0] * len(step) + [-1] * len(step), dtype=torch.int64, device=DEV)))
        kept = last.clone()
        for segs in tables:
            last.copy_(kept)
            rows = torch.cat([x, x + 100.0]) if segs.singles is None else x
            got, _, _ = F.sum_norm(rows.to(DEV), None, None, w.to(DEV), 1e-5, dtype, False, shift=F.TokenShift(mu.to(DEV), last, segs))
            close(got[:, :len(x)], torch.cat([want[i][:, at[i]:at[i] + n] for i, n in step], 1), tol(dtype, 1e-5))
        for i, n in step:
            at[i] += n
            close(last[slots[i]], normed[i][at[i] - 1], 1e-5)
    assert at == [150, 40, 7] and bool((last[[1, 3]] == 7.0).all())


@BOTH
@pytest.mark.parametrize("T,K,F_", [(3, 128, 16), (200, 2048, 64), (700, 256, 128), (33, 44, 13)])
def test_linear_with_tanh(T, K, F_, dtype):
    x, w = rnd(T, K, seed=1, scale=2.0, dtype=dtype), rnd(F_, K, seed=2, scale=K ** -0.5, dtype=dtype)
    want = torch.tanh(x.double() @ w.double().T)
    close(gemm.linear(x.to(DEV), w.to(DEV), tanh=True), want, tol(dtype, 1e-5, 2e-2))
    close(gemm.linear(x.to(DEV), w.to(DEV), tanh=True, out_dtype=torch.float32), want, 2e-5)


# ---- recurrence ---------------------------------------------------------------------------------------------------------
class Wkv:
    """Random inputs of one sequence, the oracle's output [T, H D] and state."""

    def __init__(self, H, D, T, dtype, seed=0, decay=0.0):
        r = lambda *s, k=0: rnd(*s, seed=seed * 100 + k)
        self.dtype = dtype
        self.q, self.k, self.v, self.gate = (r(T, H * D, k=i).to(dtype) for i in range(4))
        self.z, w0, u, nw = r(T, H * D, k=5), r(H * D, k=6) + decay - 1.0, r(H, D, k=7), 1 + 0.3 * r(H * D, k=8)
        dv = lambda t: t.to(DEV).contiguous()
        self.r = Recurrence(H, H, D, D, False, dv(w0), dv(nw), 1e-5, exp_decay=True, bonus=dv(u), qscale=1.0, shift_width=8)
        d = lambda t: t.double().view(T, H, D)
        o, self.state = oracle.bonus_recurrence(d(self.q), d(self.k), d(self.v), -torch.exp(d(self.z) + w0.double().view(H, D)),
                                                u.double(), with_state=True)
        self.want = oracle.rms(o, 1e-5).reshape(T, -1) * nw.double() * oracle.silu(self.gate.double())


def run_steps(seqs, schedule, n_slots, slots, implicit=False, state=None):
    """``schedule``: steps of (sequence, tokens); returns each sequence's outputs. Sequence i lives in slot slots[i]."""
    state = state or seqs[0].r.new_state(n_slots, seqs[0].dtype, DEV)
    state.S.fill_(7.0)                          # slots that were used before
    at, out = [0] * len(seqs), [[] for _ in seqs]
    for step in schedule:
        cat = lambda name: torch.cat([getattr(seqs[i], name)[at[i]:at[i] + n] for i, n in step]).to(DEV)
        pos = torch.cat([torch.arange(at[i], at[i] + n) for i, n in step]).int()
        row = torch.cat([torch.full((n,), slots[i]) for i, n in step]).int()
        segs = decode_segments(pos.to(DEV), row.to(DEV), torch.zeros(len(pos), dtype=torch.int64, device=DEV)) if implicit else \
            build_segments(row, pos, DEV)
        y = recurrent_attention(seqs[0].r, cat("q"), cat("k"), cat("v"), cat("gate"), None, cat("z"), state, segs).cpu()
        o = 0
        for i, n in step:
            out[i].append(y[o:o + n])
            o, at[i] = o + n, at[i] + n
    return [torch.cat(x) if x else None for x in out]


SHAPES = [(3, 64), (2, 128), (1, 32), (5, 16), (2, 48), (3, 7), (2, 20), (1, 256)]


@BOTH
@pytest.mark.parametrize("H,D", SHAPES)
def test_wkv_cuts(H, D, dtype):
    s = Wkv(H, D, 150, dtype)
    for cuts in ([150], [64, 64, 22], [2] * 20 + [3, 61, 1, 1, 44], [63, 1, 1, 65, 20], [1] * 12 + [2, 136]):
        assert sum(cuts) == 150
        got, = run_steps([s], [[(0, n)] for n in cuts], 3, [1])
        close(got, s.want, tol(dtype, 2e-4, 6e-2))


@BOTH
@pytest.mark.parametrize("H,D", SHAPES)
@pytest.mark.parametrize("decay", [-6.0, -1.0, 1.0, 3.0])
def test_wkv_state_is_fp32(H, D, decay, dtype):
    """Read-outs and the state after prompts, portions and single tokens, from decays that hardly fade anything to decays that
    wipe the state within a token: fp32 accuracy of the state also where the activations are bf16."""
    s = Wkv(H, D, 200, dtype, seed=5, decay=decay)
    for cuts in ([200], [129, 1, 70], [1] * 30 + [100, 2, 68]):
        state = s.r.new_state(2, dtype, DEV)
        got, = run_steps([s], [[(0, n)] for n in cuts], 2, [1], state=state)
        assert torch.isfinite(got).all()
        close(got, s.want, tol(dtype, 3e-4, 6e-2))
        close(state.S[1], s.state, 3e-4)


@pytest.mark.parametrize("H,D", SHAPES)
def test_wkv_mixed_batch(H, D):
    seqs = [Wkv(H, D, n, torch.bfloat16, seed=2) for n in (100, 40, 7)]
    for s in seqs[1:]:
        s.r = seqs[0].r                         # same weights: same seed
    steps = [[(0, 30), (1, 1)], [(1, 2), (2, 1), (0, 1)], [(0, 1), (1, 30), (2, 1)], [(0, 66), (2, 5)], [(1, 1)],
             [(0, 1), (1, 6)], [(0, 1)]]
    for got, s in zip(run_steps(seqs, steps, 5, [4, 0, 2]), seqs):
        close(got, s.want, 6e-2)


@BOTH
@pytest.mark.parametrize("H,D", SHAPES)
def test_wkv_decode_only(H, D, dtype):
    """Long decoding of several sequences through the path that CUDA graphs capture; one joins late in a used slot."""
    seqs = [Wkv(H, D, n, dtype, seed=3) for n in (70, 70, 30)]
    for s in seqs[1:]:
        s.r = seqs[0].r
    steps = [[(0, 1), (1, 1)]] * 40 + [[(1, 1), (2, 1), (0, 1)]] * 30
    for got, s in zip(run_steps(seqs, steps, 4, [2, 3, 0], implicit=True), seqs):
        close(got, s.want, tol(dtype, 2e-4, 6e-2))


@pytest.mark.parametrize("place", [0, 63, 64, 127, 140])
def test_wkv_remembers_one_far_token(place):
    """One token's write stands out; without decay it dominates every later read-out, through the state and within its chunk."""
    s = Wkv(2, 64, 200, torch.bfloat16, seed=6, decay=-12.0)
    s.k[place] *= 64.0
    T, d = 200, lambda t: t.double().view(200, 2, 64)
    o = oracle.bonus_recurrence(d(s.q), d(s.k), d(s.v), -torch.exp(d(s.z) + s.r.z_bias.double().cpu().view(2, 64)),
                                s.r.bonus.double().cpu())
    want = oracle.rms(o, 1e-5).reshape(T, -1) * s.r.norm_w.double().cpu() * oracle.silu(s.gate.double())
    for cuts in ([200], [place + 1, 199 - place], [150] + [1] * 50, [2] * 100):
        close(run_steps([s], [[(0, n)] for n in cuts if n], 1, [0])[0], want, 6e-2)


# ---- attention ----------------------------------------------------------------------------------------------------------
@BOTH
@pytest.mark.parametrize("n_q,n_kv,dk,dv,rot", [(6, 3, 64, 64, 32), (4, 4, 64, 32, 16), (3, 1, 10, 10, 6), (8, 2, 128, 128, 128),
                                                (2, 2, 64, 64, 8), (5, 5, 64, 64, None)])
def test_half_rotation_with_tied_values(n_q, n_kv, dk, dv, rot, dtype):
    T, bs, blocks = 40, 16, 6
    row = rnd(T, (n_q + n_kv) * dk, seed=5, dtype=dtype)
    slots = torch.randperm(bs * blocks, generator=torch.Generator().manual_seed(1))[:T]
    slots[11] = -1
    kc, vc = (torch.zeros(blocks, bs, n_kv, d, dtype=dtype, device=DEV) for d in (dk, dv))
    g = row.to(DEV)
    spec = RotarySpec(rot, 700.0) if rot else None
    F.qk_norm_rope(g, torch.arange(T, dtype=torch.int32, device=DEV), slots.to(DEV), kc, vc, n_q, n_kv, dk, dv,
                   F.rope_freq_table(spec, 64, DEV), None, None, 1e-5, tied=True)
    d, ok = row.double().view(T, n_q + n_kv, dk), slots >= 0
    turned = oracle.rotate(d, rot and {"dims": rot, "base": 700.0})
    close(g[:, :n_q * dk].view(T, n_q, dk), turned[:, :n_q], tol(dtype))
    close(kc.view(-1, n_kv, dk)[slots[ok].to(DEV)], turned[ok, n_q:], tol(dtype))
    assert torch.equal(vc.view(-1, n_kv, dv)[slots[ok].to(DEV)].cpu(), row.view(T, n_q + n_kv, dk)[ok, n_q:, :dv])


def attend(q, k, v, scale, chunk):
    """Vectorised form of oracle.attend."""
    T, H = q.shape[:2]
    g = H // k.shape[1]
    s = torch.einsum("ihd,jhd->hij", q.double(), k.double().repeat_interleave(g, 1)) * scale
    i, j = torch.arange(T)[:, None], torch.arange(T)[None]
    s = s.masked_fill((j > i) | (j < (i // chunk * chunk if chunk else 0)), -1e30)
    return torch.einsum("hij,jhv->ihv", torch.softmax(s, -1), v.double().repeat_interleave(g, 1))


def test_vectorised_oracle():
    q, k, v = rnd(20, 4, 8).double(), rnd(20, 2, 8, seed=1).double(), rnd(20, 2, 6, seed=2).double()
    for chunk in (None, 1, 6):
        close(attend(q, k, v, 0.3, chunk), oracle.attend(q, k, v, 0.3, oracle.chunk_start(chunk)), 1e-10)


@BOTH
@pytest.mark.parametrize("H,G,D,V", [(8, 2, 64, 32), (6, 6, 64, 64), (12, 1, 128, 128), (4, 2, 128, 64), (3, 3, 20, 20)])
@pytest.mark.parametrize("chunk", [1, 16, 37, 64, 100, 1000])
def test_chunked_attention(chunk, H, G, D, V, dtype):
    """The key just inside and just outside the chunk of some queries stands out."""
    T, bs = 210, 16
    q, k, v = rnd(T, H, D, seed=1, dtype=dtype), rnd(T, G, D, seed=2, dtype=dtype), rnd(T, G, V, seed=3, dtype=dtype)
    for n, i in enumerate(range(2, T, 3)):
        j = i // chunk * chunk - n % 2           # the first key of the query's chunk, or the one before it
        if 0 <= j < i:
            k[j] = (3 * q[i].view(G, -1, D)[:, 0].float()).to(dtype)
    want = attend(q, k, v, D ** -0.5, chunk)
    blocks = torch.randperm(14, generator=torch.Generator().manual_seed(2)).to(torch.int32)
    kc, vc = torch.zeros(14, bs, G, D, dtype=dtype), torch.zeros(14, bs, G, V, dtype=dtype)
    t = torch.arange(T)
    kc[blocks[t // bs].long(), t % bs], vc[blocks[t // bs].long(), t % bs] = k, v
    kc, vc, qd, bt = kc.to(DEV), vc.to(DEV), q.reshape(T, H * D).to(DEV), blocks[None].to(DEV)
    rows, ctx = torch.zeros(T, dtype=torch.int32), torch.arange(1, T + 1, dtype=torch.int32)
    opt = dict(chunk=chunk, fp32_weights=True)
    for splits in (1, 3):
        got = F.paged_attention(qd, kc, vc, bt, rows.to(DEV), ctx.to(DEV), H, G, D, splits=splits, **opt)
        heads_close(got.view(T, H, V), want, tol(dtype, 1e-4))
    if not F.attention_on_tensor_cores(dtype, H, G, D, V):
        return
    for start in (0, 1, 63, 101):                # whole prompt, and portions that continue one
        tiles, _ = F.build_prefill_tiles(rows[start:], ctx[start:] - 1, F.prefill_tile_tokens(H, G))
        out = torch.full((T - start + 1, H * V), 7.0, dtype=dtype, device=DEV)
        F.prefill_attention(qd[start:], kc, vc, bt, tiles.to(DEV), len(tiles), H, G, D, out, **opt)
        heads_close(out[:-1].view(T - start, H, V), want[start:], tol(dtype, 1e-4))
        assert bool((out[-1] == 7.0).all())


@BOTH
@pytest.mark.parametrize("H,D,R,V,K", [(4, 32, 16, 48, 32), (16, 128, 64, 128, 512), (5, 9, 6, 11, 21), (35, 16, 8, 16, 264)])
def test_gated_latent_attention(H, D, R, V, K, dtype):
    """Every path over one sequence: all rows on their own, prompt runs that start in the middle, and both in one batch. One
    far key stands out for some queries through its rotated part."""
    T, bs, eps = 170, 16, 1e-5
    rot, spec = RotarySpec(R, 5000.0, interleaved=True), {"dims": R, "base": 5000.0}
    m = LatentAttentionSpec(H, D, R, V, K, (D + R) ** -0.5, rot, gate=True)
    lay = latent_layout(m)
    q, d, gate = rnd(T, H, D + R, seed=1, dtype=dtype), rnd(T, K + R, seed=2, dtype=dtype), rnd(T, H, seed=7, scale=2.0, dtype=dtype)
    uk, uv = rnd(H * D, K, seed=3, scale=K ** -0.5, dtype=dtype), rnd(H * V, K, seed=4, scale=K ** -0.5, dtype=dtype)
    nw = 1 + 0.3 * rnd(K, seed=5)
    turn = parallel_stack.rotate_pairs
    for i, j in ((169, 0), (150, 15), (140, 16), (100, 2)):
        at = lambda x, p: torch.cat([torch.zeros(p, 1, R, dtype=torch.float64), x.double().view(1, 1, R)])
        target = turn(at(q[i, 0, D:], i), spec)[i]              # what the rotated key should be: turn it back by the key's position
        flip = torch.tensor([1.0, -1.0], dtype=torch.float64).repeat(R // 2)
        back = turn(at(target[0] * flip, j), spec)[j, 0] * flip
        d[j, K:] = (5 * back).to(dtype)
    dd = d.double()
    c = oracle.rms(dd[:, :K], eps) * nw
    key = torch.cat([(c @ uk.double().T).view(T, H, D), turn(dd[:, None, K:], spec).expand(T, H, R)], -1)
    qq = torch.cat([q[..., :D].double(), turn(q[..., D:].double(), spec)], -1)
    want = attend(qq, key, (c @ uv.double().T).view(T, H, V), m.scale, None) * oracle.sigmoid(gate.double())[..., None]
    hp = (H + 7) // 8 * 8
    y = torch.zeros(T, H * lay.qd + lay.kd + hp, dtype=dtype)
    yq = y[:, :H * lay.qd].view(T, H, lay.qd)
    yq[..., :D], yq[..., lay.dimp:lay.dimp + R] = q[..., :D], q[..., D:]
    y[:, H * lay.qd:H * lay.qd + K], y[:, H * lay.qd + lay.rankp:H * lay.qd + lay.rankp + R] = d[:, :K], d[:, K:]
    y[:, H * lay.qd + lay.kd:H * lay.qd + lay.kd + H] = gate
    up = lambda w, n, p: torch.nn.functional.pad(w.view(H, n, K), (0, lay.rankp - K, 0, p - n)).to(DEV)
    wk, wv = up(uk, D, lay.dimp), up(uv, V, lay.vdimp)
    blocks = torch.randperm(11, generator=torch.Generator().manual_seed(2)).to(torch.int32)
    cache = torch.zeros(11, bs, lay.row, dtype=dtype, device=DEV)
    bt, table = blocks[None].to(DEV), F.rope_freq_table(rot, 256, DEV)
    for cuts in ([T], [1] * 3 + [T - 3], [130, 2, 38], [20, 150]):
        at = 0
        cache.zero_()
        for n in cuts:
            pos = torch.arange(at, at + n)
            rows, ctx = torch.zeros(n, dtype=torch.int32), (pos + 1).int()
            slots = (blocks[pos // bs].long() * bs + pos % bs).to(DEV)
            t = LatentTables.prefill(m, rows, pos, torch.device(DEV), dtype)
            g = y[at:at + n].to(DEV)
            gc = g[:, H * lay.qd + lay.kd:H * lay.qd + lay.kd + H]
            xq, qa = F.latent_prep(g, pos.int().to(DEV), slots, cache, lay, table, nw.to(DEV), eps, t.loose, t.n_loose, True, gc, t.recs)
            out = torch.full((n + 1, H * lay.vdimp), 7.0, dtype=dtype, device=DEV)
            base = torch.tensor([out.data_ptr()], dtype=torch.int64, device=DEV)
            if t.n_loose:
                gemm.grouped_linear(xq.view(-1, lay.dimp), wk.transpose(1, 2).contiguous(), t.offs, out=qa.view(-1, lay.row)[:, :lay.rankp])
                o = F.latent_attention(qa, cache, bt, rows.to(DEV), ctx.to(DEV), t.rows, lay, m.scale)
                gemm.grouped_combine(o.view(-1, lay.rankp), wv, t.offs, t.recs, base, lay.vdimp)
            if t.n_tiles:
                lat = F.latent_gather(cache, bt, t.keys, t.n_keys)
                kv = gemm.linear(lat[:, :lay.rankp], torch.cat([wk, wv], 1).reshape(-1, lay.rankp))
                F.latent_prefill(g, kv, lat, t.tiles, t.base, t.n_tiles, lay, m.scale, None, None, out, gc)
            assert bool((out[-1] == 7.0).all())
            full = want.clone()                                # the errors are relative to the whole sequence's size
            full[at:at + n] = out[:n].view(n, H, lay.vdimp)[..., :V].double().cpu()
            heads_close(full, want, tol(dtype, 1e-4, 6e-2))
            at += n
    assert gemm.check_status(DEV) == 0


# ---- router -------------------------------------------------------------------------------------------------------------
ROUTERS = [(8, 3, 2, 1), (16, 3, 4, 2), (64, 6, 8, 3), (256, 8, 8, 4), (5, 5, 1, 1), (6, 2, 6, 3), (9, 3, 3, 2), (1, 1, 1, 1), (64, 4, 64, 9)]


@BOTH
@pytest.mark.parametrize("n", [1, 33, 200, 700])
@pytest.mark.parametrize("E,K,groups,keep", ROUTERS)
def test_grouped_sigmoid_router(E, K, groups, keep, n, dtype):
    W = 64
    x, w, gate = rnd(n, W, seed=1), 1 + 0.3 * rnd(W, seed=2), rnd(E, W, seed=3, scale=0.4, dtype=dtype)
    corr = rnd(E, seed=4, scale=0.8) - 0.7                       # many choice scores below zero
    counts = torch.zeros(E, dtype=torch.int32, device=DEV)
    r = F.Router(gate.to(DEV), K, True, counts, True, corr.to(DEV), groups, keep, 1.7)
    h, ids, wts = F.sum_norm(x.to(DEV), None, None, w.to(DEV), 1e-6, dtype, False, router=r)
    spec = {"top": K, "scale": 1.7, "groups": {"count": groups, "keep": keep}}
    want, s = oracle.route(h.double().cpu(), gate.double(), corr.double(), spec)
    same = (ids.cpu().long() == want).all(-1)
    assert float(same.float().mean()) > 0.98 or int((~same).sum()) <= 1      # close calls may go the other way
    close(wts.cpu()[same], s[same], 1e-4)
    assert all(len(set(i)) == K for i in ids.tolist())
    assert len({tuple(sorted({e // (E // groups) for e in i})) for i in ids.tolist()}) >= (1 if groups == keep or n == 1 else 2)
    assert torch.equal(counts.cpu(), torch.bincount(ids.reshape(-1).cpu(), minlength=E).int())


@BOTH
def test_router_takes_the_groups_literally(dtype):
    """One hidden dimension per expert, so that scores are set by hand: the group of the single best expert loses against the
    group with the two best sum; equal sums go to the lower group, negative choice scores stay eligible."""
    E, W = 8, 8
    logits = torch.tensor([[4.0, -6, -6, -6, 2, 2, -6, -6], [1, 1, 0, 0, 1, 1, 0, 0], [-3, -3, -9, -9, -4, -4, -9, -9]])
    x = logits                                                  # norm(x) * w = x below
    w = torch.ones(W)
    scale = torch.sqrt((x * x).mean(-1, keepdim=True) + 1e-6)
    gate = torch.eye(E, dtype=dtype)
    r = F.Router(gate.to(DEV), 2, True, None, True, torch.full((E,), -2.0, device=DEV), 2, 1, 1.0)
    _, ids, wts = F.sum_norm(x.to(DEV), None, None, w.to(DEV), 1e-6, dtype, False, router=r)
    want, s = oracle.route(x.double() / scale.double(), gate.double(), torch.full((E,), -2.0).double(),
                           {"top": 2, "scale": 1.0, "groups": {"count": 2, "keep": 1}})
    assert [set(i) for i in ids.tolist()] == [set(i) for i in want.tolist()] and ids.tolist()[0] == [4, 5] and ids.tolist()[1] == [0, 1]
    close(wts, s, 1e-2)


@BOTH
@pytest.mark.parametrize("T,W,E,K,ff,groups,keep", [(1, 64, 4, 2, 64, 2, 1), (70, 128, 8, 3, 40, 2, 2), (33, 44, 6, 3, 13, 3, 2), (300, 256, 16, 4, 128, 4, 2)])
def test_experts(T, W, E, K, ff, groups, keep, dtype):
    sd = {f"m.e{e}.{n}": rnd(*s, seed=10 * e + i, scale=s[1] ** -0.5, dtype=dtype)
          for e in range(E) for i, (n, s) in enumerate((("gate", (ff, W)), ("up", (ff, W)), ("down", (W, ff))))}
    sd["m.router"], sd["m.correction"] = rnd(E, W, seed=999, dtype=dtype), rnd(E, seed=998, scale=0.4, dtype=dtype)
    spec = RoutedSpec(E, K, ff, renormalize=True, scoring="sigmoid", correction=True, groups=groups, keep=keep, scale=1.4)
    ffn, buf = RoutedFeedForward(sd, "m.", spec, torch.device(DEV), dtype), RoutedBuffers(T, W, E, K, DEV, dtype)
    x, w = rnd(T, W, seed=5), torch.ones(W)
    for _ in range(2):                            # the histogram is left clean
        h, ids, wts = F.sum_norm(x.to(DEV), None, None, w.to(DEV), 1e-5, dtype, False, router=ffn.router(buf))
        got = ffn(h, ids, wts, buf).float().sum(1)
        want = oracle.experts(h.double().cpu(), {n: t.double() for n, t in sd.items()}, "m.",
                              {"router": {"experts": E, "top": K, "scale": 1.4, "groups": {"count": groups, "keep": keep}}})
        close(got, want, tol(dtype, 2e-5, 0.1))
    assert gemm.check_status(DEV) == 0
