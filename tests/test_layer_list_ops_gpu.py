"""Kernels of the layer-list decoders, one mechanism at a time, against the oracle's functions."""
import pytest
import torch

from disagmoe_b200.config import RotarySpec
from disagmoe_b200.ops import functional as F
from disagmoe_b200.ops import gemm
from disagmoe_b200.ops.recurrent import Recurrence, build_segments, decode_segments, recurrent_attention
from oracles import layer_stack as oracle

pytestmark = pytest.mark.gpu
DEV = "cuda"
BOTH = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])


def rnd(*shape, seed=0, scale=1.0, dtype=torch.float32):
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale).to(dtype)


def close(got, want, tol):
    want = want.double().cpu()
    err = (got.double().cpu() - want).abs().max() / want.pow(2).mean().sqrt()
    assert float(err) < tol, f"max error {float(err):.3g} of the rms"


def tol(dtype, f32=2e-5, bf16=3e-2):
    return f32 if dtype == torch.float32 else bf16


@BOTH
@pytest.mark.parametrize("W", [96, 100, 2048, 8192, 5])
def test_resid_norm(W, dtype):
    x, y = rnd(9, W, seed=1, scale=3.0), rnd(9, W, seed=2, dtype=dtype)
    post, pre = 1 + 0.3 * rnd(W, seed=3), 1 + 0.3 * rnd(W, seed=4)
    new = x.double() + oracle.rms(y.double(), 1e-5) * post
    h = oracle.rms(new, 1e-5) * pre * 0.3
    rows = torch.tensor([8, 0, 3], dtype=torch.int32)
    g = x.to(DEV)
    got = F.resid_norm(g, y.to(DEV), post.to(DEV), pre.to(DEV), 1e-5, dtype, 0.3, rows.to(DEV))
    close(got, h[rows.long()], tol(dtype, 1e-5))
    assert torch.equal(g.cpu(), x)
    got = F.resid_norm(g, y.to(DEV), post.to(DEV), pre.to(DEV), 1e-5, dtype, 0.3)
    close(got, h, tol(dtype, 1e-5))
    close(g, new, 1e-5)
    close(F.resid_norm(g, None, None, pre.to(DEV), 1e-5, dtype), oracle.rms(new, 1e-5) * pre, tol(dtype, 1e-5))


@BOTH
def test_scaled_embedding(dtype):
    t, ids = rnd(50, 37, dtype=dtype), torch.tensor([49, 0, 7, 7], dtype=torch.int32)
    out = torch.empty(4, 37, device=DEV)
    F.embed_f32(ids.to(DEV), t.to(DEV), 11.5, out)
    close(out, t.double()[ids.long()] * 11.5, 1e-6)


@BOTH
@pytest.mark.parametrize("T,F_,K", [(1, 7, 5), (70, 130, 33), (129, 64, 256)])
def test_linear_of_any_alignment(T, F_, K, dtype):
    x, w = rnd(T, K, seed=1, dtype=dtype), rnd(F_, K, seed=2, dtype=dtype)
    close(gemm.linear(x.to(DEV), w.to(DEV), out_dtype=torch.float32), x.double() @ w.double().T, 1e-5)
    gu = x.double() @ rnd(2 * F_, K, seed=3, dtype=dtype).double().T
    got = gemm.swiglu_linear(x.to(DEV), rnd(2 * F_, K, seed=3, dtype=dtype).to(DEV))
    close(got, oracle.silu(gu[:, :F_]) * gu[:, F_:], tol(dtype, 1e-5, 0.08))


@BOTH
@pytest.mark.parametrize("n_q,n_kv,dk,dv,rot", [(4, 2, 64, 64, RotarySpec(64, 1e4, 4.0, 100)), (3, 1, 10, 14, RotarySpec(6, 300.0)),
                                               (2, 0, 20, 20, RotarySpec(20, 50.0)), (5, 5, 128, 96, None)])
def test_qk_norm_and_rotation(n_q, n_kv, dk, dv, rot, dtype):
    T, bs, blocks = 40, 16, 6
    row = rnd(T, n_q * dk + n_kv * (dk + dv), seed=5, dtype=dtype)
    qw, kw = 1 + 0.3 * rnd(dk, seed=6), 1 + 0.3 * rnd(dk, seed=7)
    slots = torch.randperm(bs * blocks, generator=torch.Generator().manual_seed(1))[:T]
    slots[11] = -1
    kc, vc = (torch.zeros(blocks, bs, max(n_kv, 1), d, dtype=dtype, device=DEV) for d in (dk, dv))
    table = F.rope_freq_table(rot, 64, DEV)
    g = row.to(DEV)
    F.qk_norm_rope(g, torch.arange(T, dtype=torch.int32, device=DEV), slots.to(DEV), kc, vc, n_q, n_kv, dk, dv, table,
                   qw.to(DEV), kw.to(DEV), 1e-5)
    spec = rot and {"dims": rot.dims, "base": rot.base, "scaling": rot.factor and
                    {"factor": rot.factor, "original": rot.original, "fast": rot.fast, "slow": rot.slow}}
    turn = lambda x, w: oracle.rotate(oracle.rms(x, 1e-5) * w.double(), spec)
    d = row.double()
    close(g[:, :n_q * dk], turn(d[:, :n_q * dk].view(T, n_q, dk), qw).reshape(T, -1), tol(dtype))
    if n_kv:
        k = turn(d[:, n_q * dk:(n_q + n_kv) * dk].view(T, n_kv, dk), kw)
        ok = slots >= 0
        close(kc.view(-1, n_kv, dk)[slots[ok].to(DEV)], k[ok], tol(dtype))
        close(vc.view(-1, n_kv, dv)[slots[ok].to(DEV)], d[ok][:, (n_q + n_kv) * dk:].reshape(-1, n_kv, dv), 1e-6)
        used = torch.zeros(bs * blocks, dtype=torch.bool)
        used[slots[ok]] = True
        assert not kc.view(-1, n_kv, dk)[(~used).to(DEV)].any()


def test_rotation_angles_far_out():
    spec = RotarySpec(64, 1e4)
    t = F.rope_freq_table(spec, 100_000, DEV)[99_999].double().cpu()
    a = 99_999 * oracle.inverse_frequencies({"dims": 64, "base": 1e4})[0]
    assert float((t - torch.stack([a.cos(), a.sin()], -1)).abs().max()) < 1e-7


def _planted(T, H, G, D, V, window, dtype):
    """q, k, v of one sequence where the keys just inside and just outside the reach of some queries would take nearly all
    the weight if they were seen."""
    q, k, v = rnd(T, H, D, seed=1, dtype=dtype), rnd(T, G, D, seed=2, dtype=dtype), rnd(T, G, V, seed=3, dtype=dtype)
    for n, i in enumerate(range(window, T, 5)):
        j = i - window + (1 if n % 2 else 0)      # outside, inside, outside, ...
        k[j] = (3 * q[i].view(G, H // G, D)[:, 0].float()).to(dtype)
    return q, k, v


SHAPES = [(4, 2, 64, 64), (8, 1, 128, 128), (2, 2, 64, 64), (4, 1, 128, 128), (6, 2, 20, 12), (3, 3, 64, 64), (2, 1, 80, 80)]


@BOTH
@pytest.mark.parametrize("softcap", [None, 5.0, 50.0])
@pytest.mark.parametrize("H,G,D,V", SHAPES)
@pytest.mark.parametrize("window", [1, 16, 37, 64, 100, 1000])
def test_windowed_attention(window, H, G, D, V, softcap, dtype):
    T, bs = 150, 16
    q, k, v = _planted(T, H, G, D, V, window, dtype)
    want = oracle_attention(q, k, v, D ** -0.5, softcap, window)
    blocks = torch.randperm(10, generator=torch.Generator().manual_seed(2)).to(torch.int32)
    kc, vc = torch.zeros(10, bs, G, D, dtype=dtype), torch.zeros(10, bs, G, V, dtype=dtype)
    for t in range(T):
        kc[blocks[t // bs], t % bs], vc[blocks[t // bs], t % bs] = k[t], v[t]
    kc, vc, qd, bt = kc.to(DEV), vc.to(DEV), q.reshape(T, H * D).to(DEV), blocks[None].to(DEV)
    rows, ctx = torch.zeros(T, dtype=torch.int32), torch.arange(1, T + 1, dtype=torch.int32)
    opt = dict(window=window, softcap=softcap, fp32_weights=True)
    for splits in (1, 3):
        got = F.paged_attention(qd, kc, vc, bt, rows.to(DEV), ctx.to(DEV), H, G, D, splits=splits, **opt)
        close(got, want, tol(dtype, 1e-4, 4e-2))
    if not F.attention_on_tensor_cores(dtype, H, G, D, V):
        return
    for start in (0, 1, 63, 70):      # whole prompt, and portions that continue one
        tiles, _ = F.build_prefill_tiles(rows[start:], ctx[start:] - 1, F.prefill_tile_tokens(H, G))
        out = torch.zeros(T - start, H * V, dtype=dtype, device=DEV)
        F.prefill_attention(qd[start:], kc, vc, bt, tiles.to(DEV), len(tiles), H, G, D, out, **opt)
        close(out, want[start:], tol(dtype, 1e-4, 4e-2))


def oracle_attention(q, k, v, scale, softcap, window):
    """Vectorised form of oracle.softmax_attention (checked against it on one head)."""
    T, H, D = q.shape
    g = H // k.shape[1]
    k, v, q = k.double().repeat_interleave(g, 1), v.double().repeat_interleave(g, 1), q.double()
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    if softcap:
        s = softcap * torch.tanh(s / softcap)
    d = torch.arange(T)[:, None] - torch.arange(T)[None]
    p = torch.softmax(s.masked_fill((d < 0) | (d >= window), float("-inf")), -1)
    out = torch.einsum("hij,jhd->ihd", p, v)
    one = oracle.softmax_attention(q[:, :1], k[:, :1], v[:, :1], scale, softcap, window)
    assert float((out[:, :1] - one).abs().max()) < 1e-9
    return out.reshape(T, -1)


# ---- recurrences ------------------------------------------------------------------------------------------------------
class Recur:
    """Random inputs of one sequence for one recurrent layer, and the oracle's output [T, H V]."""

    def __init__(self, kind, H, G, D, V, taps, T, dtype, seed=0, decay=1.0):
        r = lambda *s, k=0, scale=1.0: rnd(*s, seed=seed * 100 + k, scale=scale)
        self.kind, self.dtype, self.T = kind, dtype, T
        lin = lambda n, k: r(T, n, k=k).to(dtype)
        self.q, self.k, self.v = lin(G * D, 1), lin(G * D, 2), lin(H * V, 3)
        self.gate, self.beta, self.z = lin(H * V, 4), lin(H, 5), r(T, H * D, k=6)
        zb, nw = r(H * D, k=7) * decay, 1 + 0.3 * r(V, k=8)
        alog = 0.5 * r(H, k=9) + (decay - 1)
        conv = r(2 * G * D + H * V, taps, k=10, scale=taps ** -0.5) if taps else None
        dv = lambda t: None if t is None else t.to(DEV).contiguous()
        self.r = Recurrence(H, G, D, V, kind == "delta", dv(zb), dv(nw), 1e-5, a_log=dv(alog) if kind == "delta" else None,
                            tau=3.0 / decay, conv_w=dv(conv), sigmoid_gate=kind == "delta")
        d = lambda t: t.double()
        q, k, v = d(self.q), d(self.k), d(self.v)
        if taps:
            c = [(0, G * D, q), (G * D, 2 * G * D, k), (2 * G * D, 2 * G * D + H * V, v)]
            q, k, v = (oracle.silu(oracle.short_conv(x, d(conv[a:b]))).to(dtype).double() for a, b, x in c)
        q, k, v = (x.view(T, n, m) for x, n, m in ((q, G, D), (k, G, D), (v, H, V)))
        z = (d(self.z) + d(zb)).view(T, H, D)
        if kind == "delta":
            unit = lambda x: (x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)).repeat_interleave(H // G, 1)
            o, S = oracle.delta_recurrence(unit(q) * D ** -0.5, unit(k), v, -torch.exp(d(alog))[:, None] * oracle.softplus(z),
                                           oracle.sigmoid(d(self.beta)), with_state=True)
            g = oracle.sigmoid(d(self.gate))
        else:
            o, S = oracle.gla_recurrence(q * D ** -0.5, k, v, oracle.log_sigmoid(z) / self.r.tau, with_state=True)
            g = oracle.silu(d(self.gate))
        self.state = S
        self.want = ((oracle.rms(o, 1e-5) * d(nw)).reshape(T, -1) * g)

    def rows(self, a, b):
        cut = lambda t: t[a:b]
        return [cut(t) for t in (self.q, self.k, self.v, self.gate, self.beta, self.z)]


def run_steps(seqs, schedule, n_slots, slots, implicit=False, state=None):
    """``schedule``: steps of (sequence, tokens); returns each sequence's outputs. Sequence i lives in slot slots[i]."""
    r0 = seqs[0]
    state = state or r0.r.new_state(n_slots, r0.dtype, DEV)
    for t in state.tensors():
        t.fill_(7.0)                        # a slot that was used before
    at, out = [0] * len(seqs), [[] for _ in seqs]
    for step in schedule:
        parts = [seqs[i].rows(at[i], at[i] + n) for i, n in step]
        # columns of one wider matrix, as the fused projection hands them over
        q, k, v, gate, beta, z = (torch.cat(c).to(DEV) for c in zip(*parts))
        pad = lambda t: torch.nn.functional.pad(t, (8, 8))[:, 8:8 + t.shape[1]]
        pos = torch.cat([torch.arange(at[i], at[i] + n) for i, n in step]).int()
        row = torch.cat([torch.full((n,), slots[i]) for i, n in step]).int()
        if implicit:
            segs = decode_segments(pos.to(DEV), row.to(DEV), torch.zeros(len(pos), dtype=torch.int64, device=DEV))
        else:
            segs = build_segments(row, pos, DEV)
        y = recurrent_attention(r0.r, pad(q), pad(k), pad(v), pad(gate), pad(beta) if r0.kind == "delta" else None, pad(z),
                                state, segs).cpu()
        o = 0
        for i, n in step:
            out[i].append(y[o:o + n])
            o, at[i] = o + n, at[i] + n
    return [torch.cat(x) if x else None for x in out]


HEADS = [("gla", 3, 3, 48, 32, 0), ("gla", 2, 2, 128, 128, 0), ("gla", 2, 2, 6, 9, 0), ("gla", 1, 1, 64, 256, 0),
         ("gla", 2, 2, 256, 64, 0), ("delta", 4, 2, 32, 64, 4), ("delta", 2, 2, 128, 128, 4), ("delta", 3, 1, 20, 7, 2),
         ("delta", 2, 1, 16, 16, 1), ("delta", 2, 2, 64, 128, 8)]


@BOTH
@pytest.mark.parametrize("kind,H,G,D,V,taps", HEADS)
def test_recurrence_cuts(kind, H, G, D, V, taps, dtype):
    s = Recur(kind, H, G, D, V, taps, 150, dtype)
    for cuts in ([150], [64, 64, 22], [2] * 20 + [3, 61, 1, 1, 44], [63, 1, 1, 65, 20], [1] * 12 + [2, 136]):
        assert sum(cuts) == 150
        got, = run_steps([s], [[(0, n)] for n in cuts], 3, [1])
        close(got, s.want, tol(dtype, 2e-4, 6e-2))


@BOTH
@pytest.mark.parametrize("kind,H,G,D,V,taps", [h for h in HEADS if h[5] == 0] + [("delta", 4, 2, 32, 64, 0), ("delta", 2, 2, 128, 128, 0),
                                              ("delta", 1, 1, 96, 40, 0), ("delta", 2, 2, 8, 8, 0)])
@pytest.mark.parametrize("decay", [0.05, 1.0, 20.0])
def test_state_is_fp32(kind, H, G, D, V, taps, decay, dtype):
    """The state after prompts, portions and single tokens, with inputs that are exact in both formats: fp32 accuracy also
    where the activations are bf16."""
    s = Recur(kind, H, G, D, V, taps, 200, dtype, seed=5, decay=decay)
    for cuts in ([200], [129, 1, 70], [1] * 30 + [100, 2, 68]):
        state = s.r.new_state(2, dtype, DEV)
        run_steps([s], [[(0, n)] for n in cuts], 2, [1], state=state)
        close(state.S[1], s.state, 3e-4)


@pytest.mark.parametrize("kind,H,G,D,V,taps", HEADS)
def test_recurrence_mixed_batch(kind, H, G, D, V, taps):
    dtype = torch.bfloat16
    seqs = [Recur(kind, H, G, D, V, taps, n, dtype, seed=2) for n in (100, 40, 7)]
    for s in seqs[1:]:
        s.r = seqs[0].r                     # same weights: same seed
    steps = [[(0, 30), (1, 1)], [(1, 2), (2, 1), (0, 1)], [(0, 1), (1, 30), (2, 1)], [(0, 66), (2, 5)], [(1, 1)],
             [(0, 1), (1, 6)], [(0, 1)]]
    for got, s in zip(run_steps(seqs, steps, 5, [4, 0, 2]), seqs):
        close(got, s.want, 6e-2)


@BOTH
@pytest.mark.parametrize("kind,H,G,D,V,taps", HEADS)
def test_recurrence_decode_only(kind, H, G, D, V, taps, dtype):
    """Long decoding of several sequences through the path that CUDA graphs capture; one joins late in a used slot."""
    seqs = [Recur(kind, H, G, D, V, taps, n, dtype, seed=3) for n in (70, 70, 30)]
    for s in seqs[1:]:
        s.r = seqs[0].r
    steps = [[(0, 1), (1, 1)]] * 40 + [[(1, 1), (2, 1), (0, 1)]] * 30
    for got, s in zip(run_steps(seqs, steps, 4, [2, 3, 0], implicit=True), seqs):
        close(got, s.want, tol(dtype, 2e-4, 6e-2))


@pytest.mark.parametrize("decay", [0.05, 4.0, 30.0])
@pytest.mark.parametrize("kind,H,G,D,V,taps", [("gla", 2, 2, 64, 64, 0), ("delta", 2, 2, 64, 64, 3)])
def test_recurrence_slow_and_fast_decays(kind, H, G, D, V, taps, decay):
    """States that hardly fade, and states that are wiped within a token or two: no overflow, no lost history."""
    s = Recur(kind, H, G, D, V, taps, 140, torch.bfloat16, seed=4, decay=decay)
    for cuts in ([140], [70, 1, 69]):
        got, = run_steps([s], [[(0, n)] for n in cuts], 1, [0])
        assert torch.isfinite(got).all()
        close(got, s.want, 8e-2)


def test_padding_rows_leave_the_state_alone():
    s = Recur("delta", 2, 1, 32, 32, 4, 4, torch.bfloat16)
    state = s.r.new_state(2, s.dtype, DEV)
    for t in state.tensors():
        t.fill_(0.5)
    args = [t.to(DEV) for t in s.rows(0, 4)]
    segs = decode_segments(torch.full((4,), 5, dtype=torch.int32, device=DEV), torch.zeros(4, dtype=torch.int32, device=DEV),
                           torch.full((4,), -1, dtype=torch.int64, device=DEV))
    recurrent_attention(s.r, *args, state, segs)
    assert all(bool((t == 0.5).all()) for t in state.tensors())
