"""Plain PyTorch restatements of every device op (any device, any float dtype; math in fp32).

They are the numerical reference of the CUDA kernels' tests, the building blocks of the fp32 CPU oracle model
and the CPU path of the ops in :mod:`disagmoe_b200.ops.functional`.
"""
from __future__ import annotations

import math
from typing import List, Optional, Tuple

import torch


def rmsnorm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    xf = x.float()
    inv = torch.rsqrt(xf.pow(2).mean(-1, keepdim=True) + eps)
    return (xf * inv * w.float()).to(x.dtype)


def add_rmsnorm(resid: Optional[torch.Tensor], adds: List[torch.Tensor], w: torch.Tensor, eps: float
                ) -> Tuple[torch.Tensor, torch.Tensor]:
    """new_resid = resid + sum(adds) (rounded to the storage dtype); y = rmsnorm(new_resid) * w."""
    acc = None if resid is None else resid.float()
    for a in adds:
        acc = a.float() if acc is None else acc + a.float()
    dtype = resid.dtype if resid is not None else adds[0].dtype
    new = acc.to(dtype)
    return new, rmsnorm(new, w, eps)


def rope_neox(x: torch.Tensor, positions: torch.Tensor, n_heads: int, hd: int, theta: float) -> torch.Tensor:
    """x [T, n_heads*hd]; rotates pairs (d, d + hd/2) by positions * theta^(-2d/hd)."""
    T = x.shape[0]
    xf = x.float().view(T, n_heads, hd)
    half = hd // 2
    inv_freq = theta ** (-torch.arange(0, half, device=x.device, dtype=torch.float32) * 2.0 / hd)
    ang = positions.float()[:, None] * inv_freq[None, :]
    c, s = ang.cos()[:, None, :], ang.sin()[:, None, :]
    a, b = xf[..., :half], xf[..., half:]
    out = torch.cat([a * c - b * s, b * c + a * s], dim=-1)
    return out.reshape(T, n_heads * hd).to(x.dtype)


def rope_kv_append(qkv: torch.Tensor, positions: torch.Tensor, slots: Optional[torch.Tensor], kcache: torch.Tensor,
                   vcache: torch.Tensor, n_q: int, n_kv: int, hd: int, theta: float) -> None:
    """In place: RoPE on q and k heads of qkv rows [q | k | v]; append k, v at flat slot ids of the paged cache
    (cache shape [num_blocks, block_size, n_kv, hd])."""
    qd, kd = n_q * hd, n_kv * hd
    qkv[:, :qd] = rope_neox(qkv[:, :qd], positions, n_q, hd, theta)
    qkv[:, qd:qd + kd] = rope_neox(qkv[:, qd:qd + kd], positions, n_kv, hd, theta)
    if slots is not None:
        ok = slots >= 0
        kflat = kcache.view(-1, n_kv * hd)
        vflat = vcache.view(-1, n_kv * hd)
        kflat[slots[ok]] = qkv[ok, qd:qd + kd].to(kcache.dtype)
        vflat[slots[ok]] = qkv[ok, qd + kd:qd + 2 * kd].to(vcache.dtype)


def paged_attention(q: torch.Tensor, kcache: torch.Tensor, vcache: torch.Tensor, block_tables: torch.Tensor,
                    bt_row: Optional[torch.Tensor], ctx_len: torch.Tensor, n_q: int, n_kv: int, hd: int,
                    scale: Optional[float] = None, window: Optional[int] = None, softcap: Optional[float] = None,
                    sink: Optional[torch.Tensor] = None, chunk: Optional[int] = None, q_temp=None,
                    gate: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Token t attends to the first ctx_len[t] cached tokens of block-table row bt_row[t] (default t), or to the last
    ``window`` of them, or to those in the same ``chunk`` of positions as the last one; ``softcap``: scores become cap * tanh(score / cap); ``sink`` [n_q]: the softmax denominator has
    exp(sink) in addition; ``q_temp`` (coef, every): scores times the query temperature of position ctx_len - 1; ``gate`` [T, n_q]:
    every head's output times sigmoid(gate)."""
    T = q.shape[0]
    block_size = kcache.shape[1]
    scale = scale if scale is not None else 1.0 / math.sqrt(hd)
    vd = vcache.shape[-1]
    out = torch.zeros(T, n_q * vd, dtype=torch.float32, device=q.device)
    gq = n_q // n_kv
    for t in range(T):
        L = int(ctx_len[t])
        if L == 0:
            continue
        row = int(bt_row[t]) if bt_row is not None else t
        nb = (L + block_size - 1) // block_size
        blocks = block_tables[row, :nb].long()
        k = kcache[blocks].reshape(nb * block_size, n_kv, hd)[:L].float()
        v = vcache[blocks].reshape(nb * block_size, n_kv, vd)[:L].float()
        if window:
            k, v = k[-window:], v[-window:]
        if chunk:
            n = (L - 1) % chunk + 1
            k, v = k[-n:], v[-n:]
        qt = q[t].float().view(n_kv, gq, hd)
        s = torch.einsum("kgd,lkd->kgl", qt, k) * scale
        if q_temp is not None:
            s = s * (1.0 + q_temp.coef * math.log(L // q_temp.every + 1))
        if softcap:
            s = softcap * torch.tanh(s / softcap)
        if sink is not None:
            s = torch.cat([s, sink.view(n_kv, gq, 1).to(s.dtype)], -1)
        p = torch.softmax(s, dim=-1)[..., :k.shape[0]]
        o = torch.einsum("kgl,lkd->kgd", p, v)
        out[t] = o.reshape(-1)
    if gate is not None:
        out = (out.view(T, n_q, vd) * torch.sigmoid(gate.float())[..., None]).reshape(T, -1)
    return out.to(q.dtype)


def route(x: torch.Tensor, norm_w: Optional[torch.Tensor], eps: float, gate_w: torch.Tensor, top_k: int,
          renormalize: bool, logit_bias: Optional[torch.Tensor] = None
          ) -> Tuple[torch.Tensor, torch.Tensor, torch.Tensor, torch.Tensor]:
    """(y, topk_ids int32 [T,k], topk_w fp32 [T,k], logits fp32): y = rmsnorm(x) (or x), softmax -> top-k."""
    y = rmsnorm(x, norm_w, eps) if norm_w is not None else x
    logits = y.float() @ gate_w.float().T
    if logit_bias is not None:
        logits = logits + logit_bias.float().to(logits.device)
    probs = torch.softmax(logits, dim=-1)
    w, ids = torch.topk(probs, top_k, dim=-1)
    if renormalize:
        w = w / w.sum(-1, keepdim=True)
    return y, ids.int(), w.float(), logits


def sigmoid_route(h: torch.Tensor, r) -> Tuple[torch.Tensor, torch.Tensor]:
    """(ids int32 [T, top], weights fp32 [T, top]) of a sigmoid :class:`disagmoe_b200.ops.functional.Router`."""
    s = torch.sigmoid(h.float() @ r.weight.float().T)
    choice = s if r.correction is None else s + r.correction
    T, E = s.shape
    if r.keep < r.groups:
        grouped = choice.view(T, r.groups, E // r.groups)
        rank = grouped.topk(min(2, E // r.groups), dim=-1).values.sum(-1)
        open_ = torch.zeros_like(rank, dtype=torch.bool).scatter_(1, rank.topk(r.keep, dim=-1).indices, True)
        choice = grouped.masked_fill(~open_[..., None], float("-inf")).reshape(T, E)
    ids = choice.topk(r.top, dim=-1).indices
    w = s.gather(1, ids)
    if r.renormalize:
        w = w / (w.sum(-1, keepdim=True) + 1e-20)
    return ids.int(), w * r.scale


def expert_offsets(topk_ids: torch.Tensor, num_experts: int) -> torch.Tensor:
    counts = torch.bincount(topk_ids.reshape(-1).long(), minlength=num_experts)
    offs = torch.zeros(num_experts + 1, dtype=torch.int32, device=topk_ids.device)
    offs[1:] = counts.cumsum(0).int()
    return offs


def sort_by_expert(topk_ids: torch.Tensor) -> torch.Tensor:
    """Stable counting sort of the flattened (token-major) [T*k] expert ids; returns dst position of every pair."""
    flat = topk_ids.reshape(-1).long()
    order = torch.sort(flat, stable=True).indices
    pos = torch.empty_like(order)
    pos[order] = torch.arange(flat.numel(), device=flat.device)
    return pos.int()


def swiglu(h: torch.Tensor, act: str = "silu", limit: float = 0.0) -> torch.Tensor:
    I = h.shape[-1] // 2
    g = h[..., :I].float()
    if act == "clamped":
        g = g.clamp(max=limit)
        return g * torch.sigmoid(1.702 * g) * (h[..., I:].float().clamp(-limit, limit) + 1.0)
    g = torch.nn.functional.silu(g) if act == "silu" else torch.nn.functional.gelu(g, approximate="tanh")
    return g * h[..., I:].float()


def moe_experts(y: torch.Tensor, topk_ids: torch.Tensor, topk_w: torch.Tensor, w13: torch.Tensor, w2: torch.Tensor
                ) -> torch.Tensor:
    """Weighted sum over the top-k experts; w13 [E, 2I, H] (gate rows then up rows), w2 [E, H, I]. fp32 result."""
    T, H = y.shape
    out = torch.zeros(T, H, dtype=torch.float32, device=y.device)
    E = w13.shape[0]
    yf = y.float()
    for e in range(E):
        tok, slot = (topk_ids == e).nonzero(as_tuple=True)
        if tok.numel() == 0:
            continue
        h = swiglu(yf[tok] @ w13[e].float().T).to(y.dtype).float()
        o = (h @ w2[e].float().T).to(y.dtype).float()
        out.index_add_(0, tok, o * topk_w[tok, slot][:, None].float())
    return out


def permute_rows(src: torch.Tensor, mapping: torch.Tensor, repeat: int = 1, gather: bool = False,
                 n_out: Optional[int] = None) -> torch.Tensor:
    n = mapping.numel()
    m = mapping.long()
    if gather:
        out = torch.zeros(n, src.shape[1], dtype=src.dtype, device=src.device)
        ok = m >= 0
        out[ok] = src[m[ok]]
        return out
    out = torch.zeros(n_out if n_out is not None else n, src.shape[1], dtype=src.dtype, device=src.device)
    idx = torch.arange(n, device=src.device) // repeat
    ok = m >= 0
    out[m[ok]] = src[idx[ok]]
    return out


# ---- decoders with an fp32 residual stream ---------------------------------------------------------------------------
def _rms_scale(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def resid_norm(resid, y, post, pre, eps, dtype, out_scale=1.0, rows=None):
    """resid (+)= norm(y) * post; returns norm(resid) * pre * out_scale (of ``rows`` only, resid untouched)."""
    if rows is not None:
        resid, y = resid[rows.long()], (y[rows.long()] if y is not None else None)
    x = resid
    if y is not None:
        x = resid + _rms_scale(y.float(), eps) * post
        if rows is None:
            resid.copy_(x)
    return None if pre is None else (_rms_scale(x, eps) * pre * out_scale).to(dtype)


def sum_norm(resid, y, parts, w, eps, dtype, centred, rows=None, mult=1.0, bias=None, gate=None, sides=None):
    """resid += mult * (y + parts.sum(1)) (either may be None; ``rows``: only these rows are returned, resid untouched); returns the
    RMS norm of resid times w, or with ``centred`` its layer norm (mean taken off) times w, plus ``bias``. ``gate``: what is added is
    multiplied by sigmoid(gate.z + gate.bias) first. ``sides``: y is the scaled sum of two rows, each normed with its weight."""
    x = resid if rows is None else resid[rows.long()]
    pick = lambda a: a if rows is None else a[rows.long()]
    g = mult if gate is None else mult * torch.sigmoid(pick(gate.z).float() + gate.bias)
    if sides is not None:
        y = sides.scale * sum(_rms_scale(sides.rows[i].float(), eps) * sides.weights[i] for i in range(2))
    for a in (y, parts):
        if a is not None:
            a = pick(a)
            x = x + g * (a.float() if a.dim() == 2 else a.float().sum(1))
    if rows is None:
        resid.copy_(x)
    if centred:
        x = x - x.mean(-1, keepdim=True)
    h = _rms_scale(x, eps) * w
    return (h if bias is None else h + bias).to(dtype)


def _turn(x, table, positions, interleaved):
    """Rotation of the leading dimensions of x [T, heads, d] by (cos, sin) rows of ``table``."""
    if table is None:
        return x
    rot = 2 * table.shape[1]
    c, s = (table[positions.long()][:, None, :, j] for j in (0, 1))
    if interleaved:
        u, v = x[..., 0:rot:2], x[..., 1:rot:2]
        return torch.cat([torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2), x[..., rot:]], -1)
    u, v = x[..., :rot // 2], x[..., rot // 2:rot]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., rot:]], -1)


def qk_norm_rope(qkv, positions, slots, kcache, vcache, n_q, n_kv, dk, dv, table, qw, kw, eps, interleaved=False,
                 v_first=None, v_lambda=0.0, tied=False, v_norm=0) -> None:
    """Per-head norm (where weights are given) + partial rotation of q (in place) and k, K / V append at slots >= 0; with
    ``v_first`` [T, n_kv, >= dv] the values appended are (1 - v_lambda) v + v_lambda v_first, ``tied`` those of the raw keys,
    ``v_norm`` > 0: divided by their root mean square over that many dimensions."""
    T = qkv.shape[0]

    def turn(x, w):
        x = x.float() if w is None else _rms_scale(x.float(), eps) * w
        return _turn(x, table, positions, interleaved)

    qs, ks = n_q * dk, n_kv * dk
    q = turn(qkv[:, :qs].reshape(T, n_q, dk), qw).to(qkv.dtype)
    if n_kv:
        k = turn(qkv[:, qs:qs + ks].reshape(T, n_kv, dk), kw).to(qkv.dtype)
        ok = slots >= 0
        kcache.view(-1, n_kv, dk)[slots[ok]] = k[ok]
        v = qkv[ok][:, qs:qs + ks].reshape(-1, n_kv, dk)[..., :dv] if tied else \
            qkv[ok][:, qs + ks:qs + ks + n_kv * dv].reshape(-1, n_kv, dv)
        if v_first is not None:
            v = ((1.0 - v_lambda) * v.float() + v_lambda * v_first[ok][..., :dv].float()).to(v.dtype)
        if v_norm:
            v = (v.float() / torch.sqrt(v.float().pow(2).sum(-1, keepdim=True) / v_norm + eps)).to(v.dtype)
        vcache.view(-1, n_kv, dv)[slots[ok]] = v
    qkv[:, :qs] = q.reshape(T, qs).clone()


def latent_prep(y, positions, slots, cache, lay, table, norm_w, eps, loose, n_loose, interleaved, gate=None, recs=None):
    """See :func:`disagmoe_b200.ops.functional.latent_prep`."""
    T, H = y.shape[0], lay.heads
    q = y[:, :H * lay.qd].reshape(T, H, lay.qd)
    d = y[:, H * lay.qd:H * lay.qd + lay.kd]
    c = (_rms_scale(d[:, :lay.rank].float(), eps) * norm_w).to(y.dtype)
    kr = _turn(d[:, None, lay.rankp:lay.rankp + lay.rot].float(), table, positions, interleaved)[:, 0].to(y.dtype)
    ok = slots >= 0
    flat = cache.view(-1, lay.row)
    flat[slots[ok], :lay.rank] = c[ok]
    flat[slots[ok], lay.rankp:lay.rankp + lay.rot] = kr[ok]
    qr = _turn(q[..., lay.dimp:lay.dimp + lay.rot].float(), table, positions, interleaved).to(y.dtype)
    xq, qa = y.new_zeros(H, n_loose, lay.dimp), y.new_zeros(H, n_loose, lay.row)
    idx = torch.arange(T) if loose is None else loose.long()
    on = idx >= 0
    xq[:, idx[on]] = q[on][..., :lay.dimp].transpose(0, 1)
    qa[:, idx[on], lay.rankp:lay.rankp + lay.rot] = qr[on].transpose(0, 1)
    if gate is not None and n_loose:
        g = torch.zeros(H, n_loose)
        g[:, idx[on]] = torch.sigmoid(gate[on].float()).T
        recs[:, 2] = g.reshape(-1).view(torch.int32)
    y[:, :H * lay.qd] = torch.cat([q[..., :lay.dimp], qr, q[..., lay.dimp + lay.rot:]], -1).reshape(T, -1)
    return xq, qa


# ---- linear recurrences ----------------------------------------------------------------------------------------------
def conv_segment(x: torch.Tensor, w: torch.Tensor, ring: Optional[torch.Tensor], pos0: int) -> torch.Tensor:
    """Causal depthwise convolution + silu of one segment's rows x [n, C] that start at position pos0; ``ring`` [taps, C]
    holds earlier inputs at their position modulo taps and takes this segment's last ones."""
    n, taps = x.shape[0], w.shape[1]
    hist = [ring[(pos0 - j) % taps] if pos0 - j >= 0 else torch.zeros_like(x[0]) for j in range(taps - 1, 0, -1)]
    full = torch.cat([torch.stack(hist), x]) if hist else x
    acc = sum(full[j:j + n].float() * w[:, j] for j in range(taps))
    for j in range(max(0, n - taps + 1), n):
        ring[(pos0 + j) % taps] = x[j]
    return torch.nn.functional.silu(acc).to(x.dtype)


def seq_conv(x, w, ring, segs, in_bias, out_bias, residual):
    """See :func:`disagmoe_b200.ops.functional.seq_conv`: fp32 [T, C]."""
    taps, out = w.shape[0], torch.zeros(x.shape, dtype=torch.float32)
    add = 0.0 if in_bias is None else in_bias
    for a, n, slot, pos0 in segs.table():
        hist = [ring[slot, (pos0 - j) % taps].float() + add if pos0 - j >= 0 else torch.zeros(x.shape[1]) for j in range(taps - 1, 0, -1)]
        seg = x[a:a + n].float() + add
        full = torch.cat([torch.stack(hist), seg]) if hist else seg
        acc = sum(full[j:j + n] * w[j] for j in range(taps))
        if out_bias is not None:
            acc = acc + out_bias
        out[a:a + n] = seg + acc if residual else acc
        for j in range(max(0, n - taps + 1), n):
            ring[slot, (pos0 + j) % taps] = x[a + j]
    return out


def diagonal_segment(u, r, i, decay, state, pos0):
    """u, r, i [n, C] fp32, decay [C] (log decay of an open gate); ``state`` [C] is read (zero where pos0 = 0) and updated."""
    S = state.clone() if pos0 > 0 else torch.zeros_like(state)
    out = []
    for t in range(u.shape[0]):
        log_a = decay * r[t]
        S = torch.exp(log_a) * S + torch.sqrt(-torch.expm1(2.0 * log_a)) * (i[t] * u[t])
        out.append(S)
    state.copy_(S)
    return torch.stack(out)


def memory_segment(q, k, v, i, f, S, n, m, pos0, qscale):
    """q, k [T, H, D], v [T, H, V], i, f [T, H] logs of the gates; the state S [H, D, V], n [H, D] and the running maxima
    m [2, H] (at the position's parity) are read (zero where pos0 = 0) and updated. Returns fp32 read-outs [T, H, V]."""
    q, k, v = q.float() * qscale, k.float(), v.float()
    zero = pos0 == 0
    A, b, top = (torch.zeros_like(t) if zero else t.clone() for t in (S, n, m[(pos0 - 1) % 2]))
    out = []
    for t in range(q.shape[0]):
        new = torch.maximum(f[t] + top, i[t])
        keep, put = torch.exp(f[t] + top - new), torch.exp(i[t] - new)
        A = keep[:, None, None] * A + put[:, None, None] * k[t][..., None] * v[t][:, None, :]
        b = keep[:, None] * b + put[:, None] * k[t]
        top = new
        size = torch.maximum((b * q[t]).sum(-1).abs(), torch.exp(-top)) + 1e-6
        out.append(torch.einsum("hdv,hd->hv", A, q[t]) / size[:, None])
    S.copy_(A)
    n.copy_(b)
    m[(pos0 + q.shape[0] - 1) % 2] = top
    return torch.stack(out)


def token_shift(h: torch.Tensor, mu: torch.Tensor, last: torch.Tensor, segs) -> torch.Tensor:
    """See :func:`disagmoe_b200.ops.functional.token_shift`: fp32 [n, T, W]."""
    before = torch.zeros_like(h)
    for a, n, slot, pos0 in segs.table():
        before[a + 1:a + n] = h[a:a + n - 1]
        if pos0 > 0:
            before[a] = last[slot]
        last[slot] = h[a + n - 1]
    return h + (before - h) * mu[:, None]


def recur_segment(q, k, v, beta, logd, state: torch.Tensor, pos0: int, delta: bool, qscale: float, bonus=None) -> torch.Tensor:
    """Token-by-token recurrence of one segment: q, k, logd [n, H, D], v [n, H, V], beta [n, H] (delta); ``state``
    [H, D, V] is read (zero where pos0 = 0) and updated. ``bonus`` [H, D]: the read-out precedes decay and write, and the
    token's own write enters it with that weight. Returns fp32 read-outs [n, H, V]."""
    q, k, v = q.float(), k.float(), v.float()
    if delta:
        q = q / torch.sqrt(q.pow(2).sum(-1, keepdim=True) + 1e-6)
        k = k / torch.sqrt(k.pow(2).sum(-1, keepdim=True) + 1e-6)
    q = q * qscale
    S = state.clone() if pos0 > 0 else torch.zeros_like(state)
    out = []
    for t in range(q.shape[0]):
        if bonus is not None:
            kv = k[t][..., None] * v[t][:, None, :]
            out.append(torch.einsum("hdv,hd->hv", S + bonus[..., None] * kv, q[t]))
            S = S * torch.exp(logd[t])[..., None] + kv
            continue
        S = S * torch.exp(logd[t])[..., None]
        u = v[t]
        if delta:
            u = torch.sigmoid(beta[t].float())[:, None] * (u - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][..., None] * u[:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    state.copy_(S)
    return torch.stack(out)


def gate_norm(o: torch.Tensor, gate: torch.Tensor, norm_w: torch.Tensor, eps: float, sigmoid_gate: bool) -> torch.Tensor:
    """o [n, H, V] fp32 -> norm over V * norm_w * (sigmoid | silu)(gate)."""
    g = gate.float()
    return _rms_scale(o, eps) * norm_w * (torch.sigmoid(g) if sigmoid_gate else torch.nn.functional.silu(g))
