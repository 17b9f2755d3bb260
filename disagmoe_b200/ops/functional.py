"""Device ops of the decoder other than the GEMMs: CUDA tensors run the sm_100a kernels of
``csrc/kernels/{elementwise,attention,moe}.cu``; CPU tensors run the PyTorch restatements of
:mod:`disagmoe_b200.ops.reference` (fp32 CPU configuration, tests).
"""
from __future__ import annotations

import ctypes
import math
from dataclasses import dataclass
from typing import Optional, Tuple

import torch

from . import _lib, reference
from .gemm import scratch

c_ll = ctypes.c_longlong
c_int = ctypes.c_int
c_float = ctypes.c_float
c_vp = ctypes.c_void_p


def _vp(t):
    return c_vp(0 if t is None else t.data_ptr())


def _st():
    return c_vp(_lib.stream_ptr())


def add_rmsnorm(resid: Optional[torch.Tensor], add: Optional[torch.Tensor], w: torch.Tensor, eps: float,
                resid_out: Optional[torch.Tensor] = None, y: Optional[torch.Tensor] = None,
                want_resid: bool = True) -> Tuple[Optional[torch.Tensor], torch.Tensor]:
    """new_resid = resid + add.sum(1); y = rmsnorm(new_resid) * w.

    resid [T, H] or None; add None, [T, H] or [T, P, H] (P partial outputs per token, e.g. one per top-k slot).
    Returns (new_resid or None, y).
    """
    ref = resid if resid is not None else add
    T, H = ref.shape[0], ref.shape[-1]
    if add is not None and add.dim() == 2:
        add = add.unsqueeze(1)
    if not ref.is_cuda:
        adds = [] if add is None else [add[:, p] for p in range(add.shape[1])]
        new, yy = reference.add_rmsnorm(resid, adds, w, eps)
        if resid_out is not None:
            resid_out.copy_(new)
            new = resid_out
        if y is not None:
            y.copy_(yy)
            yy = y
        return (new if want_resid else None), yy
    if y is None:
        y = torch.empty(T, H, dtype=torch.bfloat16, device=ref.device)
    need_resid_out = want_resid and (add is not None)
    if need_resid_out and resid_out is None:
        resid_out = torch.empty(T, H, dtype=torch.bfloat16, device=ref.device)
    n_add = 0 if add is None else add.shape[1]
    _lib.check(_lib.lib().dmoe_add_rmsnorm(
        _vp(resid), _vp(add), c_int(n_add), c_ll(add.stride(0) if add is not None else 0),
        c_ll(add.stride(1) if add is not None else 0), _vp(w), c_float(eps), _vp(resid_out if need_resid_out else None),
        _vp(y), c_int(T), c_int(H), c_ll(resid.stride(0) if resid is not None else 0),
        c_ll(resid_out.stride(0) if need_resid_out else 0), c_ll(y.stride(0)), _st()), "dmoe_add_rmsnorm")
    if not want_resid:
        return None, y
    return (resid_out if need_resid_out else resid), y


def rmsnorm(x: torch.Tensor, w: torch.Tensor, eps: float, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    return add_rmsnorm(x, None, w, eps, y=out, want_resid=False)[1]


def rope_kv_append(qkv: torch.Tensor, positions: torch.Tensor, slots: Optional[torch.Tensor], kcache: torch.Tensor,
                   vcache: torch.Tensor, n_q: int, n_kv: int, hd: int, theta: float) -> None:
    """In place neox RoPE on the q/k heads of qkv rows [q | k | v], then append k, v to the paged cache
    ([num_blocks, block_size, n_kv, hd]) at flat slots (int64, < 0 = skip)."""
    if not qkv.is_cuda:
        return reference.rope_kv_append(qkv, positions, slots, kcache, vcache, n_q, n_kv, hd, theta)
    assert qkv.dtype == torch.bfloat16 and qkv.stride(1) == 1 and positions.dtype == torch.int32
    assert slots is None or slots.dtype == torch.int64
    assert kcache.is_contiguous() and vcache.is_contiguous()
    _lib.check(_lib.lib().dmoe_rope_kv_append(
        _vp(qkv), c_ll(qkv.stride(0)), _vp(positions), _vp(slots), _vp(kcache), _vp(vcache), c_int(qkv.shape[0]),
        c_int(n_q), c_int(n_kv), c_int(hd), c_float(theta), _st()), "dmoe_rope_kv_append")


def pick_attn_splits(T: int, n_kv: int, max_ctx: int, block_size: int) -> int:
    from .gemm import num_sms
    sms = num_sms()
    ctas = max(1, T * n_kv)
    if ctas >= 2 * sms or max_ctx <= 256:
        return 1
    want = (4 * sms + ctas - 1) // ctas
    return max(1, min(want, (max_ctx + 255) // 256, 64))


_attn_ws = {}


# (key size, value size) of the tensor-core kernels over the paged cache: with options (window, soft cap, sink, fp32 softmax
# weights) for query groups of any size up to 64 heads, without for equal sizes and groups of 1, 2, 4 or 8.
ATTN_TILES = ((64, 32), (64, 64), (64, 128), (128, 64), (128, 128))


def attention_on_tensor_cores(dtype, n_q: int, n_kv: int, hd: int, vd: int) -> bool:
    """Shapes of the tensor-core attention kernels; the others (and fp32) run on the CUDA cores."""
    return dtype == torch.bfloat16 and (hd, vd) in ATTN_TILES and n_q % n_kv == 0 and n_q // n_kv <= 64


def attention_tile(dtype, device, n_q: int, n_kv: int, hd: int, vd: int) -> Tuple[int, int]:
    """Head sizes to keep queries / keys and values in: those of the smallest tensor-core kernel that holds them (the rest of
    a head is zeros), or (hd, vd) where there is none."""
    if torch.device(device).type == "cuda":
        for k, v in ATTN_TILES:
            if hd <= k and vd <= v and attention_on_tensor_cores(dtype, n_q, n_kv, k, v):
                return k, v
    return hd, vd


def _attn_workspace(device, need: int) -> torch.Tensor:
    key = device.index or 0
    ws = _attn_ws.get(key)
    if ws is None or ws.numel() < need:
        ws = torch.empty(max(need, 1 << 22), dtype=torch.float32, device=device)
        _attn_ws[key] = ws
    return ws


def _check_sink(sink, n_q: int) -> None:
    assert sink is None or (sink.dtype == torch.float32 and sink.numel() == n_q and sink.is_contiguous())


def paged_attention(q: torch.Tensor, kcache: torch.Tensor, vcache: torch.Tensor, block_tables: torch.Tensor,
                    bt_row: Optional[torch.Tensor], ctx_len: torch.Tensor, n_q: int, n_kv: int, hd: int,
                    out: Optional[torch.Tensor] = None, splits: int = 1, scale: Optional[float] = None,
                    window: Optional[int] = None, softcap: Optional[float] = None, fp32_weights: bool = False,
                    sink: Optional[torch.Tensor] = None, chunk: Optional[int] = None, q_temp=None,
                    gate: Optional[torch.Tensor] = None) -> torch.Tensor:
    """out[t] = softmax(q[t] K^T * scale) V over the first ctx_len[t] cached tokens of block-table row bt_row[t], or the
    last ``window`` of them, or those from the start of the last one's ``chunk`` (of so many positions, counted from position
    0) on; ``softcap``: scores are soft-capped, cap * tanh(score / cap); ``sink`` (fp32 [n_q]): the softmax
    denominator has exp(sink) of the head in addition. ``fp32_weights`` keeps the softmax weights at fp32 accuracy in the
    product with V (implied by the options before). ``q_temp`` (:class:`disagmoe_b200.config.QueryTemperature`): scores are multiplied by the query's
    temperature at its position; ``gate`` ([T, n_q], columns of a wider matrix are fine): every head's output is multiplied by
    sigmoid(gate). Value heads may have another size than key heads
    (``vcache.shape[-1]``)."""
    if not q.is_cuda:
        o = reference.paged_attention(q, kcache, vcache, block_tables, bt_row, ctx_len, n_q, n_kv, hd, scale, window, softcap,
                                      sink, chunk, q_temp, gate)
        if out is not None:
            out.copy_(o)
            return out
        return o
    T = q.shape[0]
    scale = scale if scale is not None else 1.0 / math.sqrt(hd)
    vd = vcache.shape[-1]
    if out is None:
        out = torch.empty(T, n_q * vd, dtype=q.dtype, device=q.device)
    _check_sink(sink, n_q)
    if not attention_on_tensor_cores(q.dtype, n_q, n_kv, hd, vd):
        return _any_attention(q, hd, q.stride(0), kcache, vcache, block_tables, bt_row, None, ctx_len, T, n_q, n_kv, hd, vd,
                              scale, window, softcap, sink, out, vd, out.stride(0), chunk, q_temp, gate)
    assert block_tables.dtype == torch.int32 and ctx_len.dtype == torch.int32 and block_tables.stride(1) == 1
    ws = _attn_workspace(q.device, T * n_q * splits * (vd + 1)) if splits > 1 else None
    if window or chunk or softcap or fp32_weights or sink is not None or q_temp is not None or gate is not None or hd != vd or \
            n_q // n_kv not in (1, 2, 4, 8):
        x = _attn_extra(q_temp, gate, q.dtype)
        _lib.check(_lib.lib().dmoe_paged_attention_ext(
            _vp(q), c_ll(q.stride(0)), _vp(kcache), _vp(vcache), _vp(block_tables), c_int(block_tables.stride(0)),
            _vp(bt_row), _vp(ctx_len), c_int(kcache.shape[1]), c_int(T), c_int(n_q), c_int(n_kv), c_int(hd), c_int(vd),
            c_float(scale), c_int(window or 0), c_int(chunk or 0), c_float(softcap or 0.0), _vp(sink), c_int(splits), _vp(out),
            c_ll(out.stride(0)), _vp(ws), ctypes.byref(x) if x else None, _st()), "dmoe_paged_attention_ext")
        return out
    _lib.check(_lib.lib().dmoe_paged_attention(
        _vp(q), c_ll(q.stride(0)), _vp(kcache), _vp(vcache), _vp(block_tables), c_int(block_tables.stride(0)),
        _vp(bt_row), _vp(ctx_len), c_int(kcache.shape[1]), c_int(T), c_int(n_q), c_int(n_kv), c_int(hd),
        c_float(scale), c_int(splits), _vp(out), c_ll(out.stride(0)), _vp(ws), _st()), "dmoe_paged_attention")
    return out


def _attn_extra(q_temp, gate, dtype) -> Optional[_lib.DmoeAttnExtra]:
    if q_temp is None and gate is None:
        return None
    assert gate is None or (gate.dtype == dtype and gate.stride(1) == 1)
    return _lib.DmoeAttnExtra(_lib.ptr(gate), gate.stride(0) if gate is not None else 0, q_temp.coef if q_temp else 0.0,
                              q_temp.every if q_temp else 0)


def _any_attention(q, q_head, q_row, kcache, vcache, block_tables, bt_row, rows, ctx_len, T, n_q, n_kv, hd, vd, scale, window,
                   softcap, sink, out, o_head, o_row, chunk=None, q_temp=None, gate=None):
    """CUDA-core attention with free strides: query t of head h at q + t * q_row + h * q_head, likewise the output; the
    cached heads of a token are contiguous, tokens ``stride(1)`` apart. Query t has the context of batch row rows[t]
    (None: t)."""
    assert q.dtype == kcache.dtype == vcache.dtype == out.dtype
    x = _attn_extra(q_temp, gate, q.dtype)
    assert kcache.stride(0) == kcache.shape[1] * kcache.stride(1) and vcache.stride(0) == vcache.shape[1] * vcache.stride(1)
    _lib.check(_lib.lib().dmoe_any_attention(
        c_int(int(q.dtype == torch.float32)), _vp(q), c_ll(q_head), c_ll(q_row), _vp(kcache), c_ll(kcache.stride(1)),
        _vp(vcache), c_ll(vcache.stride(1)), _vp(block_tables), c_int(block_tables.stride(0)), _vp(bt_row), _vp(rows),
        _vp(ctx_len), c_int(kcache.shape[1]), c_int(T), c_int(n_q), c_int(n_kv), c_int(hd), c_int(vd), c_float(scale),
        c_int(window or 0), c_int(chunk or 0), c_float(softcap or 0.0), _vp(sink), _vp(out), c_ll(o_head), c_ll(o_row),
        ctypes.byref(x) if x else None, _st()), "dmoe_any_attention")
    return out


def embed(ids: torch.Tensor, table: torch.Tensor, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    if not table.is_cuda:
        o = table[ids.long()]
        if out is not None:
            out.copy_(o)
            return out
        return o
    T, (V, H) = ids.shape[0], table.shape
    if out is None:
        out = torch.empty(T, H, dtype=table.dtype, device=table.device)
    assert ids.dtype == torch.int32 and table.dtype == torch.bfloat16 and table.is_contiguous()
    _lib.check(_lib.lib().dmoe_embed(_vp(ids), _vp(table), _vp(out), c_int(T), c_int(H), c_int(V), c_ll(out.stride(0)),
                                     _st()), "dmoe_embed")
    return out


def argmax(logits: torch.Tensor, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Greedy sampling: int32 ids of the row maxima (first maximum wins)."""
    if not logits.is_cuda:
        o = logits.float().argmax(-1).int()
        if out is not None:
            out.copy_(o)
            return out
        return o
    T, V = logits.shape
    if out is None:
        out = torch.empty(T, dtype=torch.int32, device=logits.device)
    assert logits.stride(1) == 1 and logits.dtype in (torch.float32, torch.bfloat16)
    _lib.check(_lib.lib().dmoe_argmax(_vp(logits), c_int(logits.dtype == torch.float32), c_ll(logits.stride(0)),
                                      c_int(T), c_int(V), _vp(out), _st()), "dmoe_argmax")
    return out


def permute_rows(src: torch.Tensor, mapping: torch.Tensor, repeat: int = 1, gather: bool = False,
                 out: Optional[torch.Tensor] = None, n_out: Optional[int] = None) -> torch.Tensor:
    """scatter: out[mapping[i]] = src[i // repeat]; gather: out[i] = src[mapping[i]]. mapping int32, < 0 skipped."""
    n = mapping.numel()
    if not src.is_cuda:
        o = reference.permute_rows(src, mapping, repeat, gather, n_out)
        if out is not None:
            out.copy_(o)
            return out
        return o
    H = src.shape[1]
    if out is None:
        out = torch.zeros(n_out if n_out is not None else n, H, dtype=src.dtype, device=src.device)
    assert mapping.dtype == torch.int32 and src.dtype == torch.bfloat16 and src.stride(1) == 1
    _lib.check(_lib.lib().dmoe_permute_rows(_vp(src), c_ll(src.stride(0)), _vp(out), c_ll(out.stride(0)), _vp(mapping),
                                            c_int(n), c_int(H), c_int(repeat), c_int(int(gather)), _st()),
               "dmoe_permute_rows")
    return out


def gather_ptrs(ptrs: torch.Tensor, n: int, H: int, out: torch.Tensor) -> torch.Tensor:
    """out[i] = the bf16 row of H elements at device address ptrs[i] (int64 device tensor)."""
    assert ptrs.is_cuda and ptrs.dtype == torch.int64
    _lib.check(_lib.lib().dmoe_gather_ptrs(_vp(ptrs), _vp(out), c_ll(out.stride(0)), c_int(n), c_int(H), _st()),
               "dmoe_gather_ptrs")
    return out


def route(x: torch.Tensor, norm_w: Optional[torch.Tensor], eps: float, gate_w: torch.Tensor, top_k: int,
          renormalize: bool = True, y: Optional[torch.Tensor] = None, counts: Optional[torch.Tensor] = None,
          want_logits: bool = False, logit_bias: Optional[torch.Tensor] = None):
    """(RMSNorm ->) gate -> softmax -> top-k. Returns (y, topk_ids int32 [T,k], topk_w fp32 [T,k], logits or None).
    ``counts`` (int32 [E], device) is incremented per routed (token, k) pair. ``logit_bias`` (fp32 [E]) is added to
    the gate logits (synthetic popularity skew)."""
    if not x.is_cuda:
        yy, ids, w, logits = reference.route(x, norm_w, eps, gate_w, top_k, renormalize, logit_bias)
        if counts is not None:
            counts += torch.bincount(ids.reshape(-1).long(), minlength=gate_w.shape[0]).int()
        if y is not None:
            y.copy_(yy)
            yy = y
        return yy, ids, w, (logits if want_logits else None)
    T, H = x.shape
    E = gate_w.shape[0]
    if y is None:
        y = torch.empty(T, H, dtype=torch.bfloat16, device=x.device)
    ids = torch.empty(T, top_k, dtype=torch.int32, device=x.device)
    w = torch.empty(T, top_k, dtype=torch.float32, device=x.device)
    logits = torch.empty(T, E, dtype=torch.float32, device=x.device) if want_logits else None
    assert gate_w.is_contiguous() and gate_w.dtype == torch.bfloat16 and x.stride(1) == 1
    assert logit_bias is None or (logit_bias.dtype == torch.float32 and logit_bias.is_cuda and logit_bias.numel() == E)
    _lib.check(_lib.lib().dmoe_route(
        _vp(x), c_ll(x.stride(0)), _vp(norm_w), c_float(eps), _vp(gate_w), c_int(T), c_int(H), c_int(E), c_int(top_k),
        c_int(int(renormalize)), _vp(y), c_ll(y.stride(0)), _vp(ids), _vp(w), _vp(logits), _vp(counts),
        _vp(logit_bias), _st()), "dmoe_route")
    return y, ids, w, logits


class DispatchBuffers:
    """Device buffers of the local (single GPU) expert dispatch: sorted rows, token records, offsets, scratch. Rows are bf16
    of a size that is a multiple of 16 bytes, or anything else of 2 or 4 bytes per element."""

    def __init__(self, capacity: int, H: int, E: int, device, dtype=torch.bfloat16):
        self.capacity, self.H, self.E = capacity, H, E
        self.xs = torch.zeros(capacity, H, dtype=dtype, device=device)
        self.recs = torch.zeros(capacity, 4, dtype=torch.int32, device=device)
        self.offs = torch.zeros(E + 1, dtype=torch.int32, device=device)
        self.ws = torch.zeros(2 * E + 8, dtype=torch.int32, device=device)
        self.x_bases = torch.tensor([self.xs.data_ptr()], dtype=torch.int64, device=device)
        self.rec_bases = torch.tensor([self.recs.data_ptr()], dtype=torch.int64, device=device)

    @property
    def counts(self):
        return self.ws[: self.E]


def dispatch_local(y: torch.Tensor, topk_ids: torch.Tensor, topk_w: torch.Tensor, buf: DispatchBuffers) -> None:
    """Copies every routed (token, k) row of y into ``buf.xs`` sorted by expert, writes ``buf.offs`` ([E+1]) and the
    token records ``buf.recs`` = (rank 0, dst row t*k+j, weight bits, expert). ``buf.counts`` must hold the histogram
    produced by :func:`route`; it is cleared for the next layer."""
    T, K = topk_ids.shape
    if not y.is_cuda:
        pos = reference.sort_by_expert(topk_ids).long()
        buf.offs.copy_(reference.expert_offsets(topk_ids, buf.E))
        src = torch.arange(T * K) // K
        buf.xs[pos] = y[src]
        buf.recs[pos, 0] = 0
        buf.recs[pos, 1] = torch.arange(T * K, dtype=torch.int32)
        buf.recs[pos, 2] = topk_w.reshape(-1).contiguous().view(torch.int32)
        buf.recs[pos, 3] = topk_ids.reshape(-1)
        buf.counts.zero_()
        return
    assert T * K <= buf.capacity and y.dtype == buf.xs.dtype
    s = scratch(y.device)
    if y.dtype != torch.bfloat16 or buf.H % 8 or y.stride(0) % 8:
        _lib.check(_lib.lib().dmoe_dispatch_local_any(
            c_int(y.element_size()), _vp(y), c_ll(y.stride(0)), _vp(topk_ids), _vp(topk_w), c_int(T), c_int(K), c_int(buf.H),
            c_int(buf.E), _vp(buf.ws), _vp(buf.offs), _vp(buf.x_bases), c_ll(buf.xs.stride(0)), _vp(buf.rec_bases),
            c_int(buf.capacity), _vp(s.status), _st()), "dmoe_dispatch_local_any")
        return
    _lib.check(_lib.lib().dmoe_dispatch_local(
        _vp(y), c_ll(y.stride(0)), _vp(topk_ids), _vp(topk_w), c_int(T), c_int(K), c_int(buf.H), c_int(buf.E),
        c_int(buf.E), c_int(0), _vp(buf.ws), _vp(buf.offs), _vp(buf.x_bases), c_ll(buf.xs.stride(0)),
        _vp(buf.rec_bases), c_int(buf.capacity), _vp(s.status), _st()), "dmoe_dispatch_local")


# ---- fused attention-side senders (csrc/kernels/sender.cu); CUDA only -------------------------------------------------
def norm_gather(resid: Optional[torch.Tensor], add: Optional[torch.Tensor], w: torch.Tensor, eps: float,
                resid_out: Optional[torch.Tensor], dst_ptrs: torch.Tensor, n_dst: int, dst_row0: int, ld_dst: int,
                T: int, H: int, wait_flags: Optional[torch.Tensor] = None, n_wait: int = 0,
                wait_epoch: Optional[torch.Tensor] = None, signal_ptrs: Optional[torch.Tensor] = None,
                n_signal: int = 0, signal_slot: int = 0, signal_epoch: Optional[torch.Tensor] = None,
                ticket: Optional[torch.Tensor] = None, status: Optional[torch.Tensor] = None) -> None:
    """[wait for ``wait_flags``] resid_out = resid + add.sum(1); rmsnorm(resid_out) * w is stored to rows
    [dst_row0, dst_row0 + T) of every buffer named in ``dst_ptrs`` (int64 device tensor of n_dst addresses, peers
    included); then the flags in ``signal_ptrs`` are released. ``add`` is [T, P, H] (or [T, H]) bf16."""
    d = _lib.DmoeNormGather()
    if add is not None and add.dim() == 2:
        add = add.unsqueeze(1)
    d.resid_in, d.add, d.w, d.resid_out = _lib.ptr(resid), _lib.ptr(add), w.data_ptr(), _lib.ptr(resid_out)
    d.dst_ptrs, d.n_dst, d.dst_row0, d.ld_dst = dst_ptrs.data_ptr(), n_dst, dst_row0, ld_dst
    d.ld_in = resid.stride(0) if resid is not None else 0
    d.ld_out = resid_out.stride(0) if resid_out is not None else 0
    d.n_add = 0 if add is None else add.shape[1]
    d.add_row_stride = add.stride(0) if add is not None else 0
    d.add_part_stride = add.stride(1) if add is not None else 0
    d.eps, d.T, d.H = eps, T, H
    d.wait_flags, d.n_wait, d.wait_epoch = _lib.ptr(wait_flags), n_wait, _lib.ptr(wait_epoch)
    d.signal_ptrs, d.n_signal, d.signal_slot = _lib.ptr(signal_ptrs), n_signal, signal_slot
    d.signal_epoch, d.ticket, d.status = _lib.ptr(signal_epoch), _lib.ptr(ticket), _lib.ptr(status)
    _lib.check(_lib.lib().dmoe_norm_gather(ctypes.byref(d), _st()), "dmoe_norm_gather")


def route_dispatch(resid: torch.Tensor, norm_w: torch.Tensor, eps: float, gate_w: Optional[torch.Tensor], top_k: int,
                   renormalize: bool, T: int, *, add: Optional[torch.Tensor] = None, n_add: int = 0,
                   add_slot_stride: int = 0, ld_add: int = 0, y: Optional[torch.Tensor] = None,
                   topk_ids: Optional[torch.Tensor] = None, topk_w: Optional[torch.Tensor] = None,
                   logit_bias: Optional[torch.Tensor] = None, x_bases=None, rec_bases=None, cnt_bases=None,
                   flag_bases=None, ld_dst: int = 0, experts_per_rank: int = 1, n_dst: int = 0, my_rank: int = 0,
                   ret_rank: Optional[int] = None,
                   region_cap: int = 0, disp_epoch=None, wait_flags=None, n_wait: int = 0, wait_epoch=None, ticket=None,
                   status=None) -> None:
    """One launch for the post-attention half of a layer on an attention GPU: [wait for the TP peers' o_proj flags]
    resid[:T] += the ``n_add`` partial-row slots of ``add``; RMSNorm; gate; softmax; top-k; dispatch of every routed row
    into its expert's receive region on the owning GPU (peer stores) with a release flag per expert GPU."""
    H = resid.shape[1]
    d = _lib.DmoeRouteDispatch()
    d.resid, d.ld_resid, d.add, d.n_add = resid.data_ptr(), resid.stride(0), _lib.ptr(add), n_add
    d.add_slot_stride, d.ld_add = add_slot_stride, ld_add
    d.norm_w, d.eps, d.gate_w, d.logit_bias = norm_w.data_ptr(), eps, _lib.ptr(gate_w), _lib.ptr(logit_bias)
    d.T, d.H, d.E, d.K, d.renorm = T, H, (gate_w.shape[0] if gate_w is not None else 0), top_k, int(renormalize)
    d.y, d.ld_y = _lib.ptr(y), (y.stride(0) if y is not None else 0)
    d.topk_ids, d.topk_w = _lib.ptr(topk_ids), _lib.ptr(topk_w)
    d.x_bases, d.rec_bases, d.cnt_bases, d.flag_bases = (_lib.ptr(t) for t in (x_bases, rec_bases, cnt_bases, flag_bases))
    d.ld_dst, d.experts_per_rank, d.n_dst, d.my_rank, d.region_cap = ld_dst, experts_per_rank, n_dst, my_rank, region_cap
    d.ret_rank, d.ret_rank_set = (ret_rank, 1) if ret_rank is not None else (0, 0)
    d.disp_epoch, d.wait_flags, d.n_wait, d.wait_epoch = _lib.ptr(disp_epoch), _lib.ptr(wait_flags), n_wait, _lib.ptr(wait_epoch)
    d.ticket, d.status = _lib.ptr(ticket), _lib.ptr(status)
    _lib.check(_lib.lib().dmoe_route_dispatch(ctypes.byref(d), _st()), "dmoe_route_dispatch")


def ids_gather(src: torch.Tensor, n: int, dst_ptrs: torch.Tensor, n_dst: int, dst0: int,
               signal_ptrs: Optional[torch.Tensor] = None, signal_slot: int = 0,
               signal_epoch: Optional[torch.Tensor] = None) -> None:
    """The first n int32 of ``src`` are stored at offset dst0 of every buffer in ``dst_ptrs``; then one flag per
    destination is released (the all-gather of a TP group's sampled ids)."""
    _lib.check(_lib.lib().dmoe_ids_gather(_vp(src), c_int(n), _vp(dst_ptrs), c_int(n_dst), c_int(dst0), _vp(signal_ptrs),
                                          c_int(signal_slot), _vp(signal_epoch), _st()), "dmoe_ids_gather")


def wait_flags(flags: torch.Tensor, n: int, epoch: torch.Tensor, status: Optional[torch.Tensor]) -> None:
    """Stand-alone bounded wait: flags[i] >= epoch + 1 for i < n; advances the device-resident epoch."""
    _lib.check(_lib.lib().dmoe_wait_flags(_vp(flags), c_int(n), _vp(epoch), _vp(status), _st()), "dmoe_wait_flags")


# ---- tiled causal attention for prompt tokens (csrc/kernels/attention.cu: prefill_attn_kernel) -----------------------
def prefill_tile_tokens(n_q: int, n_kv: int) -> int:
    """Prompt tokens per tile of :func:`prefill_attention` (64 query rows = tokens x query heads per kv head)."""
    return 64 // (n_q // n_kv) if n_q % n_kv == 0 else 0


def token_runs(bt_row, positions):
    """(first row, end row) of every run of consecutive rows of one sequence at consecutive positions."""
    import numpy as np
    rows, pos = np.asarray(bt_row, dtype=np.int64), np.asarray(positions, dtype=np.int64)
    if len(rows) == 0:
        return []
    brk = np.nonzero((rows[1:] != rows[:-1]) | (pos[1:] != pos[:-1] + 1))[0] + 1
    return list(zip([0] + brk.tolist(), brk.tolist() + [len(rows)]))


def build_prefill_tiles(bt_row, positions, tile_tokens: int, min_len: int = 8):
    """Finds the prompt segments of a flat token batch on the host and cuts them into attention tiles.

    bt_row / positions: int sequences (lists, numpy arrays or CPU tensors) of the batch's rows. A segment is a run of
    consecutive rows of one sequence (same block-table row) at consecutive positions; runs of at least ``min_len``
    rows go to the tiled kernel. Returns (tiles int32 CPU tensor [n, 4] = (first row, tokens, block-table row, first
    position), covered bool CPU tensor [T]): rows not covered stay with the per-token kernel."""
    import numpy as np
    rows = np.asarray(bt_row, dtype=np.int64)
    pos = np.asarray(positions, dtype=np.int64)
    T = len(rows)
    covered = np.zeros(T, dtype=bool)
    tiles = []
    if T == 0 or tile_tokens <= 0:
        return torch.zeros(0, 4, dtype=torch.int32), torch.from_numpy(covered)
    for a, b in token_runs(rows, pos):
        if b - a < min_len:
            continue
        covered[a:b] = True
        for t0 in range(a, b, tile_tokens):
            tiles.append((t0, min(tile_tokens, b - t0), int(rows[a]), int(pos[t0])))
    t = torch.tensor(tiles, dtype=torch.int32).reshape(-1, 4)
    return t, torch.from_numpy(covered)


def prefill_attention(q: torch.Tensor, kcache: torch.Tensor, vcache: torch.Tensor, block_tables: torch.Tensor,
                      tiles: torch.Tensor, n_tiles: int, n_q: int, n_kv: int, hd: int, out: torch.Tensor,
                      scale: Optional[float] = None, window: Optional[int] = None, softcap: Optional[float] = None,
                      fp32_weights: bool = False, sink: Optional[torch.Tensor] = None,
                      chunk: Optional[int] = None, q_temp=None, gate: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Causal attention of the prompt tokens named by ``tiles`` (device int32 [>= n_tiles, 4], see
    :func:`build_prefill_tiles`) over the paged cache, which already holds their own K / V; writes their rows of
    ``out``. Every tile streams its sequence's K / V once (the per-token kernel streams it once per row)."""
    if n_tiles == 0:
        return out
    assert q.is_cuda and tiles.is_cuda and tiles.dtype == torch.int32 and tiles.is_contiguous()
    scale = scale if scale is not None else 1.0 / math.sqrt(hd)
    vd = vcache.shape[-1]
    _check_sink(sink, n_q)
    if window or chunk or softcap or fp32_weights or sink is not None or q_temp is not None or gate is not None or hd != vd or \
            n_q // n_kv not in (1, 2, 4, 8):
        x = _attn_extra(q_temp, gate, q.dtype)
        _lib.check(_lib.lib().dmoe_prefill_attention_ext(
            _vp(q), c_ll(q.stride(0)), _vp(kcache), _vp(vcache), _vp(block_tables), c_int(block_tables.stride(0)),
            _vp(tiles), c_int(n_tiles), c_int(kcache.shape[1]), c_int(n_q), c_int(n_kv), c_int(hd), c_int(vd), c_float(scale),
            c_int(window or 0), c_int(chunk or 0), c_float(softcap or 0.0), _vp(sink), _vp(out), c_ll(out.stride(0)),
            ctypes.byref(x) if x else None, _st()), "dmoe_prefill_attention_ext")
        return out
    _lib.check(_lib.lib().dmoe_prefill_attention(
        _vp(q), c_ll(q.stride(0)), _vp(kcache), _vp(vcache), _vp(block_tables), c_int(block_tables.stride(0)), _vp(tiles),
        c_int(n_tiles), c_int(kcache.shape[1]), c_int(n_q), c_int(n_kv), c_int(hd), c_float(scale), _vp(out),
        c_ll(out.stride(0)), _st()), "dmoe_prefill_attention")
    return out


# ---- decoders with an fp32 residual stream (csrc/kernels/layer_ops.cu) ------------------------------------------------
def _f32(dtype) -> c_int:
    assert dtype in (torch.float32, torch.bfloat16)
    return c_int(int(dtype == torch.float32))


def embed_f32(ids: torch.Tensor, table: torch.Tensor, scale: float, out: torch.Tensor, positions: Optional[torch.Tensor] = None,
              pos_table: Optional[torch.Tensor] = None) -> torch.Tensor:
    """out (fp32) = table[ids] * scale (+ pos_table[positions])."""
    if not table.is_cuda:
        out.copy_(table[ids.long()].float() * scale)
        if pos_table is not None:
            out += pos_table[positions.long()].float()
        return out
    assert pos_table is None or (pos_table.dtype == table.dtype and pos_table.is_contiguous() and positions.dtype == torch.int32 and
                                 pos_table.shape[1] == table.shape[1])
    assert ids.dtype == torch.int32 and table.is_contiguous() and out.is_contiguous() and out.dtype == torch.float32
    _lib.check(_lib.lib().dmoe_embed_f32(_vp(ids), _vp(table), _f32(table.dtype), c_float(scale), _vp(out),
                                         c_int(ids.shape[0]), c_int(table.shape[1]), c_int(table.shape[0]),
                                         _vp(positions if pos_table is not None else None), _vp(pos_table),
                                         c_int(0 if pos_table is None else pos_table.shape[0]), _st()), "dmoe_embed_f32")
    return out


def resid_norm(resid: torch.Tensor, y: Optional[torch.Tensor], post: Optional[torch.Tensor], pre: Optional[torch.Tensor],
               eps: float, dtype: torch.dtype, out_scale: float = 1.0, rows: Optional[torch.Tensor] = None
               ) -> Optional[torch.Tensor]:
    """One step of a residual stream kept in fp32: resid += norm(y) * post (where y is given), then returns
    norm(resid) * pre * out_scale in ``dtype`` (None where pre is None). ``rows`` (int32) picks the rows to return; resid
    itself is then left as it is. post / pre: fp32 weights as multiplied (offsets from one already added)."""
    if not resid.is_cuda:
        return reference.resid_norm(resid, y, post, pre, eps, dtype, out_scale, rows)
    n, W = (resid.shape[0] if rows is None else rows.shape[0]), resid.shape[1]
    h = torch.empty(n, W, dtype=dtype, device=resid.device) if pre is not None else None
    assert resid.dtype == torch.float32 and resid.is_contiguous() and (y is None or (y.dtype == dtype and y.stride(1) == 1))
    assert rows is None or rows.dtype == torch.int32
    _lib.check(_lib.lib().dmoe_resid_norm(
        _f32(dtype), _vp(resid), _vp(y), c_ll(y.stride(0) if y is not None else 0), _vp(post), _vp(pre), c_float(out_scale),
        c_float(eps), _vp(rows), _vp(h), c_ll(W), c_int(n), c_int(W), _st()), "dmoe_resid_norm")
    return h


@dataclass
class Router:
    """Router over rows that are already normalised: ``weight`` [experts, width] in the activations' dtype. ``sigmoid``: scores
    sigmoid(logit) instead of softmax; then ``correction`` (fp32 [experts]) is added for the choice alone, and of ``groups`` equal
    groups of neighbouring experts only the ``keep`` whose two best choice scores have the largest sum are open. The ``top``
    experts with the largest (choice) scores are chosen; their weights are the scores, with ``renormalize`` divided by their
    sum, times ``scale``. ``counts`` (int32 [experts]) is the histogram that :func:`dispatch_local` reads and clears."""
    weight: torch.Tensor
    top: int
    renormalize: bool = False
    counts: Optional[torch.Tensor] = None
    sigmoid: bool = False
    correction: Optional[torch.Tensor] = None
    groups: int = 1
    keep: int = 1
    scale: float = 1.0

    MAX_EXPERTS, MAX_TOP = 256, 32


@dataclass
class TokenShift:
    """Mixes of every row with the row before it in its sequence: h + (before - h) mu_s. ``mu`` fp32 [n, W]; ``last`` fp32
    [slots, W] keeps the last row of every sequence from step to step (not read at position 0); ``segs``: the segments of the
    step (:class:`disagmoe_b200.ops.recurrent.SegmentTables`)."""
    mu: torch.Tensor
    last: torch.Tensor
    segs: "SegmentTables"                        # noqa: F821

    def descriptor(self, T: int) -> _lib.DmoeShift:
        d, s = _lib.DmoeShift(), self.segs
        n, W = self.mu.shape
        assert self.mu.dtype == self.last.dtype == torch.float32 and self.mu.is_contiguous() and self.last.is_contiguous()
        assert self.last.shape[1] == W
        d.mu, d.last, d.singles = self.mu.data_ptr(), self.last.data_ptr(), _lib.ptr(s.singles) if s.n_single else 0
        d.positions, d.rows, d.kv_slots = _lib.ptr(s.positions), _lib.ptr(s.rows), _lib.ptr(s.kv_slots)
        d.mix_stride, d.n_mix, d.n_slots, d.n_single = T * W, n, self.last.shape[0], s.n_single
        return d


def token_shift(h: torch.Tensor, shift: TokenShift, dtype: torch.dtype) -> torch.Tensor:
    """fp32 rows h [T, W] -> the mixes [n, T, W] in ``dtype``; ``shift.last`` takes the last row of every segment."""
    if not h.is_cuda:
        return reference.token_shift(h, shift.mu, shift.last, shift.segs).to(dtype)
    T, W = h.shape
    s, n = shift.segs, shift.mu.shape[0]
    assert h.dtype == torch.float32 and h.is_contiguous()
    out = torch.empty(n, T, W, dtype=dtype, device=h.device)
    d = shift.descriptor(T)
    _lib.check(_lib.lib().dmoe_token_shift(_f32(dtype), _vp(h), ctypes.byref(d), _vp(s.multi), c_int(s.n_multi), _vp(s.chunks),
                                           c_int(s.n_chunks), _vp(out), c_ll(W), c_int(W), _st()), "dmoe_token_shift")
    return out


@dataclass
class ResidualGate:
    """What joins the residual stream is multiplied, number by number, by sigmoid(z + bias): z [T, W], bias fp32 [W]."""
    z: torch.Tensor
    bias: torch.Tensor


@dataclass
class Sides:
    """Outputs of two mixers on the same rows, ``rows`` [2, T, W]; together they are scale * the sum of their RMS norms over the
    width, each times its weights (fp32 [2, W])."""
    rows: torch.Tensor
    weights: torch.Tensor
    scale: float = 0.5


@dataclass
class InputConv:
    """h + causal convolution of h per channel: ``w`` fp32 [taps, W] (the last row belongs to the token itself); ``ring`` [slots,
    taps, W] keeps a sequence's last rows by position modulo taps (not read before position 0); ``segs``: the step's segments."""
    w: torch.Tensor
    ring: torch.Tensor
    segs: "SegmentTables"                        # noqa: F821

    def descriptor(self) -> _lib.DmoeConv:
        return _conv_descriptor(self.w, self.ring, self.segs)


def _conv_descriptor(w, ring, segs, in_bias=None, out_bias=None, residual=True, blocks=1, padded=0) -> _lib.DmoeConv:
    d, (taps, C) = _lib.DmoeConv(), w.shape
    assert w.dtype == torch.float32 and w.is_contiguous() and ring.is_contiguous() and ring.shape[1:] == (taps, C)
    assert all(b is None or (b.dtype == torch.float32 and b.numel() == C) for b in (in_bias, out_bias))
    d.w, d.in_bias, d.out_bias, d.ring = w.data_ptr(), _lib.ptr(in_bias), _lib.ptr(out_bias), ring.data_ptr()
    d.singles = _lib.ptr(segs.singles) if segs.n_single else 0
    d.positions, d.rows, d.kv_slots = _lib.ptr(segs.positions), _lib.ptr(segs.rows), _lib.ptr(segs.kv_slots)
    d.n_single, d.n_slots, d.taps, d.residual, d.blocks, d.padded = segs.n_single, ring.shape[0], taps, int(residual), blocks, padded
    return d


def seq_conv(x: torch.Tensor, w: torch.Tensor, ring: torch.Tensor, segs, in_bias: Optional[torch.Tensor] = None,
             out_bias: Optional[torch.Tensor] = None, residual: bool = False, blocks: int = 0,
             out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Causal convolution over time of every column of x [T, C] + in_bias within its segment: sum_j w[j] x_(t - taps + 1 + j) +
    out_bias, with ``residual`` plus x itself. ``ring`` [slots, taps, C] keeps the last rows of x of every sequence by position modulo
    taps. blocks > 0: returns the equal blocks of columns one after the other, [blocks, T, n] with n = C / blocks padded with
    zeros to a multiple of 8."""
    T, C = x.shape
    n = C // max(1, blocks)
    padded = (n + 7) // 8 * 8 if blocks else n
    if not x.is_cuda:
        y = reference.seq_conv(x, w, ring, segs, in_bias, out_bias, residual).to(x.dtype)
        if blocks:
            y = torch.nn.functional.pad(y.view(T, blocks, n).transpose(0, 1), (0, padded - n)).contiguous()
        if out is not None:
            return out.copy_(y)
        return y
    if out is None:
        shape = (blocks, T, padded) if blocks else (T, C)
        out = (torch.empty if padded == n else torch.zeros)(shape, dtype=x.dtype, device=x.device)
    assert x.stride(1) == 1 and ring.dtype == x.dtype == out.dtype and out.stride(-1) == 1 and C == w.shape[1]
    d = _conv_descriptor(w, ring, segs, in_bias, out_bias, residual, max(1, blocks), padded)
    _lib.check(_lib.lib().dmoe_seq_conv(_f32(x.dtype), _vp(x), c_ll(x.stride(0)), ctypes.byref(d), _vp(segs.multi), c_int(segs.n_multi),
                                        _vp(segs.chunks), c_int(segs.n_chunks), _vp(out), c_ll(out.stride(-2)),
                                        c_ll(out.stride(0) if blocks else 0), c_int(C), _st()), "dmoe_seq_conv")
    return out


def sum_norm(resid: torch.Tensor, y, parts: Optional[torch.Tensor], w: torch.Tensor, eps: float,
             dtype: torch.dtype, centred: bool, rows: Optional[torch.Tensor] = None, router: Optional[Router] = None,
             mult: float = 1.0, shift: Optional[TokenShift] = None, bias: Optional[torch.Tensor] = None,
             gate: Optional[ResidualGate] = None, conv: Optional[InputConv] = None):
    """One step of a residual stream kept in fp32: resid += mult * (y + parts.sum(1)) (y [T, W] or :class:`Sides`, parts [T, P, W] or
    [T, W], each may be None; with a ``gate`` multiplied by its sigmoid), then h = norm(resid) * w (+ bias, fp32 [W]) in ``dtype``; ``centred``: layer norm, otherwise RMS norm. ``rows`` (int32)
    picks the rows to return; resid itself is then left as it is. Returns (h, expert ids [T, top], weights [T, top]), the last
    two None without a ``router``, which sees h. With a token ``shift``, h (kept in fp32 on the way) becomes its mixes
    [n, T, W]; where every segment has one token (decoding) that is one launch. With an input ``conv``, h becomes [2, T, W]: h and
    its convolved rows, likewise in one launch where every segment has one token."""
    y, sides = (None, y) if isinstance(y, Sides) else (y, None)
    if not resid.is_cuda:
        h = reference.sum_norm(resid, y, parts, w, eps, torch.float32 if shift else dtype, centred, rows, mult, bias, gate, sides)
        if conv is not None:
            return torch.stack([h, seq_conv(h, conv.w, conv.ring, conv.segs, residual=True)]), None, None
        if shift is not None:
            return token_shift(h, shift, dtype), None, None
        if router is None:
            return h, None, None
        if router.sigmoid:
            ids, wts = reference.sigmoid_route(h, router)
        else:
            _, ids, wts, _ = reference.route(h, None, eps, router.weight, router.top, router.renormalize)
            wts = wts * router.scale
        if router.counts is not None:
            router.counts += torch.bincount(ids.reshape(-1).long(), minlength=router.weight.shape[0]).int()
        return h, ids, wts
    n, W = (resid.shape[0] if rows is None else rows.shape[0]), resid.shape[1]
    if parts is not None and parts.dim() == 2:
        parts = parts.unsqueeze(1)
    two_steps = shift is not None and shift.segs.n_multi > 0
    shape = (2, n, W) if conv is not None else (n, W) if shift is None or two_steps else (shift.mu.shape[0], n, W)
    h = torch.empty(shape, dtype=torch.float32 if two_steps else dtype, device=resid.device)
    assert resid.dtype == torch.float32 and resid.is_contiguous() and w.dtype == torch.float32
    assert all(a is None or (a.dtype == dtype and a.stride(-1) == 1) for a in (y, parts)) and (rows is None or rows.dtype == torch.int32)
    ids = wts = rd = sd = None
    if router is not None:
        E, K = router.weight.shape[0], router.top
        assert rows is None and shift is None and router.weight.dtype == dtype and router.weight.is_contiguous()
        c = router.correction
        assert c is None or (router.sigmoid and c.dtype == torch.float32 and c.numel() == E and c.is_contiguous())
        ids = torch.empty(n, K, dtype=torch.int32, device=resid.device)
        wts = torch.empty(n, K, dtype=torch.float32, device=resid.device)
        rd = _lib.DmoeRouter(router.weight.data_ptr(), _lib.ptr(c), ids.data_ptr(), wts.data_ptr(), _lib.ptr(router.counts), E, K,
                             int(router.renormalize), int(router.sigmoid), router.groups, router.keep, router.scale)
    if shift is not None and not two_steps:
        sd = shift.descriptor(n)
    x = cd = None
    if bias is not None or gate is not None or sides is not None or conv is not None:
        x = _lib.DmoeSumExtra()
        assert bias is None or (bias.dtype == torch.float32 and bias.numel() == W)
        x.bias = _lib.ptr(bias)
        if gate is not None:
            assert gate.z.dtype == dtype and gate.z.stride(1) == 1 and gate.bias.dtype == torch.float32 and gate.z.shape[1] == W
            x.gate_z, x.gate_bias, x.ld_gate = gate.z.data_ptr(), gate.bias.data_ptr(), gate.z.stride(0)
        if sides is not None:
            s = sides.rows
            assert s.dtype == dtype and s.stride(2) == 1 and s.shape[2] == W and sides.weights.dtype == torch.float32 and \
                sides.weights.is_contiguous()
            x.side, x.side_w, x.ld_side, x.side_stride, x.side_scale = s.data_ptr(), sides.weights.data_ptr(), s.stride(1), \
                s.stride(0), sides.scale
        if conv is not None:
            assert rows is None and router is None and shift is None and conv.w.shape[1] == W and conv.ring.dtype == dtype
            if conv.segs.n_multi == 0:
                cd = conv.descriptor()
                x.conv = ctypes.addressof(cd)
    _lib.check(_lib.lib().dmoe_sum_norm(
        _f32(dtype), _vp(resid), _vp(y), c_ll(y.stride(0) if y is not None else 0), _vp(parts),
        c_int(parts.shape[1] if parts is not None else 0), c_ll(parts.stride(0) if parts is not None else 0),
        c_ll(parts.stride(1) if parts is not None else 0), c_float(mult), _vp(w), c_int(int(centred)), c_float(eps), _vp(rows),
        _vp(h), c_int(int(two_steps)), c_ll(W), c_int(n), c_int(W), ctypes.byref(rd) if rd else None,
        ctypes.byref(sd) if sd else None, ctypes.byref(x) if x else None, _st()), "dmoe_sum_norm")
    if conv is not None and cd is None:
        seq_conv(h[0], conv.w, conv.ring, conv.segs, residual=True, out=h[1])
    return (token_shift(h, shift, dtype) if two_steps else h), ids, wts


def rope_frequencies(dims: int, base: float, factor: Optional[float] = None, original: float = 0.0, fast: float = 32.0,
                     slow: float = 1.0):
    """(list of dims / 2 inverse frequencies, factor on cos and sin). With ``factor``: YaRN (Peng et al., "YaRN: Efficient
    Context Window Extension of Large Language Models"): dimensions that turn more than ``fast`` times over the original
    context keep their frequency, those below ``slow`` turns are slowed down by ``factor``, a linear ramp in between."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if factor is None:
        return f, 1.0
    turn_dim = lambda turns: dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(turn_dim(fast)), 0), min(math.ceil(turn_dim(slow)), dims - 1)
    width = max(hi - lo, 0.001)
    ramp = [min(max((i - lo) / width, 0.0), 1.0) for i in range(dims // 2)]
    return [x / factor * r + x * (1.0 - r) for x, r in zip(f, ramp)], 0.1 * math.log(factor) + 1.0


_freq_tables = {}


def rope_freq_table(spec, max_pos: int, device) -> Optional[torch.Tensor]:
    """fp32 [max_pos, dims / 2, 2] = (cos, sin) of a :class:`disagmoe_b200.config.RotarySpec`, from double-precision
    angles; cached per (device, positions, spec)."""
    if spec is None:
        return None
    device = torch.device(device)
    key = (device.type, device.index or 0, max_pos, spec)
    if key not in _freq_tables:
        f, m = rope_frequencies(spec.dims, spec.base, spec.factor, spec.original, spec.fast, spec.slow)
        freq = torch.tensor(f, dtype=torch.float64, device=device)
        if device.type == "cuda":
            t = torch.empty(max_pos, len(f), 2, dtype=torch.float32, device=device)
            _lib.check(_lib.lib().dmoe_rope_freq_table(_vp(t), c_int(max_pos), c_int(len(f)), _vp(freq), c_float(m), _st()),
                       "dmoe_rope_freq_table")
            torch.cuda.current_stream().synchronize()     # `freq` may be freed from here on
        else:
            ang = torch.arange(max_pos, dtype=torch.float64)[:, None] * freq
            t = (torch.stack([ang.cos(), ang.sin()], -1) * m).float()
        _freq_tables[key] = t
    return _freq_tables[key]


def qk_norm_rope(qkv: torch.Tensor, positions: torch.Tensor, slots: torch.Tensor, kcache: Optional[torch.Tensor],
                 vcache: Optional[torch.Tensor], n_q: int, n_kv: int, dk: int, dv: int, table: Optional[torch.Tensor],
                 qw: Optional[torch.Tensor], kw: Optional[torch.Tensor], eps: float, interleaved: bool = False,
                 v_first: Optional[torch.Tensor] = None, v_lambda: float = 0.0, tied: bool = False, v_norm: int = 0) -> None:
    """RMS norm of every q / k head (weights fp32 [dk]; None: no norm) and rotation by ``table`` (:func:`rope_freq_table`,
    None: no rotation; ``interleaved``: of neighbouring dimensions) on rows [q | k | v]; q in place, k and v to the paged
    caches at ``slots``. n_kv = 0: q only (a layer that reads another layer's cache). ``v_first`` [T, n_kv, >= dv]: the
    values become (1 - v_lambda) v + v_lambda v_first on their way to the cache. ``tied``: rows [q | k], the values are the first
    dv dimensions of the keys before their norm and rotation. ``v_norm`` > 0: every value head is divided by its root mean square over that
    many dimensions (the rest of it is padding)."""
    if not qkv.is_cuda:
        return reference.qk_norm_rope(qkv, positions, slots, kcache, vcache, n_q, n_kv, dk, dv, table, qw, kw, eps,
                                      interleaved, v_first, v_lambda, tied, v_norm)
    assert positions.dtype == torch.int32 and slots.dtype == torch.int64 and qkv.stride(1) == 1
    assert n_kv == 0 or (kcache.is_contiguous() and vcache.is_contiguous() and kcache.dtype == qkv.dtype)
    rot, max_pos = (2 * table.shape[1], table.shape[0]) if table is not None else (0, 1 << 30)
    _lib.check(_lib.lib().dmoe_qk_norm_rope(
        _f32(qkv.dtype), _vp(qkv), c_ll(qkv.stride(0)), _vp(positions), _vp(slots), _vp(kcache), _vp(vcache),
        c_int(qkv.shape[0]), c_int(n_q), c_int(n_kv), c_int(dk), c_int(dv), c_int(rot), c_int(int(interleaved)), _vp(table),
        c_int(max_pos), _vp(qw), _vp(kw), c_float(eps), _vp(v_first), c_ll(v_first.stride(0) if v_first is not None else 0),
        c_int(v_first.stride(1) if v_first is not None else 0), c_float(v_lambda), c_int(int(tied)), c_int(v_norm),
        _st()), "dmoe_qk_norm_rope")


# ---- latent attention (csrc/kernels/latent_attention.cu) ---------------------------------------------------------------
def _pad8(n: int) -> int:
    return (n + 7) // 8 * 8


@dataclass(frozen=True)
class LatentLayout:
    """Sizes of a latent attention layer as its kernels see them: every part of a row is padded to a multiple of 8 (zeros).

    projection row   [heads x (q unrotated | q rotated) | latent | rotated key part (| one gate per head)]
    cache row        [latent | rotated key part], an odd multiple of 8 elements from one row to the next: tiles that are copied
                     to shared memory as they are read without bank conflicts
    """
    heads: int
    dim: int
    rot: int
    vdim: int
    rank: int

    @property
    def dimp(self) -> int:
        return _pad8(self.dim)

    @property
    def rotp(self) -> int:
        return _pad8(self.rot)

    @property
    def vdimp(self) -> int:
        return _pad8(self.vdim)

    @property
    def rankp(self) -> int:
        return _pad8(self.rank)

    @property
    def qd(self) -> int:
        return self.dimp + self.rotp

    @property
    def kd(self) -> int:
        return self.rankp + self.rotp

    @property
    def row(self) -> int:
        return self.kd + (8 if self.kd % 16 == 0 else 0)

    def min_run(self) -> int:
        """Prompt tokens from which expanding the latents of all visible keys pays: it costs rank * (dim + vdim) per key and
        head once, and saves 2 rank + rot - (dim + rot + vdim) per key, head and query."""
        saves = max(1, 2 * self.rank + self.rot - (self.dim + self.rot + self.vdim))
        return min(128, max(16, self.rank * (self.dim + self.vdim) // saves))

    def tiled(self, dtype) -> bool:
        """Is there a prompt kernel for these head sizes?"""
        return dtype == torch.bfloat16 and any(self.qd <= k and self.vdimp <= v for k, v in LATENT_TILES)


LATENT_TILES = ((96, 64), (128, 128), (192, 128))     # (key, value) sizes of the prompt kernel
LATENT_MAX_RANK, LATENT_MAX_KEY = 512, 640            # of the tensor-core kernel over the latent cache


def latent_prep(y: torch.Tensor, positions: torch.Tensor, slots: torch.Tensor, cache: torch.Tensor, lay: LatentLayout,
                table: Optional[torch.Tensor], norm_w: torch.Tensor, eps: float, loose: Optional[torch.Tensor], n_loose: int,
                interleaved: bool = True, gate: Optional[torch.Tensor] = None,
                recs: Optional[torch.Tensor] = None) -> Tuple[torch.Tensor, torch.Tensor]:
    """From projection rows y (:class:`LatentLayout`): RMS norm of the latent (weight fp32 [rank]), rotation of the shared
    key part, both to the paged ``cache`` [blocks, block_size, row] at ``slots``; rotation of the queries, in place. Rows with
    loose[t] = i >= 0 (None: row t is i = t) are attended over the latents themselves, so their queries are also written
    head by head: returns (unrotated part [heads, n_loose, dimp], [heads, n_loose, row] with the rotated part in place and
    the latent part still to be filled). ``gate`` (columns of y, [T, heads]): sigmoid(gate) becomes the weight of the loose rows'
    records ``recs`` [heads * n_loose, 4] (:func:`disagmoe_b200.ops.gemm.grouped_combine`)."""
    if not y.is_cuda:
        return reference.latent_prep(y, positions, slots, cache, lay, table, norm_w, eps, loose, n_loose, interleaved, gate, recs)
    assert positions.dtype == torch.int32 and slots.dtype == torch.int64 and y.stride(1) == 1 and cache.is_contiguous()
    assert gate is None or (gate.dtype == y.dtype and gate.stride(1) == 1 and gate.stride(0) == y.stride(0))
    assert gate is None or n_loose == 0 or (recs.is_contiguous() and recs.shape == (lay.heads * n_loose, 4))
    assert y.shape[1] >= lay.heads * lay.qd + lay.kd and cache.dtype == y.dtype and norm_w.dtype == torch.float32
    xq = torch.empty(lay.heads, n_loose, lay.dimp, dtype=y.dtype, device=y.device)
    qa = torch.empty(lay.heads, n_loose, lay.row, dtype=y.dtype, device=y.device)
    rot, max_pos = (2 * table.shape[1], table.shape[0]) if table is not None else (0, 1 << 30)
    _lib.check(_lib.lib().dmoe_latent_prep(
        _f32(y.dtype), _vp(y), c_ll(y.stride(0)), _vp(positions), _vp(slots), _vp(cache), c_int(y.shape[0]), c_int(lay.heads),
        c_int(lay.dim), c_int(lay.rot), c_int(lay.rank), c_int(lay.row), c_int(rot), c_int(int(interleaved)), _vp(table), c_int(max_pos),
        _vp(norm_w), c_float(eps), _vp(loose), c_int(n_loose), _vp(xq), _vp(qa), _vp(gate), _vp(recs), _st()), "dmoe_latent_prep")
    return xq, qa


def latent_attention(qa: torch.Tensor, cache: torch.Tensor, block_tables: torch.Tensor, bt_row: torch.Tensor,
                     ctx_len: torch.Tensor, rows: Optional[torch.Tensor], lay: LatentLayout, scale: float,
                     window: Optional[int] = None, sink: Optional[torch.Tensor] = None, max_ctx: int = 1 << 30) -> torch.Tensor:
    """Attention over the cached latents: queries qa [heads, n, row] (latent part already multiplied by the key map), values
    are the latents. Query i belongs to batch row rows[i] (None: i). Returns [heads, n, rankp]."""
    H, n, row = qa.shape
    k3 = cache.unsqueeze(2)
    if not qa.is_cuda:
        idx = slice(None) if rows is None else rows.long()
        o = reference.paged_attention(qa.transpose(0, 1).reshape(n, H * row), k3, k3[..., :lay.rankp], block_tables,
                                      bt_row[idx], ctx_len[idx], H, 1, row, scale, window, None, sink)
        return o.view(n, H, lay.rankp).transpose(0, 1).contiguous()
    out = torch.empty(H, n, lay.rankp, dtype=qa.dtype, device=qa.device)
    _check_sink(sink, H)
    if qa.dtype == torch.float32 or lay.rankp > LATENT_MAX_RANK or lay.kd > LATENT_MAX_KEY or cache.shape[1] % 16:
        return _any_attention(qa, n * row, row, k3, k3[..., :lay.rankp], block_tables, bt_row, rows, ctx_len, n, H, 1, lay.kd,
                              lay.rankp, scale, window, None, sink, out, n * lay.rankp, lay.rankp)
    reach = min(max_ctx, window or max_ctx)
    splits = pick_latent_splits(n, H, reach)
    ws = _attn_workspace(qa.device, H * n * splits * (lay.rankp + 1)) if splits > 1 else None
    _lib.check(_lib.lib().dmoe_latent_attention(
        _vp(qa), _vp(cache), _vp(block_tables), c_int(block_tables.stride(0)), _vp(bt_row), _vp(rows), _vp(ctx_len),
        c_int(cache.shape[1]), c_int(n), c_int(H), c_int(lay.rankp), c_int(lay.kd), c_int(row), c_float(scale), c_int(window or 0), _vp(sink),
        c_int(splits), _vp(out), _vp(ws), _vp(scratch(qa.device).status), _st()), "dmoe_latent_attention")
    return out


def pick_latent_splits(n: int, heads: int, reach: int) -> int:
    """Key ranges per (query token, group of heads) of :func:`latent_attention`: the number whose waves of CTAs (one per SM, 16
    heads and 64 keys at a time, or 32 and 32), with some start and merge per CTA, are done first."""
    from .gemm import num_sms
    slots, ctas = num_sms(), max(1, n * ((heads + 31) // 32))
    keys = 64 if heads <= 16 else 32
    cost = lambda s: -(-ctas * s // slots) * (-(-reach // (keys * s)) + (3 if s == 1 else 5))
    return min(range(1, max(1, min(64, reach // 64)) + 1), key=cost)


def latent_gather(cache: torch.Tensor, block_tables: torch.Tensor, keys: torch.Tensor, n_keys: int) -> torch.Tensor:
    """Rows [n_keys, row] of the cached tokens named by ``keys`` (int32 [>= n_keys, 2] = block-table row, position)."""
    out = torch.empty(n_keys, cache.shape[2], dtype=cache.dtype, device=cache.device)
    assert keys.dtype == torch.int32 and keys.is_contiguous() and cache.shape[2] % 8 == 0 and cache.dtype == torch.bfloat16
    _lib.check(_lib.lib().dmoe_latent_gather(_vp(cache), _vp(block_tables), c_int(block_tables.stride(0)), _vp(keys),
                                             c_int(n_keys), c_int(cache.shape[1]), c_int(cache.shape[2]), _vp(out), _st()),
               "dmoe_latent_gather")
    return out


def latent_prefill(q: torch.Tensor, kv: torch.Tensor, lat: torch.Tensor, tiles: torch.Tensor, base: torch.Tensor, n_tiles: int,
                   lay: LatentLayout, scale: float, window: Optional[int], sink: Optional[torch.Tensor],
                   out: torch.Tensor, gate: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Causal attention of the prompt tokens named by ``tiles`` over expanded keys and values: kv [keys, heads x (key
    unrotated | value)], rotated key parts in the gathered cache rows ``lat`` [keys, row]; the key at position p of tile i's
    sequence is row base[i] + p. q: projection rows with rotated queries. Writes the tokens' rows of out [T, heads x vdimp], scaled by sigmoid(gate)
    per head where ``gate`` [T, heads] is given."""
    _check_sink(sink, lay.heads)
    assert gate is None or (gate.dtype == torch.bfloat16 and gate.stride(1) == 1)
    assert tiles.dtype == base.dtype == torch.int32 and kv.stride(1) == lat.stride(1) == 1
    _lib.check(_lib.lib().dmoe_latent_prefill(
        _vp(q), c_ll(q.stride(0)), _vp(kv), c_ll(kv.stride(0)), _vp(lat), c_ll(lat.stride(0)), _vp(tiles), _vp(base),
        c_int(n_tiles), c_int(lay.heads), c_int(lay.dimp), c_int(lay.rotp), c_int(lay.rankp), c_int(lay.vdimp), c_float(scale),
        c_int(window or 0), _vp(sink), _vp(gate), c_ll(gate.stride(0) if gate is not None else 0), _vp(out), c_ll(out.stride(0)),
        _st()), "dmoe_latent_prefill")
    return out
