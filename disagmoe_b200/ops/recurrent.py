"""Linear recurrences with a matrix state per head (``csrc/kernels/recurrent.cu``, ``recurrent_chunk.cu``): gated linear
attention, the gated delta rule and RWKV-style time mixing, with one decay per head and key channel; lightning attention, with a
constant decay per head; the matrix memory of xLSTM, with a decay per head and token and a normaliser beside the state. And the
real-gated diagonal recurrence of Griffin's block (``diag_recurrent.cu``). CUDA tensors run the kernels, CPU tensors the PyTorch
restatements.

A step's rows fall into segments (consecutive rows of one sequence). One-token segments (decoding) take one launch from
the projections to the gated, normalised output; longer ones (prompts and portions of prompts) are convolved and then run
chunk by chunk on the tensor cores, or token by token where fp32 is asked for or the head shape has no chunk kernel.
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Optional

import numpy as np
import torch

from . import _lib, reference
from .functional import token_runs
from .gemm import num_sms, scratch

CHUNK = 64          # tokens of a chunk
MAX_TAPS = 8        # longest short convolution
WORKSPACE = 512 << 20   # bytes of scratch the chunked kernels may use; more heads than fit run in groups


@dataclass
class SegmentTables:
    """Segments of one step. ``singles`` / ``multi``: int32 [n, 4] = (first row, tokens, slot, first position); ``chunks``:
    int32 [n, 4] = (first row, tokens, index into ``multi``, number in the segment). ``singles`` None with n_single > 0:
    every row is a segment of its own (decode step), described by ``positions``, ``rows`` (slots) and ``kv_slots``."""
    n_single: int = 0
    n_multi: int = 0
    n_chunks: int = 0
    max_multi: int = 0                              # tokens of the longest segment
    singles: Optional[torch.Tensor] = None
    multi: Optional[torch.Tensor] = None
    chunks: Optional[torch.Tensor] = None
    positions: Optional[torch.Tensor] = None
    rows: Optional[torch.Tensor] = None
    kv_slots: Optional[torch.Tensor] = None

    def table(self):
        """(first row, tokens, slot, first position) of every segment that is not padding (reads the tables back)."""
        if self.singles is None and self.n_single:
            return [(i, 1, int(self.rows[i]), int(self.positions[i])) for i in range(self.n_single) if self.kv_slots[i] >= 0]
        return self.singles.tolist() + self.multi.tolist()


def build_segments(bt_row, positions, device) -> SegmentTables:
    """Tables of a batch given on the host (rows of one sequence are consecutive, as every scheduler emits them)."""
    rows, pos = np.asarray(bt_row), np.asarray(positions)
    singles, multi, chunks = [], [], []
    for a, b in token_runs(rows, pos):
        seg = (a, b - a, int(rows[a]), int(pos[a]))
        if b - a == 1:
            singles.append(seg)
            continue
        chunks += [(c, min(CHUNK, b - c), len(multi), i) for i, c in enumerate(range(a, b, CHUNK))]
        multi.append(seg)
    table = torch.tensor(singles + multi + chunks, dtype=torch.int32).reshape(-1, 4)
    if torch.device(device).type == "cuda":
        table = table.to(device)
    s, m = len(singles), len(multi)
    return SegmentTables(s, m, len(chunks), max((x[1] for x in multi), default=0), table[:s], table[s:s + m], table[s + m:])


def decode_segments(positions: torch.Tensor, rows: torch.Tensor, kv_slots: torch.Tensor) -> SegmentTables:
    """Every row one token (padding rows have kv_slots < 0); no host work, so a captured graph can hold it."""
    return SegmentTables(n_single=positions.shape[0], positions=positions, rows=rows, kv_slots=kv_slots)


@dataclass
class RecurrentState:
    """Per-layer state pool: S fp32 [slots, heads, dim, vdim]; with a short convolution the ring of its last inputs [slots,
    taps, channels]; with a token shift the last input row, fp32 [slots, width]; of a matrix memory the normaliser ``n`` fp32 [slots,
    heads, dim] and the running maximum ``m`` fp32 [slots, 2, heads], kept at the parity of its position. A diagonal recurrence has S
    [slots, width]. A slot needs no clearing: a segment at position 0 starts from zero."""
    S: torch.Tensor
    ring: Optional[torch.Tensor] = None
    last: Optional[torch.Tensor] = None
    n: Optional[torch.Tensor] = None
    m: Optional[torch.Tensor] = None

    def tensors(self):
        return [t for t in (self.S, self.ring, self.last, self.n, self.m) if t is not None]


@dataclass
class Recurrence:
    """Constants of one recurrent layer (weights fp32). ``delta``: the gated delta rule with unit-norm q / k and
    log a = -exp(a_log) softplus(z + z_bias); otherwise the plain write with log a = log sigmoid(z + z_bias) / tau or,
    ``exp_decay``, log a = -exp(z + z_bias). ``bonus`` [heads, dim]: the read-out precedes decay and write, and the token's own
    write enters it weighed by the bonus. ``norm_w``: [vdim], or [heads * vdim] with a weight per head; ``qscale``: factor of q
    (None: dim ** -0.5); ``shift_width``: width of the token shift whose last row belongs to the state (0: none).
    ``head_decay`` [heads]: constant logs of the decays (no z). ``gate_bias`` [2 heads]: matrix memory; z is then the logits
    [T, 2 heads] of the input and the forget gates, soft-capped at ``gate_cap`` after the bias. ``joint_norm``: all heads' read-outs
    are normed together (norm_w [heads * vdim])."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    delta: bool
    z_bias: Optional[torch.Tensor]
    norm_w: torch.Tensor
    eps: float
    a_log: Optional[torch.Tensor] = None
    tau: float = 1.0
    conv_w: Optional[torch.Tensor] = None            # [2 kv_heads dim + heads vdim, taps]
    sigmoid_gate: bool = False
    exp_decay: bool = False
    bonus: Optional[torch.Tensor] = None
    qscale: Optional[float] = None
    shift_width: int = 0
    head_decay: Optional[torch.Tensor] = None
    gate_bias: Optional[torch.Tensor] = None
    gate_cap: float = 1.0
    joint_norm: bool = False

    @property
    def decay_kind(self) -> int:
        return 4 if self.gate_bias is not None else 3 if self.head_decay is not None else 2 if self.exp_decay else int(self.delta)

    @property
    def norm_ld(self) -> int:
        return 0 if self.norm_w.numel() == self.vdim else self.vdim

    @property
    def q_factor(self) -> float:
        return self.dim ** -0.5 if self.qscale is None else self.qscale

    @property
    def taps(self) -> int:
        return 0 if self.conv_w is None else self.conv_w.shape[1]

    @property
    def channels(self) -> int:
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim

    def new_state(self, slots: int, dtype, device) -> RecurrentState:
        S = torch.zeros(slots, self.heads, self.dim, self.vdim, dtype=torch.float32, device=device)
        ring = torch.zeros(slots, self.taps, self.channels, dtype=dtype, device=device) if self.taps else None
        last = torch.zeros(slots, self.shift_width, dtype=torch.float32, device=device) if self.shift_width else None
        n = m = None
        if self.gate_bias is not None:
            n = torch.zeros(slots, self.heads, self.dim, dtype=torch.float32, device=device)
            m = torch.zeros(slots, 2, self.heads, dtype=torch.float32, device=device)
        return RecurrentState(S, ring, last, n, m)


def _descriptor(r: Recurrence, q, k, v, gate, beta, z, state: RecurrentState) -> _lib.DmoeRecur:
    d = _lib.DmoeRecur()
    if r.gate_bias is not None:
        assert z is None or (z.stride(1) == 1 and z.dtype == torch.float32 and z.shape[1] == 2 * r.heads)
        d.gates, d.ldgates, d.gate_bias, d.gate_cap = _lib.ptr(z), 0 if z is None else z.stride(0), r.gate_bias.data_ptr(), r.gate_cap
        d.norm_state, d.max_state = state.n.data_ptr(), state.m.data_ptr()
        z = None
    d.head_decay = _lib.ptr(r.head_decay)
    for name, t in (("q", q), ("k", k), ("v", v), ("gate", gate), ("beta", beta), ("z", z)):
        assert t is None or (t.stride(1) == 1 and t.dtype == (torch.float32 if name == "z" else q.dtype))
        setattr(d, name, _lib.ptr(t))
    for name, t in (("ldq", q), ("ldk", k), ("ldv", v), ("ldg", gate), ("ldb", beta), ("ldz", z)):
        setattr(d, name, 0 if t is None else t.stride(0))
    d.z_bias, d.a_log, d.norm_w = _lib.ptr(r.z_bias), _lib.ptr(r.a_log), _lib.ptr(r.norm_w)
    d.state, d.n_slots = _lib.ptr(state.S), state.S.shape[0]
    d.heads, d.kv_heads, d.dim, d.vdim = r.heads, r.kv_heads, r.dim, r.vdim
    d.delta, d.decay_kind, d.gate_kind = int(r.delta), r.decay_kind, int(r.sigmoid_gate)
    d.bonus, d.norm_ld = _lib.ptr(r.bonus), r.norm_ld
    d.is_f32 = int(q.dtype == torch.float32)
    d.qscale, d.inv_tau, d.eps = r.q_factor, 1.0 / r.tau, r.eps
    d.status = scratch(q.device).status.data_ptr()
    return d


def _gate_norm(r: Recurrence, table, n, max_tokens, raw, gate, out, scale=None) -> None:
    v, ll, i = ctypes.c_void_p, ctypes.c_longlong, ctypes.c_int
    heads, vdim, norm_ld = (1, r.heads * r.vdim, 0) if r.joint_norm else (r.heads, r.vdim, r.norm_ld)
    _lib.check(_lib.lib().dmoe_gate_norm(
        i(int(out.dtype == torch.float32)), v(_lib.ptr(table)), i(n), i(max_tokens), v(raw.data_ptr()), ll(raw.stride(0)),
        v(gate.data_ptr()), ll(gate.stride(0)), v(r.norm_w.data_ptr()), i(norm_ld), ctypes.c_float(r.eps), i(int(r.sigmoid_gate)),
        v(out.data_ptr()), ll(out.stride(0)), i(heads), i(vdim), v(_lib.ptr(scale)), v(_lib.stream_ptr())), "dmoe_gate_norm")


def recurrent_attention(r: Recurrence, q, k, v, gate, beta, z, state: RecurrentState, segs: SegmentTables) -> torch.Tensor:
    """q, k [T, kv_heads dim], v, gate [T, heads vdim], beta [T, heads] (delta) straight from the projections (columns of
    one wider matrix are fine), z fp32 [T, heads dim] (constant decays: None; matrix memory: gate logits [T, 2 heads]). Returns [T,
    heads vdim]: the recurrence's read-outs, normalised per head (or together), weighed and gated. Convolution inputs and states of the segments' slots are updated."""
    if not q.is_cuda:
        return _reference(r, q, k, v, gate, beta, z, state, segs)
    T = q.shape[0]
    lib, st = _lib.lib(), ctypes.c_void_p(_lib.stream_ptr())
    out = torch.empty(T, r.heads * r.vdim, dtype=q.dtype, device=q.device)
    vt = lib.dmoe_recur_value_tile(r.dim, r.vdim)
    assert vt > 0, "head too large for the recurrence kernels"
    raw = scale = None
    memory = r.gate_bias is not None

    def raw_rows(d):
        """Read-outs go to fp32 rows, a matrix memory's with the factor of every row and head beside them."""
        nonlocal raw, scale
        if raw is None:
            raw = torch.empty(T, r.heads * r.vdim, dtype=torch.float32, device=q.device)
            scale = torch.empty(T, r.heads, dtype=torch.float32, device=q.device) if memory else None
        d.raw, d.ldraw, d.scale = raw.data_ptr(), raw.stride(0), _lib.ptr(scale)
    if segs.n_single:
        d = _descriptor(r, q, k, v, gate, beta, z, state)
        if r.taps:
            d.conv_w, d.ring, d.taps = r.conv_w.data_ptr(), state.ring.data_ptr(), r.taps
        d.segs, d.n_segs, d.one_token = _lib.ptr(segs.singles), segs.n_single, 1
        d.positions, d.rows, d.kv_slots = _lib.ptr(segs.positions), _lib.ptr(segs.rows), _lib.ptr(segs.kv_slots)
        svt = vt
        # few heads in flight: deal the value columns to more CTAs, at the price of a second (norm) launch
        while svt >= 32 and svt % 8 == 0 and segs.n_single * r.heads * ((r.vdim + svt - 1) // svt) < num_sms(q.device):
            svt //= 2
        fused = svt >= r.vdim and not r.joint_norm
        if fused:
            d.out, d.ldo = out.data_ptr(), out.stride(0)
        else:
            raw_rows(d)
        _lib.check(lib.dmoe_recur_step(ctypes.byref(d), ctypes.c_int(svt), st), "dmoe_recur_step")
        if not fused:
            _gate_norm(r, segs.singles, segs.n_single, 1, raw, gate, out, scale)
    if segs.n_multi:
        qs, vs = r.kv_heads * r.dim, r.heads * r.vdim
        if r.taps:
            act = torch.empty(T, r.channels, dtype=q.dtype, device=q.device)
            d = _descriptor(r, q, k, v, None, None, None, state)
            d.conv_w, d.ring, d.taps = r.conv_w.data_ptr(), state.ring.data_ptr(), r.taps
            d.segs, d.n_segs = segs.multi.data_ptr(), segs.n_multi
            _lib.check(lib.dmoe_conv_chunks(ctypes.byref(d), ctypes.c_void_p(segs.chunks.data_ptr()),
                                            ctypes.c_int(segs.n_chunks), ctypes.c_void_p(act.data_ptr()),
                                            ctypes.c_longlong(act.stride(0)), st), "dmoe_conv_chunks")
            q, k, v = act[:, :qs], act[:, qs:2 * qs], act[:, 2 * qs:]
        d = _descriptor(r, q, k, v, gate, beta, z, state)
        d.segs, d.n_segs = segs.multi.data_ptr(), segs.n_multi
        raw_rows(d)
        if memory:
            steps = torch.empty(3, r.heads, T, dtype=torch.float32, device=q.device)
            d.keep, d.put, d.run_max, d.ldsteps = *(t.data_ptr() for t in steps), T
            _lib.check(lib.dmoe_memory_gates(ctypes.byref(d), st), "dmoe_memory_gates")
        if q.dtype == torch.bfloat16 and lib.dmoe_recur_chunk_ok(r.dim, r.vdim):
            per_head = lib.dmoe_recur_chunk_bytes(r.dim, r.vdim, int(r.delta), segs.n_chunks)
            ws = torch.empty(max(per_head, min(per_head * r.heads, WORKSPACE)), dtype=torch.uint8, device=q.device)
            _lib.check(lib.dmoe_recur_chunks(ctypes.byref(d), ctypes.c_void_p(segs.chunks.data_ptr()),
                                             ctypes.c_int(segs.n_chunks), ctypes.c_void_p(ws.data_ptr()),
                                             ctypes.c_longlong(ws.numel()), st), "dmoe_recur_chunks")
        else:
            _lib.check(lib.dmoe_recur_step(ctypes.byref(d), ctypes.c_int(vt), st), "dmoe_recur_step")
        _gate_norm(r, segs.chunks, segs.n_chunks, CHUNK, raw, gate, out, scale)
    return out


def _reference(r: Recurrence, q, k, v, gate, beta, z, state: RecurrentState, segs: SegmentTables) -> torch.Tensor:
    T, H, G, D, V = q.shape[0], r.heads, r.kv_heads, r.dim, r.vdim
    zb = None if z is None or r.gate_bias is not None else z.float() + r.z_bias
    if r.gate_bias is not None:
        i, f = (r.gate_cap * torch.tanh((z + r.gate_bias) / r.gate_cap)).split(H, 1)
        f = torch.nn.functional.logsigmoid(f)
    logd = None if r.gate_bias is not None else r.head_decay[:, None].expand(T, H, D) if zb is None else -torch.exp(zb).view(T, H, D) if r.exp_decay else (-torch.exp(r.a_log)[:, None] * torch.nn.functional.softplus(zb).view(T, H, D)) if r.delta else \
        torch.nn.functional.logsigmoid(zb).view(T, H, D) / r.tau
    out = torch.zeros(T, H * V, dtype=q.dtype)
    for a, n, slot, pos0 in segs.table():
        x = torch.cat([q[a:a + n], k[a:a + n], v[a:a + n]], 1)
        if r.taps:
            x = reference.conv_segment(x, r.conv_w, state.ring[slot], pos0)
        qq, kk = (x[:, j * G * D:(j + 1) * G * D].view(n, G, D).repeat_interleave(H // G, 1) for j in (0, 1))
        if r.gate_bias is not None:
            o = reference.memory_segment(qq, kk, x[:, 2 * G * D:].view(n, H, V), i[a:a + n], f[a:a + n], state.S[slot], state.n[slot],
                                         state.m[slot], pos0, r.q_factor)
        else:
            o = reference.recur_segment(qq, kk, x[:, 2 * G * D:].view(n, H, V), None if beta is None else beta[a:a + n],
                                        logd[a:a + n], state.S[slot], pos0, r.delta, r.q_factor, r.bonus)
        if r.joint_norm:
            o = reference.gate_norm(o.reshape(n, H * V), gate[a:a + n], r.norm_w, r.eps, r.sigmoid_gate)
        else:
            o = reference.gate_norm(o, gate[a:a + n].view(n, H, V), r.norm_w.view(-1, V), r.eps, r.sigmoid_gate)
        out[a:a + n] = o.reshape(n, H * V).to(q.dtype)
    return out


# ---- real-gated diagonal recurrence ------------------------------------------------------------------------------------
@dataclass
class GatedUnit:
    """Constants of Griffin's block (fp32): convolution ``conv_w`` [taps, width], ``conv_b``, bias ``in_b`` of its input; ``gate_b`` [blocks,
    2, padded] biases of the two gates (padded = width / blocks rounded up to a multiple of 8); ``decay`` [width] log decay where the
    recurrence gate is open; ``y_b`` bias of the gelu branch."""
    width: int
    blocks: int
    conv_w: torch.Tensor
    conv_b: torch.Tensor
    in_b: torch.Tensor
    gate_b: torch.Tensor
    decay: torch.Tensor
    y_b: torch.Tensor

    @property
    def padded(self) -> int:
        return self.gate_b.shape[2]

    def new_state(self, slots: int, dtype, device) -> RecurrentState:
        ring = torch.zeros(slots, self.conv_w.shape[0], self.width, dtype=dtype, device=device)
        return RecurrentState(torch.zeros(slots, self.width, dtype=torch.float32, device=device), ring)


def unit_recurrence(g: GatedUnit, u: torch.Tensor, gates: torch.Tensor, y: torch.Tensor, state: RecurrentState,
                    segs: SegmentTables) -> torch.Tensor:
    """u [blocks, T, padded], gate logits fp32 [blocks, T, 2, padded] without their bias, y [T, width] (columns of a wider matrix are
    fine) before bias and gelu -> [T, width]: S gelu(y), with log a = decay sigmoid(r), S <- a S + sqrt(1 - a^2) sigmoid(i) u per
    channel. ``state.S`` of the segments' slots is updated."""
    T, C = y.shape
    if not u.is_cuda:
        n = C // g.blocks
        flat = lambda t: t[..., :n].transpose(0, 1).reshape(T, C).float()
        r, i = (torch.sigmoid(flat(gates[:, :, j] + g.gate_b[:, None, j])) for j in (0, 1))
        out, uu = torch.zeros(T, C, dtype=y.dtype), flat(u)
        gel = torch.nn.functional.gelu(y.float() + g.y_b, approximate="tanh")
        for a, k, slot, pos0 in segs.table():
            S = reference.diagonal_segment(uu[a:a + k], r[a:a + k], i[a:a + k], g.decay, state.S[slot], pos0)
            out[a:a + k] = (S * gel[a:a + k]).to(y.dtype)
        return out
    out = torch.empty(T, C, dtype=y.dtype, device=y.device)
    assert u.is_contiguous() and gates.is_contiguous() and gates.dtype == torch.float32 and y.stride(1) == 1 and u.dtype == y.dtype
    assert u.shape == (g.blocks, T, g.padded) and gates.shape == (g.blocks, T, 2, g.padded) and state.S.shape[1] == C
    d = _lib.DmoeUnit()
    d.u, d.gates, d.gate_bias, d.decay, d.y, d.y_bias = (t.data_ptr() for t in (u, gates, g.gate_b, g.decay, y, g.y_b))
    d.state, d.out, d.multi = state.S.data_ptr(), out.data_ptr(), _lib.ptr(segs.multi)
    d.singles = _lib.ptr(segs.singles) if segs.n_single else 0
    d.positions, d.rows, d.kv_slots = _lib.ptr(segs.positions), _lib.ptr(segs.rows), _lib.ptr(segs.kv_slots)
    d.ldy, d.ldo, d.block_rows = y.stride(0), out.stride(0), T
    d.n_single, d.n_multi, d.n_slots, d.width, d.blocks, d.padded = segs.n_single, segs.n_multi, state.S.shape[0], C, g.blocks, g.padded
    _lib.check(_lib.lib().dmoe_unit_recurrence(ctypes.c_int(int(y.dtype == torch.float32)), ctypes.byref(d),
                                               ctypes.c_void_p(_lib.stream_ptr())), "dmoe_unit_recurrence")
    return out
