"""Token mixers and feed-forwards of layer-list decoders (:class:`disagmoe_b200.config.LayerListConfig`).

Each module loads its tensors by the checkpoint's names, fuses the projections that read the same rows into one weight
(row blocks padded to multiples of 8, so that every block of the output can be the TMA operand of a following GEMM) and
maps the normalised rows of a step to the sublayer's output. Attention reads and writes the paged KV cache; recurrences
keep their state in the slot pool (:class:`disagmoe_b200.ops.recurrent.RecurrentState`), indexed by block-table row.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, List, Optional, Tuple

import numpy as np
import torch

from ..config import (AttentionSpec, ChannelDeltaSpec, GatedLinearSpec, GatedUnitSpec, HeadDecaySpec, LatentAttentionSpec,
                      LayerListConfig, MatrixMemorySpec, SideBySideSpec, WkvSpec)
from ..ops import functional as F
from ..ops import gemm
from ..ops.recurrent import (GatedUnit, Recurrence, RecurrentState, SegmentTables, recurrent_attention, unit_recurrence)
from .attention import AttnMeta
from .experts import ExpertStack
from .weights import WKV_MIXES, StateDict


@dataclass
class StepMeta(AttnMeta):
    """Attention metadata of a step plus the segments the recurrent layers run over, the row tables of the latent attention
    layers, the values that value-mixing layers mix in (set by the first of them) and, by number of blocks, the row offsets of
    grouped GEMMs over equal blocks of a step's rows."""
    segments: Optional[SegmentTables] = None
    latent: Dict[Tuple, "LatentTables"] = field(default_factory=dict)
    latent_out: Dict[int, "ScatterRows"] = field(default_factory=dict)      # by row size
    v_first: Optional[torch.Tensor] = None
    block_offs: Dict[int, torch.Tensor] = field(default_factory=dict)       # int32: 0, T, 2T, ...


class ScatterRows:
    """Rows that a combine epilogue scatters to, and the device table of their address (made once: graphs replay on it)."""

    def __init__(self, cap: int, size: int, device, dtype):
        self.rows = torch.zeros(cap, size, dtype=dtype, device=device)
        self.base = torch.tensor([self.rows.data_ptr()], dtype=torch.int64, device=device)


@dataclass
class LatentTables:
    """How one step's rows go through latent attention layers of one kind: prompt runs long enough to expand the latents of
    their visible keys are tiled, the other ("loose") rows attend over the latents."""
    n_loose: int
    loose: Optional[torch.Tensor] = None      # int32 [T]: place of a row among the loose ones, -1 = tiled; None: all are loose
    rows: Optional[torch.Tensor] = None       # int32 [n_loose]: the batch rows of the loose ones; None: the identity
    offs: Optional[torch.Tensor] = None       # int32 [heads + 1]: row groups (heads) of the per-head GEMMs
    recs: Optional[torch.Tensor] = None       # int32 [heads * n_loose, 4]: where their output rows go, see ops.gemm
    tiles: Optional[torch.Tensor] = None      # int32 [n_tiles, 4], see ops.functional.build_prefill_tiles
    base: Optional[torch.Tensor] = None       # int32 [n_tiles]: workspace row of position 0 of the tile's sequence
    n_tiles: int = 0
    keys: Optional[torch.Tensor] = None       # int32 [n_keys, 2] = (block-table row, position) of every workspace row
    n_keys: int = 0

    @staticmethod
    def key(m: LatentAttentionSpec) -> Tuple:
        return m.heads, m.window, latent_layout(m).min_run(), m.gate      # gated layers write the weights of the records

    @staticmethod
    def _per_head(rows: torch.Tensor, heads: int, device):
        """Tables of the per-head GEMMs over [heads, n, .] rows whose outputs go to rows (batch row, head)."""
        n = len(rows)
        recs = torch.zeros(heads * n, 4, dtype=torch.int32)
        recs[:, 1] = (rows[None].long() * heads + torch.arange(heads)[:, None]).reshape(-1).int()
        recs[:, 2] = torch.ones(1).view(torch.int32)
        return (torch.arange(heads + 1, dtype=torch.int32) * n).to(device), recs.to(device)

    @classmethod
    def decode(cls, m: LatentAttentionSpec, T: int, device) -> "LatentTables":
        return cls(T, None, None, *cls._per_head(torch.arange(T), m.heads, device))

    @classmethod
    def prefill(cls, m: LatentAttentionSpec, bt_row, positions, device, dtype) -> "LatentTables":
        lay, T = latent_layout(m), len(positions)
        if not (device.type == "cuda" and lay.tiled(dtype)):
            return cls.decode(m, T, device)
        tiles, covered = F.build_prefill_tiles(bt_row, positions, 64, lay.min_run())
        if len(tiles) == 0:
            return cls.decode(m, T, device)
        rows = (~covered).nonzero()[:, 0].int()
        loose = torch.full((T,), -1, dtype=torch.int32)
        loose[rows.long()] = torch.arange(len(rows), dtype=torch.int32)
        # runs of tiles: the keys of a run start a window before its first token and end with its last
        tl = tiles.numpy()
        n, row, pos = tl[:, 1], tl[:, 2], tl[:, 3]
        begins = np.nonzero(np.r_[True, (row[1:] != row[:-1]) | (pos[1:] != pos[:-1] + n[:-1])])[0]
        ends = np.r_[begins[1:], len(tl)] - 1
        lo = np.maximum(0, pos[begins] - m.window + 1) if m.window else np.zeros_like(begins)
        hi = pos[ends] + n[ends]
        at = np.r_[0, np.cumsum(hi - lo)]
        keys = np.empty((at[-1], 2), dtype=np.int32)
        for i, (a, b) in enumerate(zip(at[:-1], at[1:])):
            keys[a:b, 0], keys[a:b, 1] = row[begins[i]], np.arange(lo[i], hi[i])
        base = torch.from_numpy(np.repeat(at[:-1] - lo, ends - begins + 1).astype(np.int32))
        keys = torch.from_numpy(keys)
        t = cls(len(rows), loose.to(device), rows.to(device), None, None, tiles.to(device),
                base.to(device), len(tiles), keys.to(device), len(keys))
        if len(rows):
            t.offs, t.recs = cls._per_head(rows, m.heads, device)
        return t


def latent_layout(m: LatentAttentionSpec) -> F.LatentLayout:
    return F.LatentLayout(m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank)


def _pad8(n: int) -> int:
    return (n + 7) // 8 * 8


def _pad_rows(w: torch.Tensor, rows: int) -> torch.Tensor:
    return w if w.shape[0] == rows else torch.cat([w, w.new_zeros(rows - w.shape[0], w.shape[1])])


def _pad_heads(w: torch.Tensor, heads: int, sizes: List[Tuple[int, int]]) -> torch.Tensor:
    """Rows of w are ``heads`` blocks with parts of the given (size, padded size): zero rows fill every part up."""
    w = w.reshape(heads, -1, w.shape[1])
    parts, at = [], 0
    for n, full in sizes:
        parts += [w[:, at:at + n], w.new_zeros(heads, full - n, w.shape[2])]
        at += n
    return torch.cat(parts, 1).reshape(-1, w.shape[2])


def _pad_head_cols(w: torch.Tensor, heads: int, n: int, full: int) -> torch.Tensor:
    """The same for the columns of a map from concatenated heads of size n."""
    return w if n == full else _pad_heads(w.T.contiguous(), heads, [(n, full)]).T


def _pad_cols(w: torch.Tensor, cols: int) -> torch.Tensor:
    return w if w.shape[1] == cols else torch.cat([w, w.new_zeros(w.shape[0], cols - w.shape[1])], 1)


class FusedProjection:
    """Several linear maps of the same rows as one GEMM; ``split`` names the column blocks of its output."""

    def __init__(self, parts: List[Tuple[str, torch.Tensor]], pad: bool = True):
        rows = [_pad8(w.shape[0]) if pad else w.shape[0] for _, w in parts]
        self.weight = torch.cat([_pad_rows(w, n) for (_, w), n in zip(parts, rows)]).contiguous()
        self.cols: Dict[str, Tuple[int, int, int]] = {}
        at = 0
        for (name, w), n in zip(parts, rows):
            self.cols[name] = (at, w.shape[0], n)
            at += n

    def __call__(self, h: torch.Tensor) -> torch.Tensor:
        return gemm.linear(h, self.weight)

    def block(self, y: torch.Tensor, name: str, padded: bool = False) -> torch.Tensor:
        at, n, full = self.cols[name]
        return y[:, at:at + (full if padded else n)]


class Mixer(torch.nn.Module):
    def __init__(self, cfg: LayerListConfig, layer_id: int, device, dtype, spec=None, prefix: str = ""):
        """``spec``, ``prefix``: of a mixer inside another one (default: the layer's own, whose tensors have no further prefix)."""
        super().__init__()
        self.cfg, self.layer_id, self.spec, self.prefix = cfg, layer_id, spec or cfg.layers[layer_id].mixer, prefix
        self.device, self.dtype = torch.device(device), dtype
        self.eps = cfg.rms_norm_eps

    def shift(self, memory, meta: StepMeta) -> Optional[F.TokenShift]:
        """The token shift that the mixer's input goes through (forward then takes its mixes), if it has one."""
        return None

    def blocks(self) -> int:
        """Equal blocks of rows that a grouped GEMM of the mixer runs over (0: it has none)."""
        return 0

    def attention(self) -> Optional["SoftmaxAttention"]:
        """The softmax attention over paged keys and values in this mixer."""
        return None

    def _get(self, sd: StateDict, name: str, dtype=None) -> torch.Tensor:
        return sd[f"l{self.layer_id}.mix.{self.prefix}{name}"].to(device=self.device, dtype=dtype or self.dtype).contiguous()


class RecurrentMixer(Mixer):
    """Gated linear attention or the channel-wise gated delta rule."""

    def load_weights(self, sd: StateDict) -> None:
        m, delta = self.spec, isinstance(self.spec, ChannelDeltaSpec)
        names = ["q", "k", "v", "a1", "b", "g1"] if delta else ["q", "k", "v", "g", "a1"]
        self.proj = FusedProjection([(n, self._get(sd, n)) for n in names])
        self.a2 = _pad_cols(self._get(sd, "a2"), _pad8(m.rank)).contiguous()
        self.g2 = _pad_cols(self._get(sd, "g2"), _pad8(m.gate_rank)).contiguous() if delta else None
        self.o = self._get(sd, "o")
        f32 = lambda n: self._get(sd, n, torch.float32)
        kw = dict(heads=m.heads, dim=m.dim, vdim=m.vdim, norm_w=f32("norm"), eps=self.eps, delta=delta)
        if delta:
            conv = torch.cat([f32(n + ".conv") for n in ("q", "k", "v")]).contiguous()
            self.recur = Recurrence(kv_heads=m.kv_heads, z_bias=f32("dt_bias"), a_log=f32("A_log"), conv_w=conv,
                                    sigmoid_gate=True, **kw)
        else:
            self.recur = Recurrence(kv_heads=m.heads, z_bias=f32("a2.b"), tau=m.tau, **kw)

    def forward(self, h: torch.Tensor, state: RecurrentState, meta: StepMeta) -> torch.Tensor:
        y = self.proj(h)
        part = lambda n, padded=False: self.proj.block(y, n, padded)
        z = gemm.linear(part("a1", True), self.a2, out_dtype=torch.float32)
        gate = part("g") if self.g2 is None else gemm.linear(part("g1", True), self.g2)
        o = recurrent_attention(self.recur, part("q"), part("k"), part("v"), gate,
                                part("b") if self.recur.delta else None, z, state, meta.segments)
        return gemm.linear(o, self.o)


class WkvMixer(Mixer):
    """RWKV-style time mixing. The maps of the mixes to r, k, v and the gate run as one grouped GEMM, the map to the decays as
    two small ones with tanh in the epilogue of the first."""

    def load_weights(self, sd: StateDict) -> None:
        m = self.spec
        f32 = lambda n: self._get(sd, n, torch.float32)
        self.mu = torch.stack([f32("mu." + n) for n in WKV_MIXES]).contiguous()
        self.rkvg = torch.stack([self._get(sd, n) for n in WKV_MIXES[:4]]).contiguous()
        rank = _pad8(m.rank)
        self.w1 = _pad_rows(self._get(sd, "w1"), rank).contiguous()
        self.w2 = _pad_cols(self._get(sd, "w2"), rank).contiguous()
        self.o = self._get(sd, "o")
        self.recur = Recurrence(m.heads, m.heads, m.dim, m.dim, False, f32("w0"), f32("norm"), self.eps, exp_decay=True,
                                bonus=f32("u"), qscale=1.0, shift_width=self.cfg.hidden_size)

    def blocks(self) -> int:
        return 4

    def shift(self, memory: RecurrentState, meta: StepMeta) -> F.TokenShift:
        return F.TokenShift(self.mu, memory.last, meta.segments)

    def forward(self, mixes: torch.Tensor, state: RecurrentState, meta: StepMeta) -> torch.Tensor:
        T, n = mixes.shape[1], self.rkvg.shape[1]
        bn = gemm.pick_even_bn(T, n, 4) if mixes.is_cuda else 0
        r, k, v, gate = gemm.grouped_linear(mixes[:4].reshape(4 * T, -1), self.rkvg, meta.block_offs[4], bn=bn).view(4, T, n)
        z = gemm.linear(gemm.linear(mixes[4], self.w1, tanh=True), self.w2, out_dtype=torch.float32)
        return gemm.linear(recurrent_attention(self.recur, r, k, v, gate, None, z, state, meta.segments), self.o)


class HeadDecayMixer(Mixer):
    """Lightning attention. Queries, keys and values leave the projection with their silu."""

    def load_weights(self, sd: StateDict) -> None:
        m = self.spec
        self.proj = FusedProjection([(n, self._get(sd, n)) for n in ("q", "k", "v", "g")])
        self.o = self._get(sd, "o")
        # logs from doubles; a decay of 0 (nothing stays) as one that leaves nothing in fp32
        logs = torch.tensor(m.decay, dtype=torch.float64).clamp(min=1e-40).log().to(torch.float32).to(self.device)
        self.recur = Recurrence(m.heads, m.heads, m.dim, m.vdim, False, None, self._get(sd, "norm", torch.float32), self.eps,
                                sigmoid_gate=True, qscale=1.0, head_decay=logs, joint_norm=True)

    def forward(self, h: torch.Tensor, state: RecurrentState, meta: StepMeta) -> torch.Tensor:
        y = gemm.linear(h, self.proj.weight, silu_cols=self.proj.cols["g"][0])
        q, k, v, g = (self.proj.block(y, n) for n in ("q", "k", "v", "g"))
        return gemm.linear(recurrent_attention(self.recur, q, k, v, g, None, None, state, meta.segments), self.o)


class MatrixMemory(Mixer):
    """The matrix memory of xLSTM; projections come from the mixer that holds it."""

    def parts(self, sd: StateDict) -> List[Tuple[str, torch.Tensor]]:
        return [(n, self._get(sd, n)) for n in ("q", "k", "v", "g")]

    def load_weights(self, sd: StateDict) -> None:
        m = self.spec
        f32 = lambda n: self._get(sd, n, torch.float32)
        self.gates = torch.cat([self._get(sd, "i"), self._get(sd, "f")]).contiguous()
        self.o = self._get(sd, "o")
        self.recur = Recurrence(m.heads, m.heads, m.dim, m.vdim, False, None, f32("norm"), self.eps, sigmoid_gate=True,
                                gate_bias=torch.cat([f32("i.b"), f32("f.b")]).contiguous(), gate_cap=m.gate_cap)

    def recall(self, h, q, k, v, g, state: RecurrentState, meta: StepMeta, out: torch.Tensor) -> None:
        z = gemm.linear(h, self.gates, out_dtype=torch.float32)
        gemm.linear(recurrent_attention(self.recur, q, k, v, g, None, z, state, meta.segments), self.o, out=out)


class GatedUnitMixer(Mixer):
    """Griffin's block: one GEMM for both branches, the convolution, one grouped GEMM for the two gates of all blocks, the
    recurrence with the gelu branch."""

    def blocks(self) -> int:
        return self.spec.blocks

    def load_weights(self, sd: StateDict) -> None:
        m = self.spec
        n, p = m.width // m.blocks, _pad8(m.width // m.blocks)
        f32 = lambda name: self._get(sd, name, torch.float32)
        self.proj = FusedProjection([(b, self._get(sd, b)) for b in ("x", "y")])
        self.o = self._get(sd, "o")
        pad = torch.nn.functional.pad
        # [blocks, 2 p, p]: rows of the recurrence gate, then of the input gate
        self.gates = torch.cat([pad(self._get(sd, g), (0, p - n, 0, p - n)) for g in ("ra", "ri")], 1).contiguous()
        decay = -8.0 * torch.nn.functional.softplus(self._get(sd, "lam", torch.float64), threshold=1e3)
        self.recur = GatedUnit(m.width, m.blocks, f32("conv").T.contiguous(), f32("conv.b"), f32("x.b"),
                               torch.stack([pad(f32(g + ".b"), (0, p - n)) for g in ("ra", "ri")], 1).contiguous(),
                               decay.float().contiguous(), f32("y.b"))

    def forward(self, h: torch.Tensor, state: RecurrentState, meta: StepMeta) -> torch.Tensor:
        r, y = self.recur, self.proj(h)
        T, B, p = h.shape[0], r.blocks, r.padded
        u = F.seq_conv(self.proj.block(y, "x"), r.conv_w, state.ring, meta.segments, r.in_b, r.conv_b, blocks=B).view(B * T, p)
        bn = gemm.pick_even_bn(T, 2 * p, B) if h.is_cuda else 0
        z = gemm.grouped_linear(u, self.gates, meta.block_offs[B], bn=bn, out_dtype=torch.float32)
        out = unit_recurrence(r, u.view(B, T, p), z.view(B, T, 2, p), self.proj.block(y, "y"), state, meta.segments)
        return gemm.linear(out, self.o)


class SoftmaxAttention(Mixer):
    """Softmax attention over the layer's own paged cache or, with ``kv_from``, an earlier layer's: optional per-head query /
    key norm, rotation, window or chunks, score soft cap, sink, value mixing, values tied to the keys, value norm, query
    temperature, a gate per head. Head sizes without a tensor-core kernel are kept
    padded with zeros to those of the next one (not where heads are normed)."""

    def __init__(self, cfg: LayerListConfig, layer_id: int, device, dtype, spec=None, prefix: str = ""):
        super().__init__(cfg, layer_id, device, dtype, spec, prefix)
        m = self.spec
        self.dk, self.dv = (m.dim, m.vdim) if m.qk_norm or m.kv_from is not None else \
            F.attention_tile(dtype, self.device, m.heads, m.kv_heads, m.dim, m.vdim)

    def kv_shapes(self) -> Tuple[Tuple[int, ...], ...]:
        """Per token: shapes of what the layer caches."""
        return (self.spec.kv_heads, self.dk), (self.spec.kv_heads, self.dv)

    def attention(self) -> "SoftmaxAttention":
        return self

    def tiled(self) -> bool:
        return self.device.type == "cuda" and \
            F.attention_on_tensor_cores(self.dtype, self.spec.heads, self.spec.kv_heads, self.dk, self.dv)

    def parts(self, sd: StateDict) -> List[Tuple[str, torch.Tensor]]:
        m = self.spec
        own = m.kv_from is None
        # contiguous head blocks [q | k | v]: the norm + rotation kernel walks them as one row of heads
        heads = [("q", m.heads, m.dim, self.dk)] + ([("k", m.kv_heads, m.dim, self.dk)] if own else []) + \
            ([("v", m.kv_heads, m.vdim, self.dv)] if own and not m.tied_values else [])
        qkv = torch.cat([_pad_heads(self._get(sd, n), h, [(d, p)]) for n, h, d, p in heads])
        return [("qkv", qkv)] + ([("g", self._get(sd, "g"))] if m.gate else [])

    def load_weights(self, sd: StateDict, project: bool = True) -> None:
        """``project`` False: the projections come from the mixer that holds this one."""
        m = self.spec
        own = m.kv_from is None
        if project:
            self.proj = FusedProjection(self.parts(sd), pad=m.gate)
        self.o = _pad_head_cols(self._get(sd, "o"), m.heads, m.vdim, self.dv).contiguous()
        self.q_norm = self._get(sd, "q.norm", torch.float32) if m.qk_norm else None
        self.k_norm = self._get(sd, "k.norm", torch.float32) if m.qk_norm and own else None
        self.sink = self._get(sd, "sink", torch.float32) if m.sink else None
        mixes = m.v_mix and self.layer_id != self.cfg.first_v_mix
        self.v_lambda = float(sd[f"l{self.layer_id}.mix.vmix"].float()) if mixes else None
        self.rope = F.rope_freq_table(m.rot, self.cfg.max_seq_len, self.device)

    def forward(self, h: torch.Tensor, kv: Tuple[torch.Tensor, torch.Tensor], meta: StepMeta) -> torch.Tensor:
        y = self.proj(h)
        gate = self.proj.block(y, "g") if self.spec.gate else None
        return gemm.linear(self.attend(self.proj.block(y, "qkv"), gate, kv, meta), self.o)

    def attend(self, qkv: torch.Tensor, gate: Optional[torch.Tensor], kv: Tuple[torch.Tensor, torch.Tensor],
               meta: StepMeta) -> torch.Tensor:
        """Projection rows [q | k | v] -> the heads' outputs (k and v go to the cache)."""
        m, (kc, vc) = self.spec, kv
        n_kv = 0 if m.kv_from is not None else m.kv_heads
        first = meta.v_first if self.v_lambda is not None else None
        F.qk_norm_rope(qkv, meta.positions, meta.slots, kc, vc, m.heads, n_kv, self.dk, self.dv, self.rope, self.q_norm,
                       self.k_norm, self.eps, m.rot is not None and m.rot.interleaved, first, self.v_lambda or 0.0,
                       m.tied_values, m.vdim if m.value_norm else 0)
        if m.v_mix and self.v_lambda is None:
            meta.v_first = qkv[:, (m.heads + n_kv) * self.dk:].view(-1, n_kv, self.dv)
        q = qkv[:, :m.heads * self.dk]
        opt = dict(scale=m.scale, window=m.window, chunk=m.chunk, softcap=m.softcap, fp32_weights=True, sink=self.sink,
                   q_temp=m.q_temp, gate=gate)
        cuda = self.tiled()
        tiles, n_tiles = meta.prefill_tiles.get(F.prefill_tile_tokens(m.heads, m.kv_heads), (None, 0)) \
            if cuda and meta.prefill_tiles else (None, 0)
        splits = 1
        if cuda:
            reach = min(meta.max_ctx, m.window or meta.max_ctx, m.chunk or meta.max_ctx)
            splits = F.pick_attn_splits(q.shape[0], m.kv_heads, reach, kc.shape[1])
        attn = None
        if n_tiles == 0 or meta.num_decode_tokens > 0:
            attn = F.paged_attention(q, kc, vc, meta.block_tables, meta.bt_row,
                                     meta.ctx_len_decode if n_tiles else meta.ctx_len, m.heads, m.kv_heads, self.dk,
                                     splits=splits, **opt)
        if n_tiles:
            if attn is None:
                attn = torch.empty(q.shape[0], m.heads * self.dv, dtype=q.dtype, device=q.device)
            F.prefill_attention(q, kc, vc, meta.block_tables, tiles, n_tiles, m.heads, m.kv_heads, self.dk, attn, **opt)
        return attn


class SideBySideMixer(Mixer):
    """Attention and a matrix memory on the same rows: all projections that stay in the activations' dtype are one GEMM."""

    def __init__(self, cfg: LayerListConfig, layer_id: int, device, dtype):
        super().__init__(cfg, layer_id, device, dtype)
        self.left = SoftmaxAttention(cfg, layer_id, device, dtype, self.spec.left, "left.")
        self.right = MatrixMemory(cfg, layer_id, device, dtype, self.spec.right, "right.")

    def attention(self) -> SoftmaxAttention:
        return self.left

    def kv_shapes(self) -> Tuple[Tuple[int, ...], ...]:
        return self.left.kv_shapes()

    @property
    def recur(self) -> Recurrence:
        return self.right.recur

    def load_weights(self, sd: StateDict) -> None:
        self.proj = FusedProjection([("left." + n, w) for n, w in self.left.parts(sd)] +
                                    [("right." + n, w) for n, w in self.right.parts(sd)])
        self.left.load_weights(sd, project=False)
        self.right.load_weights(sd)
        self.out = torch.stack([self._get(sd, s + ".out", torch.float32) for s in ("left", "right")]).contiguous()

    def forward(self, h: torch.Tensor, memory, meta: StepMeta) -> F.Sides:
        kv, state = memory
        y = self.proj(h)
        part = lambda n: self.proj.block(y, n)
        rows = torch.empty(2, *h.shape, dtype=h.dtype, device=h.device)
        attn = self.left.attend(part("left.qkv"), part("left.g") if self.left.spec.gate else None, kv, meta)
        gemm.linear(attn, self.left.o, out=rows[0])
        self.right.recall(h, *(part("right." + n) for n in "qkvg"), state, meta, rows[1])
        return F.Sides(rows, self.out)


class LatentAttention(Mixer):
    """Attention over cached latents. Rows on their own (decoding, short portions) multiply the key map into the query and
    attend over the latents themselves, one shared key and value head; long prompt runs expand the latents of their visible
    keys into per-head keys and values first, which is cheaper from some tens of queries per key on."""

    def __init__(self, cfg: LayerListConfig, layer_id: int, device, dtype):
        super().__init__(cfg, layer_id, device, dtype)
        self.lay = latent_layout(self.spec)

    def kv_shapes(self) -> Tuple[Tuple[int, ...], ...]:
        return ((self.lay.row,),)

    def load_weights(self, sd: StateDict) -> None:
        m, lay = self.spec, self.lay
        H = m.heads
        q = _pad_heads(self._get(sd, "q"), H, [(m.dim, lay.dimp), (m.rot_dim, lay.rotp)])
        dkv = _pad_heads(self._get(sd, "dkv"), 1, [(m.kv_rank, lay.rankp), (m.rot_dim, lay.rotp)])
        self.proj = FusedProjection([("q", q), ("dkv", dkv)] + ([("g", self._get(sd, "g"))] if m.gate else []))
        uk = _pad_cols(_pad_heads(self._get(sd, "uk"), H, [(m.dim, lay.dimp)]), lay.rankp).view(H, lay.dimp, lay.rankp)
        uv = _pad_cols(_pad_heads(self._get(sd, "uv"), H, [(m.vdim, lay.vdimp)]), lay.rankp).view(H, lay.vdimp, lay.rankp)
        self.absorb, self.expand_v = uk.transpose(1, 2).contiguous(), uv.contiguous()
        self.expand = torch.cat([uk, uv], 1).reshape(-1, lay.rankp).contiguous() if lay.tiled(self.dtype) and \
            self.device.type == "cuda" else None
        self.o = _pad_head_cols(self._get(sd, "o"), H, m.vdim, lay.vdimp).contiguous()
        self.norm = self._get(sd, "dkv.norm", torch.float32)
        self.sink = self._get(sd, "sink", torch.float32) if m.sink else None
        self.rope = F.rope_freq_table(m.rot, self.cfg.max_seq_len, self.device)

    def forward(self, h: torch.Tensor, kv: Tuple[torch.Tensor], meta: StepMeta) -> torch.Tensor:
        m, lay, cache = self.spec, self.lay, kv[0]
        T, t = h.shape[0], meta.latent[LatentTables.key(m)]
        y = self.proj(h)
        gate = self.proj.block(y, "g") if m.gate else None
        xq, qa = F.latent_prep(y, meta.positions, meta.slots, cache, lay, self.rope, self.norm, self.eps, t.loose, t.n_loose,
                               m.rot is not None and m.rot.interleaved, gate, t.recs)
        out = meta.latent_out[m.heads * lay.vdimp]
        attn = out.rows[:T]
        if t.n_loose:
            bn = lambda F_: gemm.pick_even_bn(t.n_loose, F_, m.heads) if h.is_cuda else 0
            gemm.grouped_linear(xq.view(-1, lay.dimp), self.absorb, t.offs, out=qa.view(-1, lay.row)[:, :lay.rankp],
                                bn=bn(lay.rankp))
            o = F.latent_attention(qa, cache, meta.block_tables, meta.bt_row, meta.ctx_len, t.rows, lay, m.scale, m.window,
                                   self.sink, meta.max_ctx)
            gemm.grouped_combine(o.view(-1, lay.rankp), self.expand_v, t.offs, t.recs, out.base, lay.vdimp,
                                 bn=bn(lay.vdimp), outs=[attn.view(-1, lay.vdimp)])
        if t.n_tiles:
            lat = F.latent_gather(cache, meta.block_tables, t.keys, t.n_keys)
            kvx = gemm.linear(lat[:, :lay.rankp], self.expand)
            F.latent_prefill(y, kvx, lat, t.tiles, t.base, t.n_tiles, lay, m.scale, m.window, self.sink, attn, gate)
        return gemm.linear(attn, self.o)


def _gated_stack(sd: StateDict, prefixes: List[str], ff: int, device, dtype) -> Tuple[torch.Tensor, torch.Tensor]:
    """(w13 [n, 2 I, H], w2 [n, H, I]) of gated feed-forwards; the inner width I is ff padded to a multiple of 8 with zero
    rows / columns."""
    I = _pad8(ff)
    get = lambda p, n: sd[p + n].to(device=device, dtype=dtype)
    H = sd[prefixes[0] + "down"].shape[0]
    w13 = torch.zeros(len(prefixes), 2 * I, H, dtype=dtype, device=device)
    w2 = torch.zeros(len(prefixes), H, I, dtype=dtype, device=device)
    for i, p in enumerate(prefixes):
        w13[i, :ff], w13[i, I:I + ff], w2[i, :, :ff] = get(p, "gate"), get(p, "up"), get(p, "down")
    return w13, w2


class GatedFeedForward:
    """down(act(gate h) * (up h))"""

    def __init__(self, sd: StateDict, prefix: str, ff: int, act: str, device, dtype):
        w13, w2 = _gated_stack(sd, [prefix], ff, device, dtype)
        self.w13, self.w2, self.act = w13[0], w2[0], act

    def __call__(self, h: torch.Tensor) -> torch.Tensor:
        return gemm.linear(gemm.swiglu_linear(h, self.w13, act=self.act), self.w2)


class RoutedBuffers:
    """Activations of the routed feed-forwards of one shape for up to ``cap`` tokens, shared by the layers that have it:
    dispatched rows and the weighted output rows [cap, top, width] of the chosen experts."""

    def __init__(self, cap: int, H: int, experts: int, top: int, device, dtype):
        self.dispatch = F.DispatchBuffers(cap * top, H, experts, device, dtype)
        self.out = ScatterRows(cap * top, H, device, dtype)
        self.parts = self.out.rows.view(cap, top, H)


class RoutedFeedForward:
    """Experts on the device that has the attention: sort by expert, grouped GEMMs, weighted rows per (token, choice)."""

    def __init__(self, sd: StateDict, prefix: str, spec, device, dtype):
        if spec.experts > F.Router.MAX_EXPERTS or spec.top > F.Router.MAX_TOP:
            raise ValueError(f"more than {F.Router.MAX_EXPERTS} experts or {F.Router.MAX_TOP} per token are not supported")
        w13, w2 = _gated_stack(sd, [f"{prefix}e{e}." for e in range(spec.experts)], spec.ff, device, dtype)
        self.spec = spec
        self.stack = ExpertStack(spec.experts, w2.shape[1], w2.shape[2], device, dtype, spec.act, limit=spec.limit,
                                 weigh_input=spec.weigh_input)
        self.stack.set_weights(w13, w2)
        self.router_w = sd[prefix + "router"].to(device=device, dtype=dtype).contiguous()
        self.correction = sd[prefix + "correction"].to(device=device, dtype=torch.float32).contiguous() if spec.correction else None

    def router(self, buf: RoutedBuffers) -> F.Router:
        s = self.spec
        return F.Router(self.router_w, s.top, s.renormalize, buf.dispatch.counts, s.scoring == "sigmoid", self.correction,
                        s.groups, s.keep, s.scale)

    def __call__(self, h: torch.Tensor, ids: torch.Tensor, weights: torch.Tensor, buf: RoutedBuffers) -> torch.Tensor:
        """Output rows [T, top, width], to be summed over the choices."""
        T, d = h.shape[0], buf.dispatch
        F.dispatch_local(h, ids, weights, d)
        n, H = T * self.spec.top, h.shape[1]
        self.stack.forward_combine(n, d.xs[:n], d.offs, d.recs[:n], buf.out.base, H, outs=[buf.out.rows])
        return buf.parts[:T]


MIXERS = {AttentionSpec: SoftmaxAttention, LatentAttentionSpec: LatentAttention, GatedLinearSpec: RecurrentMixer,
          ChannelDeltaSpec: RecurrentMixer, WkvSpec: WkvMixer, HeadDecaySpec: HeadDecayMixer, GatedUnitSpec: GatedUnitMixer,
          SideBySideSpec: SideBySideMixer}


def make_mixer(cfg: LayerListConfig, layer_id: int, device, dtype) -> Mixer:
    return MIXERS[type(cfg.layers[layer_id].mixer)](cfg, layer_id, device, dtype)
