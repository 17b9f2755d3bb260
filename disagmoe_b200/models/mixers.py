"""Token mixers and the gated feed-forward of layer-list decoders (:class:`disagmoe_b200.config.LayerListConfig`).

Each module loads its tensors by the checkpoint's names, fuses the projections that read the same rows into one weight
(row blocks padded to multiples of 8, so that every block of the output can be the TMA operand of a following GEMM) and
maps the normalised rows of a step to the sublayer's output. Attention reads and writes the paged KV cache; recurrences
keep their state in the slot pool (:class:`disagmoe_b200.ops.recurrent.RecurrentState`), indexed by block-table row.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple

import torch

from ..config import AttentionSpec, ChannelDeltaSpec, GatedLinearSpec, LayerListConfig
from ..ops import functional as F
from ..ops import gemm
from ..ops.recurrent import Recurrence, RecurrentState, SegmentTables, recurrent_attention
from .attention import AttnMeta
from .weights import StateDict


@dataclass
class StepMeta(AttnMeta):
    """Attention metadata of a step plus the segments the recurrent layers run over."""
    segments: Optional[SegmentTables] = None


def _pad8(n: int) -> int:
    return (n + 7) // 8 * 8


def _pad_rows(w: torch.Tensor, rows: int) -> torch.Tensor:
    return w if w.shape[0] == rows else torch.cat([w, w.new_zeros(rows - w.shape[0], w.shape[1])])


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
    def __init__(self, cfg: LayerListConfig, layer_id: int, device, dtype):
        super().__init__()
        self.cfg, self.layer_id, self.spec = cfg, layer_id, cfg.layers[layer_id].mixer
        self.device, self.dtype = torch.device(device), dtype
        self.eps = cfg.rms_norm_eps

    def _get(self, sd: StateDict, name: str, dtype=None) -> torch.Tensor:
        return sd[f"l{self.layer_id}.mix.{name}"].to(device=self.device, dtype=dtype or self.dtype).contiguous()


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


class NormedAttention(Mixer):
    """Softmax attention with per-head query / key norm, partial rotation, optional window and score soft cap, over the
    layer's own paged cache or, with ``kv_from``, an earlier layer's."""

    def load_weights(self, sd: StateDict) -> None:
        m = self.spec
        own = m.kv_from is None
        # contiguous head blocks [q | k | v]: the norm + rotation kernel walks them as one row of heads
        self.proj = FusedProjection([(n, self._get(sd, n)) for n in (("q", "k", "v") if own else ("q",))], pad=False)
        self.o = self._get(sd, "o")
        self.q_norm = self._get(sd, "q.norm", torch.float32)
        self.k_norm = self._get(sd, "k.norm", torch.float32) if own else None
        self.rope = F.rope_freq_table(m.rot, self.cfg.max_seq_len, self.device)

    def forward(self, h: torch.Tensor, kv: Tuple[torch.Tensor, torch.Tensor], meta: StepMeta) -> torch.Tensor:
        m, (kc, vc) = self.spec, kv
        qkv = self.proj(h)
        F.qk_norm_rope(qkv, meta.positions, meta.slots, kc, vc, m.heads, 0 if m.kv_from is not None else m.kv_heads, m.dim,
                       m.vdim, self.rope, self.q_norm, self.k_norm, self.eps)
        q = qkv[:, :m.heads * m.dim]
        opt = dict(scale=m.scale, window=m.window, softcap=m.softcap, fp32_weights=True)
        cuda = q.is_cuda and F.attention_on_tensor_cores(q.dtype, m.heads, m.kv_heads, m.dim, m.vdim)
        tiles, n_tiles = meta.prefill_tiles.get(F.prefill_tile_tokens(m.heads, m.kv_heads), (None, 0)) \
            if cuda and meta.prefill_tiles else (None, 0)
        splits = 1
        if cuda:
            reach = min(meta.max_ctx, m.window or meta.max_ctx)
            splits = F.pick_attn_splits(q.shape[0], m.kv_heads, reach, kc.shape[1])
        attn = None
        if n_tiles == 0 or meta.num_decode_tokens > 0:
            attn = F.paged_attention(q, kc, vc, meta.block_tables, meta.bt_row,
                                     meta.ctx_len_decode if n_tiles else meta.ctx_len, m.heads, m.kv_heads, m.dim,
                                     splits=splits, **opt)
        if n_tiles:
            if attn is None:
                attn = torch.empty(q.shape[0], m.heads * m.vdim, dtype=q.dtype, device=q.device)
            F.prefill_attention(q, kc, vc, meta.block_tables, tiles, n_tiles, m.heads, m.kv_heads, m.dim, attn, **opt)
        return gemm.linear(attn, self.o)


class GatedFeedForward:
    """down(silu(gate h) * (up h)); the inner width is padded to a multiple of 8 with zero rows / columns."""

    def __init__(self, sd: StateDict, prefix: str, device, dtype):
        get = lambda n: sd[prefix + n].to(device=device, dtype=dtype)
        gate, up, down = get("gate"), get("up"), get("down")
        n = _pad8(gate.shape[0])
        self.w13 = torch.cat([_pad_rows(gate, n), _pad_rows(up, n)]).contiguous()
        self.w2 = _pad_cols(down, n).contiguous()

    def __call__(self, h: torch.Tensor) -> torch.Tensor:
        return gemm.linear(gemm.swiglu_linear(h, self.w13), self.w2)


MIXERS = {AttentionSpec: NormedAttention, GatedLinearSpec: RecurrentMixer, ChannelDeltaSpec: RecurrentMixer}


def make_mixer(cfg: LayerListConfig, layer_id: int, device, dtype) -> Mixer:
    return MIXERS[type(cfg.layers[layer_id].mixer)](cfg, layer_id, device, dtype)
