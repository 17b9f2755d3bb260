"""Whole-iteration executor of layer-list decoders (:class:`disagmoe_b200.config.LayerListConfig`).

    sandwich  embed * scale -> per layer [ norm -> mixer -> norm + add (-> norm -> gated feed-forward -> norm + add) ]
    parallel  embed * scale -> per layer [ norm (+ router) -> mixer, feed-forward or experts on the same rows -> add both ]
              -> norm -> head -> argmax
    prenorm   embed * scale (+ position) -> per layer [ norm (+ token shift or input convolution) -> mixer -> (gate,) add
              (-> norm + router -> experts or feed-forward -> (gate,) add) ] -> norm -> head -> argmax

The residual stream is fp32; what stands between two sublayers (norm after, residual add, norm before, and the router of a
layer with experts) is one launch. Two kinds of per-sequence memory: pages for the attention layers that have keys and values
of their own (layers that read another layer's have none; latent attention keeps one latent row per token), and for recurrent
layers one state slot per sequence (layers that share weights have caches and states of their own), numbered like its row of the block table, so the block manager's row allocation is the
slot allocation. A layer that has both (attention beside a recurrence) has both kinds, and with input convolutions
every layer has the last rows of its input in the slot. As in the MoE executor, a decode iteration is one chain of launches captured per batch-size bucket, prompts
run eagerly, and CPU tensors run the PyTorch restatements.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional, Tuple

import torch

from ..config import AttentionSpec, LatentAttentionSpec, SideBySideSpec
from ..models import weights as W
from ..models.mixers import (GatedFeedForward, LatentTables, RoutedBuffers, RoutedFeedForward, ScatterRows, StepMeta,
                             make_mixer)
from ..ops import functional as F
from ..ops import gemm
from ..ops.recurrent import MAX_TAPS, RecurrentState, SegmentTables, build_segments, decode_segments
from .step import StepExecutor, TokenBuffers


class LayerListBuffers(TokenBuffers):
    def __init__(self, cfg, cap: int, device, dtype, logit_rows: int, mixers):
        super().__init__(cfg, cap, device, logit_rows)
        self.routed: Dict[Tuple[int, int], RoutedBuffers] = {}
        for r in {(l.routed.experts, l.routed.top) for l in cfg.layers if l.routed}:
            self.routed[r] = RoutedBuffers(cap, cfg.hidden_size, *r, device, dtype)
        self.latent_out: Dict[int, ScatterRows] = {}
        for size in {m.lay.heads * m.lay.vdimp for m in mixers if hasattr(m, "lay")}:
            self.latent_out[size] = ScatterRows(cap, size, device, dtype)
        self.latent: Dict[Tuple, LatentTables] = {}          # of a prefill step
        self.block_offs: Dict[int, torch.Tensor] = {}        # likewise
        self.resid = torch.zeros(cap, cfg.hidden_size, dtype=torch.float32, device=device)
        self.segments: Optional[SegmentTables] = None        # None: decode step, every row its own segment
        self.prefill_tiles: Dict[int, Tuple[torch.Tensor, int]] = {}    # tokens per tile -> (table, tiles)
        self.ctx_len_decode: Optional[torch.Tensor] = None
        self.n_untiled = 0


class LayerListExecutor(StepExecutor):
    def _load(self, state_dict: Optional[W.StateDict]) -> None:
        cfg, dev, dt = self.cfg, self.device, self.dtype
        assert self.layer_ids == list(range(cfg.num_layers)), "a layer-list decoder runs whole"
        if any(getattr(l.mixer, "conv", 0) > MAX_TAPS for l in cfg.layers) or cfg.input_conv > MAX_TAPS:
            raise ValueError(f"short convolutions longer than {MAX_TAPS} taps are not supported")
        # without a checkpoint: seeded random weights, created on the device tensor by tensor
        sd = state_dict if state_dict is not None else W.init_state_dict(cfg, dev, dt)
        # RMS norms are stored as offsets from one
        plus = 0.0 if cfg.block == "parallel" or cfg.layer_norm else 1.0
        f32 = lambda n: sd[n].to(device=dev, dtype=torch.float32).contiguous()
        norm = lambda n: plus + f32(n)
        bias = lambda n: f32(n + ".b") if cfg.layer_norm else None
        weight = lambda n: sd[n].to(device=dev, dtype=dt).contiguous()
        self.embed_w = weight("embed")
        self.head_w = self.embed_w if cfg.tied_head else weight("head")
        self.pos_w = weight("pos") if cfg.positions else None
        self.final_norm, self.final_bias = norm("final.norm"), bias("final.norm")
        mixers, ffs, norms, biases, gates, convs = {}, {}, {}, {}, {}, {}
        for i, layer in enumerate(cfg.layers):
            if layer.weights_of is not None:
                continue
            mixers[i] = make_mixer(cfg, i, dev, dt)
            mixers[i].load_weights(sd)
            p = f"l{i}.mlp."
            ffs[i] = RoutedFeedForward(sd, p, layer.routed, dev, dt) if layer.routed else \
                GatedFeedForward(sd, p, layer.ff, layer.act, dev, dt) if layer.ff else None
            names = W.layer_norm_names(cfg, i)
            norms[i] = {n: norm(f"l{i}.{n}") for n in names}
            biases[i] = {n: bias(f"l{i}.{n}") for n in names}
            # the gate of a sublayer goes with its norm
            gates[i] = {n: (weight(f"l{i}.{g}"), f32(f"l{i}.{g}.b")) for n, g in zip(names, ("rg1", "rg2"))} if cfg.residual_gate else {}
            convs[i] = f32(f"l{i}.canon1").T.contiguous() if cfg.input_conv else None
        owners = [cfg.weight_layer(i) for i in range(cfg.num_layers)]
        self.mixers, self.ffs, self.norms, self.biases, self.gates, self.convs = \
            ([x[j] for j in owners] for x in (mixers, ffs, norms, biases, gates, convs))
        self.attentions = [a for a in (m.attention() for m in self.mixers) if a is not None]
        self.blocks_of_rows = {m.blocks() for m in self.mixers} - {0}
        self.latent_specs = {LatentTables.key(l.mixer): l.mixer for l in cfg.layers if isinstance(l.mixer, LatentAttentionSpec)}
        self.decode_tables: Dict[int, Tuple[Dict[Tuple, LatentTables], Dict[int, torch.Tensor]]] = {}

    # ---- cache and state ------------------------------------------------------------------------------------------
    def _owns_kv(self, i: int) -> bool:
        m = self.cfg.layers[i].mixer
        return isinstance(m, (LatentAttentionSpec, SideBySideSpec)) or isinstance(m, AttentionSpec) and m.kv_from is None

    def _cache_bytes_per_block(self) -> int:
        el = torch.empty((), dtype=self.dtype).element_size()
        return sum(self.block_size * math.prod(s) * el for i, m in enumerate(self.mixers) if self._owns_kv(i)
                   for s in m.kv_shapes())

    def _allocate_cache(self) -> None:
        z = lambda *s: torch.zeros(*s, dtype=self.dtype, device=self.device)
        self.kv: Dict[int, Tuple[torch.Tensor, ...]] = {}
        self.states: Dict[int, RecurrentState] = {}
        # rings of the input convolutions, by position modulo taps
        self.inputs: List[torch.Tensor] = [z(self.max_batch_size, self.cfg.input_conv, self.cfg.hidden_size)
                                           for _ in self.cfg.layers] if self.cfg.input_conv else []
        for i, layer in enumerate(self.cfg.layers):
            m = layer.mixer
            if self._owns_kv(i):
                self.kv[i] = tuple(z(self.num_blocks, self.block_size, *s) for s in self.mixers[i].kv_shapes())
            elif isinstance(m, AttentionSpec):
                self.kv[i] = self.kv[m.kv_from]
            if hasattr(self.mixers[i], "recur"):
                self.states[i] = self.mixers[i].recur.new_state(self.max_batch_size, self.dtype, self.device)

    def _slot_tensors(self) -> List[torch.Tensor]:
        """Everything that is indexed by a sequence's slot."""
        return [t for i in sorted(self.states) for t in self.states[i].tensors()] + self.inputs

    def state_bytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in self._slot_tensors())

    def export_sequence(self, blocks: List[int], row: int) -> dict:
        idx = torch.tensor(blocks, device=self.device)
        return dict(pages=[t[idx].cpu() for i in sorted(self.kv) if self._owns_kv(i) for t in self.kv[i]],
                    state=[t[row].cpu() for t in self._slot_tensors()])

    def import_sequence(self, blocks: List[int], row: int, data: dict) -> None:
        caches = [t for i in sorted(self.kv) if self._owns_kv(i) for t in self.kv[i]]
        for t, p in zip(caches, data["pages"]):
            n = min(p.shape[0], len(blocks))
            t[torch.tensor(blocks[:n], device=self.device)] = p[:n].to(self.device)
        for t, s in zip(self._slot_tensors(), data["state"]):
            t[row] = s.to(self.device)

    def _make_buffers(self, cap: int) -> LayerListBuffers:
        # prompts sample one row per sequence; a step that wants more rows allocates its logits
        return LayerListBuffers(self.cfg, cap, self.device, self.dtype, min(cap, self.max_batch_size), self.mixers)

    # ---- one iteration ----------------------------------------------------------------------------------------------
    def _begin_prefill(self, buf: LayerListBuffers, T: int, positions, ctx_len, bt_row) -> None:
        buf.segments = build_segments(bt_row, positions, self.device)
        buf.prefill_tiles, buf.ctx_len_decode, buf.n_untiled = {}, None, T
        buf.latent = {k: LatentTables.prefill(m, bt_row, positions, self.device, self.dtype)
                      for k, m in self.latent_specs.items()}
        buf.block_offs = self._block_offs(T)
        for mixer in self.attentions:
            m = mixer.spec
            if not mixer.tiled():
                continue
            n = F.prefill_tile_tokens(m.heads, m.kv_heads)
            if n in buf.prefill_tiles:
                continue
            tiles, covered = F.build_prefill_tiles(bt_row, positions, n)
            if len(tiles):
                buf.prefill_tiles[n] = (tiles.to(self.device), len(tiles))
                cd = torch.as_tensor(ctx_len).clone()
                cd[covered] = 0              # which rows are tiled does not depend on the tile size
                buf.ctx_len_decode, buf.n_untiled = cd.to(self.device), int((~covered).sum())

    def _end_prefill(self, buf: LayerListBuffers) -> None:
        buf.segments, buf.prefill_tiles, buf.ctx_len_decode, buf.latent, buf.block_offs = None, {}, None, {}, {}

    def _block_offs(self, T: int) -> Dict[int, torch.Tensor]:
        return {n: (torch.arange(n + 1, dtype=torch.int32) * T).to(self.device) for n in self.blocks_of_rows}

    def _decode_tables(self, T: int) -> Tuple[Dict[Tuple, LatentTables], Dict[int, torch.Tensor]]:
        """Latent tables and block offsets, made once per batch size: graphs replay on them."""
        if T not in self.decode_tables:
            self.decode_tables[T] = ({k: LatentTables.decode(m, T, self.device) for k, m in self.latent_specs.items()},
                                     self._block_offs(T))
        return self.decode_tables[T]

    def _forward(self, buf: LayerListBuffers, T: int, max_ctx: int, want_logits: bool):
        cfg = self.cfg
        pos, slots, rows = buf.positions[:T], buf.slots[:T], buf.bt_row[:T]
        segs = buf.segments if buf.segments is not None else decode_segments(pos, rows, slots)
        prompts = buf.segments is not None
        latent, block_offs = (buf.latent, buf.block_offs) if prompts else self._decode_tables(T)
        meta = StepMeta(pos, slots, self.block_tables, rows, buf.ctx_len[:T], max_ctx=max_ctx,
                        num_decode_tokens=buf.n_untiled if prompts else T,
                        prefill_tiles=buf.prefill_tiles if prompts else None,
                        ctx_len_decode=buf.ctx_len_decode, segments=segs,
                        latent=latent, latent_out=buf.latent_out, block_offs=block_offs)
        resid = buf.resid[:T]
        F.embed_f32(buf.ids[:T], self.embed_w, cfg.embed_scale, resid, pos, self.pos_w)
        h = getattr(self, f"_{cfg.block}_blocks")(buf, resid, meta)
        n_out = h.shape[0]
        logits = gemm.linear(h, self.head_w, out=buf.logits[:n_out] if n_out <= buf.logits.shape[0] else None,
                             out_dtype=torch.float32)
        F.argmax(logits, out=buf.next_ids[:n_out])
        return buf.next_ids[:n_out], (logits if want_logits else None)

    def _memory(self, i: int):
        if i in self.states and i in self.kv:
            return self.kv[i], self.states[i]
        return self.states[i] if i in self.states else self.kv[i]

    def _sandwich_blocks(self, buf: LayerListBuffers, resid: torch.Tensor, meta: StepMeta) -> torch.Tensor:
        """All layers; returns the head's input rows."""
        cfg, eps, dt = self.cfg, self.cfg.rms_norm_eps, self.dtype
        h = F.resid_norm(resid, None, None, self.norms[0]["norm1"], eps, dt)
        for i, (mixer, ff, n) in enumerate(zip(self.mixers, self.ffs, self.norms)):
            y, post = mixer(h, self._memory(i), meta), n["norm1b"]
            if ff is not None:
                h = F.resid_norm(resid, y, post, n["norm2"], eps, dt)
                y, post = ff(h), n["norm2b"]
            if i + 1 == len(self.mixers):
                # the head's input carries the logit scale; only the rows that are sampled get that far
                return F.resid_norm(resid, y, post, self.final_norm, eps, dt, out_scale=cfg.logit_scale, rows=buf.out_rows)
            h = F.resid_norm(resid, y, post, self.norms[i + 1]["norm1"], eps, dt)

    def _parallel_blocks(self, buf: LayerListBuffers, resid: torch.Tensor, meta: StepMeta) -> torch.Tensor:
        eps, dt = self.cfg.rms_norm_eps, self.dtype
        y = z = None
        for i, (mixer, ff, n) in enumerate(zip(self.mixers, self.ffs, self.norms)):
            r = self.cfg.layers[i].routed
            rb = buf.routed[r.experts, r.top] if r else None
            h, ids, weights = F.sum_norm(resid, y, z, n["norm1"], eps, dt, True, router=ff.router(rb) if r else None)
            y = mixer(h, self._memory(i), meta)
            z = ff(h, ids, weights, rb) if r else ff(h) if ff is not None else None
        return F.sum_norm(resid, y, z, self.final_norm, eps, dt, True, rows=buf.out_rows)[0]

    def _prenorm_blocks(self, buf: LayerListBuffers, resid: torch.Tensor, meta: StepMeta) -> torch.Tensor:
        cfg, eps, dt = self.cfg, self.cfg.rms_norm_eps, self.dtype
        centred, mult = cfg.layer_norm, cfg.residual_mult
        y = z = gate = None             # what the last sublayer left to be added: rows, or rows per chosen expert, and their gate

        def gate_of(i, name, h):
            if name not in self.gates[i]:
                return None
            w, b = self.gates[i][name]
            return F.ResidualGate(gemm.linear(h, w), b)
        for i, (mixer, ff, n, b) in enumerate(zip(self.mixers, self.ffs, self.norms, self.biases)):
            memory = self._memory(i)
            conv = F.InputConv(self.convs[i], self.inputs[i], meta.segments) if self.inputs else None
            h, _, _ = F.sum_norm(resid, y, z, n["norm1"], eps, dt, centred, mult=mult, shift=mixer.shift(memory, meta),
                                 bias=b["norm1"], gate=gate, conv=conv)
            gate = gate_of(i, "norm1", h if conv is None else h[0])
            y, z = mixer(h if conv is None else h[1], memory, meta), None
            r = cfg.layers[i].routed
            rb = buf.routed[r.experts, r.top] if r else None
            if ff is not None:
                h, ids, weights = F.sum_norm(resid, y, None, n["norm2"], eps, dt, centred, mult=mult,
                                             router=ff.router(rb) if r else None, bias=b["norm2"], gate=gate)
                gate = gate_of(i, "norm2", h)
                y, z = (None, ff(h, ids, weights, rb)) if r else (ff(h), None)
        return F.sum_norm(resid, y, z, self.final_norm, eps, dt, centred, rows=buf.out_rows, mult=mult, bias=self.final_bias,
                          gate=gate)[0]
