"""Whole-iteration executor of a colocated worker: every layer's attention and experts on one device.

This is the one-GPU point of the throughput curve (the reference's ``ColocatePlacement`` + ``dual_module_loop``,
disagmoe/utils/placement.py:467-508, disagmoe/frontend/engine.py:873-904), restructured for Blackwell: a decode
iteration is one chain of kernels with no host round trip between the router and the expert GEMMs (the expert
histogram, offsets, sort and token records stay on the device), captured in a CUDA graph per batch-size bucket.

    embed -> L x [ add+RMSNorm -> QKV (tcgen05) -> RoPE + KV append -> paged attention -> o_proj + residual
                   -> RMSNorm + gate + top-k -> sort-by-expert dispatch -> grouped GEMM-1 + SwiGLU
                   -> grouped GEMM-2 with combine epilogue (router weight, un-permute) ]
          -> add+RMSNorm -> LM head -> argmax

The same code runs on CPU tensors (fp32) through the PyTorch restatements of the ops, which is how it is checked
against the oracle without a GPU.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..config import CacheConfig, ModelConfig
from ..models import weights as W
from ..models.attention import AttnMeta, MoEAttention
from ..models.experts import MoEExperts
from ..ops import functional as F
from ..ops import gemm
from .step import StepExecutor, TokenBuffers


class StepBuffers(TokenBuffers):
    """The token buffers plus the activations of the MoE decoder."""

    def __init__(self, cfg: ModelConfig, cap: int, device, dtype):
        super().__init__(cfg, cap, device, cap)
        H, k, E = cfg.hidden_size, cfg.top_k, cfg.num_experts
        z = lambda *s, dt=dtype: torch.zeros(*s, dtype=dt, device=device)
        self.resid = z(cap, H)
        self.parts = z(cap, k, H)
        self.dispatch = F.DispatchBuffers(cap * k, H, E, device, dtype)
        self.parts_base = torch.tensor([self.parts.data_ptr()], dtype=torch.int64, device=device)
        # prompt segments of the current step for the tiled causal attention kernel (filled by prefill())
        self.prefill_tiles = z(cap, 4, dt=torch.int32)
        self.ctx_len_decode = z(cap, dt=torch.int32)
        self.n_prefill_tiles = 0


class FusedModelExecutor(StepExecutor):
    def _load(self, state_dict: Optional[W.StateDict]) -> None:
        cfg = self.cfg
        self.attn: Dict[int, MoEAttention] = {}
        self.experts: Dict[int, MoEExperts] = {}
        for l in self.layer_ids:
            a = MoEAttention(cfg, l, device=self.device, dtype=self.dtype)
            a.load_weights(state_dict) if state_dict is not None else a.init_weights()
            self.attn[l] = a
            if not cfg.is_dense_layer(l):
                e = MoEExperts(cfg, l, device=self.device, dtype=self.dtype)
                e.load_weights(state_dict) if state_dict is not None else e.init_weights()
                self.experts[l] = e
        names = ["embed_tokens.weight", "norm.weight", "lm_head.weight"]
        sd = state_dict if state_dict is not None else W.init_state_dict(cfg, self.device, self.dtype, names)
        self.embed_w = sd["embed_tokens.weight"].to(device=self.device, dtype=self.dtype).contiguous()
        self.norm_w = sd["norm.weight"].to(device=self.device, dtype=self.dtype)
        self.lm_head_w = sd["lm_head.weight"].to(device=self.device, dtype=self.dtype).contiguous()

    def _cache_bytes_per_block(self) -> int:
        return len(self.layer_ids) * 2 * self.block_size * self.attn[self.layer_ids[0]].num_kv_heads * \
            self.cfg.head_dim * torch.empty((), dtype=self.dtype).element_size()

    def _allocate_cache(self) -> None:
        kv_heads = self.attn[self.layer_ids[0]].num_kv_heads
        # [layers, 2, num_blocks, block_size, kv_heads, head_dim] (reference: disagmoe/executor/executor.py:81-83)
        self.kv_cache = torch.zeros(len(self.layer_ids), 2, self.num_blocks, self.block_size, kv_heads, self.cfg.head_dim,
                                    dtype=self.dtype, device=self.device)

    def _make_buffers(self, cap: int) -> StepBuffers:
        return StepBuffers(self.cfg, cap, self.device, self.dtype)

    def export_sequence(self, blocks: List[int], row: int) -> dict:
        return dict(pages=self.kv_cache[:, :, torch.tensor(blocks, device=self.device)].cpu())

    def import_sequence(self, blocks: List[int], row: int, data: dict) -> None:
        pages = data["pages"]
        n = min(pages.shape[2], len(blocks))
        self.kv_cache[:, :, torch.tensor(blocks[:n], device=self.device)] = pages[:, :, :n].to(self.device)

    def kv_of(self, local_idx: int):
        return self.kv_cache[local_idx, 0], self.kv_cache[local_idx, 1]

    # ---- one iteration -------------------------------------------------------------------------------------------
    def _forward(self, buf: StepBuffers, T: int, max_ctx: int, want_logits: bool):
        cfg = self.cfg
        meta = AttnMeta(buf.positions[:T], buf.slots[:T], self.block_tables, buf.bt_row[:T], buf.ctx_len[:T],
                        max_ctx=max_ctx, prefill_tiles=buf.prefill_tiles, n_prefill_tiles=buf.n_prefill_tiles,
                        ctx_len_decode=buf.ctx_len_decode[:T])
        resid = buf.resid[:T]
        F.embed(buf.ids[:T], self.embed_w, out=resid)
        parts = None
        d = buf.dispatch
        for i, l in enumerate(self.layer_ids):
            a = self.attn[l]
            a.counts = d.counts
            out = a.forward(resid, parts, self.kv_of(i), meta)   # updates `resid` in place
            if out.expert_input is None:
                parts = None
                continue
            F.dispatch_local(out.expert_input, out.topk_ids, out.topk_weights, d)
            n = T * cfg.top_k
            if resid.is_cuda:
                self.experts[l].forward_combine(n, d.xs[:n], d.offs, d.recs[:n], buf.parts_base, cfg.hidden_size)
            else:
                self.experts[l].forward_combine(n, d.xs[:n], d.offs, d.recs[:n], None, cfg.hidden_size,
                                                outs=[buf.parts.view(-1, cfg.hidden_size)])
            parts = buf.parts[:T]
        _, h = F.add_rmsnorm(resid, parts, self.norm_w, cfg.rms_norm_eps, resid_out=resid)
        if buf.out_rows is not None:
            h = h.index_select(0, buf.out_rows)
            T = h.shape[0]
        logits = gemm.linear(h, self.lm_head_w, out=buf.logits[:T], out_dtype=torch.float32)
        F.argmax(logits, out=buf.next_ids[:T])
        return buf.next_ids[:T], (logits if want_logits else None)

    def _begin_prefill(self, buf: StepBuffers, T: int, positions, ctx_len, bt_row) -> None:
        buf.n_prefill_tiles = 0
        if self.device.type == "cuda":
            a0 = self.attn[self.layer_ids[0]]
            tiles, covered = F.build_prefill_tiles(bt_row, positions, F.prefill_tile_tokens(a0.num_heads, a0.num_kv_heads))
            if len(tiles):
                buf.n_prefill_tiles = len(tiles)
                buf.prefill_tiles[:len(tiles)].copy_(tiles, non_blocking=True)
                cd = torch.as_tensor(ctx_len).clone()
                cd[covered] = 0
                buf.ctx_len_decode[:T].copy_(cd, non_blocking=True)

    def _end_prefill(self, buf: StepBuffers) -> None:
        buf.n_prefill_tiles = 0
