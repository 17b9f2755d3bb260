"""What every whole-iteration executor shares: static per-token input buffers, the device block table, packed prefill,
decode and its CUDA graphs per batch-size bucket. A model family derives from :class:`StepExecutor` and supplies its
weights, its cache and ``_forward``.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..config import CacheConfig, ModelConfig
from ..ops import _lib
from ..utils.utils import get_graph_batch_size, graph_batch_sizes


class TokenBuffers:
    """Static inputs and outputs for up to ``cap`` tokens (CUDA graphs replay on fixed addresses)."""

    def __init__(self, cfg: ModelConfig, cap: int, device, logit_rows: int):
        self.cap = cap
        z = lambda *s, dt=torch.int32: torch.zeros(*s, dtype=dt, device=device)
        self.ids, self.positions, self.ctx_len, self.bt_row, self.next_ids = (z(cap) for _ in range(5))
        self.slots = z(cap, dt=torch.int64)
        self.logits = z(logit_rows, cfg.vocab_size, dt=torch.float32)
        self.out_rows: Optional[torch.Tensor] = None      # rows whose logits are wanted (None: all), set per step


class StepExecutor:
    def __init__(self, cfg: ModelConfig, cache_cfg: CacheConfig, device="cuda", dtype: Optional[torch.dtype] = None,
                 max_batch_size: int = 256, max_prefill_tokens: int = 4096, state_dict=None,
                 num_blocks: Optional[int] = None, enable_cuda_graph: bool = True, layer_ids: Optional[List[int]] = None):
        self.cfg, self.cache_cfg = cfg, cache_cfg
        self.device = torch.device(device)
        self.dtype = dtype or cfg.dtype
        self.block_size = cache_cfg.block_size
        self.max_batch_size = max_batch_size
        self.max_blocks_per_seq = (cfg.max_seq_len + self.block_size - 1) // self.block_size
        self.layer_ids = list(range(cfg.num_layers)) if layer_ids is None else layer_ids
        self.enable_cuda_graph = enable_cuda_graph and self.device.type == "cuda"
        self._load(state_dict)
        self.num_blocks = num_blocks or cache_cfg.num_gpu_blocks or self._profile_num_blocks()
        self._allocate_cache()
        self.block_tables = torch.zeros(max_batch_size, self.max_blocks_per_seq, dtype=torch.int32, device=self.device)
        self.decode_buf = self._make_buffers(max_batch_size)
        self.prefill_buf = self._make_buffers(max_prefill_tokens) if max_prefill_tokens > max_batch_size else self.decode_buf
        self.graphs: Dict[int, torch.cuda.CUDAGraph] = {}
        self.graph_sizes: List[int] = []
        self.graph_launches: Dict[int, int] = {}

    # ---- supplied by a model family -----------------------------------------------------------------------------
    def _load(self, state_dict) -> None:
        raise NotImplementedError

    def _cache_bytes_per_block(self) -> int:
        raise NotImplementedError

    def _allocate_cache(self) -> None:
        raise NotImplementedError

    def _make_buffers(self, cap: int) -> TokenBuffers:
        raise NotImplementedError

    def _forward(self, buf: TokenBuffers, T: int, max_ctx: int, want_logits: bool):
        """Runs the first T rows of ``buf``; returns (next ids, logits or None) of ``buf.out_rows`` (or of all rows)."""
        raise NotImplementedError

    def _begin_prefill(self, buf: TokenBuffers, T: int, positions, ctx_len, bt_row) -> None:
        """Host-side tables of a packed batch of prompt (and decode) rows."""

    def _end_prefill(self, buf: TokenBuffers) -> None:
        """Undoes ``_begin_prefill``: the decode path (and its graphs) may share the buffers."""

    def export_sequence(self, blocks: List[int], row: int) -> dict:
        """CPU copies of everything cached for one sequence (KV pages, recurrent state)."""
        raise NotImplementedError

    def import_sequence(self, blocks: List[int], row: int, data: dict) -> None:
        raise NotImplementedError

    # ---- memory -------------------------------------------------------------------------------------------------
    def _profile_num_blocks(self) -> int:
        if self.device.type != "cuda":
            return 512
        free, total = torch.cuda.mem_get_info(self.device)
        budget = free - (1.0 - self.cache_cfg.gpu_memory_utilization) * total - (6 << 30)
        return max(64, int(budget // max(1, self._cache_bytes_per_block())))

    # ---- one iteration -------------------------------------------------------------------------------------------
    def _fill(self, buf, T, ids, positions, slots, ctx_len, bt_row):
        nb = self.device.type == "cuda"
        buf.ids[:T].copy_(ids, non_blocking=nb)
        buf.positions[:T].copy_(positions, non_blocking=nb)
        buf.slots[:T].copy_(slots, non_blocking=nb)
        buf.ctx_len[:T].copy_(ctx_len, non_blocking=nb)
        buf.bt_row[:T].copy_(bt_row, non_blocking=nb)

    def set_block_table_row(self, row: int, blocks: List[int]) -> None:
        t = torch.tensor(blocks, dtype=torch.int32)
        self.block_tables[row, :len(blocks)].copy_(t)

    def prefill(self, ids, positions, slots, ctx_len, bt_row, want_logits=False, out_rows: Optional[List[int]] = None):
        """Eager pass over prompt tokens (any number of sequences packed together, decode rows among them). Host tensors
        in, device out. ``out_rows``: the rows to sample (and whose logits to return), in this order; None = all."""
        T = ids.shape[0]
        assert T <= self.prefill_buf.cap, f"{T} prefill tokens exceed the buffer ({self.prefill_buf.cap})"
        buf = self.prefill_buf
        self._fill(buf, T, ids, positions, slots, ctx_len, bt_row)
        self._begin_prefill(buf, T, positions, ctx_len, bt_row)
        if out_rows is not None:
            buf.out_rows = torch.tensor(out_rows, dtype=torch.int32).to(self.device)
        try:
            return self._forward(buf, T, int(ctx_len.max()), want_logits)
        finally:
            buf.out_rows = None
            self._end_prefill(buf)

    def capture(self, sizes: Optional[List[int]] = None) -> None:
        """Warm-up (compiles nothing, but sizes scratch buffers and sets kernel attributes) and graph capture."""
        if not self.enable_cuda_graph:
            return
        sizes = sizes or graph_batch_sizes(self.max_batch_size, self.cfg.graph_stride * 4)
        buf = self.decode_buf
        buf.ctx_len.fill_(1)
        buf.slots.fill_(-1)
        side = torch.cuda.Stream(self.device)
        for b in sorted(set(sizes), reverse=True):
            side.wait_stream(torch.cuda.current_stream())
            with torch.cuda.stream(side):
                for _ in range(2):
                    self._forward(buf, b, self.cfg.max_seq_len, False)
            torch.cuda.current_stream().wait_stream(side)
            torch.cuda.synchronize()
            g = torch.cuda.CUDAGraph()
            n0 = _lib.LAUNCHES
            with torch.cuda.graph(g):
                self._forward(buf, b, self.cfg.max_seq_len, False)
            self.graphs[b] = g
            self.graph_launches[b] = _lib.LAUNCHES - n0
        self.graph_sizes = sorted(self.graphs)
        torch.cuda.synchronize()

    def decode(self, ids, positions, slots, ctx_len, bt_row=None, want_logits=False):
        """One decode iteration for B sequences (one token each). Inputs are host (pinned) or device tensors of
        length B; returns the device tensor of greedy next-token ids (and logits when asked; they are overwritten by the
        next step)."""
        B = ids.shape[0]
        buf = self.decode_buf
        if bt_row is None:
            bt_row = torch.arange(B, dtype=torch.int32)
        if self.graph_sizes and B <= self.graph_sizes[-1]:
            _, b = get_graph_batch_size(B, self.graph_sizes)
            self._fill(buf, B, ids, positions, slots, ctx_len, bt_row)
            if b > B:
                # padding rows: no KV append, no state update, attend to nothing
                buf.slots[B:b].fill_(-1)
                buf.ctx_len[B:b].fill_(0)
                buf.ids[B:b].fill_(0)
            self.graphs[b].replay()
            _lib.add_launches(self.graph_launches[b])
            return buf.next_ids[:B], (buf.logits[:B] if want_logits else None)
        self._fill(buf, B, ids, positions, slots, ctx_len, bt_row)
        return self._forward(buf, B, int(ctx_len.max()) if not ctx_len.is_cuda else self.cfg.max_seq_len, want_logits)
