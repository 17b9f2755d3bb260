"""Single-GPU serving engine: every layer's attention and experts colocated on one device.

The in-process counterpart of a one-worker ``ColocatePlacement`` deployment (reference: disagmoe/utils/placement.py:
467-508, disagmoe/frontend/engine.py:873-904): continuous batching over the whole-iteration executor that the model
registry picks for the configuration (MoE decoders: :class:`disagmoe_b200.executor.fused.FusedModelExecutor`, layer-list
decoders: :class:`disagmoe_b200.executor.layer_list.LayerListExecutor`), the native paged-KV ``BlockManager`` with a
device-resident block table that is patched incrementally, pinned host staging for the per-step inputs and a
device->host read of the sampled ids (the sampler lives on the host, as in the reference).
"""
from __future__ import annotations

import time
from dataclasses import dataclass, field
from typing import Dict, List, Optional, Sequence, Tuple

import torch

from .. import disagmoe_c as C
from ..config import CacheConfig, ModelConfig
from ..models.registry import make_executor
from ..utils.constants import EOS_TOKEN_ID


@dataclass
class _Seq:
    req_id: int
    prompt: List[int]
    max_new_tokens: int
    length: int = 0                 # tokens whose K/V are cached
    last_token: int = 0             # next input token
    outputs: List[int] = field(default_factory=list)
    t_arrival: float = 0.0
    t_tokens: List[float] = field(default_factory=list)


class ColocatedEngine:
    def __init__(self, cfg: ModelConfig, cache_cfg: Optional[CacheConfig] = None, device="cuda", max_batch_size: int = 256,
                 max_prefill_tokens: int = 4096, state_dict=None, num_blocks: Optional[int] = None,
                 enable_cuda_graph: bool = True, ignore_eos: bool = True, dtype=None):
        self.cfg = cfg
        self.cache_cfg = cache_cfg or CacheConfig()
        self.device = torch.device(device)
        self.max_batch_size = max_batch_size
        self.ignore_eos = ignore_eos
        self.executor = make_executor(cfg, self.cache_cfg, device=device, dtype=dtype, max_batch_size=max_batch_size,
                                      max_prefill_tokens=max_prefill_tokens, state_dict=state_dict,
                                      num_blocks=num_blocks, enable_cuda_graph=enable_cuda_graph)
        self.block_size = self.cache_cfg.block_size
        self.block_mgr = C.BlockManager(self.block_size, self.executor.num_blocks - self.cache_cfg.num_reserved_blocks,
                                        self.cache_cfg.num_reserved_blocks, max_batch_size)
        self.waiting: List[_Seq] = []
        self.running: Dict[int, _Seq] = {}    # insertion ordered
        self.finished: Dict[int, _Seq] = {}
        self.fed: Dict[int, int] = {}         # sequences driven by feed(): tokens cached so far
        pin = self.device.type == "cuda"
        B = max(max_batch_size, max_prefill_tokens)
        mk = lambda dt: torch.zeros(B, dtype=dt, pin_memory=pin)
        self._h_ids, self._h_pos, self._h_ctx, self._h_row = mk(torch.int32), mk(torch.int32), mk(torch.int32), mk(torch.int32)
        self._h_slots = mk(torch.int64)
        self._h_out = torch.zeros(B, dtype=torch.int32, pin_memory=pin)
        self._h_patch = torch.zeros(3, 4 * B + 1024, dtype=torch.int64, pin_memory=pin)
        self.h2d_bytes_last = 0
        self.d2h_bytes_last = 0
        self.steps = 0
        self._last_was_prefill = False
        self.profile_events = False     # when set, every decode step appends a (start, end) CUDA event pair
        self.event_pairs = []

    # ---- requests -----------------------------------------------------------------------------------------------
    def add_request(self, req_id: int, prompt_ids: List[int], max_new_tokens: int) -> None:
        assert len(prompt_ids) >= 1 and len(prompt_ids) + max_new_tokens <= self.cfg.max_seq_len
        self.waiting.append(_Seq(req_id, list(prompt_ids), max_new_tokens, t_arrival=time.time()))

    def add_synthetic_request(self, req_id: int, context_len: int, next_token: int, max_new_tokens: int) -> None:
        """A sequence that already has ``context_len`` cached tokens (whatever the KV cache holds at its blocks):
        used by benchmarks that measure decode throughput at a given context length without running the prefill."""
        assert len(self.running) < self.max_batch_size
        s = _Seq(req_id, [], max_new_tokens, length=context_len, last_token=next_token, t_arrival=time.time())
        self.block_mgr.allocate(req_id, context_len + 1)
        self.running[req_id] = s
        self._apply_block_table_patches()

    def has_unfinished(self) -> bool:
        return bool(self.waiting or self.running)

    # ---- block table --------------------------------------------------------------------------------------------
    def _apply_block_table_patches(self) -> int:
        ups = self.block_mgr.drain_updates()
        if not ups:
            return 0
        n = len(ups)
        if n > self._h_patch.shape[1]:
            self._h_patch = torch.zeros(3, 2 * n, dtype=torch.int64, pin_memory=self._h_patch.is_pinned())
        t = torch.tensor(ups, dtype=torch.int64)          # [n, 3] rows, cols, blocks
        self._h_patch[:, :n] = t.T
        d = self._h_patch[:, :n].to(self.device, non_blocking=True)
        self.executor.block_tables.index_put_((d[0], d[1]), d[2].int())
        return 3 * 8 * n

    # ---- steps --------------------------------------------------------------------------------------------------
    def _execute(self, ids, pos, rows, slots, out_rows: Optional[List[int]] = None, decode_only: bool = False,
                 want_logits: bool = False):
        """One pass of the executor over a batch of rows (token ids, positions, block-table rows, KV slots): staging,
        block-table patches, then the decode path (one token per sequence) or the general one. Returns device tensors
        (next ids, logits or None) of ``out_rows``, or of every row."""
        T = len(ids)
        h2d = self._apply_block_table_patches()
        self._h_ids.numpy()[:T] = ids
        self._h_pos.numpy()[:T] = pos
        self._h_ctx.numpy()[:T] = self._h_pos.numpy()[:T] + 1
        self._h_row.numpy()[:T] = rows
        self._h_slots.numpy()[:T] = slots
        self.h2d_bytes_last += h2d + T * 24
        args = (self._h_ids[:T], self._h_pos[:T], self._h_slots[:T], self._h_ctx[:T], self._h_row[:T])
        if not decode_only:
            return self.executor.prefill(*args, want_logits=want_logits, out_rows=out_rows)
        nxt, logits = self.executor.decode(*args, want_logits=want_logits)
        if out_rows is None or out_rows == list(range(T)):
            return nxt, logits
        pick = torch.tensor(out_rows, dtype=torch.long, device=nxt.device)
        return nxt[pick], (logits[pick] if logits is not None else None)

    def _slots(self, req_id: int, start: int, n: int) -> List[int]:
        """KV slots of positions start .. start + n - 1 of a sequence."""
        blocks, bs = self.block_mgr.get_seq_block_list(req_id), self.block_size
        return [blocks[p // bs] * bs + p % bs for p in range(start, start + n)]

    def feed(self, entries: Sequence[Tuple[int, Sequence[int], Sequence[int]]]) -> torch.Tensor:
        """One engine step over given tokens instead of sampled ones: ``entries`` = (sequence id, its next tokens, places
        among them whose logits are wanted); all entries run as one batch, portions of prompts beside single decode tokens,
        from what earlier steps left in the cache and the state. Sequences are admitted at their first entry and hold their
        pages and slot until :meth:`end_fed`. Returns the wanted logits [n, vocab] in the order of entries and places."""
        if len(set(self.fed) | {sid for sid, _, _ in entries}) > self.max_batch_size:
            raise ValueError(f"more than {self.max_batch_size} live sequences")
        ids, pos, rows, slots, want = [], [], [], [], []
        for sid, tokens, places in entries:
            n, start = len(tokens), self.fed.get(sid)
            if n == 0:
                continue
            if (start or 0) + n > self.cfg.max_seq_len:
                raise ValueError(f"sequence {sid} would grow beyond {self.cfg.max_seq_len} tokens")
            if start is None:
                start = 0
                self.block_mgr.allocate(sid, n)
            else:
                self.block_mgr.append_tokens(sid, start, n)
            want += [len(ids) + p for p in places]
            ids += tokens
            pos += range(start, start + n)
            rows += [self.block_mgr.row_of(sid)] * n
            slots += self._slots(sid, start, n)
            self.fed[sid] = start + n
        if not ids:
            return torch.empty(0, self.cfg.vocab_size)
        decode_only = all(len(tokens) <= 1 for _, tokens, _ in entries)
        _, logits = self._execute(ids, pos, rows, slots, out_rows=want or [0], decode_only=decode_only, want_logits=True)
        if self.device.type == "cuda":
            torch.cuda.current_stream().synchronize()      # the staging buffers are free again
        return logits[:len(want)]

    def end_fed(self, seq_ids: Sequence[int]) -> None:
        """Gives back the pages and slots of sequences driven by :meth:`feed`."""
        for sid in seq_ids:
            if self.fed.pop(sid, None) is not None:
                self.block_mgr.release(sid)

    def _blocks(self, tokens: int) -> int:
        return (tokens + self.block_size - 1) // self.block_size

    def _prefill(self) -> List[Tuple[int, int]]:
        ex = self.executor
        batch: List[_Seq] = []
        total = 0
        # blocks the running sequences will still take before they finish stay free: a decode step never finds the
        # pool empty (there is no preemption)
        reserve = sum(max(0, self._blocks(max(len(s.prompt), s.length) + s.max_new_tokens - len(s.outputs)) -
                          len(self.block_mgr.get_seq_block_list(s.req_id))) for s in self.running.values())
        while self.waiting and len(self.running) + len(batch) < self.max_batch_size:
            s = self.waiting[0]
            need = self._blocks(len(s.prompt) + s.max_new_tokens)
            if total + len(s.prompt) > ex.prefill_buf.cap or self.block_mgr.num_free_blocks() - reserve < need:
                break
            reserve += need - self._blocks(len(s.prompt) + 1)
            self.waiting.pop(0)
            self.block_mgr.allocate(s.req_id, len(s.prompt) + 1)
            batch.append(s)
            total += len(s.prompt)
        if not batch:
            return []
        ids, pos, rows, slots, ends = [], [], [], [], []
        for s in batch:
            n = len(s.prompt)
            ids += s.prompt
            pos += range(n)
            rows += [self.block_mgr.row_of(s.req_id)] * n
            slots += self._slots(s.req_id, 0, n)
            ends.append(len(ids) - 1)
        nxt, _ = self._execute(ids, pos, rows, slots, out_rows=ends)
        out = nxt.cpu()
        res = []
        now = time.time()
        for i, s in enumerate(batch):
            s.length = len(s.prompt)
            tok = int(out[i])
            self._record(s, tok, now)
            res.append((s.req_id, tok))
        self.d2h_bytes_last += len(batch) * 4
        return res

    def _record(self, s: _Seq, tok: int, now: float) -> None:
        s.outputs.append(tok)
        s.t_tokens.append(now)
        s.last_token = tok
        done = len(s.outputs) >= s.max_new_tokens or (not self.ignore_eos and tok == EOS_TOKEN_ID)
        if done:
            self.block_mgr.release(s.req_id)
            self.finished[s.req_id] = s
            self.running.pop(s.req_id, None)
        else:
            self.running[s.req_id] = s

    def _decode(self) -> List[Tuple[int, int]]:
        seqs = list(self.running.values())
        B = len(seqs)
        if B == 0:
            return []
        lens = [s.length for s in seqs]
        rs = self.block_mgr.step_decode([s.req_id for s in seqs], lens)
        ev = None
        if self.profile_events and self.device.type == "cuda":
            ev = (torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True))
            ev[0].record()
        nxt, _ = self._execute([s.last_token for s in seqs], lens, rs[:B], rs[B:], decode_only=True)
        self._h_out[:B].copy_(nxt, non_blocking=True)
        if ev is not None:
            ev[1].record()
            self.event_pairs.append(ev)
        if self.device.type == "cuda":
            torch.cuda.current_stream().synchronize()
        toks = self._h_out[:B].tolist()
        now = time.time()
        res = []
        for s, tok in zip(seqs, toks):
            s.length += 1
            self._record(s, tok, now)
            res.append((s.req_id, tok))
        self.d2h_bytes_last += B * 4
        return res

    def step(self) -> List[Tuple[int, int]]:
        """One engine iteration: prefill newly admitted requests (if any), else one decode token for every running
        sequence. Returns (req_id, token) pairs produced by this step."""
        self.h2d_bytes_last = self.d2h_bytes_last = 0
        self.steps += 1
        # prefill and decode steps alternate while both have work, so a burst of arrivals cannot stall the running
        # sequences for more than one prefill step (bounds the inter-token latency tail)
        want_prefill = self.waiting and len(self.running) < self.max_batch_size
        if want_prefill and not (self._last_was_prefill and self.running):
            out = self._prefill()
            if out:
                self._last_was_prefill = True
                return out
        self._last_was_prefill = False
        return self._decode()

    # ---- serving-state snapshot ----------------------------------------------------------------------------------
    def save_state(self, path: str) -> None:
        """Writes the request table and the KV pages (and recurrent state) of every live sequence (between two steps). A new engine with the
        same weights continues from it with :meth:`load_state` and produces the same tokens."""
        seqs = []
        for s in self.running.values():
            blocks = self.block_mgr.get_seq_block_list(s.req_id)
            cached = self.executor.export_sequence(blocks, self.block_mgr.row_of(s.req_id))
            seqs.append(dict(req_id=s.req_id, prompt=s.prompt, max_new_tokens=s.max_new_tokens, length=s.length,
                             last_token=s.last_token, outputs=list(s.outputs), cached=cached))
        waiting = [dict(req_id=s.req_id, prompt=s.prompt, max_new_tokens=s.max_new_tokens) for s in self.waiting]
        finished = {r: list(s.outputs) for r, s in self.finished.items()}
        tmp = path + ".tmp"
        torch.save(dict(running=seqs, waiting=waiting, finished=finished, block_size=self.block_size), tmp)
        import os
        os.replace(tmp, path)

    def load_state(self, path: str) -> None:
        st = torch.load(path, map_location="cpu", weights_only=True)   # plain containers + tensors only
        assert st["block_size"] == self.block_size and not self.running and not self.waiting
        for d in st["running"]:
            s = _Seq(d["req_id"], d["prompt"], d["max_new_tokens"], length=d["length"], last_token=d["last_token"],
                     outputs=list(d["outputs"]), t_arrival=time.time())
            self.block_mgr.allocate(s.req_id, s.length + 1)
            blocks = self.block_mgr.get_seq_block_list(s.req_id)
            self.executor.import_sequence(blocks, self.block_mgr.row_of(s.req_id), d["cached"])
            self.running[s.req_id] = s
        for d in st["waiting"]:
            self.add_request(d["req_id"], d["prompt"], d["max_new_tokens"])
        for r, outs in st["finished"].items():
            self.finished[r] = _Seq(r, [], len(outs), outputs=list(outs))
        self._apply_block_table_patches()

    def launch_count(self) -> int:
        from ..ops import _lib
        return _lib.LAUNCHES

    def tokens_per_step(self) -> int:
        return len(self.running)

    def run_until_done(self, max_steps: int = 1 << 30) -> Dict[int, List[int]]:
        n = 0
        while self.has_unfinished() and n < max_steps:
            self.step()
            n += 1
        return {r: s.outputs for r, s in self.finished.items()}
