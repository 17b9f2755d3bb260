"""Trace replay: given token ids instead of sampled ones, step by step, with the logits as output.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps.jsonl

DIR is a checkpoint folder (config.json, model.safetensors). Every input line is one engine step,

    {"step": 7, "entries": [{"id": "q1", "tokens": [311, 8], "want": [1]}, {"id": "q2", "tokens": [42], "want": [0]}], "end": ["q2"]}

whose entries run as one batch (portions of prompts beside single tokens) from the cache and state that earlier steps
left; ``want`` are the places among an entry's tokens whose logits are written, in order, to ``<out>/<step>.f32``
(little-endian fp32, [wanted, vocab]); the requests in ``end`` are finished after the step and give back their pages and
slot. After every step the line ``done <step>`` is printed. The engine is the serving engine
(:class:`disagmoe_b200.frontend.colocated.ColocatedEngine`) with a pool for ``--max-tokens`` tokens and slots for
``--max-requests`` live requests; nothing is sampled.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict, IO, Iterable

import torch

from ..config import CacheConfig
from ..models.registry import load_model
from .colocated import ColocatedEngine

BLOCK = 16


class TraceReplay:
    def __init__(self, model_dir: str, dtype: torch.dtype, max_tokens: int, max_requests: int = 4, device="cuda"):
        if torch.device(device).type == "cuda" and not torch.cuda.is_available():
            raise RuntimeError("no CUDA device")
        blocks = (max_tokens + BLOCK - 1) // BLOCK
        cfg, sd = load_model(model_dir, dtype, max_seq_len=blocks * BLOCK)
        self.engine = ColocatedEngine(cfg, CacheConfig(block_size=BLOCK), device=device, max_batch_size=max_requests,
                                      max_prefill_tokens=max(blocks * BLOCK, max_requests), state_dict=sd,
                                      num_blocks=blocks, dtype=dtype)
        self.engine.executor.capture(list(range(1, max_requests + 1)))
        self.ids: Dict[str, int] = {}
        self.next_id = 0

    def _sid(self, name: str) -> int:
        if name not in self.ids:
            self.ids[name] = self.next_id
            self.next_id += 1
        return self.ids[name]

    def step(self, entries, end) -> torch.Tensor:
        """Wanted logits of one step, fp32 on the CPU."""
        logits = self.engine.feed([(self._sid(e["id"]), e["tokens"], e["want"]) for e in entries]).float().cpu()
        self.engine.end_fed([self.ids.pop(name) for name in end if name in self.ids])
        return logits

    def replay(self, lines: Iterable[str], out_dir: str, stream: IO[str]) -> None:
        for line in lines:
            if not line.strip():
                continue
            s = json.loads(line)
            logits = self.step(s["entries"], s.get("end", ()))
            if logits.shape[0]:
                path = os.path.join(out_dir, "%d.f32" % s["step"])
                with open(path + ".tmp", "wb") as f:
                    f.write(logits.contiguous().numpy().astype("<f4").tobytes())
                os.replace(path + ".tmp", path)
            stream.write("done %d\n" % s["step"])
            stream.flush()


def main(argv=None) -> int:
    p = argparse.ArgumentParser(prog="trace_run", description="replay token ids through a model and write logits")
    p.add_argument("--model", required=True, help="checkpoint folder: config.json and model.safetensors")
    p.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"],
                   help="bfloat16: as served; float32: every product and activation in fp32")
    p.add_argument("--out", required=True, help="folder for <step>.f32")
    p.add_argument("--max-tokens", type=int, required=True, help="size of the KV pool in tokens")
    p.add_argument("--max-requests", type=int, default=4, help="state slots / live requests")
    args = p.parse_args(argv)
    os.makedirs(args.out, exist_ok=True)
    replay = TraceReplay(args.model, getattr(torch, args.dtype), args.max_tokens, args.max_requests)
    replay.replay(sys.stdin, args.out, sys.stdout)
    return 0
