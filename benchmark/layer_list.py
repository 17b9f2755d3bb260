"""Prefill and decode throughput of layer-list decoders beside the closest decoder of the package at equal size.

    python bench.py --layer-list [rurunex | supinex | vufinex | panarax] [--steps K --warmup W]

Both run through the same engine classes with random weights.
  rurunex  repeats (gated linear attention, channel-wise delta rule, windowed attention), every layer with a gated
           feed-forward; beside the MoE decoder with a dense feed-forward in every layer and full attention: same width, heads,
           feed-forward and number of layers
  supinex  repeats (attention over everything, windowed latent attention), experts in every layer but the first; beside the MoE
           decoder with the same width, heads, experts and number of layers
  vufinex  repeats (RWKV-style time mixing, gated latent attention, chunked attention), experts in every layer; beside the MoE
           decoder with the same width, heads, experts and number of layers
  panarax  repeats (attention beside a matrix memory with a dense feed-forward, gated diagonal recurrence, lightning attention, both
           with experts); beside the MoE decoder with the same width, heads, experts and numbers of dense and expert layers
Prints one JSON line per (size, phase, model): tokens/s from device-timed steps (CUDA events, L2 flushed between steps), and
one per (size, phase) with the device time per kernel.
"""
from __future__ import annotations

import json
import math
import statistics
from typing import Dict, List

import torch

from disagmoe_b200.config import (AttentionSpec, CacheConfig, ChannelDeltaSpec, GatedLinearSpec, GatedUnitSpec, HeadDecaySpec,
                                  LatentAttentionSpec, LayerListConfig, LayerSpec, MatrixMemorySpec, ModelConfig, QueryTemperature,
                                  RotarySpec, RoutedSpec, SideBySideSpec, WkvSpec)
from disagmoe_b200.frontend.colocated import ColocatedEngine
from disagmoe_b200.ops import _lib, gemm

# name: width, heads, kv heads, head size, feed-forward, layers
SIZES = {"1024": (1024, 8, 2, 128, 2816, 6), "2048": (2048, 16, 4, 128, 5632, 6), "4096": (4096, 32, 8, 128, 11264, 6)}
# the same, then: latent rank, experts, experts per token (the feed-forward is an expert's; the dense first layer has 4 of them)
MOE_SIZES = {"1024": (1024, 8, 2, 128, 768, 6, 256, 32, 4), "2048": (2048, 16, 4, 128, 1408, 6, 512, 64, 6),
             "4096": (4096, 32, 8, 128, 4096, 6, 512, 16, 2)}
VOCAB = 32000


def hybrid_config(size: str, window: int = 1024, max_seq_len: int = 8192) -> LayerListConfig:
    W, H, G, D, ff, n = SIZES[size]
    layers: List[LayerSpec] = []
    for i in range(0, n, 3):
        attn = AttentionSpec(H, G, D, D, D ** -0.5, RotarySpec(D, 1e6, 4.0, 8192), window, 30.0, 2 if i else None)
        layers += [LayerSpec(GatedLinearSpec(H, D, D, 16.0, 16), ff), LayerSpec(ChannelDeltaSpec(H, H, D, D, 4, D, D), ff),
                   LayerSpec(attn, ff)]
    return LayerListConfig.make(W, VOCAB, layers, max_seq_len=max_seq_len, embed_scale=32.0, name="rurunex-" + size)


def dense_config(size: str, max_seq_len: int = 8192) -> ModelConfig:
    W, H, G, D, ff, n = SIZES[size]
    return ModelConfig(hidden_size=W, num_layers=n, num_heads=H, num_kv_heads=G, num_experts=1, intermediate_size=ff,
                       dtype=torch.bfloat16, ep_size=1, top_k=1, vocab_size=VOCAB, head_dim=D, rope_theta=1e6,
                       first_k_dense=n, dense_intermediate_size=ff, max_seq_len=max_seq_len, name="dense-" + size)


def parallel_config(size: str, window: int = 1024, max_seq_len: int = 8192) -> LayerListConfig:
    W, H, G, D, ff, n, rank, E, K = MOE_SIZES[size]
    attn = AttentionSpec(H, G, D, D, D ** -0.5, RotarySpec(D, 5e5, interleaved=True), qk_norm=False, sink=True, v_mix=True)
    lat = LatentAttentionSpec(H, D, D // 2, D, rank, (D + D // 2) ** -0.5, window=window, sink=True,
                              rot=RotarySpec(D // 2, 1e6, 4.0, 8192, interleaved=True))
    moe = RoutedSpec(E, K, ff)
    layers = [LayerSpec(attn if i % 2 == 0 else lat, routed=moe) if i else LayerSpec(attn, 4 * ff, "gelu_tanh") for i in range(n)]
    return LayerListConfig.make(W, VOCAB, layers, max_seq_len=max_seq_len, block="parallel", name="supinex-" + size)


def prenorm_config(size: str, chunk: int = 1024, max_seq_len: int = 8192) -> LayerListConfig:
    W, H, G, D, ff, n, rank, E, K = MOE_SIZES[size]
    moe = RoutedSpec(E, K, ff, renormalize=True, scoring="sigmoid", correction=True, groups=8, keep=4, scale=2.0)
    mixers = (WkvSpec(2 * H, D // 2, D // 2),
              LatentAttentionSpec(H, D, D // 2, D, rank, (D + D // 2) ** -0.5, RotarySpec(D // 2, 1e6, interleaved=True), gate=True),
              AttentionSpec(H, G, D, D, D ** -0.5, RotarySpec(D // 2, 5e5), qk_norm=False, chunk=chunk, tied_values=True))
    return LayerListConfig.make(W, VOCAB, [LayerSpec(mixers[i % 3], routed=moe) for i in range(n)], max_seq_len=max_seq_len,
                                block="prenorm", embed_scale=32.0, residual_mult=0.5, name="vufinex-" + size)


def gated_config(size: str, max_seq_len: int = 8192) -> LayerListConfig:
    W, H, G, D, ff, n, _, E, K = MOE_SIZES[size]
    moe = RoutedSpec(E, K, ff, act="clamped", scoring="sigmoid", limit=7.0, weigh_input=True)
    both = SideBySideSpec(AttentionSpec(H, G, D, D, D ** -0.5, qk_norm=False, value_norm=True, gate=True, q_temp=QueryTemperature(0.1, 1024)),
                          MatrixMemorySpec(H // 2, D, D, 15.0))
    decays = HeadDecaySpec(H, D, D, tuple(math.exp(-2.0 ** (-8.0 * (i + 1) / H)) for i in range(H)))
    layers = [LayerSpec(both, 4 * ff), LayerSpec(GatedUnitSpec(H * D, H, 4), routed=moe), LayerSpec(decays, routed=moe)]
    return LayerListConfig.make(W, VOCAB, layers * (n // 3), max_seq_len=max_seq_len, block="prenorm", layer_norm=True, residual_gate=True,
                                input_conv=4, positions=max_seq_len, tied_head=True, name="panarax-" + size)


def moe_config(size: str, max_seq_len: int = 8192, dense_layers: int = 1) -> ModelConfig:
    W, H, G, D, ff, n, _, E, K = MOE_SIZES[size]
    return ModelConfig(hidden_size=W, num_layers=n, num_heads=H, num_kv_heads=G, num_experts=E, intermediate_size=ff,
                       dtype=torch.bfloat16, ep_size=1, top_k=K, vocab_size=VOCAB, head_dim=D, rope_theta=5e5,
                       norm_topk_prob=False, first_k_dense=dense_layers, dense_intermediate_size=4 * ff, max_seq_len=max_seq_len,
                       name="moe-" + size)


def make_engine(cfg, batch: int, prompt_tokens: int, ctx: int, steps: int) -> ColocatedEngine:
    blocks = max(batch * ((ctx + steps + 32) // 16 + 1), prompt_tokens // 16 + 64)
    eng = ColocatedEngine(cfg, CacheConfig(block_size=16), device="cuda", max_batch_size=batch,
                          max_prefill_tokens=max(batch, prompt_tokens), num_blocks=blocks)
    ex = eng.executor
    if hasattr(ex, "kv_cache"):
        ex.kv_cache.normal_(0, 0.5)
    else:
        for t in (t for kv in ex.kv.values() for t in kv):
            t.normal_(0, 0.5)
        for s in ex.states.values():
            s.S.normal_(0, 0.1)
    ex.capture([batch])
    return eng


class Flush:
    """Overwrites a buffer larger than L2 between timed steps."""

    def __init__(self):
        self.buf = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")

    def __call__(self):
        self.buf.zero_()


def timed(fn, steps: int, warmup: int, flush) -> float:
    """Median device milliseconds of fn."""
    out = []
    for i in range(warmup + steps):
        flush()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        fn()
        b.record()
        torch.cuda.synchronize()
        if i >= warmup:
            out.append(a.elapsed_time(b))
    return statistics.median(out)


def kernel_times(fn) -> Dict[str, list]:
    fn()
    torch.cuda.synchronize()
    _lib.start_timeline()
    fn()
    return {k: [n, round(ms, 4)] for k, (n, ms) in sorted(_lib.stop_timeline().items(), key=lambda kv: -kv[1][1])}


def rows_of(n_seqs: int, length: int, block: int = 16):
    """Host tensors of n_seqs prompts of one length, each in its own pages and row."""
    pos = torch.arange(length, dtype=torch.int32).repeat(n_seqs)
    row = torch.arange(n_seqs, dtype=torch.int32).repeat_interleave(length)
    per = (length + block - 1) // block * block
    slots = row.long() * per + pos.long()
    ids = torch.randint(0, VOCAB, (n_seqs * length,), generator=torch.Generator().manual_seed(0), dtype=torch.int32)
    return ids, pos, slots, pos + 1, row, per // block


def main(args) -> int:
    flush = Flush()
    for size in (args.layer_list_sizes or "1024,2048,4096").split(","):
        for phase, n, length in (("prefill", 1, 4096), ("prefill", 4, 2048), ("decode", 16, 2048), ("decode", 256, 1024)):
            for cfg in {"rurunex": lambda: (hybrid_config(size), dense_config(size)),
                        "supinex": lambda: (parallel_config(size), moe_config(size)),
                        "vufinex": lambda: (prenorm_config(size), moe_config(size, dense_layers=0)),
                        "panarax": lambda: (gated_config(size), moe_config(size, dense_layers=2))}[args.layer_list]():
                B = n if phase == "decode" else 8
                eng = make_engine(cfg, B, n * length if phase == "prefill" else B, length if phase == "decode" else 16, 8)
                ex = eng.executor
                if phase == "prefill":
                    ids, pos, slots, ctx, row, nb = rows_of(n, length)
                    for r in range(n):
                        ex.set_block_table_row(r, list(range(r * nb, (r + 1) * nb)))
                    ends = [(r + 1) * length - 1 for r in range(n)]
                    step = eager = lambda: ex.prefill(ids, pos, slots, ctx, row, out_rows=ends)
                else:
                    nb = length // 16 + 1
                    for r in range(n):
                        ex.set_block_table_row(r, list(range(r * nb, (r + 1) * nb)))
                    pos = torch.full((n,), length - 1, dtype=torch.int32)
                    row = torch.arange(n, dtype=torch.int32)
                    slots = row.long() * nb * 16 + length - 1
                    ids = torch.zeros(n, dtype=torch.int32)
                    step = lambda: ex.decode(ids, pos, slots, pos + 1, row)

                    def eager():
                        sizes, ex.graph_sizes = ex.graph_sizes, []
                        ex.decode(ids, pos, slots, pos + 1, row)
                        ex.graph_sizes = sizes
                ms = timed(step, max(3, args.steps), max(3, args.warmup), flush)
                toks = n * length if phase == "prefill" else n
                print(json.dumps({"model": cfg.name, "phase": phase, "sequences": n, "length": length, "ms": round(ms, 3),
                                  "tokens_per_s": round(toks / ms * 1e3, 1), "launches": ex.graph_launches.get(n),
                                  "kernel_status": gemm.check_status("cuda")}), flush=True)
                print(json.dumps({"kernels_ms": kernel_times(eager)}), flush=True)
                del eng, ex, step, eager
                torch.cuda.empty_cache()
    return 0
