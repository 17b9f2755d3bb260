"""Kernels of latent attention layers on their own, against the bytes they have to move and the FLOPs they have to do.

    python -m benchmark.ops.latent_attention [--heads 16 --rank 512 --window 1024] [--only attention|decode|prefill]

decode: 256 sequences, one query each, over ``--window`` cached tokens. prefill: one run of 4096 tokens (expansion GEMM and
attention). Device times from CUDA events, L2 flushed before every launch.
"""
from __future__ import annotations

import argparse
import json

import torch

from benchmark.layer_list import Flush, timed
from disagmoe_b200.config import LatentAttentionSpec, RotarySpec
from disagmoe_b200.models.mixers import LatentTables, latent_layout
from disagmoe_b200.ops import functional as F
from disagmoe_b200.ops import gemm


def peaks():
    try:
        with open("MEASURED_PEAKS.json") as f:
            p = json.load(f)
        return p["hbm_gbs"], p["bf16_tflops"]
    except OSError:
        return 6650.0, 1590.0


def main(argv=None) -> None:
    ap = argparse.ArgumentParser()
    ap.add_argument("--heads", type=int, default=16)
    ap.add_argument("--dim", type=int, default=128)
    ap.add_argument("--rot", type=int, default=64)
    ap.add_argument("--rank", type=int, default=512)
    ap.add_argument("--window", type=int, default=1024)
    ap.add_argument("--batch", type=int, default=256)
    ap.add_argument("--prompt", type=int, default=4096)
    ap.add_argument("--steps", type=int, default=10)
    ap.add_argument("--splits", type=int, default=0)
    ap.add_argument("--only", default="")
    a = ap.parse_args(argv)
    dev, dt, H, B, N = torch.device("cuda"), torch.bfloat16, a.heads, a.batch, a.window
    m = LatentAttentionSpec(H, a.dim, a.rot, a.dim, a.rank, 0.05, RotarySpec(a.rot, 1e4, interleaved=True), a.window, True)
    lay, flush = latent_layout(m), Flush()
    hbm, flops = peaks()
    sink = torch.zeros(H, device=dev)
    rnd = lambda *s: torch.randn(*s, device=dev).to(dt)

    def report(name, ms, nbytes, nflops):
        bound = max(nbytes / hbm / 1e6, nflops / flops / 1e9)
        print(json.dumps({"kernel": name, "us": round(ms * 1e3, 1), "MB": round(nbytes / 1e6, 1), "GFLOP": round(nflops / 1e9, 2),
                          "of_measured_roofline": round(bound / ms, 3)}), flush=True)

    if a.only in ("", "decode", "attention"):
        blocks = N // 16
        cache = rnd(B * blocks, 16, lay.row)
        bt = torch.arange(B * blocks, dtype=torch.int32, device=dev).view(B, blocks)
        ctx, qa = torch.full((B,), N, dtype=torch.int32, device=dev), rnd(H, B, lay.row)
        row = torch.arange(B, dtype=torch.int32, device=dev)
        if a.splits:
            F.pick_latent_splits = lambda *_: a.splits
        run = lambda: F.latent_attention(qa, cache, bt, row, ctx, None, lay, m.scale, a.window, sink, N)
        report("latent_attention (decode)", timed(run, a.steps, 3, flush), (B * N + 2 * H * B) * lay.row * 2,
               2.0 * B * N * H * (lay.row + lay.rankp))
    if a.only in ("", "decode"):
        y, pos = rnd(B, H * lay.qd + lay.kd), ctx - 1
        slots, table, nw = row.long() * N, F.rope_freq_table(m.rot, N, dev), torch.ones(a.rank, device=dev)
        report("latent_prep (decode)", timed(lambda: F.latent_prep(y, pos, slots, cache, lay, table, nw, 1e-6, None, B), a.steps, 3, flush),
               B * (2 * H * lay.qd + 2 * lay.row) * 2, 0)
        t = LatentTables.decode(m, B, dev)
        xq, w = rnd(H * B, lay.dimp), rnd(H, lay.rankp, lay.dimp)
        report("key map into the query (grouped GEMM)", timed(lambda: gemm.grouped_linear(xq, w, t.offs, out=qa.view(-1, lay.row)[:, :lay.rankp], bn=gemm.pick_even_bn(B, lay.rankp, H)), a.steps, 3, flush),
               (xq.numel() + w.numel() + H * B * lay.rankp) * 2, 2.0 * H * B * lay.dimp * lay.rankp)
        o, wv, out = rnd(H * B, lay.rankp), rnd(H, lay.vdimp, lay.rankp), rnd(B, H * lay.vdimp)
        base = torch.tensor([out.data_ptr()], dtype=torch.int64, device=dev)
        report("value map of the outputs (grouped GEMM)", timed(lambda: gemm.grouped_combine(o, wv, t.offs, t.recs, base, lay.vdimp, bn=gemm.pick_even_bn(B, lay.vdimp, H)), a.steps, 3, flush),
               (o.numel() + wv.numel() + out.numel()) * 2, 2.0 * H * B * lay.vdimp * lay.rankp)
    if a.only in ("", "prefill"):
        T = a.prompt
        pos = torch.arange(T)
        t = LatentTables.prefill(m, torch.zeros(T, dtype=torch.int32), pos, dev, dt)
        cache, bt = rnd(T // 16, 16, lay.row), torch.arange(T // 16, dtype=torch.int32, device=dev)[None]
        y, out = rnd(T, H * lay.qd + lay.kd), torch.empty(T, H * lay.vdimp, dtype=dt, device=dev)
        w = rnd(H * (lay.dimp + lay.vdimp), lay.rankp) * 0.05
        slots, table, nw = pos.to(dev), F.rope_freq_table(m.rot, T, dev), torch.ones(a.rank, device=dev)
        pos = pos.int().to(dev)
        report("latent_prep (prompt)", timed(lambda: F.latent_prep(y, pos, slots, cache, lay, table, nw, 1e-6, t.loose, t.n_loose), a.steps, 3, flush),
               T * (2 * H * lay.rotp + 2 * lay.row) * 2, 0)
        lat = F.latent_gather(cache, bt, t.keys, t.n_keys)
        report("latent_gather", timed(lambda: F.latent_gather(cache, bt, t.keys, t.n_keys), a.steps, 3, flush), 2 * T * lay.row * 2, 0)
        kv = gemm.linear(lat[:, :lay.rankp], w)
        report("expansion GEMM", timed(lambda: gemm.linear(lat[:, :lay.rankp], w), a.steps, 3, flush), (lat.numel() + w.numel() + kv.numel()) * 2,
               2.0 * T * w.numel())
        pairs = sum(min(i + 1, a.window) for i in range(T))
        report("latent_prefill", timed(lambda: F.latent_prefill(y, kv, lat, t.tiles, t.base, t.n_tiles, lay, m.scale, a.window, sink, out), a.steps, 3, flush),
               (kv.numel() + y.numel() + out.numel()) * 2, 2.0 * pairs * H * (lay.qd + lay.vdimp))


if __name__ == "__main__":
    main()
