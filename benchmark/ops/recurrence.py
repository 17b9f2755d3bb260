"""Recurrent layers alone: prompts (chunked kernels) and decode steps; gated linear attention, the channel-wise delta rule,
RWKV-style time mixing (wkv, with its token shift on its own), lightning attention, the matrix memory, and Griffin's block (unit: its
convolution and its recurrence).

    python -m benchmark.ops.recurrence [--kinds gla,delta,wkv,lightning,memory,unit] [--heads 16] [--dim 128] [--tokens 4096] [--batch 256]

Device time (CUDA events, L2 flushed in between) beside the bytes the operation has to move: projections in, output out and,
for a decode step, every state read and written once.
"""
import argparse
import json
import os
import statistics
import sys

import torch

sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__)))))

from disagmoe_b200.ops import functional as F
from disagmoe_b200.ops.recurrent import (GatedUnit, Recurrence, build_segments, decode_segments, recurrent_attention,
                                         unit_recurrence)


def layer(kind, H, D, V, dev="cuda"):
    r = lambda *s: torch.randn(*s, device=dev)
    if kind == "gla":
        return Recurrence(H, H, D, V, False, r(H * D) + 2.0, 1 + 0.1 * r(V), 1e-6, tau=16.0)
    if kind == "wkv":
        return Recurrence(H, H, D, V, False, r(H * D) - 3.0, 1 + 0.1 * r(H * D), 1e-6, exp_decay=True, bonus=0.5 * r(H, D), qscale=1.0,
                          shift_width=H * D)
    if kind == "lightning":
        return Recurrence(H, H, D, V, False, None, 1 + 0.1 * r(H * V), 1e-6, sigmoid_gate=True, qscale=1.0, joint_norm=True,
                          head_decay=-torch.exp2(-8.0 * (torch.arange(H, device=dev) + 1) / H))
    if kind == "memory":
        return Recurrence(H, H, D, V, False, None, 1 + 0.1 * r(H * V), 1e-6, sigmoid_gate=True, gate_cap=15.0,
                          gate_bias=torch.cat([r(H), r(H) + 4.0]))
    if kind == "unit":
        C = H * D
        return GatedUnit(C, H, 0.5 * r(4, C), r(C), r(C), r(H, 2, D), -8.0 * torch.nn.functional.softplus(r(C) - 4.0), r(C))
    return Recurrence(H, H, D, V, True, 0.5 * r(H * D) - 4.0, 1 + 0.1 * r(V), 1e-6, a_log=0.3 * r(H),
                      conv_w=0.5 * r(2 * H * D + H * V, 4), sigmoid_gate=True)


def main():
    p = argparse.ArgumentParser()
    p.add_argument("--heads", type=int, default=16)
    p.add_argument("--dim", type=int, default=128)
    p.add_argument("--tokens", type=int, default=4096, help="prompt tokens")
    p.add_argument("--prompts", type=int, default=1)
    p.add_argument("--batch", type=int, default=256, help="decoding sequences")
    p.add_argument("--iters", type=int, default=10)
    p.add_argument("--only", default="", help="prompt | decode")
    p.add_argument("--kinds", default="gla,delta,wkv,lightning,memory,unit")
    a = p.parse_args()
    H, D = a.heads, a.dim
    flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")
    peak = json.load(open("MEASURED_PEAKS.json"))["hbm_gbs"] if os.path.exists("MEASURED_PEAKS.json") else 6650.0
    for kind in a.kinds.split(","):
        r = layer(kind, H, D, D)
        for phase in ("prompt", "decode"):
            if a.only not in ("", phase):
                continue
            T = a.tokens if phase == "prompt" else a.batch
            b = lambda n: torch.randn(T, n, device="cuda").bfloat16()
            x = b(4 * H * D + H)
            q, k, v, gate, beta = (x[:, i * H * D:(i + 1) * H * D] for i in range(4)), None, None, None, x[:, 4 * H * D:]
            q, k, v, gate = q
            z = torch.randn(T, H * D, device="cuda")
            state = r.new_state(a.batch if phase == "decode" else a.prompts, torch.bfloat16, "cuda")
            if phase == "prompt":
                n = T // a.prompts
                segs = build_segments(torch.arange(a.prompts).repeat_interleave(n), torch.arange(n).repeat(a.prompts), "cuda")
            else:
                i = torch.arange(T, device="cuda")
                segs = decode_segments(torch.full((T,), 100, dtype=torch.int32, device="cuda"), i.int(), i)
            if kind == "memory":
                z = z[:, :2 * H].contiguous()
            if kind == "unit":
                u, zz = torch.randn(H, T, D, device="cuda").bfloat16(), torch.randn(H, T, 2, D, device="cuda")
            cases = [] if kind == "unit" else [(kind, T * H * D * (2 * 5 + (0 if kind in ("lightning", "memory") else 4)) + (2 * state.S.numel() * 4 if phase == "decode" else 0),
                      lambda: recurrent_attention(r, q, k, v, gate, beta if kind == "delta" else None,
                                                  None if kind == "lightning" else z, state, segs))]
            if kind == "unit":
                cases = [("convolution", T * H * D * 2 * (2 if phase == "prompt" else 6),
                          lambda: F.seq_conv(q, r.conv_w, state.ring, segs, r.in_b, r.conv_b, blocks=H)),
                         ("unit", T * H * D * (2 * 3 + 8 + (8 if phase == "decode" else 0)), lambda: unit_recurrence(r, u, zz, k, state, segs))]
            if kind == "wkv":
                W = H * D
                mu, w, resid = torch.rand(5, W, device="cuda"), torch.ones(W, device="cuda"), torch.randn(T, W, device="cuda")
                shift = F.TokenShift(mu, state.last, segs)
                if phase == "prompt":
                    cases.append(("token shift", T * W * (4 + 5 * 2), lambda: F.token_shift(resid, shift, torch.bfloat16)))
                else:
                    cases.append(("norm + token shift", T * W * (4 + 5 * 2 + 8),
                                  lambda: F.sum_norm(resid, None, None, w, 1e-6, torch.bfloat16, False, shift=shift)))
            for name, moved, fn in cases:
                ms = []
                for it in range(a.iters + 3):
                    flush.zero_()
                    e = [torch.cuda.Event(enable_timing=True) for _ in range(2)]
                    e[0].record()
                    fn()
                    e[1].record()
                    torch.cuda.synchronize()
                    ms.append(e[0].elapsed_time(e[1]))
                t = statistics.median(ms[3:])
                print(json.dumps({"kind": name, "phase": phase, "tokens": T, "heads": H, "dim": D, "us": round(t * 1e3, 1),
                                  "MB": round(moved / 1e6, 1), "GB_s": round(moved / t / 1e6),
                                  "of_measured_copy": round(moved / t / 1e6 / peak, 3)}), flush=True)


if __name__ == "__main__":
    main()
