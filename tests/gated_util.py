"""Small gated-residual models (Panarax design) for the tests; engines and comparisons as for the other layer lists."""
import torch

from disagmoe_b200.config import CacheConfig
from disagmoe_b200.frontend.colocated import ColocatedEngine
from disagmoe_b200.frontend.colocated_mixed import MixedBatchEngine
from disagmoe_b200.models.registry import panarax_config_from_json


def unit(width, blocks, conv=4, mlp=None):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}, "mlp": mlp}


def lightning(dim, vdim, decay, mlp=None):
    return {"type": "lightning", "mixer": {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay)}, "mlp": mlp}


def left(heads, kv_heads, dim, vdim, scale=None, q_temp=(0.4, 16)):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5}
    if q_temp:
        m["q_temp"] = {"coef": q_temp[0], "every": q_temp[1]}
    return m


def right(heads, dim, vdim, cap=8.0):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def both(left, right, mlp=None):
    return {"type": "parallel", "mixer": {"left": left, "right": right}, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit=1.5):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def model(width, vocab, layers, taps=4, positions=1200, eps=1e-5):
    return {"architecture": "Panarax", "width": width, "vocab": vocab, "layers": layers, "norm": {"eps": eps},
            "canon": {"taps": taps}, "max_positions": positions}


MODELS = {
    # tensor-core shapes; grouped queries; every mixer with either kind of feed-forward
    "even": model(128, 320, [both(left(4, 2, 64, 64), right(3, 32, 48), dense(96)), unit(96, 3, 4, moe(8, 2, 40)),
                             lightning(32, 48, (0.3, 0.95, 0.998), moe(12, 3, 64, 0.8)), unit(192, 4, 2, dense(72)),
                             both(left(6, 1, 40, 72, 0.2, (1.3, 7)), right(2, 64, 128, 3.0), moe(4, 1, 48)),
                             lightning(64, 64, (0.99, 0.7), dense(80)), lightning(128, 32, (1.0, 0.0, 0.9), None)]),
    # nothing aligned: widths, heads, vocabulary, blocks, experts; two taps
    "odd": model(44, 101, [lightning(10, 7, (0.5, 0.97, 0.999), moe(6, 3, 11, 2.5)), both(left(6, 3, 10, 14, 0.31, (0.2, 5)), right(3, 12, 9),
                           dense(37)), unit(45, 3, 3, moe(5, 5, 8)), both(left(3, 3, 20, 6, None, None), right(1, 6, 22, 20.0), None),
                           unit(26, 2, 1, dense(13)), unit(21, 1, 5, None)], taps=2),
    # one of everything: heads, blocks, experts, one tap
    "ones": model(64, 80, [unit(32, 1, 4, moe(1, 1, 16)), lightning(16, 16, (0.9,), moe(4, 4, 16)),
                           both(left(1, 1, 16, 16, 1.0, (0.7, 1)), right(1, 16, 16, 1.0), dense(24)), unit(64, 64, 2, None)], taps=1),
    # many heads, long convolutions, large states
    "wide": model(96, 90, [both(left(16, 2, 128, 128, None, (0.1, 64)), right(5, 128, 64), moe(16, 16, 32, 3.0)),
                           unit(320, 5, 8, moe(64, 1, 24)), lightning(128, 128, (0.2, 0.9, 0.99, 0.9995, 0.6), dense(200)),
                           both(left(35, 5, 24, 32), right(9, 8, 8), None)], taps=8),
}


def make_engine(raw, weights, device="cpu", dtype=torch.float32, max_seqs=4, pool=640, graph=False, mixed=False, block=16, **kw):
    cfg = panarax_config_from_json(raw, {n: tuple(t.shape) for n, t in weights.items()}, dtype=dtype, max_seq_len=pool)
    cls = MixedBatchEngine if mixed else ColocatedEngine
    eng = cls(cfg, CacheConfig(block_size=block), device=device, max_batch_size=max_seqs, max_prefill_tokens=pool,
              state_dict=weights, num_blocks=pool // block, enable_cuda_graph=graph, dtype=dtype, **kw)
    if graph:
        eng.executor.capture(list(range(1, max_seqs + 1)))
    return eng
