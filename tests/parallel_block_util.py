"""Small parallel-block models (Supinex design) for the tests; engines and comparisons as for the other layer lists."""
import torch

from disagmoe_b200.config import CacheConfig
from disagmoe_b200.frontend.colocated import ColocatedEngine
from disagmoe_b200.frontend.colocated_mixed import MixedBatchEngine
from disagmoe_b200.models.registry import supinex_config_from_json


def attn(heads, kv_heads, dim, vdim, mlp=None, v_mix=True, rot="full", scale=None, base=7000.0):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5, "v_mix": v_mix}
    if rot:
        m["rot"] = {"dims": dim if rot == "full" else rot, "base": base}
    return {"type": "attention", "mixer": m, "mlp": mlp}


YARN = {"factor": 3.0, "original": 200, "fast": 20.0, "slow": 1.0}


def latent(heads, dim, rot_dim, vdim, kv_rank, window, mlp=None, scale=None, scaling=YARN):
    rot = {"dims": rot_dim, "base": 40000.0}
    if scaling:
        rot["scaling"] = scaling
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "rot": rot,
         "scale": scale or (dim + rot_dim) ** -0.5}
    if window:
        m["mask"] = {"size": window}
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def model(width, vocab, layers, eps=1e-5):
    return {"architecture": "Supinex", "width": width, "vocab": vocab, "layers": layers, "norm": {"eps": eps}}


MODELS = {
    # tensor-core shapes, key and value sizes that differ, prompt kernel of the latent layers
    "even": model(128, 320, [latent(4, 32, 16, 48, 32, 37, moe(6, 2, 40)), attn(6, 2, 64, 32, dense(96)),
                             latent(3, 64, 64, 128, 136, 64, dense(72)), attn(8, 2, 64, 32, moe(12, 5, 64), scale=0.2),
                             attn(2, 2, 128, 64, None, v_mix=False, rot=32)]),
    # nothing aligned; padded heads; a latent of odd size; a layer without rotation
    "odd": model(44, 101, [attn(3, 3, 10, 7, moe(5, 3, 13), rot=6), latent(5, 9, 6, 11, 21, 19, None, scaling=None),
                           attn(6, 3, 12, 7, dense(37), rot=None, scale=0.31), latent(2, 12, 10, 5, 30, 50, moe(3, 3, 8))]),
    # one of everything
    "ones": model(64, 80, [attn(1, 1, 16, 16, moe(1, 1, 16)), latent(1, 8, 2, 8, 8, 1, moe(9, 1, 24)),
                           attn(1, 1, 16, 16, dense(8), v_mix=False)]),
    # many heads on one key head, more heads than one tile, a large latent, a window wider than the prompt
    "wide": model(96, 90, [attn(12, 1, 32, 32, dense(64)), latent(35, 16, 8, 16, 264, 500, moe(4, 4, 32)),
                           latent(17, 96, 32, 96, 64, None, None), attn(9, 1, 100, 80, moe(20, 8, 24), v_mix=False)]),
}


def make_engine(raw, weights, device="cpu", dtype=torch.float32, max_seqs=4, pool=640, graph=False, mixed=False, block=16, **kw):
    cfg = supinex_config_from_json(raw, {}, dtype=dtype, max_seq_len=pool)
    cls = MixedBatchEngine if mixed else ColocatedEngine
    eng = cls(cfg, CacheConfig(block_size=block), device=device, max_batch_size=max_seqs, max_prefill_tokens=pool,
              state_dict=weights, num_blocks=pool // block, enable_cuda_graph=graph, dtype=dtype, **kw)
    if graph:
        eng.executor.capture(list(range(1, max_seqs + 1)))
    return eng
