"""Small pre-norm models (Vufinex design) for the tests; engines and comparisons as for the other layer lists."""
import torch

from disagmoe_b200.config import CacheConfig
from disagmoe_b200.frontend.colocated import ColocatedEngine
from disagmoe_b200.frontend.colocated_mixed import MixedBatchEngine
from disagmoe_b200.models.registry import vufinex_config_from_json


def wkv(heads, dim, mlp=None):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim}, "mlp": mlp}


def attn(heads, kv_heads, dim, chunk, mlp=None, rot="full", scale=None, base=3000.0):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale or dim ** -0.5, "mask": {"size": chunk}}
    if rot:
        m["rot"] = {"dims": dim if rot == "full" else rot, "base": base}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def latent(heads, dim, rot_dim, vdim, kv_rank, mlp=None, scale=None, base=50000.0):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
                      "scale": scale or (dim + rot_dim) ** -0.5, "rot": {"dims": rot_dim, "base": base}}}


def moe(experts, top, ff, groups=1, keep=1, scale=1.0):
    return {"kind": "moe", "expert": {"ff": ff},
            "router": {"experts": experts, "top": top, "scale": scale, "groups": {"count": groups, "keep": keep}}}


def again(layers, i):
    """A layer that uses the weights of layer i of the list."""
    return {**layers[i], "weights_of": i}


def model(width, vocab, layers, embed=6.0, mult=0.4, eps=1e-5):
    return {"architecture": "Vufinex", "width": width, "vocab": vocab, "layers": layers, "norm": {"eps": eps},
            "embedding": {"scale": embed}, "residual_mult": mult}


def _shared(*layers, of=(0, 2)):
    layers = list(layers)
    return layers + [again(layers, i) for i in of]


MODELS = {
    # tensor-core shapes; grouped queries; every kind of layer a second time on the same weights
    "even": model(128, 320, _shared(wkv(3, 32, moe(8, 2, 40, 4, 2, 1.7)), latent(4, 32, 16, 48, 32, moe(12, 3, 64, 3, 1, 0.8)),
                                    attn(4, 2, 64, 37, moe(8, 3, 48, 2, 1, 2.0)), attn(8, 1, 128, 64, None, rot=64),
                                    wkv(1, 128, None), of=(2, 0, 1))),
    # nothing aligned: widths, heads, vocabulary, experts in groups of three; chunks of a page and of odd sizes
    "odd": model(44, 101, [attn(6, 3, 10, 19, moe(9, 2, 13, 3, 2, 1.3), rot=6), wkv(3, 7, moe(6, 3, 11, 2, 2)),
                           latent(5, 9, 6, 11, 21, None), wkv(2, 12, None), attn(3, 3, 20, 16, moe(5, 5, 8), rot=None, scale=0.31)],
                 embed=1.0, mult=1.0),
    # one of everything: heads, experts per group, a chunk of one token
    "ones": model(64, 80, [wkv(1, 16, moe(4, 1, 16, 4, 1)), attn(1, 1, 16, 1, moe(1, 1, 16)), latent(1, 8, 2, 8, 8, moe(6, 2, 24, 6, 3)),
                           attn(1, 1, 32, 500, None)], mult=0.25),
    # many heads, a large latent, a chunk wider than the prompt
    "wide": model(96, 90, [latent(35, 16, 8, 16, 264, moe(16, 8, 32, 4, 2, 3.0)), wkv(5, 64, moe(64, 6, 24, 8, 3)),
                           attn(12, 1, 100, 300, moe(4, 4, 24)), latent(17, 96, 32, 96, 64, None)], embed=20.0),
}


def make_engine(raw, weights, device="cpu", dtype=torch.float32, max_seqs=4, pool=640, graph=False, mixed=False, block=16, **kw):
    cfg = vufinex_config_from_json(raw, {n: tuple(t.shape) for n, t in weights.items()}, dtype=dtype, max_seq_len=pool)
    cls = MixedBatchEngine if mixed else ColocatedEngine
    eng = cls(cfg, CacheConfig(block_size=block), device=device, max_batch_size=max_seqs, max_prefill_tokens=pool,
              state_dict=weights, num_blocks=pool // block, enable_cuda_graph=graph, dtype=dtype, **kw)
    if graph:
        eng.executor.capture(list(range(1, max_seqs + 1)))
    return eng
