"""Small layer-list models, an engine built from them, and comparisons with the slow oracle."""
import torch

from disagmoe_b200.config import CacheConfig
from disagmoe_b200.frontend.colocated import ColocatedEngine
from disagmoe_b200.frontend.colocated_mixed import MixedBatchEngine
from disagmoe_b200.models.registry import rurunex_config_from_json
from oracles import layer_stack as oracle


def gla(heads, dim, vdim, tau=4.0, rank=8, ff=None):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau, "rank": rank}, "mlp": mlp(ff)}


def delta(heads, kv_heads, dim, vdim, conv=4, rank=8, ff=None):
    return {"type": "channel_delta", "mlp": mlp(ff),
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "rank": rank}}


def attn(heads, kv_heads, dim, vdim, window, scale=None, softcap=12.0, rot=None, kv_from=None, ff=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window},
         "scale": scale if scale is not None else dim ** -0.5, "softcap": softcap,
         "rot": rot or {"dims": dim, "base": 5000.0,
                        "scaling": {"factor": 4.0, "original": 256, "fast": 16.0, "slow": 1.0}}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp(ff)}


def mlp(ff):
    return None if ff is None else {"kind": "dense", "ff": ff}


def model(width, vocab, layers, embed=8.0, logit=0.7, eps=1e-5):
    return {"architecture": "Rurunex", "width": width, "vocab": vocab, "layers": layers, "norm": {"eps": eps},
            "embedding": {"scale": embed}, "logit_scale": logit}


PARTIAL = {"dims": 32, "base": 1000.0}
MODELS = {
    # tensor-core head sizes; shared keys under a different window; grouped delta heads; feed-forwards everywhere
    "even": model(128, 320, [gla(2, 64, 32, ff=96), delta(4, 2, 48, 32, ff=200), attn(4, 2, 64, 64, 37, ff=96),
                             attn(4, 2, 64, 64, 50, kv_from=2, softcap=30.0), gla(3, 32, 16),
                             attn(8, 1, 128, 128, 20, rot=PARTIAL, scale=0.1)]),
    # nothing aligned: widths, ranks, head and value sizes, vocabulary
    "odd": model(44, 101, [delta(3, 1, 12, 7, conv=3, rank=5), attn(6, 2, 10, 14, 19, rot={"dims": 6, "base": 300.0}, ff=37),
                           gla(5, 6, 9, tau=1.0, rank=3, ff=11), delta(2, 2, 20, 20, conv=2, rank=7),
                           attn(6, 2, 10, 14, 33, rot={"dims": 6, "base": 300.0}, kv_from=1)], embed=1.0, logit=1.0),
    # one head, one tap, a window of one token, wide states
    "ones": model(64, 80, [delta(1, 1, 128, 64, conv=1, ff=64), attn(1, 1, 64, 64, 1), gla(1, 96, 128, tau=16.0),
                           attn(3, 3, 32, 32, 500, softcap=2.0)]),
}


def tokens(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def make_engine(raw, weights, device="cpu", dtype=torch.float32, max_seqs=4, pool=640, graph=False, mixed=False, block=16,
                **kw):
    cfg = rurunex_config_from_json(raw, {n: tuple(t.shape) for n, t in weights.items()}, dtype=dtype, max_seq_len=pool)
    cls = MixedBatchEngine if mixed else ColocatedEngine
    eng = cls(cfg, CacheConfig(block_size=block), device=device, max_batch_size=max_seqs, max_prefill_tokens=pool,
              state_dict=weights, num_blocks=pool // block, enable_cuda_graph=graph, dtype=dtype, **kw)
    if graph:
        eng.executor.capture(list(range(1, max_seqs + 1)))
    return eng


def feed(eng, sid, toks, cuts, end=True):
    """Logits of every token of one sequence fed in portions of the given sizes (the last size repeats)."""
    out, at, i = [], 0, 0
    while at < len(toks):
        n = cuts[min(i, len(cuts) - 1)]
        part = toks[at:at + n]
        out.append(eng.feed([(sid, part, list(range(len(part))))]).float().cpu().clone())
        at, i = at + n, i + 1
    if end:
        eng.end_fed([sid])
    return torch.cat(out)


def error(got, want):
    """Largest row error (root mean square over the vocabulary, mean taken off) relative to the logits' own scale."""
    d = got.double() - want.double()
    d = d - d.mean(-1, keepdim=True)
    w = want.double() - want.double().mean(-1, keepdim=True)
    return float((d.pow(2).mean(-1).sqrt() / w.pow(2).mean().sqrt()).max())
