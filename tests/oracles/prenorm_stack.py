"""Slow double-precision restatement of the pre-norm decoder (Vufinex design), one function per mechanism.

As in :mod:`oracles.layer_stack`, every function takes the whole history of one sequence (rows = tokens from position 0):
no cache, no state carried between calls, no batching, no code of the package. Weights are a dict name -> tensor with the
checkpoint's names, the configuration is the plain dict of config.json.
"""
import torch

from oracles.layer_stack import centred_norm, rms, rotate, sigmoid, silu
from oracles.parallel_stack import gated, rotate_pairs


def attend(q, k, v, scale, first):
    """q [T, H, D], k [T, G, D], v [T, G, V] -> [T, H, V]; the query at i sees the keys first(i) .. i."""
    T, H = q.shape[:2]
    g = H // k.shape[1]
    kh, vh = k.repeat_interleave(g, 1), v.repeat_interleave(g, 1)
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for i in range(T):
        j = first(i)
        s = torch.einsum("jhd,hd->hj", kh[j:i + 1], q[i]) * scale
        out[i] = torch.einsum("hj,jhv->hv", torch.softmax(s, -1), vh[j:i + 1])
    return out


def chunk_start(size):
    """First key that the query at i sees if keys are shared inside chunks of ``size`` positions only."""
    return (lambda i: i // size * size) if size else (lambda i: 0)


def attention(h, w, p, m):
    """The values are the keys before their rotation."""
    T, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q, k = (h @ w[p + "q"].T).view(T, H, D), (h @ w[p + "k"].T).view(T, G, D)
    o = attend(rotate(q, m.get("rot")), rotate(k, m.get("rot")), k, m["scale"], chunk_start((m.get("mask") or {}).get("size")))
    return o.reshape(T, H * D) @ w[p + "o"].T


def latent_attention(h, w, p, m, eps):
    """Every head's output is scaled by a gate of its own."""
    T, H, D, R, V, K = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (h @ w[p + "q"].T).view(T, H, D + R)
    d = h @ w[p + "dkv"].T
    c = rms(d[:, :K], eps) * w[p + "dkv.norm"]
    k_rot = rotate_pairs(d[:, None, K:], m.get("rot")).expand(T, H, R)
    k = torch.cat([(c @ w[p + "uk"].T).view(T, H, D), k_rot], -1)
    v = (c @ w[p + "uv"].T).view(T, H, V)
    o = attend(torch.cat([q[..., :D], rotate_pairs(q[..., D:], m.get("rot"))], -1), k, v, m["scale"], chunk_start(None))
    o = o * sigmoid(h @ w[p + "g"].T)[..., None]
    return o.reshape(T, H * V) @ w[p + "o"].T


def token_shift(h, mu):
    """Every row moved towards the row before it (zeros before the first) by the factor mu of the channel."""
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * mu


def bonus_recurrence(r, k, v, log_decay, u, with_state=False):
    """r, k, log_decay [T, H, D], v [T, H, V], u [H, D]: the read-out sees the state before the token's own write, and the
    token itself weighed by u."""
    T, H, D = r.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=r.dtype)
    out = []
    for t in range(T):
        write = k[t][..., None] * v[t][:, None, :]
        out.append(((S + u[..., None] * write) * r[t][..., None]).sum(1))
        S = torch.exp(log_decay[t])[..., None] * S + write
    return (torch.stack(out), S) if with_state else torch.stack(out)


def wkv(h, w, p, m, eps):
    T, H, D = h.shape[0], m["heads"], m["dim"]
    mix = {n: token_shift(h, w[p + "mu." + n]) for n in "rkvgw"}
    r, k, v = ((mix[n] @ w[p + n].T).view(T, H, D) for n in "rkv")
    z = torch.tanh(mix["w"] @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"]
    o = bonus_recurrence(r, k, v, -torch.exp(z).view(T, H, D), w[p + "u"])
    o = rms(o, eps).reshape(T, H * D) * w[p + "norm"] * silu(mix["g"] @ w[p + "g"].T)
    return o @ w[p + "o"].T


def route(h, w, correction, router):
    """(chosen experts [T, top], their weights): sigmoid scores; the correction and the groups count for the choice alone."""
    s = sigmoid(h @ w.T)
    choice = s + correction
    T, E = s.shape
    n, keep = router["groups"]["count"], router["groups"]["keep"]
    grouped = choice.view(T, n, E // n)
    rank = grouped.sort(-1, descending=True).values[..., :2].sum(-1)
    best = torch.argsort(rank, dim=-1, descending=True, stable=True)[:, :keep]
    open_ = torch.zeros(T, n, dtype=torch.bool).scatter_(1, best, True)
    choice = grouped.masked_fill(~open_[..., None], float("-inf")).reshape(T, E)
    ids = torch.argsort(choice, dim=-1, descending=True, stable=True)[:, :router["top"]]
    wts = s.gather(1, ids)
    return ids, wts / (wts.sum(-1, keepdim=True) + 1e-20) * router["scale"]


def experts(h, w, p, m):
    ids, s = route(h, w[p + "router"], w[p + "correction"], m["router"])
    out = torch.zeros_like(h)
    for e in range(m["router"]["experts"]):
        weight = (s * (ids == e)).sum(-1)
        rows = (ids == e).any(-1).nonzero()[:, 0]
        out[rows] += weight[rows, None] * gated(h[rows], w, f"{p}e{e}.", silu)
    return out


def run(config, weights, tokens):
    """(logits [T, vocab], residual stream after every layer [layers, T, width]) in double precision."""
    w = {n: t.double() for n, t in weights.items()}
    eps, mult = config["norm"]["eps"], config["residual_mult"]
    x = w["embed"][torch.as_tensor(tokens).long()] * config["embedding"]["scale"]
    stream = []
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{layer.get('weights_of', i)}.", layer["mixer"]
        h = centred_norm(x, w[p + "norm1"], eps)
        if layer["type"] == "wkv":
            y = wkv(h, w, p + "mix.", m, eps)
        elif layer["type"] == "latent_attention":
            y = latent_attention(h, w, p + "mix.", m, eps)
        else:
            y = attention(h, w, p + "mix.", m)
        x = x + mult * y
        if layer["mlp"] is not None:
            x = x + mult * experts(centred_norm(x, w[p + "norm2"], eps), w, p + "mlp.", layer["mlp"])
        stream.append(x)
    return centred_norm(x, w["final.norm"], eps) @ w["head"].T, torch.stack(stream)


def shapes(config, rank=8):
    """Checkpoint tensor names and shapes of a configuration (``rank``: inner size of the decay maps, which only the
    checkpoint knows)."""
    W, out = config["width"], {"embed": (config["vocab"], config["width"])}
    for i, layer in enumerate(config["layers"]):
        if "weights_of" in layer:
            continue
        p, m, f = f"l{i}.", layer["mixer"], layer["mlp"]
        x, H, D = p + "mix.", m["heads"], m["dim"]
        out[p + "norm1"] = (W,)
        if layer["type"] == "wkv":
            out.update({x + "mu." + n: (W,) for n in "rkvgw"})
            out.update({x + n: (H * D, W) for n in "rkvg"})
            out.update({x + "w1": (rank, W), x + "w2": (H * D, rank), x + "w0": (H * D,), x + "u": (H, D), x + "norm": (H * D,),
                        x + "o": (W, H * D)})
        elif layer["type"] == "latent_attention":
            R, V, K = m["rot_dim"], m["vdim"], m["kv_rank"]
            out.update({x + "q": (H * (D + R), W), x + "dkv": (K + R, W), x + "dkv.norm": (K,), x + "uk": (H * D, K),
                        x + "uv": (H * V, K), x + "g": (H, W), x + "o": (W, H * V)})
        else:
            out.update({x + "q": (H * D, W), x + "k": (m["kv_heads"] * D, W), x + "o": (W, H * D)})
        if f is None:
            continue
        out[p + "norm2"] = (W,)
        E, F = f["router"]["experts"], f["expert"]["ff"]
        for e in range(E):
            q = f"{p}mlp.e{e}."
            out.update({q + "gate": (F, W), q + "up": (F, W), q + "down": (W, F)})
        out.update({p + "mlp.router": (E, W), p + "mlp.correction": (E,)})
    out.update({"final.norm": (W,), "head": (config["vocab"], W)})
    return out


def random_weights(config, seed=0, rank=8):
    """bfloat16-representable weights with lively norms, decays, mixes and corrections (float32 tensors)."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for n, s in shapes(config, rank).items():
        r = torch.randn(s, generator=g)
        leaf = n.rsplit(".", 1)[-1]
        if ".mu." in n:
            t = torch.sigmoid(r)
        elif leaf == "w0":
            t = 1.5 * r - 2.0
        elif leaf == "u":
            t = 0.7 * r
        elif leaf == "correction":
            t = 0.3 * r
        elif len(s) == 1:
            t = 1.0 + 0.3 * r if ".mix." in n else 0.2 * r
        elif leaf == "router":
            t = 2.0 * r * s[1] ** -0.5
        else:
            t = r * (0.1 if n == "embed" else s[1] ** -0.5)
        out[n] = t.bfloat16().float()
    return out
