"""Slow double-precision restatement of the parallel-block decoder (Supinex design), one function per mechanism.

As in :mod:`oracles.layer_stack`, every function takes the whole history of one sequence (rows = tokens from position 0):
no cache, no batching, no code of the package. Weights are a dict name -> tensor with the checkpoint's names, the
configuration is the plain dict of config.json.
"""
import math

import torch

from oracles.layer_stack import inverse_frequencies, rms, silu


def layer_norm(x, w, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rotate_pairs(x, rot):
    """x [T, heads, dim]: row t at position t; neighbours (2i, 2i + 1) of the first rot["dims"] dimensions are a pair."""
    if not rot:
        return x
    f, m = inverse_frequencies(rot)
    out = x.clone()
    pos = torch.arange(x.shape[0], dtype=torch.float64)
    for i in range(rot["dims"] // 2):
        c, s = (torch.cos(pos * f[i]) * m)[:, None], (torch.sin(pos * f[i]) * m)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


def sink_softmax(s, sink):
    """Softmax over the last axis whose denominator has exp(sink) in addition (sink broadcasts against s[..., 0])."""
    if sink is None:
        return torch.softmax(s, -1)
    m = torch.maximum(s.max(-1).values, sink)
    e = torch.exp(s - m[..., None])
    return e / (e.sum(-1) + torch.exp(sink - m))[..., None]


def attend(q, k, v, scale, sink=None, window=None):
    """q [T, H, D], k [T, G, D], v [T, G, V] -> [T, H, V]; a query sees itself and what is before it, ``window`` tokens
    altogether where that is given."""
    T, H = q.shape[:2]
    g = H // k.shape[1]
    kh, vh = k.repeat_interleave(g, 1), v.repeat_interleave(g, 1)
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for i in range(T):
        j = 0 if not window else max(0, i - window + 1)
        s = torch.einsum("jhd,hd->hj", kh[j:i + 1], q[i]) * scale
        out[i] = torch.einsum("hj,jhv->hv", sink_softmax(s, sink), vh[j:i + 1])
    return out


def mix_values(v, first, lam):
    return (1.0 - lam) * v + lam * first


def attention(h, w, p, m, eps, first):
    """Returns (output, values of the first value-mixing layer); ``first`` is None up to and in that layer."""
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rotate_pairs((h @ w[p + "q"].T).view(T, H, D), m.get("rot"))
    k = rotate_pairs((h @ w[p + "k"].T).view(T, G, D), m.get("rot"))
    v = (h @ w[p + "v"].T).view(T, G, V)
    if m.get("v_mix"):
        if first is None:
            first = v
        else:
            v = mix_values(v, first, w[p + "vmix"])
    o = attend(q, k, v, m["scale"], w[p + "sink"], (m.get("mask") or {}).get("size"))
    return o.reshape(T, H * V) @ w[p + "o"].T, first


def latent_attention(h, w, p, m, eps):
    T, H, D, R, V, K = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (h @ w[p + "q"].T).view(T, H, D + R)
    q_rot = rotate_pairs(q[..., D:], m.get("rot"))
    d = h @ w[p + "dkv"].T
    c = rms(d[:, :K], eps) * w[p + "dkv.norm"]
    k_rot = rotate_pairs(d[:, None, K:], m.get("rot"))
    k = torch.cat([(c @ w[p + "uk"].T).view(T, H, D), k_rot.expand(T, H, R)], -1)
    v = (c @ w[p + "uv"].T).view(T, H, V)
    o = attend(torch.cat([q[..., :D], q_rot], -1), k, v, m["scale"], w[p + "sink"], (m.get("mask") or {}).get("size"))
    return o.reshape(T, H * V) @ w[p + "o"].T


def route(h, w, top):
    """(chosen experts [T, top], their softmax scores as they are)."""
    s = torch.softmax(h @ w.T, -1)
    best = torch.argsort(s, dim=-1, descending=True, stable=True)[:, :top]
    return best, s.gather(1, best)


def gated(h, w, p, act):
    return (act(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def experts(h, w, p, m):
    ids, s = route(h, w[p + "router"], m["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(m["router"]["experts"]):
        weight = (s * (ids == e)).sum(-1)
        rows = weight.nonzero()[:, 0]
        out[rows] += weight[rows, None] * gated(h[rows], w, f"{p}e{e}.", silu)
    return out


def feed_forward(h, w, p, m):
    return gated(h, w, p, gelu_tanh) if m["kind"] == "dense" else experts(h, w, p, m)


def run(config, weights, tokens):
    """(logits [T, vocab], residual stream after every layer [layers, T, width]) in double precision."""
    w = {n: t.double() for n, t in weights.items()}
    eps = config["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens).long()]
    first, stream = None, []
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        h = layer_norm(x, w[p + "norm1"], eps)
        if layer["type"] == "latent_attention":
            y = latent_attention(h, w, p + "mix.", layer["mixer"], eps)
        else:
            y, first = attention(h, w, p + "mix.", layer["mixer"], eps, first)
        if layer["mlp"] is not None:
            y = y + feed_forward(h, w, p + "mlp.", layer["mlp"])
        x = x + y
        stream.append(x)
    return layer_norm(x, w["final.norm"], eps) @ w["head"].T, torch.stack(stream)


def shapes(config):
    """Checkpoint tensor names and shapes of a configuration."""
    W, out = config["width"], {"embed": (config["vocab"], config["width"])}
    for i, layer in enumerate(config["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer["mlp"]
        x, H, D, V = p + "mix.", m["heads"], m["dim"], m["vdim"]
        out.update({p + "norm1": (W,), x + "sink": (H,), x + "o": (W, H * V)})
        if layer["type"] == "latent_attention":
            R, K = m["rot_dim"], m["kv_rank"]
            out.update({x + "q": (H * (D + R), W), x + "dkv": (K + R, W), x + "dkv.norm": (K,), x + "uk": (H * D, K),
                        x + "uv": (H * V, K)})
        else:
            G = m["kv_heads"]
            out.update({x + "q": (H * D, W), x + "k": (G * D, W), x + "v": (G * V, W)})
            if m.get("v_mix"):
                out[x + "vmix"] = ()
        if f is None:
            continue
        one = lambda q, F: {q + "gate": (F, W), q + "up": (F, W), q + "down": (W, F)}
        if f["kind"] == "dense":
            out.update(one(p + "mlp.", f["ff"]))
        else:
            for e in range(f["router"]["experts"]):
                out.update(one(f"{p}mlp.e{e}.", f["expert"]["ff"]))
            out[p + "mlp.router"] = (f["router"]["experts"], W)
    out.update({"final.norm": (W,), "head": (config["vocab"], W)})
    return out


def random_weights(config, seed=0):
    """bfloat16-representable weights with lively norms, sinks and mixing factors (float32 tensors)."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for n, s in shapes(config).items():
        r = torch.randn(s, generator=g)
        leaf = n.rsplit(".", 1)[-1]
        if leaf == "vmix":
            t = 0.5 + 0.3 * r
        elif leaf == "sink":
            t = 1.0 + r
        elif len(s) == 1:
            t = 1.0 + 0.3 * r
        elif leaf == "router":
            t = 2.0 * r * s[1] ** -0.5
        else:
            t = r * (1.0 if n == "embed" else s[1] ** -0.5)
        out[n] = t.bfloat16().float()
    return out
