"""Slow double-precision restatement of the gated-residual decoder (Panarax design), one function per mechanism.

As in :mod:`oracles.layer_stack`, every function takes the whole history of one sequence (rows = tokens from position 0):
no cache, no state carried between calls, no batching, no code of the package. Weights are a dict name -> tensor with the
checkpoint's names, the configuration is the plain dict of config.json.
"""
import math

import torch

from oracles.layer_stack import log_sigmoid, rms, sigmoid, silu, softplus
from oracles.parallel_stack import gelu_tanh
from oracles.prenorm_stack import attend


def layer_norm(x, w, b, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def convolve(x, w):
    """x [T, C], w [C, taps]: the last column belongs to the token itself, rows before the first are zeros."""
    taps = w.shape[1]
    full = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=x.dtype), x])
    return sum(full[j:j + x.shape[0]] * w[:, j] for j in range(taps))


def input_convolution(h, w):
    return h + convolve(h, w)


def residual_gate(h, w, b):
    return sigmoid(h @ w.T + b)


# ---- mixers ------------------------------------------------------------------------------------------------------------
def unit_recurrence(u, r, i, lam, with_state=False):
    """u, r, i [T, C], lam [C]: a diagonal recurrence whose decay and write the gates r and i set."""
    S = torch.zeros_like(u[0])
    out = []
    for t in range(u.shape[0]):
        log_a = -8.0 * r[t] * softplus(lam)
        S = torch.exp(log_a) * S + torch.sqrt(1.0 - torch.exp(2.0 * log_a)) * (i[t] * u[t])
        out.append(S)
    return (torch.stack(out), S) if with_state else torch.stack(out)


def block_map(u, w, b):
    """Every one of the equal parts of u's columns through a square map of its own."""
    n, size = w.shape[:2]
    return torch.cat([u[:, j * size:(j + 1) * size] @ w[j].T + b[j] for j in range(n)], -1)


def unit_block(h, w, p, m):
    y = gelu_tanh(h @ w[p + "y"].T + w[p + "y.b"])
    u = convolve(h @ w[p + "x"].T + w[p + "x.b"], w[p + "conv"]) + w[p + "conv.b"]
    r, i = (sigmoid(block_map(u, w[p + n], w[p + n + ".b"])) for n in ("ra", "ri"))
    return (unit_recurrence(u, r, i, w[p + "lam"]) * y) @ w[p + "o"].T


def decay_recurrence(q, k, v, decay, with_state=False):
    """q, k [T, H, D], v [T, H, V], decay [H] or [T, H]."""
    T, H, D = q.shape
    decay = torch.as_tensor(decay, dtype=q.dtype).expand(T, H)
    S = torch.zeros(H, D, v.shape[-1], dtype=q.dtype)
    out = []
    for t in range(T):
        S = decay[t][:, None, None] * S + k[t][..., None] * v[t][:, None, :]
        out.append((S * q[t][..., None]).sum(1))
    return (torch.stack(out), S) if with_state else torch.stack(out)


def lightning(h, w, p, m, eps):
    T, H = h.shape[0], m["heads"]
    q, k, v = (silu(h @ w[p + n].T).view(T, H, -1) for n in "qkv")
    o = decay_recurrence(q, k, v, m["decay"]).reshape(T, -1)
    return (rms(o, eps) * w[p + "norm"] * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def memory_recurrence(q, k, v, i, f, with_state=False):
    """q, k [T, H, D], v [T, H, V], logs i, f [T, H] of the input and forget gates: matrix memory S with a normaliser n, both
    kept relative to exp(m), the running maximum m starting at 0."""
    T, H, D = q.shape
    S, n, m = torch.zeros(H, D, v.shape[-1], dtype=q.dtype), torch.zeros(H, D, dtype=q.dtype), torch.zeros(H, dtype=q.dtype)
    out = []
    for t in range(T):
        new = torch.maximum(f[t] + m, i[t])
        keep, put = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        S = keep[:, None, None] * S + put[:, None, None] * k[t][..., None] * v[t][:, None, :]
        n = keep[:, None] * n + put[:, None] * k[t]
        m = new
        size = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out.append((S * q[t][..., None]).sum(1) / size[:, None])
    return (torch.stack(out), (S, n, m)) if with_state else torch.stack(out)


def matrix_memory(h, w, p, m, eps):
    T, H, cap = h.shape[0], m["heads"], m["gate_cap"]
    q, k, v = ((h @ w[p + n].T).view(T, H, -1) for n in "qkv")
    capped = lambda n: cap * torch.tanh((h @ w[p + n].T + w[p + n + ".b"]) / cap)
    o = memory_recurrence(q * m["dim"] ** -0.5, k, v, capped("i"), log_sigmoid(capped("f")))
    o = rms(o, eps).reshape(T, -1) * w[p + "norm"] * sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


def query_temperature(positions, t):
    """The factor of the queries at ``positions``."""
    if not t:
        return torch.ones(len(positions), dtype=torch.float64)
    return torch.tensor([1.0 + t["coef"] * math.log((p + 1) // t["every"] + 1) for p in positions], dtype=torch.float64)


def attention(h, w, p, m, eps):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q, k, v = ((h @ w[p + n].T).view(T, g, -1) for n, g in (("q", H), ("k", G), ("v", G)))
    q = q * query_temperature(range(T), m.get("q_temp"))[:, None, None]
    o = attend(q, k, rms(v, eps), m["scale"], lambda i: 0)
    o = o * sigmoid(h @ w[p + "g"].T)[..., None]
    return o.reshape(T, -1) @ w[p + "o"].T


def side_by_side(left, right, w, p, eps):
    return 0.5 * (rms(left, eps) * w[p + "left.out"] + rms(right, eps) * w[p + "right.out"])


def mixer(h, w, p, layer, eps):
    m = layer["mixer"]
    if layer["type"] == "rglru":
        return unit_block(h, w, p, m)
    if layer["type"] == "lightning":
        return lightning(h, w, p, m, eps)
    return side_by_side(attention(h, w, p + "left.", m["left"], eps), matrix_memory(h, w, p + "right.", m["right"], eps), w, p, eps)


# ---- feed-forwards -----------------------------------------------------------------------------------------------------
def dense(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def clamped_expert(h, w, p, limit):
    g, u = (h @ w[p + "gate"].T).clamp(max=limit), (h @ w[p + "up"].T).clamp(-limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def experts(h, w, p, m):
    """Sigmoid scores; the score scales what an expert reads."""
    s = sigmoid(h @ w[p + "router"].T)
    ids = torch.argsort(s, dim=-1, descending=True, stable=True)[:, :m["router"]["top"]]
    out = torch.zeros_like(h)
    for e in range(m["router"]["experts"]):
        rows = (ids == e).any(-1).nonzero()[:, 0]
        out[rows] += clamped_expert(s[rows, e, None] * h[rows], w, f"{p}e{e}.", m["expert"]["limit"])
    return out


def run(config, weights, tokens):
    """(logits [T, vocab], residual stream after every layer [layers, T, width]) in double precision."""
    w = {n: t.double() for n, t in weights.items()}
    eps = config["norm"]["eps"]
    norm = lambda x, n: layer_norm(x, w[n], w[n + ".b"], eps)
    x = w["embed"][torch.as_tensor(tokens).long()] + w["pos"][:len(tokens)]
    stream = []
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        h = norm(x, p + "norm1")
        y = mixer(input_convolution(h, w[p + "canon1"]), w, p + "mix.", layer, eps)
        x = x + residual_gate(h, w[p + "rg1"], w[p + "rg1.b"]) * y
        f = layer["mlp"]
        if f is not None:
            h = norm(x, p + "norm2")
            y = dense(h, w, p + "mlp.") if f["kind"] == "dense" else experts(h, w, p + "mlp.", f)
            x = x + residual_gate(h, w[p + "rg2"], w[p + "rg2.b"]) * y
        stream.append(x)
    return norm(x, "final.norm") @ w["embed"].T, torch.stack(stream)


# ---- checkpoints of a configuration --------------------------------------------------------------------------------------
def shapes(config):
    W = config["width"]
    out = {"embed": (config["vocab"], W), "pos": (config["max_positions"], W)}

    def norm(n):
        out.update({n: (W,), n + ".b": (W,)})
    for i, layer in enumerate(config["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer["mlp"]
        x = p + "mix."
        norm(p + "norm1")
        out.update({p + "canon1": (W, config["canon"]["taps"]), p + "rg1": (W, W), p + "rg1.b": (W,)})
        if layer["type"] == "rglru":
            C, n = m["width"], m["blocks"]
            out.update({x + "y": (C, W), x + "y.b": (C,), x + "x": (C, W), x + "x.b": (C,), x + "conv": (C, m["conv"]),
                        x + "conv.b": (C,), x + "lam": (C,), x + "o": (W, C)})
            for g in ("ra", "ri"):
                out.update({x + g: (n, C // n, C // n), x + g + ".b": (n, C // n)})
        elif layer["type"] == "lightning":
            K, V = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            out.update({x + "q": (K, W), x + "k": (K, W), x + "v": (V, W), x + "g": (V, W), x + "norm": (V,), x + "o": (W, V)})
        else:
            a, r = m["left"], m["right"]
            out.update({x + "left.q": (a["heads"] * a["dim"], W), x + "left.k": (a["kv_heads"] * a["dim"], W),
                        x + "left.v": (a["kv_heads"] * a["vdim"], W), x + "left.g": (a["heads"], W),
                        x + "left.o": (W, a["heads"] * a["vdim"]), x + "left.out": (W,)})
            K, V = r["heads"] * r["dim"], r["heads"] * r["vdim"]
            out.update({x + "right.q": (K, W), x + "right.k": (K, W), x + "right.v": (V, W), x + "right.g": (V, W),
                        x + "right.norm": (V,), x + "right.o": (W, V), x + "right.out": (W,)})
            for g in "if":
                out.update({x + f"right.{g}": (r["heads"], W), x + f"right.{g}.b": (r["heads"],)})
        if f is None:
            continue
        norm(p + "norm2")
        out.update({p + "rg2": (W, W), p + "rg2.b": (W,)})
        gated = lambda q, n: out.update({q + "gate": (n, W), q + "up": (n, W), q + "down": (W, n)})
        if f["kind"] == "dense":
            gated(p + "mlp.", f["ff"])
        else:
            for e in range(f["router"]["experts"]):
                gated(f"{p}mlp.e{e}.", f["expert"]["ff"])
            out[p + "mlp.router"] = (f["router"]["experts"], W)
    norm("final.norm")
    return out


def random_weights(config, seed=0):
    """bfloat16-representable weights with lively norms, gates, decays and convolutions (float32 tensors)."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for n, s in shapes(config).items():
        r = torch.randn(s, generator=g)
        leaf = n.split(".", 1)[-1]
        if leaf == "mix.lam":
            t = 1.5 * r - 3.0
        elif leaf == "mix.right.f.b":
            t = r + 2.0
        elif leaf.endswith(".b"):
            t = 0.3 * r
        elif len(s) == 1:
            t = 1.0 + 0.3 * r
        elif leaf == "canon1" or leaf == "mix.conv":
            t = 0.4 * r
        elif leaf == "mlp.router":
            t = 1.5 * r * s[1] ** -0.5
        elif n in ("embed", "pos"):
            t = 0.5 * r
        else:
            t = r * s[-1] ** -0.5
        out[n] = t.bfloat16().float()
    return out
