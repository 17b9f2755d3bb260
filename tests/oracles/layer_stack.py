"""Slow double-precision restatement of the layer-list decoder (Rurunex design), one function per mechanism.

Every function takes the whole history of one sequence (rows = tokens from position 0) and loops where a loop is the
clearest statement: no cache, no state carried between calls, no batching, and no code of the package. Weights come as
a dict name -> tensor with the checkpoint's names, the configuration as the plain dict of config.json.
"""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def centred_norm(x, w, eps):
    """Norm whose stored weight is an offset from one."""
    return rms(x, eps) * (1.0 + w)


def silu(x):
    return x / (1.0 + torch.exp(-x))


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def softplus(x):
    return torch.clamp(x, min=0) + torch.log1p(torch.exp(-x.abs()))


def log_sigmoid(x):
    return -softplus(-x)


def inverse_frequencies(rot):
    """(frequencies [dims / 2], factor on cos and sin) of a rotation, with the YaRN ramp if it is scaled."""
    dims, base = rot["dims"], float(rot["base"])
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return torch.tensor(f, dtype=torch.float64), 1.0
    where = lambda turns: dims * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(where(sc["fast"])), 0), min(math.ceil(where(sc["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / sc["factor"] * r + fi * (1 - r))
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x, rot):
    """x [T, heads, dim]: row t is at position t."""
    if not rot:
        return x
    f, m = inverse_frequencies(rot)
    half = rot["dims"] // 2
    a = torch.arange(x.shape[0], dtype=torch.float64)[:, None, None] * f
    c, s = torch.cos(a) * m, torch.sin(a) * m
    u, v, rest = x[..., :half], x[..., half:2 * half], x[..., 2 * half:]
    return torch.cat([u * c - v * s, v * c + u * s, rest], -1)


def short_conv(x, taps):
    """Causal depthwise convolution: x [T, C], taps [C, n]; the last column weighs the current row."""
    n = taps.shape[1]
    pad = torch.cat([torch.zeros(n - 1, x.shape[1], dtype=x.dtype), x])
    return sum(pad[j:j + x.shape[0]] * taps[:, j] for j in range(n))


def gla_recurrence(q, k, v, log_decay, with_state=False):
    """q, k, log_decay [T, H, D], v [T, H, V] -> read-outs [T, H, V] (and the state after the last token)."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=q.dtype)
    out = []
    for t in range(T):
        S = torch.exp(log_decay[t])[..., None] * S + k[t][..., None] * v[t][:, None, :]
        out.append((S * q[t][..., None]).sum(1))
    return (torch.stack(out), S) if with_state else torch.stack(out)


def delta_recurrence(q, k, v, log_decay, beta, with_state=False):
    """As above, but what is written is the error of the read-out at k, scaled by beta [T, H]."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=q.dtype)
    out = []
    for t in range(T):
        S = torch.exp(log_decay[t])[..., None] * S
        u = beta[t][:, None] * (v[t] - (S * k[t][..., None]).sum(1))
        S = S + k[t][..., None] * u[:, None, :]
        out.append((S * q[t][..., None]).sum(1))
    return (torch.stack(out), S) if with_state else torch.stack(out)


def gla(h, w, p, m, eps):
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).view(T, H, D) * D ** -0.5
    k = (h @ w[p + "k"].T).view(T, H, D)
    v = (h @ w[p + "v"].T).view(T, H, V)
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]
    o = gla_recurrence(q, k, v, log_sigmoid(z).view(T, H, D) / m["tau"])
    o = rms(o, eps) * w[p + "norm"]
    return (o.reshape(T, H * V) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def channel_delta(h, w, p, m, eps):
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    act = lambda n: silu(short_conv(h @ w[p + n].T, w[p + n + ".conv"]))
    unit = lambda x: x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)
    q, k = unit(act("q").view(T, G, D)) * D ** -0.5, unit(act("k").view(T, G, D))
    q, k = q.repeat_interleave(H // G, 1), k.repeat_interleave(H // G, 1)
    v = act("v").view(T, H, V)
    beta = sigmoid(h @ w[p + "b"].T)
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]
    logd = -torch.exp(w[p + "A_log"])[:, None] * softplus(z).view(T, H, D)
    o = delta_recurrence(q, k, v, logd, beta)
    o = rms(o, eps) * w[p + "norm"]
    gate = sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T)
    return (o.reshape(T, H * V) * gate) @ w[p + "o"].T


def softmax_attention(q, k, v, scale, softcap, window):
    """q [T, H, D], k [T, G, D], v [T, G, V], all of one sequence from position 0."""
    T, H = q.shape[:2]
    g = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for i in range(T):
        j0 = 0 if not window else max(0, i - window + 1)
        for h in range(H):
            s = (k[j0:i + 1, h // g] @ q[i, h]) * scale
            if softcap:
                s = softcap * torch.tanh(s / softcap)
            out[i, h] = torch.softmax(s, 0) @ v[j0:i + 1, h // g]
    return out


def attention(h, w, p, m, eps, shared=None):
    """Returns (output, (keys, values)); ``shared`` are the keys and values of an earlier layer."""
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rotate(rms((h @ w[p + "q"].T).view(T, H, D), eps) * w[p + "q.norm"], m.get("rot"))
    if shared is None:
        k = rotate(rms((h @ w[p + "k"].T).view(T, G, D), eps) * w[p + "k.norm"], m.get("rot"))
        shared = (k, (h @ w[p + "v"].T).view(T, G, V))
    o = softmax_attention(q, *shared, m["scale"], m.get("softcap"), (m.get("mask") or {}).get("size"))
    return o.reshape(T, H * V) @ w[p + "o"].T, shared


def feed_forward(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def run(config, weights, tokens):
    """(logits [T, vocab], residual stream after every layer [layers, T, width]) in double precision."""
    w = {n: t.double() for n, t in weights.items()}
    eps = config["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens).long()] * config["embedding"]["scale"]
    kv, stream = {}, []
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = centred_norm(x, w[p + "norm1"], eps)
        if layer["type"] == "gla":
            y = gla(h, w, p + "mix.", m, eps)
        elif layer["type"] == "channel_delta":
            y = channel_delta(h, w, p + "mix.", m, eps)
        else:
            y, kv[i] = attention(h, w, p + "mix.", m, eps, kv.get(m.get("kv_from", -1)))
        x = x + centred_norm(y, w[p + "norm1b"], eps)
        if layer["mlp"] is not None:
            y = feed_forward(centred_norm(x, w[p + "norm2"], eps), w, p + "mlp.")
            x = x + centred_norm(y, w[p + "norm2b"], eps)
        stream.append(x)
    logits = centred_norm(x, w["final.norm"], eps) @ w["head"].T * config["logit_scale"]
    return logits, torch.stack(stream)


def shapes(config):
    """Checkpoint tensor names and shapes of a configuration (``rank`` of the low-rank maps: mixer['rank'], default 8)."""
    W, out = config["width"], {}
    out["embed"] = (config["vocab"], W)
    for i, layer in enumerate(config["layers"]):
        p, m, t = f"l{i}.", layer["mixer"], layer["type"]
        H, D, V = m["heads"], m["dim"], m["vdim"]
        G, r = m.get("kv_heads", H), m.get("rank", 8)
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if layer["mlp"] else ()):
            out[p + n] = (W,)
        x = p + "mix."
        if t == "gla":
            out.update({x + "q": (H * D, W), x + "k": (H * D, W), x + "v": (H * V, W), x + "g": (H * V, W),
                        x + "o": (W, H * V), x + "norm": (V,), x + "a1": (r, W), x + "a2": (H * D, r), x + "a2.b": (H * D,)})
        elif t == "channel_delta":
            for n, c in (("q", G * D), ("k", G * D), ("v", H * V)):
                out[x + n] = (c, W)
                out[x + n + ".conv"] = (c, m["conv"])
            out.update({x + "b": (H, W), x + "A_log": (H,), x + "norm": (V,), x + "a1": (r, W), x + "a2": (H * D, r),
                        x + "dt_bias": (H * D,), x + "g1": (r, W), x + "g2": (H * V, r), x + "o": (W, H * V)})
        else:
            out.update({x + "q": (H * D, W), x + "q.norm": (D,), x + "o": (W, H * V)})
            if "kv_from" not in m:
                out.update({x + "k": (G * D, W), x + "v": (G * V, W), x + "k.norm": (D,)})
        if layer["mlp"]:
            F = layer["mlp"]["ff"]
            out.update({p + "mlp.gate": (F, W), p + "mlp.up": (F, W), p + "mlp.down": (W, F)})
    out["final.norm"] = (W,)
    out["head"] = (config["vocab"], W)
    return out


def random_weights(config, seed=0):
    """bfloat16-representable weights with lively norms, gates and decays (float32 tensors)."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for n, s in shapes(config).items():
        leaf = n.split("mix.")[-1].split(".", 1)[-1] if "mix." not in n else n.split("mix.")[-1]
        r = torch.randn(*s, generator=g)
        if len(s) == 1:
            t = {"A_log": 0.5 * r, "dt_bias": r - 2.0, "a2.b": r + 1.0}.get(leaf)
            if t is None:
                t = 1.0 + 0.3 * r if leaf in ("norm", "q.norm", "k.norm") and "mix." in n else 0.2 * r
        elif leaf.endswith(".conv"):
            t = r * s[1] ** -0.5
        elif n == "embed":
            t = 0.1 * r
        else:
            t = r * s[1] ** -0.5
        out[n] = t.bfloat16().float()
    return out
