"""Checkpoint layout, seeded random initialisation, sharding and save / load.

Checkpoint ("state dict") names and shapes follow the reference's parameters:

    layers.{l}.qkv_proj.weight                 [(h + 2 kv) * hd, H]   q | k | v row blocks   (disagmoe/models/linear.py:626-712)
    layers.{l}.o_proj.weight                   [H, h * hd]                                   (linear.py:967-1014)
    layers.{l}.gate.weight                     [E, H]                                        (disagmoe/models/attention.py:159-164)
    layers.{l}.pre_attention_layernorm.weight  [H]
    layers.{l}.post_attention_layernorm.weight [H]                                           (attention.py:166-167)
    layers.{l}.experts.w13_weight              [E, H, 2 I]   gate half then up half, [in, out] (disagmoe/models/experts.py:42-55)
    layers.{l}.experts.w2_weight               [E, I, H]

plus what a real model needs and the reference mocks away: ``embed_tokens.weight [V, H]``, ``norm.weight [H]``,
``lm_head.weight [V, H]``, shared experts ``layers.{l}.shared_expert.{w13_weight [H, 2 Is], w2_weight [Is, H]}``,
``layers.{l}.shared_expert_gate.weight [1, H]`` and dense FFN layers ``layers.{l}.mlp.{w13_weight, w2_weight}``.

Sharding rules are those of the reference's weight loaders: q heads and kv heads are split over TP ranks (kv heads
replicated when tp > kv heads, linear.py:672-678), o_proj is split along its input dimension (linear.py:1016-1051),
expert tensors are sliced ``[e_lo:e_hi]`` per EP rank.

The kernels want every GEMM weight K-contiguous ("[out, in]"), so expert weights are transposed once at load time
into the runtime layout ``w13 [E, 2 I, H]`` / ``w2 [E, H, I]`` (:func:`to_runtime_expert_layout`).
"""
from __future__ import annotations

import json
import os
import struct
from typing import Dict, Iterable, List, Optional, Tuple

import torch

from ..config import (AttentionSpec, ChannelDeltaSpec, GatedLinearSpec, GatedUnitSpec, HeadDecaySpec, LatentAttentionSpec,
                      LayerListConfig, MatrixMemorySpec, ModelConfig, SideBySideSpec, WkvSpec)

StateDict = Dict[str, torch.Tensor]
WKV_MIXES = ("r", "k", "v", "g", "w")       # the mixed inputs of RWKV-style time mixing, in the order the mixer keeps them


def layer_norm_names(cfg: LayerListConfig, i: int) -> Tuple[str, ...]:
    """The residual-stream norms of layer i."""
    if cfg.block == "parallel":
        return ("norm1",)
    if cfg.block == "prenorm":
        return ("norm1", "norm2") if cfg.layers[i].ff or cfg.layers[i].routed else ("norm1",)
    return ("norm1", "norm1b") + (("norm2", "norm2b") if cfg.layers[i].ff else ())


def mixer_shapes(x: str, m, H: int) -> Dict[str, Tuple[int, ...]]:
    """Names (after the prefix x) and shapes of a mixer's tensors."""
    out: Dict[str, Tuple[int, ...]] = {}
    if isinstance(m, SideBySideSpec):
        for side, spec in (("left.", m.left), ("right.", m.right)):
            out.update(mixer_shapes(x + side, spec, H))
            out[x + side + "out"] = (H,)
        return out
    if isinstance(m, GatedUnitSpec):
        n, C = m.width // m.blocks, m.width
        for b in ("y", "x"):
            out.update({x + b: (C, H), x + b + ".b": (C,)})
        out.update({x + "conv": (C, m.conv), x + "conv.b": (C,), x + "lam": (C,), x + "o": (H, C)})
        for g in ("ra", "ri"):
            out.update({x + g: (m.blocks, n, n), x + g + ".b": (m.blocks, n)})
        return out
    vs = m.heads * m.vdim
    if isinstance(m, (HeadDecaySpec, MatrixMemorySpec)):
        ks = m.heads * m.dim
        out.update({x + "q": (ks, H), x + "k": (ks, H), x + "v": (vs, H), x + "g": (vs, H), x + "norm": (vs,)})
        if isinstance(m, MatrixMemorySpec):
            for g in ("i", "f"):
                out.update({x + g: (m.heads, H), x + g + ".b": (m.heads,)})
    elif isinstance(m, GatedLinearSpec):
        ks = m.heads * m.dim
        out.update({x + "q": (ks, H), x + "k": (ks, H), x + "v": (vs, H), x + "g": (vs, H), x + "norm": (m.vdim,),
                    x + "a1": (m.rank, H), x + "a2": (ks, m.rank), x + "a2.b": (ks,)})
    elif isinstance(m, ChannelDeltaSpec):
        ks, zs = m.kv_heads * m.dim, m.heads * m.dim
        for n, c in (("q", ks), ("k", ks), ("v", vs)):
            out.update({x + n: (c, H), x + n + ".conv": (c, m.conv)})
        out.update({x + "b": (m.heads, H), x + "A_log": (m.heads,), x + "norm": (m.vdim,), x + "a1": (m.rank, H),
                    x + "a2": (zs, m.rank), x + "dt_bias": (zs,), x + "g1": (m.gate_rank, H),
                    x + "g2": (vs, m.gate_rank)})
    elif isinstance(m, LatentAttentionSpec):
        out.update({x + "q": (m.heads * (m.dim + m.rot_dim), H), x + "dkv": (m.kv_rank + m.rot_dim, H),
                    x + "dkv.norm": (m.kv_rank,), x + "uk": (m.heads * m.dim, m.kv_rank), x + "uv": (vs, m.kv_rank)})
    elif isinstance(m, WkvSpec):
        out.update({x + "mu." + n: (H,) for n in WKV_MIXES})
        out.update({x + n: (vs, H) for n in ("r", "k", "v", "g")})
        out.update({x + "w1": (m.rank, H), x + "w2": (vs, m.rank), x + "w0": (vs,), x + "u": (m.heads, m.dim), x + "norm": (vs,)})
    else:
        own = m.kv_from is None
        out[x + "q"] = (m.heads * m.dim, H)
        if own:
            out[x + "k"] = (m.kv_heads * m.dim, H)
        if own and not m.tied_values:
            out[x + "v"] = (m.kv_heads * m.vdim, H)
        if m.qk_norm:
            out.update({x + n + ".norm": (m.dim,) for n in (("q", "k") if own else ("q",))})
        if m.v_mix:
            out[x + "vmix"] = ()
    if isinstance(m, (AttentionSpec, LatentAttentionSpec)) and m.gate:
        out[x + "g"] = (m.heads, H)
    if getattr(m, "sink", False):
        out[x + "sink"] = (m.heads,)
    out[x + "o"] = (H, vs)
    return out


def layer_list_shapes(cfg: LayerListConfig) -> Dict[str, Tuple[int, ...]]:
    """Names and shapes of a layer-list checkpoint: ``l<i>.norm1 / norm1b / norm2 / norm2b`` around the sublayers (parallel
    blocks have ``norm1`` alone, pre-norm blocks ``norm1`` and ``norm2``), ``l<i>.mix.*`` the mixer, ``l<i>.mlp.*`` the feed-forward, with ``e<j>.`` in front of an
    expert's tensors, ``l<i>.canon1`` the input convolution, ``l<i>.rg1 / rg2`` the residual gates; a bias has ``.b`` after the name of
    its weight; linear weights [out, in]. A layer that uses another one's weights has none."""
    H = cfg.hidden_size
    out: Dict[str, Tuple[int, ...]] = {"embed": (cfg.vocab_size, H)}
    if cfg.positions:
        out["pos"] = (cfg.positions, H)

    def norm(n: str) -> None:
        out.update({n: (H,), n + ".b": (H,)} if cfg.layer_norm else {n: (H,)})
    for i, layer in enumerate(cfg.layers):
        if layer.weights_of is not None:
            continue
        p = f"l{i}."
        for n in layer_norm_names(cfg, i):
            norm(p + n)
        out.update(mixer_shapes(p + "mix.", layer.mixer, H))
        if cfg.input_conv:
            out[p + "canon1"] = (H, cfg.input_conv)
        if cfg.residual_gate:
            for g in ("rg1", "rg2") if layer.ff or layer.routed else ("rg1",):
                out.update({p + g: (H, H), p + g + ".b": (H,)})
        gated = lambda q, ff: {q + "gate": (ff, H), q + "up": (ff, H), q + "down": (H, ff)}
        if layer.ff:
            out.update(gated(p + "mlp.", layer.ff))
        if layer.routed:
            for e in range(layer.routed.experts):
                out.update(gated(f"{p}mlp.e{e}.", layer.routed.ff))
            out[p + "mlp.router"] = (layer.routed.experts, H)
            if layer.routed.correction:
                out[p + "mlp.correction"] = (layer.routed.experts,)
    norm("final.norm")
    if not cfg.tied_head:
        out["head"] = (cfg.vocab_size, H)
    return out


def _init_layer_list_tensor(cfg: LayerListConfig, name: str, shape: Tuple[int, ...], gen, device) -> torch.Tensor:
    """Random values of the order a trained model has: weights of unit gain, norms near one, slow decays."""
    r = torch.randn(shape, generator=gen, device=device, dtype=torch.float32)
    leaf = name.split(".mix.")[-1]
    if leaf == "u":
        return r * 0.5
    if name.endswith(".canon1") or leaf == "conv":
        return 0.3 * r
    if leaf == "lam":
        return r - 4.0
    if leaf == "right.f.b":
        return 0.5 * r + 4.0
    if leaf.endswith(".b") and leaf != "a2.b":
        return 0.1 * r
    if len(shape) >= 2:
        return r * (0.02 if name in ("embed", "pos") else shape[-1] ** -0.5)
    if leaf == "A_log":
        return r * 0.3
    if leaf == "dt_bias":
        return r * 0.5 - 4.0
    if leaf == "a2.b":
        return r + 2.0
    if leaf.startswith("mu."):
        return torch.sigmoid(r)
    if leaf == "w0":
        return r - 3.0
    if leaf.endswith(".correction"):
        return r * 0.1
    if leaf == "vmix":
        return 0.5 + 0.1 * r
    if leaf == "sink":
        return r
    # norms of the residual stream: RMS norms store offsets from one
    return 1.0 + 0.05 * r if ".mix." in name or cfg.block == "parallel" or cfg.layer_norm else 0.05 * r


def param_shapes(cfg: ModelConfig) -> Dict[str, Tuple[int, ...]]:
    if isinstance(cfg, LayerListConfig):
        return layer_list_shapes(cfg)
    H, hd = cfg.hidden_size, cfg.head_dim
    shapes: Dict[str, Tuple[int, ...]] = {
        "embed_tokens.weight": (cfg.vocab_size, H),
        "norm.weight": (H,),
        "lm_head.weight": (cfg.vocab_size, H),
    }
    for l in range(cfg.num_layers):
        p = f"layers.{l}."
        shapes[p + "qkv_proj.weight"] = ((cfg.num_heads + 2 * cfg.num_kv_heads) * hd, H)
        shapes[p + "o_proj.weight"] = (H, cfg.num_heads * hd)
        shapes[p + "pre_attention_layernorm.weight"] = (H,)
        shapes[p + "post_attention_layernorm.weight"] = (H,)
        if cfg.is_dense_layer(l):
            shapes[p + "mlp.w13_weight"] = (H, 2 * cfg.dense_intermediate_size)
            shapes[p + "mlp.w2_weight"] = (cfg.dense_intermediate_size, H)
            continue
        shapes[p + "gate.weight"] = (cfg.num_experts, H)
        shapes[p + "experts.w13_weight"] = (cfg.num_experts, H, 2 * cfg.intermediate_size)
        shapes[p + "experts.w2_weight"] = (cfg.num_experts, cfg.intermediate_size, H)
        if cfg.num_shared_experts > 0:
            shapes[p + "shared_expert.w13_weight"] = (H, 2 * cfg.shared_intermediate_size)
            shapes[p + "shared_expert.w2_weight"] = (cfg.shared_intermediate_size, H)
            if cfg.shared_expert_gate:
                shapes[p + "shared_expert_gate.weight"] = (1, H)
    return shapes


def _name_seed(seed: int, name: str) -> int:
    h = 1469598103934665603
    for ch in name.encode():
        h = ((h ^ ch) * 1099511628211) & 0xFFFFFFFFFFFFFFFF
    return (h ^ (seed * 0x9E3779B97F4A7C15)) & 0x7FFFFFFFFFFFFFFF


def is_expert_stack(name: str) -> bool:
    return name.endswith(".experts.w13_weight") or name.endswith(".experts.w2_weight")


def init_tensor(cfg: ModelConfig, name: str, shape: Tuple[int, ...], device="cpu", dtype=None) -> torch.Tensor:
    """One parameter, N(0, init_std) (norm weights = 1), drawn from a generator seeded by (cfg.seed, name): the
    value of a tensor does not depend on which other tensors a process creates, so every worker can materialise
    only its shard's names and still agree with a single-process model. The stacked expert tensors are drawn expert
    by expert from (cfg.seed, name + "." + expert index), so an expert-parallel worker that creates only its own
    experts (:func:`init_expert`) gets exactly the slices of the full tensor. Draws on a CUDA device come from a
    different generator than CPU draws: compare models initialised on the same kind of device."""
    dtype = dtype or cfg.dtype
    if name.endswith("layernorm.weight") or name == "norm.weight":
        return torch.ones(shape, dtype=dtype, device=device)
    if is_expert_stack(name) and len(shape) == 3:
        return torch.stack([init_tensor(cfg, f"{name}.{e}", tuple(shape[1:]), device, dtype) for e in range(shape[0])])
    gen = torch.Generator(device=device)
    gen.manual_seed(_name_seed(cfg.seed, name))
    if isinstance(cfg, LayerListConfig):
        return _init_layer_list_tensor(cfg, name, shape, gen, device).to(dtype)
    t = torch.empty(shape, dtype=torch.float32 if torch.device(device).type == "cpu" else dtype, device=device)
    t.normal_(0.0, cfg.init_std, generator=gen)
    return t.to(dtype)


def init_expert(cfg: ModelConfig, layer_id: int, e: int, device="cpu", dtype=None) -> Tuple[torch.Tensor, torch.Tensor]:
    """Checkpoint-layout (w13 [H, 2I], w2 [I, H]) weights of global expert ``e`` of layer ``layer_id``: the same values
    as ``init_state_dict(cfg)["layers.<l>.experts.w13_weight"][e]`` / ``w2_weight[e]`` on the same kind of device."""
    p = f"layers.{layer_id}.experts."
    H, I = cfg.hidden_size, cfg.intermediate_size
    return (init_tensor(cfg, f"{p}w13_weight.{e}", (H, 2 * I), device, dtype),
            init_tensor(cfg, f"{p}w2_weight.{e}", (I, H), device, dtype))


def init_state_dict(cfg: ModelConfig, device="cpu", dtype=None, names: Optional[Iterable[str]] = None) -> StateDict:
    shapes = param_shapes(cfg)
    names = list(names) if names is not None else list(shapes)
    return {n: init_tensor(cfg, n, shapes[n], device, dtype) for n in names}


# ---------------------------------------------------------------------------------------------- sharding
def kv_heads_per_rank(cfg: ModelConfig, tp: int) -> int:
    return max(1, cfg.num_kv_heads // tp)


def shard_qkv(w: torch.Tensor, cfg: ModelConfig, tp: int, rank: int) -> torch.Tensor:
    """Rows of the fused qkv weight that TP rank ``rank`` owns: its q heads, then its (possibly replicated) kv heads."""
    if tp == 1:
        return w
    hd, h, kv = cfg.head_dim, cfg.num_heads, cfg.num_kv_heads
    assert h % tp == 0 and (kv % tp == 0 or tp % kv == 0)
    hq = h // tp
    q = w[rank * hq * hd:(rank + 1) * hq * hd]
    kvr = kv_heads_per_rank(cfg, tp)
    kv_idx = rank * kvr if kv >= tp else rank // (tp // kv)
    k0 = h * hd
    k = w[k0 + kv_idx * hd:k0 + (kv_idx + kvr) * hd]
    v0 = k0 + kv * hd
    v = w[v0 + kv_idx * hd:v0 + (kv_idx + kvr) * hd]
    return torch.cat([q, k, v], dim=0).contiguous()


def shard_o_proj(w: torch.Tensor, cfg: ModelConfig, tp: int, rank: int) -> torch.Tensor:
    if tp == 1:
        return w
    per = cfg.num_heads // tp * cfg.head_dim
    return w[:, rank * per:(rank + 1) * per].contiguous()


def shard_experts(w: torch.Tensor, e_lo: int, e_hi: int) -> torch.Tensor:
    return w[e_lo:e_hi]


def to_runtime_expert_layout(w13_ckpt: torch.Tensor, w2_ckpt: torch.Tensor) -> Tuple[torch.Tensor, torch.Tensor]:
    """[.., H, 2I] / [.., I, H] ([in, out]) -> K-contiguous [.., 2I, H] / [.., H, I] ([out, in])."""
    return w13_ckpt.transpose(-1, -2).contiguous(), w2_ckpt.transpose(-1, -2).contiguous()


def to_checkpoint_expert_layout(w13_rt: torch.Tensor, w2_rt: torch.Tensor) -> Tuple[torch.Tensor, torch.Tensor]:
    return w13_rt.transpose(-1, -2).contiguous(), w2_rt.transpose(-1, -2).contiguous()


# ---------------------------------------------------------------------------------------------- save / load
def save_state_dict(sd: StateDict, path: str) -> None:
    os.makedirs(os.path.dirname(os.path.abspath(path)) or ".", exist_ok=True)
    tmp = path + ".tmp"
    torch.save({k: v.detach().cpu() for k, v in sd.items()}, tmp)
    os.replace(tmp, path)


def load_state_dict(path: str, device="cpu", dtype=None) -> StateDict:
    sd = torch.load(path, map_location="cpu", weights_only=True)
    return {k: v.to(device=device, dtype=dtype or v.dtype) for k, v in sd.items()}


_SAFETENSORS_DTYPES = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16, "I32": torch.int32,
                       "I64": torch.int64}


def load_safetensors(path: str) -> StateDict:
    """Reads a safetensors file: 8-byte little-endian header length, a JSON header name -> dtype, shape, data_offsets, then
    the data. Tensors keep their stored dtype and own their memory."""
    out: StateDict = {}
    with open(path, "rb") as f:
        n = struct.unpack("<Q", f.read(8))[0]
        header = json.loads(f.read(n))
        for name, e in header.items():
            if name == "__metadata__":
                continue
            if e["dtype"] not in _SAFETENSORS_DTYPES:
                raise ValueError(f"{path}: tensor {name} has unsupported dtype {e['dtype']}")
            a, b = e["data_offsets"]
            f.seek(8 + n + a)
            data = bytearray(f.read(b - a))
            dt = _SAFETENSORS_DTYPES[e["dtype"]]
            t = torch.frombuffer(data, dtype=dt) if data else torch.empty(0, dtype=dt)
            out[name] = t.reshape(e["shape"])
    return out


def save_safetensors(sd: StateDict, path: str) -> None:
    """Writes tensors in the format :func:`load_safetensors` reads."""
    names = {v: k for k, v in _SAFETENSORS_DTYPES.items()}
    header, pos, blobs = {}, 0, []
    for name, t in sd.items():
        t = t.detach().cpu().contiguous()
        raw = t.reshape(-1).view(torch.uint8).numpy().tobytes()
        header[name] = {"dtype": names[t.dtype], "shape": list(t.shape), "data_offsets": [pos, pos + len(raw)]}
        pos += len(raw)
        blobs.append(raw)
    head = json.dumps(header).encode()
    head += b" " * (-len(head) % 8)
    tmp = path + ".tmp"
    with open(tmp, "wb") as f:
        f.write(struct.pack("<Q", len(head)) + head + b"".join(blobs))
    os.replace(tmp, path)


def check_state_dict(cfg: ModelConfig, sd: StateDict) -> List[str]:
    """Names that are missing or have the wrong shape (empty list = compatible)."""
    bad = []
    for n, shp in param_shapes(cfg).items():
        if n not in sd or tuple(sd[n].shape) != tuple(shp):
            bad.append(n)
    return bad
