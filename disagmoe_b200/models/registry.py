"""Model registry: which configuration reader, checkpoint layout and executor serve an architecture.

``load_model(path)`` reads a checkpoint folder (config.json + model.safetensors) and picks the architecture by the
``architecture`` key of config.json; ``make_executor`` builds the whole-iteration executor of a configuration, whether it
comes from a folder or from a preset.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Any, Callable, Dict, Optional, Tuple

import torch

from ..config import (AttentionSpec, ChannelDeltaSpec, GatedLinearSpec, GatedUnitSpec, HeadDecaySpec, LatentAttentionSpec,
                      LayerListConfig, LayerSpec, MatrixMemorySpec, ModelConfig, PRESETS, QueryTemperature, RotarySpec, RoutedSpec,
                      SideBySideSpec, WkvSpec, get_preset)
from . import weights as W


def _rotary(rot: Optional[dict], interleaved: bool = False) -> Optional[RotarySpec]:
    if not rot:
        return None
    sc = rot.get("scaling") or {}
    return RotarySpec(int(rot["dims"]), float(rot["base"]), interleaved=interleaved, **{k: float(v) for k, v in sc.items()})


def _window(mixer: dict) -> Optional[int]:
    return (mixer.get("mask") or {}).get("size")


# ---- Rurunex: gated linear attention, channel-wise gated delta rule and windowed attention in any order -----------------
def _rurunex_layer(i: int, layer: dict, shapes: Dict[str, Tuple[int, ...]]) -> LayerSpec:
    m, kind = layer["mixer"], layer["type"]
    rank = lambda name: shapes[f"l{i}.mix.{name}"][0] if f"l{i}.mix.{name}" in shapes else 16
    if kind == "gla":
        mixer = GatedLinearSpec(m["heads"], m["dim"], m["vdim"], float(m["tau"]), rank("a1"))
    elif kind == "channel_delta":
        mixer = ChannelDeltaSpec(m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"], rank("a1"), rank("g1"))
    elif kind == "attention":
        mixer = AttentionSpec(m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]), _rotary(m.get("rot")),
                              _window(m), m.get("softcap"), m.get("kv_from"))
    else:
        raise ValueError(f"layer {i}: unknown mixer {kind!r}")
    mlp = layer.get("mlp")
    if mlp is not None and mlp.get("kind") != "dense":
        raise ValueError(f"layer {i}: unknown feed-forward {mlp.get('kind')!r}")
    return LayerSpec(mixer, None if mlp is None else mlp["ff"])


def rurunex_config_from_json(raw: Dict[str, Any], shapes: Dict[str, Tuple[int, ...]], **kw) -> LayerListConfig:
    """``shapes``: tensor name -> shape of the checkpoint, the only place that has the ranks of the low-rank maps."""
    layers = [_rurunex_layer(i, l, shapes) for i, l in enumerate(raw["layers"])]
    return LayerListConfig.make(raw["width"], raw["vocab"], layers, rms_norm_eps=float(raw["norm"]["eps"]),
                                embed_scale=float(raw["embedding"]["scale"]), logit_scale=float(raw["logit_scale"]),
                                architecture=raw["architecture"], name=raw["architecture"].lower(), **kw)


# ---- Supinex: attention over everything and windowed latent attention in any order, dense or routed feed-forwards, both
# sublayers of a layer on one norm -----------------------------------------------------------------------------------------
def _supinex_layer(i: int, layer: dict) -> LayerSpec:
    m, kind, mlp = layer["mixer"], layer["type"], layer.get("mlp")
    rot = _rotary(m.get("rot"), interleaved=True)
    if kind == "latent_attention":
        mixer = LatentAttentionSpec(m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], float(m["scale"]), rot,
                                    _window(m), sink=True)
    elif kind == "attention":
        mixer = AttentionSpec(m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]), rot, _window(m),
                              qk_norm=False, sink=True, v_mix=bool(m.get("v_mix")))
    else:
        raise ValueError(f"layer {i}: unknown mixer {kind!r}")
    if mlp is None:
        return LayerSpec(mixer)
    if mlp["kind"] == "dense":
        return LayerSpec(mixer, mlp["ff"], "gelu_tanh")
    if mlp["kind"] != "moe":
        raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
    return LayerSpec(mixer, routed=RoutedSpec(mlp["router"]["experts"], mlp["router"]["top"], mlp["expert"]["ff"]))


def supinex_config_from_json(raw: Dict[str, Any], shapes: Dict[str, Tuple[int, ...]], **kw) -> LayerListConfig:
    layers = [_supinex_layer(i, l) for i, l in enumerate(raw["layers"])]
    return LayerListConfig.make(raw["width"], raw["vocab"], layers, rms_norm_eps=float(raw["norm"]["eps"]), block="parallel",
                                architecture=raw["architecture"], name=raw["architecture"].lower(), **kw)


# ---- Vufinex: RWKV-style time mixing, gated latent attention and chunked attention in any order, grouped sigmoid routers; layers
# may use the weights of others ---------------------------------------------------------------------------------------------
def _vufinex_layer(i: int, layer: dict, j: int, shapes: Dict[str, Tuple[int, ...]]) -> LayerSpec:
    """``j``: the layer whose tensors layer i uses."""
    m, kind, mlp = layer["mixer"], layer["type"], layer.get("mlp")
    if kind == "wkv":
        mixer = WkvSpec(m["heads"], m["dim"], shapes.get(f"l{j}.mix.w1", (16,))[0])
    elif kind == "latent_attention":
        mixer = LatentAttentionSpec(m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], float(m["scale"]),
                                    _rotary(m.get("rot"), interleaved=True), gate=True)
    elif kind == "attention":
        mixer = AttentionSpec(m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]), _rotary(m.get("rot")),
                              qk_norm=False, chunk=_window(m), tied_values=True)
    else:
        raise ValueError(f"layer {i}: unknown mixer {kind!r}")
    routed = None
    if mlp is not None:
        if mlp["kind"] != "moe":
            raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
        r = mlp["router"]
        g = r.get("groups") or {"count": 1, "keep": 1}
        routed = RoutedSpec(r["experts"], r["top"], mlp["expert"]["ff"], renormalize=True, scoring="sigmoid", correction=True,
                            groups=g["count"], keep=g["keep"], scale=float(r.get("scale", 1.0)))
    return LayerSpec(mixer, routed=routed, weights_of=layer.get("weights_of"))


def vufinex_config_from_json(raw: Dict[str, Any], shapes: Dict[str, Tuple[int, ...]], **kw) -> LayerListConfig:
    def owner(i: int) -> int:
        for _ in raw["layers"]:
            if raw["layers"][i].get("weights_of") is None:
                break
            i = raw["layers"][i]["weights_of"]
        return i
    layers = [_vufinex_layer(i, l, owner(i), shapes) for i, l in enumerate(raw["layers"])]
    return LayerListConfig.make(raw["width"], raw["vocab"], layers, rms_norm_eps=float(raw["norm"]["eps"]), block="prenorm",
                                embed_scale=float(raw["embedding"]["scale"]), residual_mult=float(raw["residual_mult"]),
                                architecture=raw["architecture"], name=raw["architecture"].lower(), **kw)


# ---- Panarax: attention beside a matrix memory, gated diagonal recurrences and lightning attention in any order, dense or
# clamped routed feed-forwards; gated residuals, input convolutions, learned positions ---------------------------------------
def _panarax_layer(i: int, layer: dict) -> LayerSpec:
    m, kind, mlp = layer["mixer"], layer["type"], layer.get("mlp")
    if kind == "rglru":
        mixer = GatedUnitSpec(m["width"], m["blocks"], m["conv"])
    elif kind == "lightning":
        mixer = HeadDecaySpec(m["heads"], m["dim"], m["vdim"], tuple(float(d) for d in m["decay"]))
    elif kind == "parallel":
        a, r = m["left"], m["right"]
        t = a.get("q_temp")
        mixer = SideBySideSpec(
            AttentionSpec(a["heads"], a["kv_heads"], a["dim"], a["vdim"], float(a["scale"]), qk_norm=False, value_norm=True, gate=True,
                          q_temp=QueryTemperature(float(t["coef"]), int(t["every"])) if t else None),
            MatrixMemorySpec(r["heads"], r["dim"], r["vdim"], float(r["gate_cap"])))
    else:
        raise ValueError(f"layer {i}: unknown mixer {kind!r}")
    if mlp is None:
        return LayerSpec(mixer)
    if mlp["kind"] == "dense":
        return LayerSpec(mixer, mlp["ff"])
    if mlp["kind"] != "moe":
        raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
    r, e = mlp["router"], mlp["expert"]
    return LayerSpec(mixer, routed=RoutedSpec(r["experts"], r["top"], e["ff"], act="clamped", scoring="sigmoid", limit=float(e["limit"]),
                                              weigh_input=True))


def panarax_config_from_json(raw: Dict[str, Any], shapes: Dict[str, Tuple[int, ...]], **kw) -> LayerListConfig:
    layers = [_panarax_layer(i, l) for i, l in enumerate(raw["layers"])]
    return LayerListConfig.make(raw["width"], raw["vocab"], layers, rms_norm_eps=float(raw["norm"]["eps"]), block="prenorm",
                                layer_norm=True, residual_gate=True, input_conv=int(raw["canon"]["taps"]),
                                positions=int(raw["max_positions"]), tied_head=True, architecture=raw["architecture"],
                                name=raw["architecture"].lower(), **kw)


@dataclass(frozen=True)
class Architecture:
    config_from_json: Callable[..., ModelConfig]


ARCHITECTURES: Dict[str, Architecture] = {
    "Rurunex": Architecture(rurunex_config_from_json),
    "Supinex": Architecture(supinex_config_from_json),
    "Vufinex": Architecture(vufinex_config_from_json),
    "Panarax": Architecture(panarax_config_from_json),
}


def load_model(path: str, dtype: Optional[torch.dtype] = None, **kw) -> Tuple[ModelConfig, W.StateDict]:
    """(configuration, weights on the CPU as stored) of a checkpoint folder. ``kw``: further configuration fields."""
    with open(os.path.join(path, "config.json")) as f:
        raw = json.load(f)
    name = raw.get("architecture")
    if name not in ARCHITECTURES:
        raise ValueError(f"unknown architecture {name!r}; known: {sorted(ARCHITECTURES)}")
    sd = W.load_safetensors(os.path.join(path, "model.safetensors"))
    cfg = ARCHITECTURES[name].config_from_json(raw, {n: tuple(t.shape) for n, t in sd.items()},
                                               dtype=dtype or torch.bfloat16, **kw)
    bad = W.check_state_dict(cfg, sd)
    if bad:
        raise ValueError(f"{path}: tensors missing or of the wrong shape: {', '.join(bad[:8])}")
    return cfg, sd


def resolve_model(name_or_path: str, dtype: Optional[torch.dtype] = None, **kw) -> Tuple[ModelConfig, Optional[W.StateDict]]:
    """A preset name -> (its configuration, None: random weights); a checkpoint folder -> :func:`load_model`."""
    if name_or_path in PRESETS:
        return get_preset(name_or_path, **({"dtype": dtype} if dtype else {}), **kw), None
    if os.path.isdir(name_or_path):
        return load_model(name_or_path, dtype, **kw)
    raise ValueError(f"{name_or_path!r} is neither a preset ({', '.join(sorted(PRESETS))}) nor a checkpoint folder")


def require_experts(cfg: ModelConfig) -> None:
    """The disaggregated paths place the MoE decoder's routed experts on GPUs of their own; layer-list models, which have
    none or keep them beside the attention, are refused there."""
    if isinstance(cfg, LayerListConfig):
        why = "keeps its experts beside the attention" if any(l.routed for l in cfg.layers) else "has no routed experts"
        raise ValueError(f"{cfg.name} {why}: serve it with the single-GPU engines (--backend colocated)")


def make_executor(cfg: ModelConfig, cache_cfg, **kw):
    """The whole-iteration executor that runs ``cfg`` on one device."""
    from ..executor.fused import FusedModelExecutor
    from ..executor.layer_list import LayerListExecutor
    cls = LayerListExecutor if isinstance(cfg, LayerListConfig) else FusedModelExecutor
    return cls(cfg, cache_cfg, **kw)
