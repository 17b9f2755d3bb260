"""Model / cache / sampling configuration and the model presets.

Field names follow the reference's dataclasses (disagmoe/config.py:8-67) so that scripts written against it keep
working; the extra fields describe what the reference mocks away (vocabulary, RoPE, shared experts, dense
layers) and what the Blackwell kernels need to know.
"""
from __future__ import annotations

from dataclasses import dataclass, field, replace
from typing import List, Optional, Tuple, Union

import torch


@dataclass
class ModelConfig:
    hidden_size: int
    num_layers: int
    num_heads: int
    num_kv_heads: int
    num_experts: int
    intermediate_size: int
    dtype: torch.dtype
    ep_size: int
    tp_size: int = 1
    dp_size: int = 1
    rank: int = 0
    layer_ids: Optional[List[int]] = None
    top_k: int = 1

    tp_enable_inter_group: bool = True
    enable_cuda_graph_attn: bool = False
    enable_cuda_graph_expert: bool = False
    enable_grouped_gemm: bool = True

    graph_stride: int = 8
    max_batch_size_attn: int = 160
    max_batch_size_expert: int = 512
    max_seq_len: int = 4096

    enable_trace: bool = False

    # ---- real-model fields (the reference serves a mocked model and has none of these) ----
    vocab_size: int = 32000
    head_dim: Optional[int] = None              # default hidden_size // num_heads
    rope_theta: float = 10000.0
    rms_norm_eps: float = 1e-5
    norm_topk_prob: bool = True                 # renormalise the top-k router weights (Mixtral: yes)
    num_shared_experts: int = 0                 # always-on experts (Qwen-MoE: 1, DeepSeek-V2-Lite: 2)
    shared_intermediate_size: int = 0           # total ffn width of the shared expert(s)
    shared_expert_gate: bool = False            # sigmoid gate on the shared expert output (Qwen-MoE)
    first_k_dense: int = 0                      # leading layers with a dense FFN instead of experts
    dense_intermediate_size: int = 0
    eos_token_id: int = 2
    init_std: float = 0.02
    seed: int = 0
    name: str = "custom"

    def __post_init__(self):
        if self.head_dim is None:
            self.head_dim = self.hidden_size // self.num_heads

    @property
    def num_experts_per_rank(self) -> int:
        return self.num_experts // self.ep_size

    @property
    def q_size(self) -> int:
        return self.num_heads * self.head_dim

    @property
    def kv_size(self) -> int:
        return self.num_kv_heads * self.head_dim

    def is_dense_layer(self, layer_id: int) -> bool:
        return layer_id < self.first_k_dense

    def clone(self, **changes) -> "ModelConfig":
        return replace(self, **changes)


ACTIVATIONS = ("silu", "gelu_tanh")             # of gated feed-forwards
EXPERT_ACTIVATIONS = ACTIVATIONS + ("clamped",)     # of experts: also min(g, limit) sigmoid(1.702 g) (clamp(u, limit) + 1)


# ---- decoders described layer by layer --------------------------------------------------------------------------------
# A layer = one token mixer (attention or a linear recurrence) and an optional feed-forward, dense or routed to experts.
# Mixers carry their own sizes, so layers of one model may differ in everything but the width. How the two sublayers sit on
# the residual stream is the model's ``block``.
@dataclass(frozen=True)
class RotarySpec:
    """Rotary embedding on the first ``dims`` dimensions of a head: pairs (i, i + dims / 2), or (2i, 2i + 1) where
    ``interleaved``; ``factor`` != None: YaRN."""
    dims: int
    base: float
    factor: Optional[float] = None
    original: float = 0.0
    fast: float = 32.0
    slow: float = 1.0
    interleaved: bool = False


@dataclass(frozen=True)
class QueryTemperature:
    """Scores of the query at position p are multiplied by 1 + coef ln(floor((p + 1) / every) + 1)."""
    coef: float
    every: int


@dataclass(frozen=True)
class AttentionSpec:
    """Softmax attention. ``window``: how many of the latest tokens, its own included, a query attends to (None: all).
    ``chunk``: positions fall into chunks of that size, counted from 0, and a query attends to its own chunk only.
    ``kv_from``: the earlier layer whose cached keys and values this layer reads (it then has none). ``qk_norm``: RMS norm
    of every query and key head. ``sink``: a learned number per head enters the softmax denominator. ``v_mix``: the values
    are mixed with those that the first such layer computed for the same token. ``tied_values``: the values are the keys before
    their rotation (vdim = dim, no map of their own). ``value_norm``: every value head is divided by its root mean square before it
    is cached. ``gate``: every head's output is scaled by the sigmoid of a linear map of the layer's input. ``q_temp``: query
    temperature by position."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Optional[RotarySpec] = None
    window: Optional[int] = None
    softcap: Optional[float] = None
    kv_from: Optional[int] = None
    qk_norm: bool = True
    sink: bool = False
    v_mix: bool = False
    chunk: Optional[int] = None
    tied_values: bool = False
    value_norm: bool = False
    gate: bool = False
    q_temp: Optional[QueryTemperature] = None


@dataclass(frozen=True)
class LatentAttentionSpec:
    """Softmax attention whose keys and values are linear maps of one latent vector of ``kv_rank`` numbers per token; beside
    it every token has one rotated key part of ``rot_dim`` numbers that all heads share. The cache holds those two. ``gate``:
    every head's output is scaled by the sigmoid of a linear map of the layer's input."""
    heads: int
    dim: int                                    # unrotated query / key size per head
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot: Optional[RotarySpec] = None
    window: Optional[int] = None
    sink: bool = False
    gate: bool = False


@dataclass(frozen=True)
class GatedLinearSpec:
    """Gated linear attention: decay sigmoid(z)^(1 / tau) per key channel, ``rank`` = inner size of the map to z."""
    heads: int
    dim: int
    vdim: int
    tau: float
    rank: int = 16


@dataclass(frozen=True)
class ChannelDeltaSpec:
    """Gated delta rule with one decay per head and key channel and short convolutions of ``conv`` taps on q, k and v;
    ``rank`` / ``gate_rank`` = inner sizes of the maps to the decay and to the output gate."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    rank: int = 16
    gate_rank: int = 16


@dataclass(frozen=True)
class WkvSpec:
    """RWKV-style time mixing: every projection reads a mix of its own of the row and the row before it; state of ``dim`` x
    ``dim`` numbers per head with decays exp(-exp(.)) per key channel, read before the token's own write, which enters with a
    bonus per channel. ``rank`` = inner size of the map to the decays."""
    heads: int
    dim: int
    rank: int = 16

    @property
    def vdim(self) -> int:
        return self.dim

    @property
    def kv_heads(self) -> int:
        return self.heads


@dataclass(frozen=True)
class HeadDecaySpec:
    """Lightning attention: linear attention with silu on queries, keys and values and one constant decay per head; all heads'
    read-outs are normed together and gated."""
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]

    @property
    def kv_heads(self) -> int:
        return self.heads


@dataclass(frozen=True)
class MatrixMemorySpec:
    """Matrix memory of xLSTM: exponential input gate and sigmoid forget gate per head and token, logits soft-capped at
    ``gate_cap``; beside the state a normaliser and a running maximum per head."""
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    @property
    def kv_heads(self) -> int:
        return self.heads


@dataclass(frozen=True)
class GatedUnitSpec:
    """Griffin's recurrent block: a branch through a short convolution of ``conv`` taps and a real-gated diagonal recurrence of
    ``width`` channels, multiplied by a gelu branch. The two gates are linear within each of the ``blocks`` equal parts."""
    width: int
    blocks: int
    conv: int

    @property
    def heads(self) -> int:
        return self.blocks

    @property
    def kv_heads(self) -> int:
        return self.blocks

    @property
    def dim(self) -> int:
        return self.width // self.blocks

    @property
    def vdim(self) -> int:
        return self.dim


@dataclass(frozen=True)
class SideBySideSpec:
    """Two mixers on the same rows; the result is half the sum of their outputs, each normed over the model width first."""
    left: AttentionSpec
    right: MatrixMemorySpec

    @property
    def heads(self) -> int:
        return max(self.left.heads, self.right.heads)

    @property
    def dim(self) -> int:
        return max(self.left.dim, self.right.dim)


@dataclass(frozen=True)
class RoutedSpec:
    """Feed-forward of ``experts`` gated feed-forwards of width ``ff``; a token uses the ``top`` ones with the largest
    scores, weighted by these scores (``renormalize``: divided by their sum) times ``scale``. ``scoring``: "softmax", or
    "sigmoid" of every logit. With sigmoid scores, ``correction``: a stored number per expert enters the choice, not the weight;
    ``groups`` / ``keep``: the list of experts is cut into ``groups`` runs of one length, ranked by the sum of their two best
    corrected scores, and a token chooses within the first ``keep`` of them. ``limit``: of the "clamped" activation.
    ``weigh_input``: the weight scales what an expert reads, not what it returns."""
    experts: int
    top: int
    ff: int
    act: str = "silu"
    renormalize: bool = False
    scoring: str = "softmax"
    correction: bool = False
    groups: int = 1
    keep: int = 1
    scale: float = 1.0
    limit: float = 0.0
    weigh_input: bool = False


@dataclass(frozen=True)
class LayerSpec:
    mixer: Union[AttentionSpec, LatentAttentionSpec, GatedLinearSpec, ChannelDeltaSpec, WkvSpec, HeadDecaySpec, GatedUnitSpec,
                 SideBySideSpec]
    ff: Optional[int] = None                    # width of the dense gated feed-forward, None = the layer has none
    act: str = "silu"                           # of the dense feed-forward: silu or gelu_tanh
    routed: Optional[RoutedSpec] = None         # experts instead of a dense feed-forward
    weights_of: Optional[int] = None            # the layer that lends this one its tensors (caches and states stay per layer)


@dataclass
class LayerListConfig(ModelConfig):
    """A decoder given as a list of :class:`LayerSpec`. The MoE fields of the base class stay at zero: experts, where
    layers have some, run beside the attention, and only the single-GPU engines serve these models.

    ``block``: how a layer's sublayers sit on the residual stream x.
      "sandwich"  x += post(mixer(pre(x))), then x += post(ff(pre(x))); RMS norms whose stored weight is an offset from one
      "parallel"  h = norm(x); x += mixer(h) + ff(h); layer norms (mean taken off) with a plain weight
      "prenorm"   x += m mixer(pre(x)), then x += m ff(pre(x)), m = ``residual_mult``; RMS norms as in "sandwich"
    Options of pre-norm blocks: ``layer_norm`` (norms take the mean off and have a plain weight and a bias), ``residual_gate`` (every
    sublayer's result is multiplied by sigmoid(W h + b), h = its normed input), ``input_conv`` taps > 0 (the mixer reads h + a
    causal convolution of h per channel). Of the whole model: ``positions`` > 0 learned position vectors, ``tied_head`` (the
    head is the embedding table).
    """
    layers: List[LayerSpec] = field(default_factory=list)
    embed_scale: float = 1.0
    logit_scale: float = 1.0
    architecture: str = ""
    block: str = "sandwich"
    residual_mult: float = 1.0
    layer_norm: bool = False
    residual_gate: bool = False
    input_conv: int = 0
    positions: int = 0
    tied_head: bool = False

    def is_dense_layer(self, layer_id: int) -> bool:
        return True

    def __post_init__(self):
        super().__post_init__()
        assert self.num_layers == len(self.layers) and self.block in ("sandwich", "parallel", "prenorm")
        if self.block != "prenorm" and (self.layer_norm or self.residual_gate or self.input_conv):
            raise ValueError("layer norms with a bias, gated residuals and input convolutions need pre-norm blocks")
        if self.positions:
            self.max_seq_len = min(self.max_seq_len, self.positions)
        for i, layer in enumerate(self.layers):
            m, r = layer.mixer, layer.routed
            if isinstance(m, HeadDecaySpec) and (len(m.decay) != m.heads or not all(0.0 <= d <= 1.0 for d in m.decay)):
                raise ValueError(f"layer {i}: {m.heads} heads need one decay in 0 .. 1 each")
            if isinstance(m, GatedUnitSpec) and m.width % m.blocks:
                raise ValueError(f"layer {i}: {m.width} channels do not make {m.blocks} equal blocks")
            if r is not None and r.act == "clamped" and r.limit <= 0.0:
                raise ValueError(f"layer {i}: clamped experts need a limit")
            if isinstance(m, SideBySideSpec):
                m = m.left
                if m.kv_from is not None or m.v_mix:
                    raise ValueError(f"layer {i}: attention beside another mixer shares no keys or values")
            if getattr(m, "q_temp", None) is not None and m.q_temp.every < 1:
                raise ValueError(f"layer {i}: the query temperature changes every {m.q_temp.every} tokens")
            if layer.act not in ACTIVATIONS or (r is not None and r.act not in EXPERT_ACTIVATIONS):
                raise ValueError(f"layer {i}: unknown activation (known: {', '.join(ACTIVATIONS)})")
            if r is not None and (layer.ff or self.block == "sandwich" or not 1 <= r.top <= r.experts):
                raise ValueError(f"layer {i}: experts need a parallel or pre-norm block, no dense feed-forward beside them and "
                                 f"1 <= top <= experts")
            if r is not None and r.scoring not in ("softmax", "sigmoid"):
                raise ValueError(f"layer {i}: unknown expert scores {r.scoring!r}")
            if r is not None and (r.experts % r.groups or not 1 <= r.keep <= r.groups or r.top > r.experts // r.groups * r.keep):
                raise ValueError(f"layer {i}: {r.top} experts of {r.keep} out of {r.groups} groups of {r.experts}")
            if r is not None and r.scoring != "sigmoid" and (r.correction or r.groups > 1):
                raise ValueError(f"layer {i}: corrections and groups of experts need sigmoid scores")
            if layer.weights_of is not None and replace(layer, weights_of=None) != \
                    replace(self.layers[self.weight_layer(i)], weights_of=None):
                raise ValueError(f"layer {i} cannot use the weights of layer {layer.weights_of}")
            rot = getattr(m, "rot", None)
            if rot is not None and (rot.dims % 2 or rot.dims > (m.rot_dim if isinstance(m, LatentAttentionSpec) else m.dim)):
                raise ValueError(f"layer {i}: {rot.dims} rotated dimensions do not fit the head")
            if isinstance(m, (GatedLinearSpec, LatentAttentionSpec, WkvSpec, HeadDecaySpec, GatedUnitSpec)):
                continue
            if getattr(m, "tied_values", False) and (m.vdim != m.dim or m.v_mix or m.kv_from is not None or m.qk_norm or m.value_norm):
                raise ValueError(f"layer {i}: values tied to the keys have their size and no norm, mixing or sharing")
            if getattr(m, "value_norm", False) and (m.v_mix or m.kv_from is not None):
                raise ValueError(f"layer {i}: normed values are neither mixed nor read from another layer")
            if m.heads % m.kv_heads:
                raise ValueError(f"layer {i}: {m.heads} heads do not share {m.kv_heads} key / value heads evenly")
            src = getattr(m, "kv_from", None)
            if src is not None:
                s = self.layers[src].mixer if 0 <= src < i else None
                if not isinstance(s, AttentionSpec) or s.kv_from is not None or \
                        (s.kv_heads, s.dim, s.vdim) != (m.kv_heads, m.dim, m.vdim):
                    raise ValueError(f"layer {i} cannot read the keys and values of layer {src}")
            first = self.first_v_mix
            if getattr(m, "v_mix", False):
                f = self.layers[first].mixer
                if m.kv_from is not None or (f.kv_heads, f.vdim) != (m.kv_heads, m.vdim):
                    raise ValueError(f"layer {i} cannot mix its values with those of layer {first}")

    def weight_layer(self, i: int) -> int:
        """The layer whose tensors layer i uses."""
        seen = {i}
        while self.layers[i].weights_of is not None:
            i = self.layers[i].weights_of
            if not 0 <= i < len(self.layers) or i in seen:
                raise ValueError(f"weights_of names no layer with weights: {i}")
            seen.add(i)
        return i

    @property
    def first_v_mix(self) -> Optional[int]:
        """The layer whose values the later value-mixing layers mix in."""
        return next((i for i, l in enumerate(self.layers) if getattr(l.mixer, "v_mix", False)), None)

    @classmethod
    def make(cls, width: int, vocab: int, layers: List[LayerSpec], dtype=torch.bfloat16, **kw) -> "LayerListConfig":
        heads = max(l.mixer.heads for l in layers)
        kw = {**dict(rms_norm_eps=1e-6, head_dim=max(l.mixer.dim for l in layers)), **kw}
        return cls(hidden_size=width, num_layers=len(layers), num_heads=heads, num_kv_heads=heads, num_experts=0,
                   intermediate_size=max((l.routed.ff if l.routed else l.ff or 0) for l in layers), dtype=dtype, ep_size=1, top_k=0, vocab_size=vocab,
                   layers=list(layers), **kw)


@dataclass
class CacheConfig:
    """Paged KV cache configuration (field names of vLLM's CacheConfig as used at disagmoe/config.py:41-61)."""
    block_size: int = 16
    gpu_memory_utilization: float = 0.8
    swap_space: float = 0
    cache_dtype: str = "auto"
    num_gpu_blocks_override: Optional[int] = None
    sliding_window: Optional[int] = None
    enable_prefix_caching: bool = False
    cpu_offload_gb: float = 0
    num_reserved_blocks: int = 0
    num_gpu_blocks: Optional[int] = None
    num_cpu_blocks: Optional[int] = None


@dataclass
class SamplingConfig:
    min_output_len: int
    max_output_len: int


mixtral_config = ModelConfig(
    hidden_size=4096, num_layers=32, num_heads=32, num_kv_heads=8, num_experts=8, intermediate_size=14336,
    dtype=torch.bfloat16, ep_size=8, top_k=2, vocab_size=32000, rope_theta=1e6, name="mixtral-8x7b",
)

duo_expert_mixtral = ModelConfig(
    hidden_size=4096, num_layers=32, num_heads=32, num_kv_heads=8, num_experts=2, intermediate_size=14336,
    dtype=torch.bfloat16, ep_size=2, vocab_size=32000, rope_theta=1e6, name="mixtral-duo",
)

# Qwen1.5-MoE-A2.7B shape: 60 routed experts (top-4, no renormalisation) + one sigmoid-gated shared expert.
qwen_moe_config = ModelConfig(
    hidden_size=2048, num_layers=24, num_heads=16, num_kv_heads=16, num_experts=60, intermediate_size=1408,
    dtype=torch.bfloat16, ep_size=6, dp_size=2, top_k=4, vocab_size=151936, head_dim=128, rope_theta=1e6,
    rms_norm_eps=1e-6, norm_topk_prob=False, num_shared_experts=1, shared_intermediate_size=5632,
    shared_expert_gate=True, name="qwen1.5-moe-a2.7b",
)

# DeepSeek-V2-Lite shape with standard attention in place of MLA: first layer dense, 64 experts top-6, 2 shared.
deepseek_v2_lite_config = ModelConfig(
    hidden_size=2048, num_layers=27, num_heads=16, num_kv_heads=16, num_experts=64, intermediate_size=1408,
    dtype=torch.bfloat16, ep_size=8, tp_size=1, top_k=6, vocab_size=102400, head_dim=128, rope_theta=1e4,
    rms_norm_eps=1e-6, norm_topk_prob=False, num_shared_experts=2, shared_intermediate_size=2 * 1408,
    first_k_dense=1, dense_intermediate_size=10944, name="deepseek-v2-lite",
)

# Tiny Mixtral-style model of the CPU / fp32 correctness configuration.
tiny_config = ModelConfig(
    hidden_size=256, num_layers=2, num_heads=4, num_kv_heads=4, num_experts=8, intermediate_size=512,
    dtype=torch.float32, ep_size=1, top_k=2, vocab_size=1024, head_dim=64, rope_theta=1e4, name="tiny-moe",
)

# Rurunex design at the size of a small production model (random weights): two recurrences for every attention layer.
def _rurunex_layers(groups: int, heads: int, dim: int, ff: int) -> List[LayerSpec]:
    gla = GatedLinearSpec(heads, dim, dim, tau=16.0, rank=16)
    delta = ChannelDeltaSpec(heads, heads, dim, dim, conv=4, rank=dim, gate_rank=dim)
    out: List[LayerSpec] = []
    for g in range(groups):
        attn = AttentionSpec(heads, max(1, heads // 4), dim, dim, scale=dim ** -0.5, window=1024, softcap=30.0,
                             rot=RotarySpec(dim, 1e6, factor=4.0, original=8192),
                             kv_from=len(out) - 1 if g % 2 else None)
        out += [LayerSpec(gla, ff), LayerSpec(delta, ff), LayerSpec(attn, ff)]
    return out


rurunex_config = LayerListConfig.make(2048, 32000, _rurunex_layers(6, 16, 128, 5632), max_seq_len=8192, embed_scale=45.25,
                                      logit_scale=0.25, architecture="Rurunex", name="rurunex-18l")

# Supinex design at the size of a small production model (random weights): grouped-query attention over the whole context
# and windowed latent attention in turn; experts in every layer but the first.
def _supinex_layers(groups: int, heads: int, dim: int, rank: int, ff: int, experts: RoutedSpec, window: int) -> List[LayerSpec]:
    rot, half = RotarySpec(dim, 5e5, interleaved=True), dim // 2
    attn = AttentionSpec(heads, max(1, heads // 4), dim, dim, scale=dim ** -0.5, rot=rot, qk_norm=False, sink=True, v_mix=True)
    latent = LatentAttentionSpec(heads, dim, half, dim, rank, scale=(dim + half) ** -0.5, window=window, sink=True,
                                 rot=RotarySpec(half, 1e6, factor=4.0, original=8192, interleaved=True))
    out: List[LayerSpec] = []
    for g in range(groups):
        out += [LayerSpec(attn, routed=experts) if g else LayerSpec(attn, ff, "gelu_tanh"), LayerSpec(latent, routed=experts)]
    return out


supinex_config = LayerListConfig.make(
    2048, 32000, _supinex_layers(8, 16, 128, 512, 5632, RoutedSpec(64, 6, 1408), 1024), max_seq_len=8192, block="parallel",
    architecture="Supinex", name="supinex-16l")

# Vufinex design at the size of a small production model (random weights): RWKV-style time mixing, gated latent attention and
# chunked attention in turn, every second attention layer on the weights of the one before it; grouped sigmoid routers.
def _vufinex_layers(groups: int, heads: int, dim: int, rank: int, experts: RoutedSpec, chunk: int) -> List[LayerSpec]:
    half = dim // 2
    wkv = WkvSpec(2 * heads, half, half)
    latent = LatentAttentionSpec(heads, dim, half, dim, rank, scale=(dim + half) ** -0.5, gate=True,
                                 rot=RotarySpec(half, 1e6, interleaved=True))
    attn = AttentionSpec(heads, max(1, heads // 4), dim, dim, scale=dim ** -0.5, rot=RotarySpec(half, 5e5), qk_norm=False,
                         chunk=chunk, tied_values=True)
    out: List[LayerSpec] = []
    for g in range(groups):
        out += [LayerSpec(m, routed=experts, weights_of=4 * (g - 1) + i if g % 2 and i == 3 else None)
                for i, m in enumerate((wkv, latent, wkv, attn))]
    return out


vufinex_config = LayerListConfig.make(
    2048, 32000, _vufinex_layers(4, 16, 128, 512, RoutedSpec(64, 6, 1408, renormalize=True, scoring="sigmoid", correction=True,
                                                             groups=8, keep=3, scale=2.5), 1024),
    max_seq_len=8192, block="prenorm", embed_scale=45.25, residual_mult=0.5, architecture="Vufinex", name="vufinex-16l")

# Panarax design at the size of a small production model (random weights): attention beside a matrix memory, a gated diagonal
# recurrence and lightning attention in turn; the first of the three has a dense feed-forward, the others experts.
def _panarax_layers(groups: int, heads: int, dim: int, ff: int, experts: RoutedSpec) -> List[LayerSpec]:
    both = SideBySideSpec(AttentionSpec(heads, max(1, heads // 4), dim, dim, scale=dim ** -0.5, qk_norm=False, value_norm=True, gate=True,
                                        q_temp=QueryTemperature(0.1, 1024)), MatrixMemorySpec(heads // 2, dim, dim, 15.0))
    unit = GatedUnitSpec(heads * dim, heads, 4)
    decays = HeadDecaySpec(heads, dim, dim, tuple(2.718281828459045 ** -(2.0 ** (-8.0 * (i + 1) / heads)) for i in range(heads)))
    return [LayerSpec(both, ff), LayerSpec(unit, routed=experts), LayerSpec(decays, routed=experts)] * groups


panarax_config = LayerListConfig.make(
    2048, 32000, _panarax_layers(5, 16, 128, 5632, RoutedSpec(32, 2, 1408, act="clamped", scoring="sigmoid", limit=7.0, weigh_input=True)),
    max_seq_len=8192, block="prenorm", layer_norm=True, residual_gate=True, input_conv=4, positions=8192, tied_head=True,
    architecture="Panarax", name="panarax-15l")

PRESETS = {
    "panarax": panarax_config,
    "vufinex": vufinex_config,
    "supinex": supinex_config,
    "rurunex": rurunex_config,
    "mixtral": mixtral_config, "mixtral-8x7b": mixtral_config, "duo": duo_expert_mixtral,
    "qwen-moe": qwen_moe_config, "deepseek-v2-lite": deepseek_v2_lite_config, "tiny": tiny_config,
}


def get_preset(name: str, **changes) -> ModelConfig:
    return PRESETS[name].clone(**changes)
