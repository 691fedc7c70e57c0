"""Model configurations.

One dataclass covers the decoder families of the reference examples: dense
Llama-style (tests/kernels/llama_decoder_dynamo.py, qwen3_embedding), Qwen3 MoE
(examples/models/qwen3/config.py:12-46) and gpt-oss
(examples/models/gpt_oss/config.py:14-68: alternating sliding-window layers,
attention sinks, biases, clamped SwiGLU, YaRN RoPE).

Decoders whose layers differ from one another (`models/hybrid.py`) list them in
`ModelConfig.layers`, one `LayerSpec` with its mixer's sizes per layer; the
uniform fields above (heads, head_dim, intermediate_size) are then unused.
"""

from __future__ import annotations

import math
from dataclasses import dataclass, field, replace
from typing import List, Optional, Tuple, Union


@dataclass(frozen=True)
class RopeSpec:
    """Rotary embedding of the first `dims` dimensions of a head.  With a factor the frequencies are scaled: by YaRN, or with
    `high` set by bands of wavelengths (Llama 3.1: kept below original / high, divided by the factor above original / low)."""
    base: float = 10000.0
    dims: int = 0
    factor: Optional[float] = None
    original: float = 0.0
    fast: float = 32.0
    slow: float = 1.0
    low: float = 0.0
    high: float = 0.0


@dataclass(frozen=True)
class MapsAttentionSpec:
    """Differential attention: two score maps of size `dim` per head over values of size `vdim`."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    diff: float                      # constant part of the second map's weight
    rope: RopeSpec = RopeSpec()
    softcap: float = 0.0             # <= 0: scores are not capped
    kind = "attention"


@dataclass(frozen=True)
class RecurrenceSpec:
    """HGRN2 linear recurrence: `dim` gated channels by `vdim` values per head."""
    heads: int
    dim: int
    vdim: int
    kind = "hgrn2"


@dataclass(frozen=True)
class LinearAttentionSpec:
    """Gated linear attention: `dim` key channels by `vdim` values per head, decays sigmoid(z)^(1 / tau) from a low-rank z
    (rank 0: as the weights have it)."""
    heads: int
    dim: int
    vdim: int
    tau: float = 16.0
    rank: int = 0
    kind = "gla"


@dataclass(frozen=True)
class TimeMixSpec:
    """RWKV-style time mixing: every projection reads its own mix of the token and the one before it, `dim` by `dim` states
    with data-dependent decays and a bonus for the current token."""
    heads: int
    dim: int
    rank: int = 0
    kind = "rwkv"


@dataclass(frozen=True)
class WindowAttentionSpec:
    """Grouped-query attention without rotation over the last `window` tokens (0: all), queries and keys normed over all
    heads together, sigmoid gate on the heads."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int
    kind = "window"


@dataclass(frozen=True)
class ParallelSpec:
    """Attention and time mixing side by side on the same input, summed with constant weights."""
    left: WindowAttentionSpec
    right: TimeMixSpec
    left_scale: float = 1.0
    right_scale: float = 1.0
    kind = "parallel"


@dataclass(frozen=True)
class ChunkAttentionSpec:
    """Grouped-query attention inside chunks of `chunk` positions: projection biases, half-split rotation, per-head norm of
    queries and keys, one gate per head.  kv_from: the keys and values are those of that layer."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int
    rope: RopeSpec = RopeSpec()
    kv_from: Optional[int] = None
    kind = "chunk"


@dataclass(frozen=True)
class LatentAttentionSpec:
    """Latent attention over the last `window` tokens with a sink and a gate per head: queries through a latent of q_rank, keys
    and values from a cached latent of kv_rank and a shared rotated part of `rot` dimensions."""
    heads: int
    dim: int
    rot: int
    vdim: int
    kv_rank: int
    q_rank: int
    scale: float
    window: int
    rope: RopeSpec = RopeSpec()
    kind = "latent"


@dataclass(frozen=True)
class GroupedAttentionSpec:
    """Grouped-query attention.  rope (None: no rotation): interleaved rotation of the first rope.dims dimensions; softcap > 0:
    scores are capped; window > 0: the last `window` tokens and the first `keep_first` ones (0: all); distance: a score loses
    r1 ln(1 + r2 distance), two numbers per head; sink, gate: one per head; bias: biases of all four projections.  kv_from: the
    keys and values are those of that layer."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float = 0.0
    rope: Optional[RopeSpec] = None
    window: int = 0
    keep_first: int = 0
    distance: bool = False
    sink: bool = False
    gate: bool = False
    bias: bool = False
    kv_from: Optional[int] = None
    kind = "grouped"


@dataclass(frozen=True)
class DeltaSpec:
    """Gated delta rule: `dim` by `vdim` states with one decay per head, short convolutions of `conv` taps on queries, keys and
    values; query / key heads are shared by heads / kv_heads heads."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    kind = "delta"


@dataclass(frozen=True)
class StateSpaceSpec:
    """Mamba-2: `state` by `vdim` states with a scalar decay per head, input and read-out vectors in `groups`, a short convolution of
    `conv` taps, gated results normed in `norm_groups` equal parts."""
    heads: int
    groups: int
    state: int
    vdim: int
    conv: int
    norm_groups: int = 1
    kind = "ssd"


@dataclass(frozen=True)
class BlendSpec:
    """Attention and a state-space mixer side by side on the same input; the mean of their results, each RMS-normed over the model's
    width."""
    left: GroupedAttentionSpec
    right: StateSpaceSpec
    kind = "blend"


@dataclass(frozen=True)
class ClampedSpec:
    """Gated feed-forward g sigmoid(1.702 g) (u + 1) with g at most `limit` and u within +-limit."""
    ff: int
    limit: float


@dataclass(frozen=True)
class ExpertsSpec:
    """Routed gated feed-forwards of width `ff`.  score "softmax": softmax over all experts, the `top` best of the `keep` best
    of `groups` equal groups (0: all), weights normalised and multiplied by `scale`; "sigmoid": the `top` largest sigmoids,
    not normalised.  limit 0: SiLU gate, otherwise the form of `ClampedSpec`.  scale_input: the weight multiplies an expert's
    input instead of its output.  shared: a feed-forward of every token, with a sigmoid gate of its own."""
    experts: int
    top: int
    ff: int
    groups: int = 0
    keep: int = 0
    scale: float = 1.0
    score: str = "softmax"
    limit: float = 0.0
    scale_input: bool = False
    shared: Optional[ClampedSpec] = None


@dataclass(frozen=True)
class LayerSpec:
    """block "gated": mixer and gated feed-forward beside each other, a sigmoid gate on both results; "pre-norm": the
    mixer, then the feed-forward (plain `act`, or `experts`), each added to the residual; "sandwich": the same with a norm after
    each of the two as well; "parallel": mixer and feed-forward (gated `act`, or `experts`) on one norm, their sum added to
    the residual, then the per-layer token input."""
    mixer: Union[MapsAttentionSpec, RecurrenceSpec, LinearAttentionSpec, ParallelSpec, ChunkAttentionSpec,
                 LatentAttentionSpec, GroupedAttentionSpec, DeltaSpec, BlendSpec]
    ff: int = 0                      # 0: no dense feed-forward
    act: str = "gelu_tanh"
    block: str = "gated"
    experts: Optional[ExpertsSpec] = None


@dataclass(frozen=True)
class LoopSpec:
    """Layers [start, stop) run `times` times in a row with the same weights."""
    start: int
    stop: int
    times: int


@dataclass
class ModelConfig:
    name: str = "llama"
    vocab_size: int = 128256
    hidden_size: int = 4096
    num_layers: int = 32
    num_heads: int = 32
    num_kv_heads: int = 8
    head_dim: int = 128
    intermediate_size: int = 14336
    rms_eps: float = 1e-5
    rope_theta: float = 500000.0
    max_position: int = 8192
    qk_norm: bool = False                 # per-head RMSNorm on q and k (Qwen3)
    attn_bias: bool = False               # qkv / o biases (gpt-oss)
    causal: bool = True
    # MoE (num_experts == 0 -> dense SwiGLU FFN)
    num_experts: int = 0
    top_k: int = 0
    moe_intermediate_size: int = 0
    router_mode: str = "softmax_topk"     # or "topk_softmax" (gpt-oss)
    router_bias: bool = False
    expert_bias: bool = False
    # gpt-oss attention features
    sliding_window: int = 0
    layer_types: Optional[List[str]] = None   # "full_attention" | "sliding_attention" per layer
    attention_sinks: bool = False
    swiglu_limit: float = 0.0             # > 0 selects the clamped (up + 1) * gate * sigmoid(alpha * gate) form
    swiglu_alpha: float = 1.702
    # YaRN
    rope_scaling_factor: float = 1.0
    rope_original_max_position: int = 0
    rope_beta_fast: float = 32.0
    rope_beta_slow: float = 1.0
    block_size: int = 32
    # layer-by-layer description (models/hybrid.py)
    layers: Optional[List[LayerSpec]] = None
    loop: Optional[LoopSpec] = None
    embedding_scale: float = 1.0
    norm_groups: int = 1
    norm_offset: float = 0.0              # added to the stored weights of the layer and final norms
    tie_embeddings: bool = False          # logits from the embedding table
    layer_norm: bool = False              # layer norms with bias instead of RMS norms
    tanh_norm: bool = False               # tanh(alpha x) * w + b instead of RMS norms
    depth_average: bool = False           # after a layer: weighted sum of the embedding output and all layers' results
    token_side: int = 0                   # width of the per-layer token input (0: none)
    logit_softcap: float = 0.0            # > 0: logits <- cap * tanh(logits / cap)

    @property
    def q_size(self) -> int:
        return self.num_heads * self.head_dim

    @property
    def kv_size(self) -> int:
        return self.num_kv_heads * self.head_dim

    @property
    def is_moe(self) -> bool:
        return self.num_experts > 0

    def window_for_layer(self, layer: int) -> int:
        if self.sliding_window <= 0:
            return 0
        if self.layer_types is None:
            return self.sliding_window
        return self.sliding_window if self.layer_types[layer] == "sliding_attention" else 0

    def scaled(self, **overrides) -> "ModelConfig":
        return replace(self, **overrides)

    def shard_shapes(self, n: int) -> "ModelConfig":
        """The configuration whose full model has the per-rank shapes of this one under n-way tensor
        (and expert) parallelism: 1/n of the heads, of the FFN width, of the experts and of the
        vocabulary.  Used to time the kernels of one rank of an n-GPU job on a single GPU."""
        if n <= 1:
            return self
        return replace(
            self, name=f"{self.name}-shard{n}", num_heads=max(1, self.num_heads // n),
            num_kv_heads=max(1, self.num_kv_heads // n), intermediate_size=self.intermediate_size // n,
            num_experts=self.num_experts // n if self.is_moe else 0,
            top_k=max(1, self.top_k // n) if self.is_moe else 0,      # same (token, expert) pairs per rank
            vocab_size=self.vocab_size // n)

    def layer_runs(self) -> List[Tuple[int, int]]:
        """(layer, pass) in execution order for a layer-by-layer configuration; pass is -1 outside the loop."""
        n = len(self.layers)
        lp = self.loop or LoopSpec(n, n, 1)
        return ([(i, -1) for i in range(lp.start)]
                + [(i, t) for t in range(lp.times) for i in range(lp.start, lp.stop)]
                + [(i, -1) for i in range(lp.stop, n)])

    def param_count(self) -> int:
        h = self.hidden_size
        if self.layers is not None:
            from .weights import hybrid_weight_shapes

            return sum(math.prod(shape) for shape in hybrid_weight_shapes(self).values())
        attn = h * (self.q_size + 2 * self.kv_size) + self.q_size * h
        if self.is_moe:
            ffn = self.num_experts * 3 * h * self.moe_intermediate_size + h * self.num_experts
        else:
            ffn = 3 * h * self.intermediate_size
        return self.num_layers * (attn + ffn + 2 * h) + 2 * self.vocab_size * h + h


def llama3_8b(**kw) -> ModelConfig:
    """Llama-3-8B-shaped dense decoder."""
    return ModelConfig(name="llama3-8b", **kw)


def qwen3_30b_a3b(**kw) -> ModelConfig:
    """Qwen3-30B-A3B-shaped MoE decoder (128 experts, top-8, expert FFN 768)."""
    base = dict(name="qwen3-30b-a3b", vocab_size=151936, hidden_size=2048, num_layers=48, num_heads=32,
                num_kv_heads=4, head_dim=128, intermediate_size=0, rms_eps=1e-6, rope_theta=1e6,
                max_position=40960, qk_norm=True, num_experts=128, top_k=8, moe_intermediate_size=768)
    base.update(kw)
    return ModelConfig(**base)


def gpt_oss_20b(**kw) -> ModelConfig:
    """gpt-oss-20b-shaped MoE decoder (32 experts, top-4, sliding window 128 on alternating layers)."""
    n = kw.get("num_layers", 24)
    base = dict(name="gpt-oss-20b", vocab_size=201088, hidden_size=2880, num_layers=n, num_heads=64,
                num_kv_heads=8, head_dim=64, intermediate_size=0, rms_eps=1e-5, rope_theta=150000.0,
                max_position=131072, attn_bias=True, num_experts=32, top_k=4, moe_intermediate_size=2880,
                router_mode="topk_softmax", router_bias=True, expert_bias=True, sliding_window=128,
                layer_types=["sliding_attention" if i % 2 == 0 else "full_attention" for i in range(n)],
                attention_sinks=True, swiglu_limit=7.0, swiglu_alpha=1.702, rope_scaling_factor=32.0,
                rope_original_max_position=4096)
    base.update(kw)
    return ModelConfig(**base)


def qwen3_embedding(size: str = "0.6b", **kw) -> ModelConfig:
    """Qwen3-Embedding-shaped dense encoder-style decoder (examples/models/qwen3_embedding/config.py:15-112)."""
    presets = {
        "0.6b": dict(hidden_size=1024, num_layers=28, num_heads=16, num_kv_heads=8, intermediate_size=3072),
        "8b": dict(hidden_size=4096, num_layers=36, num_heads=32, num_kv_heads=8, intermediate_size=12288),
    }
    base = dict(name=f"qwen3-embedding-{size}", vocab_size=151669, head_dim=128, rms_eps=1e-6, rope_theta=1e6,
                max_position=32768, qk_norm=True)
    base.update(presets[size])
    base.update(kw)
    return ModelConfig(**base)


def tiny(**kw) -> ModelConfig:
    """Small dense config for unit tests and the smoke run."""
    base = dict(name="tiny", vocab_size=512, hidden_size=256, num_layers=2, num_heads=4, num_kv_heads=2,
                head_dim=64, intermediate_size=512, max_position=512)
    base.update(kw)
    return ModelConfig(**base)


def rope_frequencies(rope: RopeSpec):
    """(frequencies [dims / 2], cos / sin multiplier) of a `RopeSpec`.  With a factor and `high`, frequencies of wavelengths
    above original / low are divided by the factor, those below original / high are kept and those in between are blended
    linearly in original / wavelength.  With a factor alone, the frequencies are blended between base^(-2i/dims) and the same divided by the factor over the pairs whose wavelengths lie between
    original / fast and original / slow tokens (bounds rounded outwards to whole pairs)."""
    import torch

    i = torch.arange(rope.dims // 2, dtype=torch.float64)
    freq = rope.base ** (-2.0 * i / max(rope.dims, 1))
    if rope.factor is None:
        return freq, 1.0
    if rope.high:
        turns = rope.original * freq / (2 * math.pi)
        s = ((turns - rope.low) / (rope.high - rope.low)).clamp(0, 1)
        return (1 - s) * freq / rope.factor + s * freq, 1.0

    def pair_of(turns):          # pair index whose angle makes `turns` full turns over the original length
        return rope.dims * math.log(rope.original / (2 * math.pi * turns)) / (2 * math.log(rope.base))

    lo = max(math.floor(pair_of(rope.fast)), 0)
    hi = min(math.ceil(pair_of(rope.slow)), rope.dims - 1)
    ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0, 1)
    return freq / rope.factor * ramp + freq * (1 - ramp), 0.1 * math.log(rope.factor) + 1.0


def tolenex_config(raw: dict, **kw) -> ModelConfig:
    """`ModelConfig` of a Tolenex config.json."""
    layers = []
    for l in raw["layers"]:
        m, mlp = l["mixer"], l.get("mlp")
        if l["type"] == "hgrn2":
            mixer = RecurrenceSpec(m["heads"], m["dim"], m["vdim"])
        elif l["type"] == "attention":
            r = m["rot"]
            sc = r.get("scaling") or {}
            mixer = MapsAttentionSpec(
                m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"], m["diff"],
                RopeSpec(r["base"], r["dims"], sc.get("factor"), sc.get("original", 0), sc.get("fast", 32.0),
                         sc.get("slow", 1.0)), m.get("softcap") or 0.0)
        else:
            raise ValueError(f"unknown layer type {l['type']!r}")
        if mlp is not None and mlp["kind"] != "dense":
            raise ValueError(f"unknown feed-forward kind {mlp['kind']!r}")
        layers.append(LayerSpec(mixer, mlp["ff"] if mlp is not None else 0))
    lp = raw.get("loop")
    base = dict(name="tolenex", vocab_size=raw["vocab"], hidden_size=raw["width"], num_layers=len(layers),
                rms_eps=raw["norm"]["eps"], norm_groups=raw["norm"]["groups"], layers=layers,
                loop=LoopSpec(lp["start"], lp["stop"], lp["times"]) if lp else None,
                embedding_scale=raw["embedding"]["scale"], max_position=0)
    base.update(kw)
    return ModelConfig(**base)


def tolenex_shape(width: int, *, layers: int, heads: int, kv_heads: int, ff: int, vocab: int = 32000,
                  dim: int = 64, vdim: int = 128, recurrent_every: int = 2, loop: Optional[LoopSpec] = None,
                  groups: int = 4, **kw) -> ModelConfig:
    """A Tolenex configuration of regular shape: every `recurrent_every`-th layer is an attention layer, the
    others are recurrences whose heads are vdim by vdim."""
    rope = RopeSpec(500000.0, dim, 4.0, 8192, 32.0, 1.0)
    specs = []
    for i in range(layers):
        if i % recurrent_every == recurrent_every - 1:
            mixer = MapsAttentionSpec(heads, kv_heads, dim, vdim, dim ** -0.5, 0.5, rope, 30.0)
        else:
            mixer = RecurrenceSpec(heads, vdim, vdim)
        specs.append(LayerSpec(mixer, ff))
    base = dict(name="tolenex", vocab_size=vocab, hidden_size=width, num_layers=layers, rms_eps=1e-5,
                norm_groups=groups, layers=specs, loop=loop, embedding_scale=1.0, max_position=0)
    base.update(kw)
    return ModelConfig(**base)


def mumilorn_config(raw: dict, **kw) -> ModelConfig:
    """`ModelConfig` of a Mumilorn config.json."""

    def mixer_of(kind, m):
        if kind == "gla":
            return LinearAttentionSpec(m["heads"], m["dim"], m["vdim"], m["tau"])
        if kind == "parallel":
            a, r = m["left"], m["right"]
            return ParallelSpec(
                WindowAttentionSpec(a["heads"], a["kv_heads"], a["dim"], a["vdim"], a["scale"], a["mask"]["size"]),
                TimeMixSpec(r["heads"], r["dim"]), m["left_scale"], m["right_scale"])
        raise ValueError(f"unknown layer type {kind!r}")

    layers = []
    for l in raw["layers"]:
        mlp, ff, experts = l.get("mlp"), 0, None
        if mlp is not None:
            if mlp["kind"] == "dense":
                ff = mlp["ff"]
            elif mlp["kind"] == "moe":
                r = mlp["router"]
                g = r.get("groups") or {}
                experts = ExpertsSpec(r["experts"], r["top"], mlp["expert"]["ff"], g.get("count", 0), g.get("keep", 0),
                                      r["scale"])
            else:
                raise ValueError(f"unknown feed-forward kind {mlp['kind']!r}")
        layers.append(LayerSpec(mixer_of(l["type"], l["mixer"]), ff, "relu2", "pre-norm", experts))
    base = dict(name="mumilorn", vocab_size=raw["vocab"], hidden_size=raw["width"], num_layers=len(layers),
                rms_eps=raw["norm"]["eps"], layers=layers, norm_offset=1.0, tie_embeddings=True, max_position=0)
    base.update(kw)
    return ModelConfig(**base)


def mumilorn_shape(width: int, *, layers: int, heads: int, kv_heads: int, ff: int, vocab: int = 32000, dim: int = 128,
                   window: int = 1024, rank: int = 64, parallel_every: int = 2, experts: int = 0, top: int = 0,
                   expert_ff: int = 0, groups: int = 0, keep: int = 0, moe_every: int = 2, **kw) -> ModelConfig:
    """A Mumilorn configuration of regular shape: every `parallel_every`-th layer has the parallel mixer, the others gated
    linear attention; with experts, every `moe_every`-th feed-forward is routed."""
    specs = []
    for i in range(layers):
        if i % parallel_every == parallel_every - 1:
            mixer = ParallelSpec(WindowAttentionSpec(heads, kv_heads, dim, dim, dim ** -0.5, window),
                                 TimeMixSpec(heads, dim, rank), 0.7, 0.7)
        else:
            mixer = LinearAttentionSpec(heads, dim, dim, 16.0, rank)
        if experts and i % moe_every == moe_every - 1:
            specs.append(LayerSpec(mixer, 0, "relu2", "pre-norm", ExpertsSpec(experts, top, expert_ff, groups, keep, 1.0)))
        else:
            specs.append(LayerSpec(mixer, ff, "relu2", "pre-norm"))
    base = dict(name="mumilorn", vocab_size=vocab, hidden_size=width, num_layers=layers, rms_eps=1e-6, layers=specs,
                norm_offset=1.0, tie_embeddings=True, max_position=0)
    base.update(kw)
    return ModelConfig(**base)


def ligizen_config(raw: dict, **kw) -> ModelConfig:
    """`ModelConfig` of a Ligizen config.json."""

    def mixer_of(kind, m):
        r = m["rot"]
        sc = r.get("scaling") or {}
        rope = RopeSpec(r["base"], r["dims"], sc.get("factor"), sc.get("original", 0), low=sc.get("low", 0.0),
                        high=sc.get("high", 0.0))
        if kind == "attention":
            return ChunkAttentionSpec(m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"], m["mask"]["size"], rope,
                                      m.get("kv_from"))
        if kind == "latent_attention":
            if r["dims"] != m["rot_dim"]:
                raise ValueError("the whole rotated part of a latent attention is rotated")
            return LatentAttentionSpec(m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"], m["scale"],
                                       m["mask"]["size"], rope)
        raise ValueError(f"unknown layer type {kind!r}")

    layers = []
    for i, l in enumerate(raw["layers"]):
        mlp, ff, experts = l.get("mlp"), 0, None
        if mlp is not None:
            if mlp["kind"] == "dense":
                ff = mlp["ff"]
            elif mlp["kind"] == "moe":
                r, sh = mlp["router"], mlp.get("shared")
                experts = ExpertsSpec(r["experts"], r["top"], mlp["expert"]["ff"], score="sigmoid",
                                      limit=mlp["expert"]["limit"], scale_input=True,
                                      shared=ClampedSpec(sh["ff"], sh["limit"]) if sh else None)
            else:
                raise ValueError(f"unknown feed-forward kind {mlp['kind']!r}")
        mixer = mixer_of(l["type"], l["mixer"])
        src = getattr(mixer, "kv_from", None)
        if src is not None and not (0 <= src < i and layers[src].mixer.kind == "chunk" and layers[src].mixer.kv_from is None):
            raise ValueError(f"layer {i} cannot read the keys of layer {src}")
        layers.append(LayerSpec(mixer, ff, "silu", "parallel", experts))
    base = dict(name="ligizen", vocab_size=raw["vocab"], hidden_size=raw["width"], num_layers=len(layers),
                rms_eps=raw["norm"]["eps"], layers=layers, embedding_scale=raw["embedding"]["scale"], layer_norm=True,
                token_side=(raw.get("token_side") or {}).get("dim", 0), logit_softcap=raw.get("logit_softcap") or 0.0,
                max_position=0)
    base.update(kw)
    return ModelConfig(**base)


def ligizen_shape(width: int, *, layers: int, heads: int, kv_heads: int, ff: int, vocab: int = 32000, dim: int = 128,
                  window: int = 1024, chunk: int = 1024, latent_dim: int = 128, rot: int = 64, kv_rank: int = 512,
                  q_rank: int = 1536, side: int = 256, experts: int = 0, top: int = 0, expert_ff: int = 0, moe_every: int = 2,
                  share_every: int = 0, **kw) -> ModelConfig:
    """A Ligizen configuration of regular shape: latent and chunked attention alternate; with experts, every `moe_every`-th
    feed-forward is routed (with a shared expert); with share_every, every share_every-th chunked layer but the first reads
    the keys and values of the chunked layer before it."""
    rope = RopeSpec(500000.0, dim, 8.0, 8192, low=1.0, high=4.0)
    specs, chunked, source = [], 0, None
    for i in range(layers):
        if i % 2 == 0:
            mixer = LatentAttentionSpec(heads, latent_dim, rot, dim, kv_rank, q_rank, (latent_dim + rot) ** -0.5, window,
                                        RopeSpec(10000.0, rot))
        else:
            chunked += 1
            shares = share_every and chunked > 1 and chunked % share_every == 0
            mixer = ChunkAttentionSpec(heads, kv_heads, dim, dim, dim ** -0.5, chunk, rope, source if shares else None)
            source = source if shares else i
        if experts and i % moe_every == moe_every - 1:
            specs.append(LayerSpec(mixer, 0, "silu", "parallel", ExpertsSpec(
                experts, top, expert_ff, score="sigmoid", limit=7.0, scale_input=True, shared=ClampedSpec(expert_ff, 7.0))))
        else:
            specs.append(LayerSpec(mixer, ff, "silu", "parallel"))
    base = dict(name="ligizen", vocab_size=vocab, hidden_size=width, num_layers=layers, rms_eps=1e-5, layers=specs,
                layer_norm=True, token_side=side, logit_softcap=50.0, max_position=0)
    base.update(kw)
    return ModelConfig(**base)


def redodra_config(raw: dict, **kw) -> ModelConfig:
    """`ModelConfig` of a Redodra config.json."""

    def attention(m, **fields):
        r, mask = m.get("rot"), m.get("mask") or {}
        return GroupedAttentionSpec(m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"], m.get("softcap") or 0.0,
                                    RopeSpec(r["base"], r["dims"]) if r else None, mask.get("size", 0),
                                    mask.get("keep_first", 0), kv_from=m.get("kv_from"), **fields)

    def mixer_of(kind, m):
        if kind == "attention":
            return attention(m, sink=True, gate=True)
        if kind == "delta":
            return DeltaSpec(m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"])
        if kind == "parallel":
            r = m["right"]
            return BlendSpec(attention(m["left"], distance=True, bias=True),
                             StateSpaceSpec(r["heads"], r["groups"], r["state"], r["vdim"], r["conv"], r["norm_groups"]))
        raise ValueError(f"unknown layer type {kind!r}")

    layers = []
    for i, l in enumerate(raw["layers"]):
        mlp = l.get("mlp")
        if mlp is not None and mlp["kind"] != "dense":
            raise ValueError(f"unknown feed-forward kind {mlp['kind']!r}")
        mixer = mixer_of(l["type"], l["mixer"])
        src = getattr(mixer, "kv_from", None)
        if src is not None and not (0 <= src < i and layers[src].mixer.kind == "grouped" and layers[src].mixer.kv_from is None):
            raise ValueError(f"layer {i} cannot read the keys of layer {src}")
        layers.append(LayerSpec(mixer, mlp["ff"] if mlp is not None else 0, "xielu", "sandwich"))
    base = dict(name="redodra", vocab_size=raw["vocab"], hidden_size=raw["width"], num_layers=len(layers),
                rms_eps=raw["norm"]["eps"], layers=layers, tanh_norm=True, depth_average=True, max_position=0)
    base.update(kw)
    return ModelConfig(**base)


def redodra_shape(width: int, *, layers: int, heads: int, kv_heads: int, ff: int, vocab: int = 32000, dim: int = 128,
                  window: int = 1024, keep_first: int = 4, state: int = 128, groups: int = 8, conv: int = 4,
                  share_every: int = 0, **kw) -> ModelConfig:
    """A Redodra configuration of regular shape: layers of the delta rule, the parallel mixer and attention take turns (delta rule and
    parallel mixer twice as often as attention); with share_every, every share_every-th attention layer but the first reads the
    keys and values of the attention layer before it."""
    specs, attended, source = [], 0, None
    for i in range(layers):
        if i % 5 in (0, 2):
            mixer = DeltaSpec(heads, heads, dim, dim, conv)
        elif i % 5 in (1, 3):
            mixer = BlendSpec(GroupedAttentionSpec(heads, kv_heads, dim, dim, dim ** -0.5, 30.0, None, window, keep_first,
                                                   distance=True, bias=True),
                              StateSpaceSpec(heads, groups, state, dim, conv, groups))
        else:
            attended += 1
            shares = share_every and attended > 1 and attended % share_every == 0
            mixer = GroupedAttentionSpec(heads, kv_heads, dim, dim, dim ** -0.5, 30.0, RopeSpec(500000.0, dim), sink=True,
                                         gate=True, kv_from=source if shares else None)
            source = source if shares else i
        specs.append(LayerSpec(mixer, ff, "xielu", "sandwich"))
    base = dict(name="redodra", vocab_size=vocab, hidden_size=width, num_layers=layers, rms_eps=1e-5, layers=specs,
                tanh_norm=True, depth_average=True, max_position=0)
    base.update(kw)
    return ModelConfig(**base)


def yarn_inv_freq(cfg: ModelConfig):
    """(inv_freq [head_dim/2], attention scaling) for the configured RoPE; plain RoPE when
    rope_scaling_factor == 1 (YaRN per examples/models/gpt_oss/config.py:64-68)."""
    import torch

    d = cfg.head_dim
    base = cfg.rope_theta
    freq = base ** (torch.arange(0, d, 2, dtype=torch.float64) / d)
    if cfg.rope_scaling_factor <= 1.0:
        return (1.0 / freq), 1.0
    factor = cfg.rope_scaling_factor
    orig = cfg.rope_original_max_position
    concentration = 0.1 * math.log(factor) + 1.0
    d_half = d / 2
    low = d_half * math.log(orig / (cfg.rope_beta_fast * 2 * math.pi)) / math.log(base)
    high = d_half * math.log(orig / (cfg.rope_beta_slow * 2 * math.pi)) / math.log(base)
    interpolation = 1.0 / (factor * freq)
    extrapolation = 1.0 / freq
    ramp = (torch.arange(d_half, dtype=torch.float64) - low) / (high - low)
    mask = 1 - ramp.clamp(0, 1)
    inv_freq = interpolation * (1 - mask) + extrapolation * mask
    return inv_freq, concentration
