"""Decoder-only LLM architecture descriptions used by the model builders, the CUDA plugin and the
benchmarks. The named configurations are the ones of the serving benchmarks (Llama-3-8B,
Llama-3-70B, Mixtral-8x7B); ``tiny`` variants keep tests fast."""
from __future__ import annotations

import math
from dataclasses import dataclass, replace
from typing import List, Optional, Tuple, Union


@dataclass(frozen=True)
class LlmConfig:
    name: str = "llama"
    vocab_size: int = 128256
    hidden_size: int = 4096
    num_layers: int = 32
    num_heads: int = 32
    num_kv_heads: int = 8
    head_dim: int = 128
    ffn_size: int = 14336
    rope_theta: float = 500000.0
    rms_eps: float = 1e-5
    num_experts: int = 0          # 0 = dense FFN
    experts_top_k: int = 2
    weight_format: str = "int4"   # "int4" (u4 asym, group scales + zero points) | "int8" | "bf16" | "fp8"
    group_size: int = 128
    sliding_window: int = 0

    @property
    def q_size(self) -> int:
        return self.num_heads * self.head_dim

    @property
    def kv_size(self) -> int:
        return self.num_kv_heads * self.head_dim

    def with_(self, **kw) -> "LlmConfig":
        return replace(self, **kw)


LLAMA3_8B = LlmConfig(name="llama-3-8b")
LLAMA3_70B = LlmConfig(name="llama-3-70b", hidden_size=8192, num_layers=80, num_heads=64, num_kv_heads=8,
                       ffn_size=28672, weight_format="fp8")
MIXTRAL_8X7B = LlmConfig(name="mixtral-8x7b", vocab_size=32000, hidden_size=4096, num_layers=32, num_heads=32,
                         num_kv_heads=8, ffn_size=14336, rope_theta=1e6, num_experts=8, experts_top_k=2,
                         weight_format="bf16")
TINY_LLAMA = LlmConfig(name="tiny-llama", vocab_size=512, hidden_size=256, num_layers=2, num_heads=4, num_kv_heads=2,
                       head_dim=128, ffn_size=512, group_size=128)
TINY_MOE = LlmConfig(name="tiny-moe", vocab_size=512, hidden_size=256, num_layers=2, num_heads=4, num_kv_heads=2,
                     head_dim=128, ffn_size=256, num_experts=4, experts_top_k=2, weight_format="bf16")

NAMED = {c.name: c for c in (LLAMA3_8B, LLAMA3_70B, MIXTRAL_8X7B, TINY_LLAMA, TINY_MOE)}


# ----------------------------------------------------------------------------------------- layered decoders
# A decoder whose layers are listed one by one: every layer names its token mixer and its feed-forward, each with sizes of its
# own. The residual stream is fp32; how sublayers and norms meet it is the configuration's ``block``. The serving program of these configurations is runtime/layered_llm.py.
@dataclass(frozen=True)
class RotarySpec:
    """Rotation of the first ``dims`` dimensions by the position (dimension i paired with i + dims / 2). ``yarn`` = (factor,
    original length, fast, slow): frequencies that turn less than ``slow`` times over the original length are divided by the
    factor, those that turn more than ``fast`` times are kept, with a linear ramp over the dimensions in between."""
    dims: int
    base: float
    yarn: Optional[Tuple[float, float, float, float]] = None

    def inv_freq(self) -> List[float]:
        freq = [self.base ** (-2.0 * i / self.dims) for i in range(self.dims // 2)]
        if self.yarn is None:
            return freq
        factor, original, fast, slow = self.yarn
        turns_at = lambda t: self.dims * math.log(original / (2.0 * math.pi * t)) / (2.0 * math.log(self.base))
        first = max(math.floor(turns_at(fast)), 0)
        last = min(math.ceil(turns_at(slow)), self.dims - 1)
        width = max(last - first, 0.001)
        keep = [1.0 - min(max((i - first) / width, 0.0), 1.0) for i in range(self.dims // 2)]
        return [f * k + f / factor * (1.0 - k) for f, k in zip(freq, keep)]

    def multiplier(self) -> float:
        """Factor of cos and sin."""
        return 1.0 if self.yarn is None else 0.1 * math.log(self.yarn[0]) + 1.0


@dataclass(frozen=True)
class AttentionSpec:
    """Grouped-query attention; ``window`` 0 = full causal attention, else a position sees itself and window - 1 before it;
    ``chunk`` > 0: a position sees only keys of its own chunk of that many positions, counted from position 0."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int = 0
    qk_norm: bool = False          # RMS norm of every query / key head, one weight of size dim for all heads
    gated: bool = False            # heads times sigmoid(W_g x) before the output projection
    rotary: Optional[RotarySpec] = None
    head_gate: bool = False        # the gate is one number per head instead of one per column
    chunk: int = 0
    sink: bool = False             # exp(sink), a number per head, joins the softmax denominator
    taps: int = 0                  # > 0: short causal convolution on every column of q, k and v, ahead of the rotation
    v_mix: bool = False            # values are mixed with those of the first layer that has this set

    @property
    def carries_state(self) -> bool:
        return self.taps > 1


@dataclass(frozen=True)
class LatentAttentionSpec:
    """Attention whose keys and values are projections of one normed low-rank row per token, plus a rotated key part that all
    heads share; those two are what is cached."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rotary: RotarySpec
    window: int = 0
    carries_state = False


@dataclass(frozen=True)
class ChannelDeltaSpec:
    """Gated delta rule with a decay per head and key channel, short convolutions with silu on q, k and v, unit-norm queries and keys, a
    norm and a low-rank sigmoid gate on every head's read-out. ``decay_rank`` / ``gate_rank``: inner sizes of the two low-rank
    projections, 0 = whatever the checkpoint's tensors have."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int
    decay_rank: int = 0
    gate_rank: int = 0
    carries_state = True


@dataclass(frozen=True)
class RgLruSpec:
    """Griffin's recurrent block: short causal convolution, block-diagonal gates, real-gated linear recurrent unit."""
    width: int
    blocks: int
    taps: int
    decay: float = 8.0             # log a = -decay * r * softplus(lambda)
    carries_state = True


@dataclass(frozen=True)
class LimitedGluSpec:
    """g = min(gate, limit), u = clamp(up, -limit, limit); g * sigmoid(slope * g) * (u + shift)."""
    ff: int
    limit: float
    slope: float = 1.702
    shift: float = 1.0


@dataclass(frozen=True)
class SquaredReluSpec:
    """W_down relu(W_up x)^2."""
    ff: int


@dataclass(frozen=True)
class LayerSpec:
    mixer: Union[AttentionSpec, LatentAttentionSpec, RgLruSpec, ChannelDeltaSpec]
    mlp: Optional[Union[LimitedGluSpec, SquaredReluSpec]] = None


# How a layer meets the residual stream x.
POST_NORM = "post_norm"            # x <- norm1(scale * x + mixer(x)), then x <- norm2(scale * x + mlp(x))
PARALLEL_NORM = "parallel_norm"    # x <- x + mixer(norm1(x)) + mlp(norm2(x))


@dataclass(frozen=True)
class LayeredConfig:
    """Layers in one of the two forms above; a norm's weight is norm_offset + what is stored."""
    name: str
    vocab_size: int
    hidden_size: int
    layers: Tuple[LayerSpec, ...]
    norm_eps: float = 1e-5
    residual_scale: float = 1.0    # POST_NORM only
    norm_offset: float = 0.0
    block: str = POST_NORM
    embed_norm: bool = False       # the embedding passes a norm of its own
    logit_softcap: float = 0.0     # > 0: logits <- cap * tanh(logits / cap)

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def has_recurrent_state(self) -> bool:
        """True when a request holds state that is not rows of the paged cache."""
        return any(l.mixer.carries_state for l in self.layers)
