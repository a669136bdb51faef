"""Configuration of hybrid decoders: a stack whose layers name their own mixer, its sizes and their feed-forward.

`HybridConfig` also carries the fields that the shared modules read from a ``TransformerConfig`` (linears, MLP, wrapper,
controller), so that those take either.
"""
from __future__ import annotations

import dataclasses
import math
from dataclasses import dataclass
from typing import Optional, Tuple, Union

import torch


@dataclass(frozen=True)
class YarnScaling:
    """Frequencies that turn often over the ``original`` context stay, slow ones are divided by ``factor``; a linear ramp
    over the pair index joins them between ``fast`` and ``slow`` turns."""

    factor: float
    original: float
    fast: float
    slow: float


@dataclass(frozen=True)
class RotaryConfig:
    base: float
    dims: int  # leading dimensions that turn, in interleaved pairs (2i, 2i + 1)
    scaling: Optional[YarnScaling] = None


@dataclass(frozen=True)
class LatentAttentionConfig:
    heads: int
    dim: int       # unrotated query / key dimensions per head
    rot_dim: int   # rotated ones; the key's are shared by all heads
    vdim: int
    kv_rank: int
    scale: float
    rot: RotaryConfig
    window: Optional[int] = None   # keys seen, the token itself included; None: all earlier ones
    kv_from: Optional[int] = None  # 0-based layer whose cached rows this layer reads instead of making its own

    def __post_init__(self):
        if self.rot.dims % 2 or not 0 <= self.rot.dims <= self.rot_dim:
            raise ValueError("rot.dims must be even and at most rot_dim")
        if self.window is not None and self.window < 1:
            raise ValueError("a window holds at least the token itself")

    def cached_row_width(self) -> int:
        return self.row_width if self.kv_from is None else 0

    def request_state(self, hidden_size: int, dtype: torch.dtype) -> Optional[dict]:
        return None

    @property
    def kv_pad(self) -> int:
        """Where the rotated part starts in a cached row."""
        return -(-self.kv_rank // 16) * 16

    @property
    def row_width(self) -> int:
        """Elements of a cached row: latent and rotated part, padded for 16-byte copies and 16 x 32 tensor-core steps."""
        return -(-(self.kv_pad + self.rot_dim) // 32) * 32


@dataclass(frozen=True)
class DeltaRuleConfig:
    heads: int
    dim: int   # key and value channels per head
    rank: int  # inner width of the decay's two-step projection
    decay_scale: float = math.exp(-0.5)  # decay = exp(-decay_scale * sigmoid(.))
    unit_eps: float = 1e-6               # inside the unit key's root

    def cached_row_width(self) -> int:
        return 0

    def request_state(self, hidden_size: int, dtype: torch.dtype) -> Optional[dict]:
        return {"state": ((self.heads, self.dim, self.dim), torch.float32)}


def _conv_state(channels: int, taps: int, dtype: torch.dtype) -> dict:
    """The inputs a short convolution looks back at."""
    return {"conv": ((taps - 1, channels), dtype)} if taps > 1 else {}


def _check_taps(taps: int) -> None:
    if not 1 <= taps <= 8:
        raise ValueError("short convolutions have 1 to 8 taps")


@dataclass(frozen=True)
class ShortConvAttentionConfig:
    """Grouped-query attention whose queries, keys and values pass a short causal convolution, with per-head norms of queries and
    keys, no rotation, and optionally a window and values mixed with those of the first mixing layer."""

    heads: int
    kv_heads: int
    dim: int                      # query / key dimensions per head
    vdim: int                     # value dimensions per head
    scale: float
    conv: int                     # taps of the convolutions
    window: Optional[int] = None  # keys seen, the token itself included; None: all earlier ones
    value_mix: bool = False

    def __post_init__(self):
        if self.heads % self.kv_heads:
            raise ValueError("heads must be a multiple of kv_heads")
        if self.window is not None and self.window < 1:
            raise ValueError("a window holds at least the token itself")
        if max(self.dim, self.vdim) > 256:
            raise ValueError("head dimensions go up to 256")
        _check_taps(self.conv)

    @property
    def conv_channels(self) -> int:
        return (self.heads + self.kv_heads) * self.dim + self.kv_heads * self.vdim

    @property
    def tensor_cores(self) -> bool:
        """Head sizes that the tensor-core kernels take."""
        return (self.dim % 8 == 0 and self.vdim % 8 == 0 and max(self.dim, self.vdim) <= 128 and self.heads // self.kv_heads <= 16)

    def cached_row_width(self) -> int:
        """Elements of a cached row: the keys of all heads, then the values."""
        return self.kv_heads * (self.dim + self.vdim)

    def request_state(self, hidden_size: int, dtype: torch.dtype) -> Optional[dict]:
        return _conv_state(self.conv_channels, self.conv, dtype)


@dataclass(frozen=True)
class WkvConfig:
    heads: int
    dim: int   # key and value channels per head
    rank: int  # inner width of the decay's two-step projection

    def __post_init__(self):
        if self.dim > 256:
            raise ValueError("recurrent heads have up to 256 channels")

    def cached_row_width(self) -> int:
        return 0

    def request_state(self, hidden_size: int, dtype: torch.dtype) -> Optional[dict]:
        return {"state": ((self.heads, self.dim, self.dim), torch.float32), "shift": ((hidden_size,), dtype)}


@dataclass(frozen=True)
class GatedDeltaConfig:
    heads: int
    kv_heads: int
    dim: int   # query / key channels per head
    vdim: int  # value channels per head
    conv: int  # taps of the convolutions
    unit_eps: float = 1e-6  # inside the unit vectors' root

    def __post_init__(self):
        if self.heads % self.kv_heads:
            raise ValueError("heads must be a multiple of kv_heads")
        if self.dim > 256:
            raise ValueError("recurrent heads have up to 256 key channels")
        _check_taps(self.conv)

    @property
    def conv_channels(self) -> int:
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim

    def cached_row_width(self) -> int:
        return 0

    def request_state(self, hidden_size: int, dtype: torch.dtype) -> Optional[dict]:
        return {"state": ((self.heads, self.vdim, self.dim), torch.float32), **_conv_state(self.conv_channels, self.conv, dtype)}


MixerConfig = Union[LatentAttentionConfig, DeltaRuleConfig, ShortConvAttentionConfig, WkvConfig, GatedDeltaConfig]


@dataclass(frozen=True)
class ExpertConfig:
    """One gated feed-forward: g' sigmoid(alpha g') (u' + 1), g' = min(g, limit), u' clamped to [-limit, limit]."""

    ff: int
    limit: float
    alpha: float = 1.702


@dataclass(frozen=True)
class MoeConfig:
    experts: int
    top: int  # experts per token; their weights are their sigmoid scores
    expert: ExpertConfig
    shared: Optional[ExpertConfig] = None  # runs for every token, times a gate of its own

    def __post_init__(self):
        if not 1 <= self.top <= min(self.experts, 64) or self.experts > 1024:
            raise ValueError("1 <= top <= experts, at most 64 of 1024")


@dataclass(frozen=True)
class HybridLayerConfig:
    mixer: MixerConfig
    ffn_hidden_size: Optional[int] = None  # width of a dense feed-forward
    moe: Optional[MoeConfig] = None        # or a mixture of experts; both None: no feed-forward


@dataclass
class HybridConfig:
    vocab_size: int
    hidden_size: int
    layers: Tuple[HybridLayerConfig, ...]
    layernorm_epsilon: float = 1e-5
    params_dtype: torch.dtype = torch.bfloat16  # bfloat16, or float32: the whole model in true 32-bit arithmetic
    activation: str = "relu2"
    gated_linear_unit: bool = False
    add_bias_linear: bool = False
    ffn_hidden_size: Optional[int] = None       # set per layer (`for_layer`)
    fp8: Optional[str] = None
    tensor_model_parallel_size: int = 1
    enable_cuda_graph: bool = False
    inference_sampling_seed: int = 42
    fuse_splitk_reduction_into_norm: bool = True
    defer_logits_gather: bool = True
    # "output_norm": sublayers one after the other with norms on their outputs, embedding norm, tied head (`HybridModel`);
    # "parallel": mixer and feed-forward side by side on two norms of the same stream, scaled embedding, a head of its own
    # (`ParallelHybridModel`)
    block: str = "output_norm"
    embedding_scale: float = 1.0
    logit_scale: float = 1.0

    def __post_init__(self):
        self.layers = tuple(self.layers)
        if self.params_dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("hybrid decoders compute in bfloat16 or float32")
        if self.tensor_model_parallel_size != 1:
            raise NotImplementedError("hybrid decoders run on one GPU")
        if self.block == "parallel":
            mixing = [x.mixer for x in self.layers if isinstance(x.mixer, ShortConvAttentionConfig) and x.mixer.value_mix]
            if len({(m.kv_heads, m.vdim) for m in mixing}) > 1:
                raise ValueError("layers whose values are mixed must agree in their number and size")
        for i, layer in enumerate(self.layers):
            m = layer.mixer
            src = getattr(m, "kv_from", None)
            if src is None:
                continue
            own = self.layers[src].mixer if 0 <= src < i else None
            if not isinstance(own, LatentAttentionConfig) or own.kv_from is not None:
                raise ValueError(f"layer {i} reads the rows of layer {src}, which is no earlier latent-attention layer with its own")
            if (own.kv_rank, own.rot_dim, own.rot) != (m.kv_rank, m.rot_dim, m.rot):
                raise ValueError(f"layers {src} and {i} share cached rows but differ in their shape or rotation")

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    def for_layer(self, index: int) -> "HybridConfig":
        """The view of layer ``index`` that per-layer modules (MLP) read."""
        return dataclasses.replace(self, ffn_hidden_size=self.layers[index].ffn_hidden_size)
