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
    halves: bool = False  # pairs are (i, i + dims / 2) instead


@dataclass(frozen=True)
class LatentAttentionConfig:
    heads: int
    dim: int       # unrotated query / key dimensions per head
    rot_dim: int   # rotated ones; the key's are shared by all heads
    vdim: int
    kv_rank: int
    scale: float
    rot: Optional[RotaryConfig] = None
    window: Optional[int] = None   # keys seen, the token itself included; None: all earlier ones
    kv_from: Optional[int] = None  # 0-based layer whose cached rows this layer reads instead of making its own
    q_rank: Optional[int] = None   # queries come from a normed latent of their own; None: straight from the layer's input
    sink: bool = False             # one more term per head in the softmax denominator
    gate: str = "head"             # sigmoid gates on the output: one per "head", or one per "value" channel of every head

    def __post_init__(self):
        if self.rot is not None and (self.rot.dims % 2 or not 0 <= self.rot.dims <= self.rot_dim):
            raise ValueError("rot.dims must be even and at most rot_dim")
        if self.q_rank is not None and self.rot_dim:
            raise ValueError("queries that come from a latent have no rotated part")
        if self.gate not in ("head", "value"):
            raise ValueError("gates belong to heads or to value channels")
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


@dataclass(frozen=True)
class DistanceBias:
    """A learned bias per head and distance class: one class per distance up to half the rows, logarithmic ones up to ``longest``."""

    rows: int
    longest: float

    def row(self, distance: int) -> int:
        half = self.rows // 2
        if distance < half:
            return distance
        if self.longest <= half:
            return self.rows - 1
        return min(self.rows - 1, half + math.floor(math.log(distance / half) / math.log(self.longest / half) * (self.rows - half)))

    def rows_by_distance(self) -> list:
        """The row of every distance, up to the first one from which on it stays the last."""
        out = [self.row(0)]
        while out[-1] < self.rows - 1:
            out.append(self.row(len(out)))
        return out


@dataclass(frozen=True)
class GroupedAttentionConfig:
    """Grouped-query attention with its parts as parameters.  ``diff`` makes it differential: two maps per head over the same values, out =
    rms-normed (a1 - lambda a2) (1 - diff)."""

    heads: int
    kv_heads: int
    dim: int                             # query / key dimensions per head (and map)
    vdim: int                            # value dimensions per head
    scale: float
    window: Optional[int] = None         # keys seen, the token itself included; None: all earlier ones
    keep_first: int = 0                  # keys at the sequence's start that a window never hides
    rot: Optional[RotaryConfig] = None
    unit_queries_keys: bool = False      # queries and keys divided by their root mean square after the rotation
    values_from_keys: bool = False       # the values are the projected keys
    biases: bool = False                 # on queries, keys and the output
    softcap: Optional[float] = None
    sink: bool = False                   # one more term per head in the softmax denominator
    distance_bias: Optional[DistanceBias] = None
    diff: Optional[float] = None
    gate: bool = False                   # value channels times sigmoid of a projection (differential attention)
    head_gate: bool = False              # heads times sigmoid of a projection, one number each (one map)
    value_mix: bool = False              # values mixed with those of the first layer that mixes them
    kv_from: Optional[int] = None        # 0-based layer whose cached rows this layer reads instead of making its own

    def __post_init__(self):
        if self.heads % self.kv_heads:
            raise ValueError("heads must be a multiple of kv_heads")
        if self.window is not None and self.window < 1:
            raise ValueError("a window holds at least the token itself")
        if max(self.dim, self.vdim) > 256:
            raise ValueError("head dimensions go up to 256")
        if self.rot is not None and (self.rot.dims % 2 or not 0 <= self.rot.dims <= self.dim):
            raise ValueError("rot.dims must be even and at most dim")
        if self.diff is None and self.gate or self.diff is not None and (self.sink or self.distance_bias is not None):
            raise ValueError("differential attention comes with a gate and without sinks or a distance bias")
        if self.diff is not None and self.head_gate:
            raise ValueError("differential attention gates value channels, not heads")
        if self.values_from_keys and (self.dim != self.vdim or self.diff is not None):
            raise ValueError("values that are keys have their size, and one map")
        if self.value_mix and (self.values_from_keys or self.kv_from is not None):
            raise ValueError("values are mixed where a layer projects its own")

    @property
    def maps(self) -> int:
        return 1 if self.diff is None else 2

    @property
    def tensor_cores(self) -> bool:
        """Head sizes that the tensor-core kernels take."""
        return self.dim % 8 == 0 and self.vdim % 8 == 0 and max(self.dim, self.vdim) <= 128 and self.heads // self.kv_heads <= 16

    @property
    def row_width(self) -> int:
        return self.kv_heads * (self.maps * self.dim + self.vdim)

    def cached_row_width(self) -> int:
        """Elements of a cached row: the keys of all heads, then the values."""
        return self.row_width if self.kv_from is None else 0

    def request_state(self, hidden_size: int, dtype: torch.dtype) -> Optional[dict]:
        return None


@dataclass(frozen=True)
class MatrixMemoryConfig:
    """Linear recurrence with scalar input and forget gates in the log domain, scaled by a running maximum, and a normaliser."""

    heads: int
    dim: int   # query / key channels per head
    vdim: int  # value channels per head
    gate_cap: float

    def __post_init__(self):
        if self.dim > 256 or self.vdim > 1023:
            raise ValueError("recurrent heads have up to 256 key and 1023 value channels")

    def cached_row_width(self) -> int:
        return 0

    def request_state(self, hidden_size: int, dtype: torch.dtype) -> Optional[dict]:
        """The matrix, its normaliser as one more value channel, and the maximum."""
        return {"state": ((self.heads, self.vdim + 1, self.dim), torch.float32), "top": ((self.heads,), torch.float32)}


@dataclass(frozen=True)
class GatedScanConfig:
    """Gated recurrence, element by element, whose gates read the current token only (minGRU)."""

    width: int

    def cached_row_width(self) -> int:
        return 0

    def request_state(self, hidden_size: int, dtype: torch.dtype) -> Optional[dict]:
        return {"state": ((self.width,), torch.float32)}


@dataclass(frozen=True)
class SideBySideConfig:
    """Mixers that read the same input and whose outputs are added up with constant factors."""

    parts: Tuple[Tuple[str, Union[GroupedAttentionConfig, MatrixMemoryConfig], float], ...]  # (checkpoint prefix, mixer, factor)

    def __post_init__(self):
        if sum(m.cached_row_width() > 0 for _, m, _ in self.parts) > 1 or sum(m.request_state(1, torch.float32) is not None for _, m, _ in self.parts) > 1:
            raise ValueError("one of the mixers caches rows, one keeps state")
        if any(getattr(m, "biases", False) or getattr(m, "kv_from", None) is not None for _, m, _ in self.parts):
            raise ValueError("mixers side by side have no biases and read no other layer's rows")

    def cached_row_width(self) -> int:
        return max(m.cached_row_width() for _, m, _ in self.parts)

    def request_state(self, hidden_size: int, dtype: torch.dtype) -> Optional[dict]:
        out = {}
        for _, m, _ in self.parts:
            out.update(m.request_state(hidden_size, dtype) or {})
        return out or None


MixerConfig = Union[LatentAttentionConfig, DeltaRuleConfig, ShortConvAttentionConfig, WkvConfig, GatedDeltaConfig, GroupedAttentionConfig,
                    MatrixMemoryConfig, GatedScanConfig, SideBySideConfig]


@dataclass(frozen=True)
class ExpertConfig:
    """One gated feed-forward: g' sigmoid(alpha g') (u' + 1), g' = min(g, limit), u' clamped to [-limit, limit]; without a limit silu(g) u.
    ``gated`` False: max(u, 0)^2 of one projection."""

    ff: int
    limit: Optional[float] = None
    alpha: float = 1.702
    gated: bool = True

    def __post_init__(self):
        if not self.gated and self.limit is not None:
            raise ValueError("limits belong to gated feed-forwards")


@dataclass(frozen=True)
class SoftmaxRouting:
    """Scores are a softmax; a learned correction takes part in the choice only; only the experts of the best groups can be chosen; the
    chosen scores, divided by their sum and times ``scale``, weigh the experts' outputs.  The last ``identity`` router outputs are
    experts whose output is their input."""

    identity: int = 0
    groups: int = 1
    keep_groups: int = 1
    scale: float = 1.0


@dataclass(frozen=True)
class ChosenSoftmaxRouting:
    """Scores are logits plus a bias; the softmax over the chosen ones alone weighs the experts' outputs."""


@dataclass(frozen=True)
class MoeConfig:
    experts: int
    top: int  # experts per token; without ``routing`` their sigmoid scores weigh their inputs
    expert: ExpertConfig
    shared: Optional[ExpertConfig] = None  # runs for every token, times a gate of its own where the scores are sigmoids
    routing: Union[SoftmaxRouting, ChosenSoftmaxRouting, None] = None

    def __post_init__(self):
        r = self.routing
        columns, reachable = self.experts, self.experts
        if (r is None) != (self.expert.limit is not None) or (isinstance(r, SoftmaxRouting) and self.shared is not None):
            raise ValueError("softmax routing goes with experts without limits, and without a shared one where groups are kept")
        if self.shared is not None and (self.shared.gated != self.expert.gated or (self.shared.limit is None) != (self.expert.limit is None)):
            raise ValueError("the shared expert has the form of the others")
        if isinstance(r, SoftmaxRouting):
            columns = self.experts + r.identity
            if r.identity < 0 or not 1 <= r.keep_groups <= r.groups or columns % r.groups:
                raise ValueError("experts and identity experts form equal groups, at least one of which is kept")
            reachable = columns // r.groups * r.keep_groups
        if not 1 <= self.top <= min(reachable, 64) or not 1 <= columns <= 1024 or self.experts < 1:
            raise ValueError("1 <= top <= experts that can be chosen, at most 64 of 1024")


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
    # (`ParallelHybridModel`); with ``input_taps`` both read ONE norm, each through a short causal filter of its own
    # "streams": sublayers one after the other with layer norms on their inputs, ``streams`` residual streams that every sublayer blends
    # and mixes (0: one plain residual stream), scaled embedding, tied head (`StreamHybridModel`)
    block: str = "output_norm"
    streams: int = 0
    embedding_scale: float = 1.0
    logit_scale: float = 1.0
    norm_offset: float = 1.0  # added to the norms' stored weights ("parallel")
    input_taps: int = 0       # taps of the filters in front of the sublayers, 0: none ("parallel")

    def __post_init__(self):
        self.layers = tuple(self.layers)
        if self.params_dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("hybrid decoders compute in bfloat16 or float32")
        if self.tensor_model_parallel_size != 1:
            raise NotImplementedError("hybrid decoders run on one GPU")
        if self.block == "parallel":
            mixing = [x.mixer for x in self.layers if getattr(x.mixer, "value_mix", False)]
            if len({(m.kv_heads, m.vdim) for m in mixing}) > 1:
                raise ValueError("layers whose values are mixed must agree in their number and size")
        if self.input_taps:
            _check_taps(self.input_taps)
            if self.block != "parallel":
                raise ValueError("input filters belong to parallel blocks")
        if self.block == "streams" and any(x.moe is not None and x.moe.shared is not None for x in self.layers):
            raise ValueError("shared experts belong to parallel blocks")
        if self.streams > 16:
            raise ValueError("at most 16 residual streams")
        for i, layer in enumerate(self.layers):
            m = layer.mixer
            src = getattr(m, "kv_from", None)
            if src is None:
                continue
            own = self.layers[src].mixer if 0 <= src < i else None
            if isinstance(m, GroupedAttentionConfig):
                if not isinstance(own, GroupedAttentionConfig) or own.kv_from is not None:
                    raise ValueError(f"layer {i} reads the rows of layer {src}, which is no earlier attention layer with its own")
                if (own.kv_heads, own.maps, own.dim, own.vdim, own.rot) != (m.kv_heads, m.maps, m.dim, m.vdim, m.rot):
                    raise ValueError(f"layers {src} and {i} share cached rows but differ in their shape or rotation")
                continue
            if not isinstance(own, LatentAttentionConfig) or own.kv_from is not None:
                raise ValueError(f"layer {i} reads the rows of layer {src}, which is no earlier latent-attention layer with its own")
            if (own.kv_rank, own.rot_dim, own.rot) != (m.kv_rank, m.rot_dim, m.rot):
                raise ValueError(f"layers {src} and {i} share cached rows but differ in their shape or rotation")

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    def mixes_values_first(self, index: int) -> bool:
        """Whether layer ``index`` is the first whose values the others' are mixed with."""
        mixing = [i for i, x in enumerate(self.layers) if getattr(x.mixer, "value_mix", False)]
        return mixing[:1] == [index]

    def request_state(self, index: int) -> Optional[dict]:
        """What layer ``index`` keeps per request: its mixer's state and the inputs its filters look back at."""
        state = self.layers[index].mixer.request_state(self.hidden_size, self.params_dtype)
        if self.input_taps == 0:
            return state
        out = dict(state or {})  # (empty: nothing to keep, but the kernels ask for the slots)
        if self.input_taps > 1:
            out["input"] = ((self.input_taps - 1, self.hidden_size), self.params_dtype)
        return out

    def for_layer(self, index: int) -> "HybridConfig":
        """The view of layer ``index`` that per-layer modules (MLP) read."""
        return dataclasses.replace(self, ffn_hidden_size=self.layers[index].ffn_hidden_size)
