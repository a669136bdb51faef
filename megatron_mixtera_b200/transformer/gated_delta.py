"""Gated delta rule: a recurrent mixer whose state forgets by one factor per head and token and corrects what it recalls for a key,
behind short convolutions of queries, keys and values."""
from __future__ import annotations

import torch

from .. import _lib, ops  # noqa: F401
from ..tensor_parallel.layers import ColumnParallelLinear, RowParallelLinear, _device
from .hybrid_config import GatedDeltaConfig, HybridConfig
from .short_conv import filter_of, short_conv_args
from .wkv import DELTA, recurrence_args


class GatedDelta(torch.nn.Module):
    def __init__(self, config: HybridConfig, mixer: GatedDeltaConfig, layer_index: int):
        super().__init__()
        self.config, self.mixer, self.layer_number = config, mixer, layer_index + 1
        m = mixer
        self.width = m.heads * m.vdim
        # one linear for everything that reads the layer's input: [q | k | v | gate | step size | decay]
        self.in_width = m.conv_channels + self.width + 2 * m.heads
        self.linear_in = ColumnParallelLinear(config.hidden_size, -(-self.in_width // 8) * 8, config=config, bias=False)

        def param(*shape):
            return torch.nn.Parameter(torch.zeros(shape, dtype=config.params_dtype, device=_device()), requires_grad=False)

        self.conv_filter = param(m.conv, m.conv_channels)
        self.decay_rate, self.decay_bias, self.norm_weight = param(m.heads), param(m.heads), param(m.vdim)
        self.linear_proj = RowParallelLinear(self.width, config.hidden_size, config=config, bias=False)

    def checkpoint_tensors(self) -> dict:
        m, H = self.mixer, self.config.hidden_size
        widths = {"q": m.kv_heads * m.dim, "k": m.kv_heads * m.dim, "v": self.width}
        out = {k: (n, H) for k, n in widths.items()}
        out.update({f"{k}.conv": (n, m.conv) for k, n in widths.items()})
        out.update({"g": (self.width, H), "b": (m.heads, H), "a": (m.heads, H), "A_log": (m.heads,), "dt_bias": (m.heads,),
                    "norm": (m.vdim,), "o": (H, self.width)})
        return out

    def load(self, get) -> None:
        w = self.linear_in.weight.data
        w.zero_()
        w[: self.in_width].copy_(torch.cat([get(k).to(w.device) for k in "qkvgba"]))
        self.conv_filter.data.copy_(filter_of(torch.cat([get(f"{k}.conv") for k in "qkv"])))
        for dst, name in ((self.decay_rate, "A_log"), (self.decay_bias, "dt_bias"), (self.norm_weight, "norm"),
                          (self.linear_proj.weight, "o")):
            dst.data.copy_(get(name))

    def forward(self, x, ctx, rope=None, step=None):
        """``x`` [T, H] -> the output linear's partial sums.  Decode steps run one fused kernel; other steps convolve all tokens
        and scan every request's."""
        m, T, dev = self.mixer, x.shape[0], x.device
        proj, _ = self.linear_in(x)
        state, conv_state = ctx.recurrent_state(self.layer_number, "state"), ctx.recurrent_state(self.layer_number, "conv")
        out = torch.empty((T, self.width), dtype=x.dtype, device=dev)
        a = recurrence_args(ctx, DELTA, self.config, m, state, T)
        g = m.conv_channels
        a.proj, a.proj_ld, a.off_r, a.off_g, a.off_b, a.off_a = proj.data_ptr(), proj.stride(0), 0, g, g + self.width, g + self.width + m.heads
        a.off_k, a.off_v = m.kv_heads * m.dim, 2 * m.kv_heads * m.dim
        a.decay_rate, a.decay_bias, a.unit_eps = self.decay_rate.data_ptr(), self.decay_bias.data_ptr(), m.unit_eps
        a.norm_weight, a.norm_per_head, a.out = self.norm_weight.data_ptr(), 0, out.data_ptr()
        a.conv_filter, a.taps = self.conv_filter.data_ptr(), m.conv
        a.conv_state = None if conv_state is None else conv_state.data_ptr()
        if ctx.is_decode_only():
            ops.struct_kernel("recurrence_decode", a, state)
        else:
            conv = torch.empty((T, m.conv_channels), dtype=x.dtype, device=dev)
            o = torch.empty((T, self.width), dtype=torch.float32, device=dev)
            c = short_conv_args(ctx, proj=proj, filter_=self.conv_filter, state=conv_state, channels=m.conv_channels, taps=m.conv, out=conv)
            ops.struct_kernel("conv_silu", c, state)
            a.conv, a.o_f32 = conv.data_ptr(), o.data_ptr()
            if ctx.padded_active_token_count != ctx.active_token_count:
                o.zero_()  # padding tokens belong to no row
            ops.struct_kernel("recurrence_scan", a, state)
            ops.struct_kernel("recurrence_finish", a, state)
        return self.linear_proj(out, defer_reduction=True)[0]
