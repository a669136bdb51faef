"""Matrix memory: a linear recurrence per head whose scalar input and forget gates live in the log domain, scaled by a running maximum, with a
normaliser beside the matrix.  A mixer part, see `JoinedMixer`."""
from __future__ import annotations

import torch

from .. import ops
from ..tensor_parallel.layers import _device
from .hybrid_config import HybridConfig, MatrixMemoryConfig
from .wkv import recurrence_args

MEMORY = 2  # B200_RECURRENCE_MEMORY


class MatrixMemory(torch.nn.Module):
    def __init__(self, config: HybridConfig, mixer: MatrixMemoryConfig, layer_index: int):
        super().__init__()
        self.config, self.mixer, self.layer_number = config, mixer, layer_index + 1
        m = mixer
        self.inputs = {"q": m.heads * m.dim, "k": m.heads * m.dim, "v": m.heads * m.vdim, "g": m.heads * m.vdim}
        self.out_width = m.heads * m.vdim

        def param(*shape):
            return torch.nn.Parameter(torch.zeros(shape, dtype=config.params_dtype, device=_device()), requires_grad=False)

        # input gates, then forget gates: a product of their own, whose fp32 partial sums the recurrence reads
        self.weight_gates = param(-(-2 * m.heads // 8) * 8, config.hidden_size)
        self.gate_bias, self.norm_weight = param(2 * m.heads), param(self.out_width)

    def checkpoint_tensors(self) -> dict:
        """Checkpoint name (below this part of the mixer) -> shape, without the input linear's weights."""
        h, H = self.mixer.heads, self.config.hidden_size
        return {"i": (h, H), "i.b": (h,), "f": (h, H), "f.b": (h,), "norm": (self.out_width,)}

    def load(self, get) -> None:
        n = 2 * self.mixer.heads
        self.weight_gates.data[:n].copy_(torch.cat([get("i"), get("f")]))
        self.gate_bias.data.copy_(torch.cat([get("i.b"), get("f.b")]))
        self.norm_weight.data.copy_(get("norm"))

    def forward(self, x, proj, column: int, out, out_column: int, scale: float, ctx, rope=None, step=None) -> None:
        """Decode steps run one fused kernel; other steps find every token's factors, scan and finish."""
        m, T, dev = self.mixer, proj.shape[0], proj.device
        state = ctx.recurrent_state(self.layer_number, "state")
        a = recurrence_args(ctx, MEMORY, self.config, m, state, T)
        a.top, a.gate_cap = ctx.recurrent_state(self.layer_number, "top").data_ptr(), m.gate_cap
        n = m.heads * m.dim
        a.proj, a.proj_ld, a.off_r, a.off_k, a.off_v, a.off_g = (proj.data_ptr(), proj.stride(0), column, column + n, column + 2 * n,
                                                                 column + 2 * n + self.out_width)
        a.decay_bias, a.norm_weight, a.norm_per_head = self.gate_bias.data_ptr(), self.norm_weight.data_ptr(), 1
        a.out, a.out_ld, a.out_scale = out.data_ptr() + out_column * out.element_size(), out.stride(0), scale
        a.z, a.z_splits = ops.partials_of(ops.linear_partials(x, self.weight_gates))
        a.z_ld = self.weight_gates.shape[0]
        if ctx.is_decode_only():
            ops.struct_kernel("recurrence_decode", a, state)
            return
        gates = torch.empty((T, m.heads, 4), dtype=torch.float32, device=dev)
        below = torch.empty((T, m.heads), dtype=torch.float32, device=dev)
        o = torch.empty((T, self.out_width), dtype=torch.float32, device=dev)
        a.gates, a.below, a.o_f32 = gates.data_ptr(), below.data_ptr(), o.data_ptr()
        if ctx.using_cuda_graph_this_step() or ctx.padded_active_token_count != ctx.active_token_count:
            o.zero_()  # padding tokens belong to no row
            below.fill_(1.0)
        ops.struct_kernel("recurrence_gates", a, state)
        ops.struct_kernel("recurrence_scan", a, state)
        ops.struct_kernel("recurrence_finish", a, state)
