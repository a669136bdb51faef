"""Gated scan (minGRU): an element-wise recurrence whose gates read the current token only, so that a prompt's tokens need not be walked one by
one.  A mixer part, see `JoinedMixer`."""
from __future__ import annotations

import torch

from .. import _lib, ops
from ..tensor_parallel.layers import _device
from .hybrid_config import GatedScanConfig, HybridConfig
from .short_conv import step_rows


class GatedScan(torch.nn.Module):
    takes_partials = True  # decode steps: the projection's unreduced partial sums

    def __init__(self, config: HybridConfig, mixer: GatedScanConfig, layer_index: int):
        super().__init__()
        self.config, self.mixer, self.layer_number = config, mixer, layer_index + 1
        self.inputs = {k: mixer.width for k in ("z", "x", "g")}
        self.out_width = mixer.width

        def param():
            return torch.nn.Parameter(torch.zeros(mixer.width, dtype=config.params_dtype, device=_device()), requires_grad=False)

        self.update_bias, self.input_bias = param(), param()

    def checkpoint_tensors(self) -> dict:
        """Checkpoint name (below this part of the mixer) -> shape, without the input linear's weights."""
        return {"z.b": (self.mixer.width,), "x.b": (self.mixer.width,)}

    def load(self, get) -> None:
        self.update_bias.data.copy_(get("z.b"))
        self.input_bias.data.copy_(get("x.b"))

    def forward(self, x, proj, column: int, out, out_column: int, scale: float, ctx, rope=None, step=None) -> None:
        """``proj`` [T, ...], or in decode steps its partial sums; ``out`` [T, ...]: the gated state from ``out_column`` on."""
        if scale != 1.0:
            raise NotImplementedError("a gated scan beside another mixer")
        state, n = ctx.recurrent_state(self.layer_number, "state"), self.mixer.width
        a = _lib.GatedScanArgs()
        step_rows(a, ctx, x.shape[0])
        if isinstance(proj, ops.GemmPartials):
            a.partials, a.num_splits = ops.partials_of(proj)
            a.proj_ld = proj.shape[-1]
        else:
            a.proj, a.proj_ld = proj.data_ptr(), proj.stride(0)
        a.off_z, a.off_u, a.off_g, a.width = column, column + n, column + 2 * n, n
        a.z_bias, a.u_bias = self.update_bias.data_ptr(), self.input_bias.data_ptr()
        a.state, a.state_slots = state.data_ptr(), state.shape[0]
        a.out, a.out_ld, a.dtype = out.data_ptr() + out_column * out.element_size(), out.stride(0), ops.dtype_code(out.dtype)
        ops.struct_kernel("gated_scan", a, state)
