"""Time mixing with a matrix-valued state: every projection reads its own blend of a token and the one before it, the state decays
per key channel by a rate computed from the token, and the current token's write counts with a bonus of its own."""
from __future__ import annotations

import torch

from .. import _lib, ops
from ..tensor_parallel.layers import RowParallelLinear, _device
from .hybrid_config import HybridConfig, WkvConfig
from .short_conv import step_rows

WKV, DELTA = 0, 1  # B200_RECURRENCE_*


def recurrence_args(ctx, kind: int, config: HybridConfig, mixer, state, num_tokens: int) -> _lib.RecurrenceArgs:
    a = _lib.RecurrenceArgs()
    step_rows(a, ctx, num_tokens)
    a.kind, a.heads, a.kv_heads, a.dim = kind, mixer.heads, getattr(mixer, "kv_heads", mixer.heads), mixer.dim
    a.vdim = getattr(mixer, "vdim", mixer.dim)
    a.state, a.state_slots, a.eps = state.data_ptr(), state.shape[0], config.layernorm_epsilon
    a.dtype = ops.dtype_code(config.params_dtype)
    return a


class Wkv(torch.nn.Module):
    def __init__(self, config: HybridConfig, mixer: WkvConfig, layer_index: int):
        super().__init__()
        self.config, self.mixer, self.layer_number = config, mixer, layer_index + 1
        H, n = config.hidden_size, mixer.heads * mixer.dim
        self.width = n

        def param(*shape):
            return torch.nn.Parameter(torch.zeros(shape, dtype=config.params_dtype, device=_device()), requires_grad=False)

        self.blend = param(5, H)         # r, k, v, gate, decay
        self.weight_in = param(4 * n, H)  # r, k, v, gate: one product each, on its own blend
        self.decay_down, self.decay_up, self.decay_bias = param(mixer.rank, H), param(n, mixer.rank), param(n)
        self.bonus, self.norm_weight = param(n), param(n)
        self.linear_proj = RowParallelLinear(n, H, config=config, bias=False)

    def checkpoint_tensors(self) -> dict:
        n, H, rank = self.width, self.config.hidden_size, self.mixer.rank
        out = {f"mu.{k}": (H,) for k in "rkvgw"}
        out.update({k: (n, H) for k in "rkvg"})
        out.update({"w1": (rank, H), "w2": (n, rank), "w0": (n,), "u": (self.mixer.heads, self.mixer.dim), "norm": (n,), "o": (H, n)})
        return out

    def load(self, get) -> None:
        self.blend.data.copy_(torch.stack([get(f"mu.{k}") for k in "rkvgw"]))
        self.weight_in.data.copy_(torch.cat([get(k) for k in "rkvg"]))
        for dst, name in ((self.decay_down, "w1"), (self.decay_up, "w2"), (self.decay_bias, "w0"), (self.norm_weight, "norm"),
                          (self.linear_proj.weight, "o")):
            dst.data.copy_(get(name))
        self.bonus.data.copy_(get("u").reshape(-1))

    def forward(self, x, ctx, rope=None, step=None):
        """``x`` [T, H] -> the output linear's partial sums."""
        m, (T, H), n, dev = self.mixer, x.shape, self.width, x.device
        # every projection's input
        blends = torch.empty((T, 4 * H), dtype=x.dtype, device=dev)
        decay_in = torch.empty((T, H), dtype=x.dtype, device=dev)
        shift = ctx.recurrent_state(self.layer_number, "shift")
        s = _lib.ShiftArgs()
        step_rows(s, ctx, T)
        s.x, s.mu, s.state, s.state_slots = x.data_ptr(), self.blend.data_ptr(), shift.data_ptr(), shift.shape[0]
        s.out, s.out_last, s.width, s.mixes, s.dtype = blends.data_ptr(), decay_in.data_ptr(), H, 5, ops.dtype_code(x.dtype)
        ops.struct_kernel("token_shift", s, x)
        proj = torch.empty((T, 4 * n), dtype=x.dtype, device=dev)
        ops.linear(blends, self.weight_in, out=proj, batch=4, x_batch=H, y_batch=n, K=H)
        state = ctx.recurrent_state(self.layer_number, "state")
        lora = torch.empty((T, m.rank), dtype=x.dtype, device=dev)
        out = torch.empty((T, n), dtype=x.dtype, device=dev)
        a = recurrence_args(ctx, WKV, self.config, m, state, T)
        a.proj, a.proj_ld, a.off_r, a.off_k, a.off_v, a.off_g = proj.data_ptr(), proj.stride(0), 0, n, 2 * n, 3 * n
        a.lora, a.rank, a.w2, a.decay_bias, a.bonus = (lora.data_ptr(), m.rank, self.decay_up.data_ptr(), self.decay_bias.data_ptr(),
                                                       self.bonus.data_ptr())
        a.norm_weight, a.norm_per_head, a.out = self.norm_weight.data_ptr(), 1, out.data_ptr()
        a.z, a.z_splits = ops.partials_of(ops.linear_partials(decay_in, self.decay_down))
        ops.struct_kernel("recurrence_lora", a, state)
        if ctx.is_decode_only():
            ops.struct_kernel("recurrence_decode", a, state)
        else:
            o = torch.empty((T, n), dtype=torch.float32, device=dev)
            a.o_f32 = o.data_ptr()
            a.z, a.z_splits = ops.partials_of(ops.linear_partials(lora, self.decay_up))
            if ctx.padded_active_token_count != ctx.active_token_count:
                o.zero_()  # padding tokens belong to no row
            ops.struct_kernel("recurrence_scan", a, state)
            ops.struct_kernel("recurrence_finish", a, state)
        return self.linear_proj(out, defer_reduction=True)[0]
