"""Generalized delta rule: a recurrent mixer with one fp32 [key channel] x [value channel] state per head and request."""
from __future__ import annotations

import torch

from .. import _lib, ops
from ..tensor_parallel.layers import ColumnParallelLinear, RowParallelLinear, _device
from .hybrid_config import DeltaRuleConfig, HybridConfig


class GeneralDeltaRule(torch.nn.Module):
    def __init__(self, config: HybridConfig, mixer: DeltaRuleConfig, layer_index: int):
        super().__init__()
        self.config, self.mixer, self.layer_number = config, mixer, layer_index + 1
        dt, dev = config.params_dtype, _device()
        self.width = mixer.heads * mixer.dim
        # one linear for everything that reads the layer's input: [r | k | v | gate | removal rate | decay, first step]
        self.in_width = 5 * self.width + mixer.rank
        self.linear_in = ColumnParallelLinear(config.hidden_size, -(-self.in_width // 8) * 8, config=config, bias=False)
        self.decay_up = torch.nn.Parameter(torch.empty(self.width, mixer.rank, dtype=dt, device=dev), requires_grad=False)

        def vector():
            return torch.nn.Parameter(torch.zeros(self.width, dtype=dt, device=dev), requires_grad=False)

        self.decay_bias, self.removal_bias, self.norm_weight = vector(), vector(), vector()
        self.linear_proj = RowParallelLinear(self.width, config.hidden_size, config=config, bias=False)

    def checkpoint_tensors(self) -> dict:
        n, H, rank = self.width, self.config.hidden_size, self.mixer.rank
        out = {k: (n, H) for k in ("r", "k", "v", "g", "a")}
        out.update({"w1": (rank, H), "w2": (n, rank), "w0": (n,), "a.b": (n,), "norm": (n,), "o": (H, n)})
        return out

    def load(self, get) -> None:
        w = self.linear_in.weight.data
        w.zero_()
        w[: self.in_width].copy_(torch.cat([get(k).to(w.device) for k in ("r", "k", "v", "g", "a", "w1")]))
        for dst, name in ((self.decay_up, "w2"), (self.decay_bias, "w0"), (self.removal_bias, "a.b"), (self.norm_weight, "norm"),
                          (self.linear_proj.weight, "o")):
            dst.data.copy_(get(name))

    def forward(self, x, ctx, rope=None):
        """``x`` [T, H] -> the output linear's partial sums.  Decode steps run one fused kernel; other steps prepare the
        decay with a GEMM and scan every request's tokens."""
        m, T, n, dev = self.mixer, x.shape[0], self.width, x.device
        proj, _ = self.linear_in(x)
        state = ctx.recurrent_state(self.layer_number, "state")
        out = torch.empty((T, n), dtype=x.dtype, device=dev)
        a = _lib.DeltaArgs()
        a.proj, a.proj_ld, a.out = proj.data_ptr(), proj.stride(0), out.data_ptr()
        a.w2, a.decay_bias, a.removal_bias = self.decay_up.data_ptr(), self.decay_bias.data_ptr(), self.removal_bias.data_ptr()
        a.norm_weight = self.norm_weight.data_ptr()
        a.state, a.state_slots = state.data_ptr(), state.shape[0]
        a.state_in, a.state_out = ctx.state_read_slots.data_ptr(), ctx.state_write_slots.data_ptr()
        a.off_r, a.off_k, a.off_v, a.off_g, a.off_a, a.off_w1 = (i * n for i in range(6))
        a.rank, a.heads, a.dim, a.num_tokens, a.num_rows = m.rank, m.heads, m.dim, T, T
        a.dtype, a.decay_scale, a.unit_eps, a.eps = ops.dtype_code(x.dtype), m.decay_scale, m.unit_eps, self.config.layernorm_epsilon
        if ctx.is_decode_only():
            ops.delta_decode(a, state)
        else:
            lora = torch.empty((T, m.rank), dtype=x.dtype, device=dev)
            o = torch.empty((T, n), dtype=torch.float32, device=dev)
            a.lora, a.o_f32 = lora.data_ptr(), o.data_ptr()
            ops.delta_lora(a, state)
            z = ops.linear(lora, self.decay_up)
            a.z, a.num_rows = z.data_ptr(), ctx.padded_active_request_count
            a.cu_tokens = ctx.cu_query_seq_lengths_cudagraph_only.data_ptr()
            ops.delta_scan(a, state)
            ops.delta_finish(a, state)
        return self.linear_proj(out, defer_reduction=True)[0]
