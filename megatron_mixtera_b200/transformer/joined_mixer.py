"""Mixer parts around one input and one output linear: a single part, or several side by side on the same input whose outputs are added up (the
output linear's sum over all of its input features does that; a part's constant factor is applied where the part writes its output)."""
from __future__ import annotations

import torch

from ..tensor_parallel.layers import ColumnParallelLinear, RowParallelLinear, _device
from .gated_scan import GatedScan
from .grouped_attention import GroupedAttention
from .hybrid_config import GatedScanConfig, GroupedAttentionConfig, HybridConfig, MatrixMemoryConfig, SideBySideConfig
from .matrix_memory import MatrixMemory

PARTS = {GatedScanConfig: GatedScan, GroupedAttentionConfig: GroupedAttention, MatrixMemoryConfig: MatrixMemory}


def _pad(n: int) -> int:
    return -(-n // 8) * 8  # 16-byte rows and starts in bf16


class JoinedMixer(torch.nn.Module):
    def __init__(self, config: HybridConfig, mixer, layer_index: int):
        super().__init__()
        self.config = config
        specs = mixer.parts if isinstance(mixer, SideBySideConfig) else (("", mixer, 1.0),)
        self.parts = torch.nn.ModuleList(PARTS[type(m)](config, m, layer_index) for _, m, _ in specs)
        self.prefixes = [name + "." if name else "" for name, _, _ in specs]
        self.scales = [float(s) for _, _, s in specs]
        self.columns, self.out_columns, n_in, n_out = [], [], 0, 0
        for p in self.parts:
            self.columns.append(n_in)
            self.out_columns.append(n_out)
            n_in += _pad(sum(p.inputs.values()))
            n_out += _pad(p.out_width)
        self.padded_outputs = any(p.out_width % 8 for p in self.parts)
        self.linear_in = ColumnParallelLinear(config.hidden_size, n_in, config=config, bias=False)
        self.linear_proj = RowParallelLinear(n_out, config.hidden_size, config=config, bias=False)
        self.output_bias = None
        if getattr(mixer, "biases", False):
            self.output_bias = torch.nn.Parameter(torch.zeros(config.hidden_size, dtype=config.params_dtype, device=_device()), requires_grad=False)

    def prefill_unit_tokens(self) -> set:
        return {p.prefill_unit_tokens() for p in self.parts if isinstance(p, GroupedAttention)}

    def checkpoint_tensors(self) -> dict:
        """Checkpoint name (below the layer's mixer) -> shape."""
        H, out = self.config.hidden_size, {}
        for pre, p in zip(self.prefixes, self.parts):
            out.update({pre + k: (n, H) for k, n in p.inputs.items()})
            out.update({pre + k: s for k, s in p.checkpoint_tensors().items()})
            out[pre + "o"] = (H, p.out_width)
        if self.output_bias is not None:
            out["o.b"] = (H,)
        return out

    def ignored_tensors(self) -> set:
        return {pre + k for pre, p in zip(self.prefixes, self.parts) for k in getattr(p, "ignored_tensors", set)()}

    def load(self, get) -> None:
        w_in, w_out = self.linear_in.weight.data, self.linear_proj.weight.data
        w_in.zero_()
        w_out.zero_()
        for pre, p, c, o in zip(self.prefixes, self.parts, self.columns, self.out_columns):
            w_in[c: c + sum(p.inputs.values())].copy_(torch.cat([get(pre + k) for k in p.inputs]))
            w_out[:, o: o + p.out_width].copy_(get(pre + "o"))
            p.load(lambda k, pre=pre: get(pre + k))
        if self.output_bias is not None:
            self.output_bias.data.copy_(get("o.b"))

    def forward(self, x, ctx, rope, step=None):
        """``x`` [T, H] -> the output linear's partial sums.  ``rope``: per part, the rotation tables (or None); ``step``: what the layers of
        one forward share."""
        takes_partials = len(self.parts) == 1 and ctx.is_decode_only() and getattr(self.parts[0], "takes_partials", False)
        proj, _ = self.linear_in(x, defer_reduction=takes_partials)
        out = torch.empty((x.shape[0], self.linear_proj.weight.shape[1]), dtype=x.dtype, device=x.device)
        if self.padded_outputs or not ctx.is_decode_only() and (
                ctx.using_cuda_graph_this_step() or ctx.padded_active_token_count != ctx.active_token_count):
            out.zero_()  # padding tokens belong to no row, padding columns to no part
        for p, c, o, s, tables in zip(self.parts, self.columns, self.out_columns, self.scales, rope):
            p(x, proj, c, out, o, s, ctx, tables, step)
        return self.linear_proj(out, defer_reduction=True)[0]
