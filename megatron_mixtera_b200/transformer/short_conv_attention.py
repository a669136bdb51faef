"""Grouped-query attention with short convolutions: queries, keys and values pass a causal convolution over time, queries and keys
a per-head RMS norm, values may be mixed with those of the first mixing layer; no rotation, softmax over a sliding window."""
from __future__ import annotations

import torch

from .. import _lib, ops
from ..tensor_parallel.layers import ColumnParallelLinear, RowParallelLinear, _device
from .attention import choose_attention_splits
from .hybrid_config import HybridConfig, ShortConvAttentionConfig
from .short_conv import filter_of, short_conv_args


class ShortConvAttention(torch.nn.Module):
    def __init__(self, config: HybridConfig, mixer: ShortConvAttentionConfig, layer_index: int):
        super().__init__()
        self.config, self.mixer, self.layer_number = config, mixer, layer_index + 1
        m, dt, dev = mixer, config.params_dtype, _device()
        self.first_values = config.mixes_values_first(layer_index)
        # one linear for queries | keys | values
        self.linear_qkv = ColumnParallelLinear(config.hidden_size, -(-m.conv_channels // 8) * 8, config=config, bias=False)

        def param(*shape):
            return torch.nn.Parameter(torch.zeros(shape, dtype=dt, device=dev), requires_grad=False)

        self.conv_filter = param(m.conv, m.conv_channels)
        self.q_norm, self.k_norm, self.mix = param(m.dim), param(m.dim), param(1)
        self.linear_proj = RowParallelLinear(m.heads * m.vdim, config.hidden_size, config=config, bias=False)

    @property
    def tensor_cores(self) -> bool:
        return self.config.params_dtype == torch.bfloat16 and self.mixer.tensor_cores

    def prefill_unit_tokens(self) -> int:
        """Query tokens that share a block of 64 query rows (0: the attention kernel works token by token)."""
        return 64 // (self.mixer.heads // self.mixer.kv_heads) if self.tensor_cores else 0

    def checkpoint_tensors(self) -> dict:
        """Checkpoint name (below the layer's mixer) -> shape."""
        m, H = self.mixer, self.config.hidden_size
        widths = {"q": m.heads * m.dim, "k": m.kv_heads * m.dim, "v": m.kv_heads * m.vdim}
        out = {k: (n, H) for k, n in widths.items()}
        out.update({f"{k}.conv": (n, m.conv) for k, n in widths.items()})
        out.update({"q.norm": (m.dim,), "k.norm": (m.dim,), "o": (H, m.heads * m.vdim)})
        if m.value_mix and not self.first_values:
            out["vmix"] = ()
        return out

    def ignored_tensors(self) -> set:
        return {"vmix"} if self.first_values else set()

    def load(self, get) -> None:
        w = self.linear_qkv.weight.data
        w.zero_()
        w[: self.mixer.conv_channels].copy_(torch.cat([get(k).to(w.device) for k in "qkv"]))
        self.conv_filter.data.copy_(filter_of(torch.cat([get(f"{k}.conv") for k in "qkv"])))
        self.q_norm.data.copy_(get("q.norm"))
        self.k_norm.data.copy_(get("k.norm"))
        if self.mixer.value_mix and not self.first_values:
            self.mix.data.copy_(get("vmix").reshape(1))
        self.linear_proj.weight.data.copy_(get("o"))

    def forward(self, x, ctx, rope=None, step=None):
        """``x`` [T, H] -> the output linear's partial sums.  ``step`` (shared by the layers of one forward) carries the first
        mixing layer's values on to the others."""
        m, T, dev = self.mixer, x.shape[0], x.device
        proj, _ = self.linear_qkv(x)
        queries = torch.empty((T, m.heads * m.dim), dtype=x.dtype, device=dev)
        pool = ctx.token_rows(self.layer_number)
        values_at = m.kv_heads * m.dim
        c = short_conv_args(ctx, proj=proj, filter_=self.conv_filter, state=ctx.recurrent_state(self.layer_number, "conv"),
                            channels=m.conv_channels, taps=m.conv, out=queries)
        c.q_norm, c.k_norm, c.eps = self.q_norm.data_ptr(), self.k_norm.data_ptr(), self.config.layernorm_epsilon
        c.k_pool, c.v_pool, c.pool_row_elems = pool.data_ptr(), pool[:, :, values_at:].data_ptr(), pool.shape[2]
        c.chunk_idx, c.local_pos = ctx.token_to_chunk_idx.data_ptr(), ctx.token_to_local_position_within_kv_chunk.data_ptr()
        c.num_chunks, c.chunk_size = pool.shape[0], pool.shape[1]
        c.heads, c.kv_heads, c.dim, c.vdim = m.heads, m.kv_heads, m.dim, m.vdim
        if self.first_values:
            step["first_values"] = torch.empty((T, m.kv_heads * m.vdim), dtype=x.dtype, device=dev)
            c.v_first_out = step["first_values"].data_ptr()
        elif m.value_mix:
            c.v_first_in, c.mix = step["first_values"].data_ptr(), self.mix.data_ptr()
        ops.struct_kernel("conv_qkv", c, pool)
        return self.linear_proj(self._attend(queries, pool, values_at, ctx), defer_reduction=True)[0]

    def _attend(self, queries, pool, values_at: int, ctx):
        m, T = self.mixer, queries.shape[0]
        out = torch.empty((T, m.heads * m.vdim), dtype=queries.dtype, device=queries.device)
        table = ctx.request_to_kv_chunk_ids_cudagraph_only
        decode = ctx.is_decode_only()
        a = _lib.AttentionArgs()
        a.separate, a.qkv, a.out = 1, queries.data_ptr(), out.data_ptr()
        a.k_cache, a.v_cache, a.pool_row_elems = pool.data_ptr(), pool[:, :, values_at:].data_ptr(), pool.shape[2]
        a.block_table, a.max_chunks_per_row = table.data_ptr(), table.shape[1]
        a.num_tokens, a.num_q_heads, a.num_kv_heads, a.head_dim, a.value_dim = T, m.heads, m.kv_heads, m.dim, m.vdim
        a.num_chunks, a.chunk_size, a.num_splits = pool.shape[0], pool.shape[1], 1
        a.softmax_scale, a.window = m.scale, m.window or 0
        a._anchor = pool
        tc = self.tensor_cores
        if decode:
            a.kv_seq_lengths, a.row_order = ctx.kv_seq_lengths_cudagraph_only.data_ptr(), ctx.attention_row_order.data_ptr()
            if tc:
                longest = ctx.max_sequence_length if m.window is None else min(ctx.max_sequence_length, m.window + 64)
                a.num_splits = choose_attention_splits(T, m.kv_heads, longest, pool.shape[1])
            ops.separate_attention(a, queries.dtype, tensor_cores=tc)
            return out
        a.kv_seq_lengths, a.row_of_token = ctx.token_kv_lengths.data_ptr(), ctx.token_to_block_table_row.data_ptr()
        if tc:
            out.zero_()  # padding tokens belong to no unit
            units, count = ctx.prefill_units_of(self.prefill_unit_tokens())
            ops.separate_attention(a, queries.dtype, units=units, num_units=count, tensor_cores=True)
        else:
            ops.separate_attention(a, queries.dtype, tensor_cores=False)
        return out
