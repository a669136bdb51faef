"""Latent attention: keys and values of all heads come from one small row per token, the only thing cached.

Two forms of the same attention.  Absorbed: the key matrix is applied to the queries instead of the cached rows and the value
matrix to the attention output, both as batched per-head GEMMs; the cached rows are read once and never expanded.  This is
how decoding runs, and portions of prompts with a long past.  Expanded: one GEMM spells out the keys and values of all heads,
which costs several times fewer products per (query, key) pair; it pays where most of the keys belong to the step itself.
"""
from __future__ import annotations

import torch

from .. import _lib, ops
from ..tensor_parallel.layers import ColumnParallelLinear, RowParallelLinear, _device
from .attention import _sm_count
from .grouped_attention import EXTRA
from .hybrid_config import HybridConfig, LatentAttentionConfig


def choose_latent_splits(num_rows: int, heads: int, window, max_sequence_length: int, blocks_per_row: int) -> int:
    """Key splits of a decode row, each of them ``blocks_per_row`` CTAs: a function of capture-time constants.  The fewest splits that
    fill the CTAs the GPU holds at once to 85 % (else the best there is), none below 256 keys at the longest visible range."""
    slots = _sm_count() * (2 if heads <= 16 else 1)
    blocks = max(1, num_rows * blocks_per_row)
    keys = max_sequence_length if window is None else min(window, max_sequence_length)
    best, best_fill = 1, 0.0
    for splits in range(1, max(1, min(keys // 256, 64)) + 1):
        length = -(-(-(-keys // splits)) // 64) * 64  # whole tiles, as the kernels cut
        units = blocks * -(-keys // length)
        fill = units / (-(-units // slots) * slots)
        if fill > best_fill:
            best, best_fill = splits, fill
        if fill >= 0.85:
            return splits
    return best


class LatentAttention(torch.nn.Module):
    def __init__(self, config: HybridConfig, mixer: LatentAttentionConfig, layer_index: int):
        super().__init__()
        self.config, self.mixer = config, mixer
        m, dt, dev = mixer, config.params_dtype, _device()
        self.cache_layer_number = (layer_index if m.kv_from is None else m.kv_from) + 1
        self.owns_rows = m.kv_from is None
        # one linear for everything that reads the layer's input: [queries or their latent | latent, shared key | gates]
        self.query_width = m.heads * (m.dim + m.rot_dim)
        self.gate_width = m.heads * (m.vdim if m.gate == "value" else 1)
        self.inputs = {"q": self.query_width} if m.q_rank is None else {"dq": m.q_rank}
        if self.owns_rows:
            self.inputs["dkv"] = m.kv_rank + m.rot_dim
        self.inputs["g"] = self.gate_width
        starts_at_vectors = m.gate == "value"  # (gates are read as vectors there)
        self.offsets, at = {}, 0
        for name, n in self.inputs.items():
            at = -(-at // 8) * 8 if starts_at_vectors else at
            self.offsets[name] = at
            at += n
        self.dkv_offset, self.gate_offset = self.offsets.get("dkv", -1), self.offsets["g"]
        self.in_width = at
        padded = -(-at // 8) * 8  # whole 16-byte vectors per row; the added rows are zero
        self.linear_in = ColumnParallelLinear(config.hidden_size, padded, config=config, bias=False)
        self.query_up = self.query_norm = self.sinks = None
        if m.q_rank is not None:
            self.query_up = torch.nn.Parameter(torch.empty(self.query_width, m.q_rank, dtype=dt, device=dev), requires_grad=False)
            self.query_norm = torch.nn.Parameter(torch.ones(m.q_rank, dtype=dt, device=dev), requires_grad=False)
        if m.sink:
            self.sinks = torch.nn.Parameter(torch.zeros(m.heads, dtype=torch.float32, device=dev), requires_grad=False)
        # absorbed: per head [latent][dim]; expanded: [keys of all heads | values of all heads] x latent
        self.key_up = torch.nn.Parameter(torch.empty(m.heads * m.kv_rank, m.dim, dtype=dt, device=dev), requires_grad=False)
        self.key_value_up = torch.nn.Parameter(torch.empty(m.heads * (m.dim + m.vdim), m.kv_rank, dtype=dt, device=dev),
                                               requires_grad=False)
        if self.owns_rows:
            self.latent_norm = torch.nn.Parameter(torch.ones(m.kv_rank, dtype=dt, device=dev), requires_grad=False)
        else:
            self.register_parameter("latent_norm", None)
        self.linear_proj = RowParallelLinear(m.heads * m.vdim, config.hidden_size, config=config, bias=False)

    def checkpoint_tensors(self) -> dict:
        """Checkpoint name (below the layer's mixer) -> shape."""
        m, H = self.mixer, self.config.hidden_size
        out = {name: (n, H) for name, n in self.inputs.items()}
        out.update({"uk": (m.heads * m.dim, m.kv_rank), "uv": (m.heads * m.vdim, m.kv_rank), "o": (H, m.heads * m.vdim)})
        if m.q_rank is not None:
            out.update({"dq.norm": (m.q_rank,), "uq": (self.query_width, m.q_rank)})
        if m.sink:
            out["sink"] = (m.heads,)
        if self.owns_rows:
            out["dkv.norm"] = (m.kv_rank,)
        return out

    def load(self, get) -> None:
        m = self.mixer
        w = self.linear_in.weight.data
        w.zero_()
        for name, n in self.inputs.items():
            w[self.offsets[name]: self.offsets[name] + n].copy_(get(name))
        if m.q_rank is not None:
            self.query_up.data.copy_(get("uq"))
            self.query_norm.data.copy_(get("dq.norm"))
        if m.sink:
            self.sinks.data.copy_(get("sink"))
        self.key_up.data.copy_(get("uk").view(m.heads, m.dim, m.kv_rank).transpose(1, 2).reshape(m.heads * m.kv_rank, m.dim))
        self.key_value_up.data.copy_(torch.cat([get("uk"), get("uv")]))
        if self.owns_rows:
            self.latent_norm.data.copy_(get("dkv.norm"))
        self.linear_proj.weight.data.copy_(get("o"))

    @property
    def value_up(self):
        return self.key_value_up[self.mixer.heads * self.mixer.dim:]

    expand_prompts = True  # False: the absorbed form everywhere

    UNIT_TOKENS = 16   # per work unit of the absorbed prompt kernel (it cuts a unit into blocks of query rows itself)
    BLOCK_TOKENS = 64  # queries, and keys of a chunk, of the prompt kernel of grouped attention

    @property
    def prompts_as_grouped(self) -> bool:
        """Whether expanded keys and values are an ordinary pool to the prompt kernel of grouped attention: nothing rotated beside them."""
        m = self.mixer
        return (self.config.params_dtype == torch.bfloat16 and m.rot_dim == 0 and m.window is None and m.dim % 8 == 0 and m.vdim % 8 == 0
                and max(m.dim, m.vdim) <= 128 and m.q_rank is not None)

    def prefill_unit_tokens(self) -> set:
        """Tokens per work unit of the prompt kernels."""
        return {self.UNIT_TOKENS} | ({self.BLOCK_TOKENS} if self.prompts_as_grouped else set())

    def _expansion(self, x, ctx):
        m = self.mixer
        if not (self.expand_prompts and x.dtype == torch.bfloat16 and ops.latent_prompt_supported(m.dim, m.rot_dim, m.vdim, m.heads)):
            return None
        return ctx.expanded_keys(m.window, self.BLOCK_TOKENS if self.prompts_as_grouped else 0)

    def _attend_grouped(self, queries, key_values, block_table, proj, out, ctx) -> None:
        """Attention of a prompt step over its expanded rows [keys of all heads | values of all heads] in whole chunks."""
        m = self.mixer
        a = _lib.AttentionArgs()
        a.separate, a.softmax_scale, a.out_scale = EXTRA, m.scale, 1.0
        a.qkv, a.q_ld, a.out, a.out_ld = queries.data_ptr(), queries.stride(0), out.data_ptr(), out.stride(0)
        a.k_cache, a.v_cache = key_values.data_ptr(), key_values.data_ptr() + m.heads * m.dim * key_values.element_size()
        a.pool_row_elems, a.num_chunks, a.chunk_size = key_values.stride(0), key_values.shape[0] // self.BLOCK_TOKENS, self.BLOCK_TOKENS
        a.block_table, a.max_chunks_per_row = block_table.data_ptr(), block_table.shape[1]
        a.num_tokens, a.num_q_heads, a.num_kv_heads, a.head_dim, a.value_dim = queries.shape[0], m.heads, m.heads, m.dim, m.vdim
        a.num_splits, a.kv_seq_lengths, a.row_of_token = 1, ctx.token_kv_lengths.data_ptr(), ctx.token_to_block_table_row.data_ptr()
        a.sinks = None if self.sinks is None else self.sinks.data_ptr()
        a.gate, a.gate_ld = proj.data_ptr() + self.gate_offset * proj.element_size(), proj.stride(0)
        a.value_gates, a._anchor = int(m.gate == "value"), key_values
        units, count = ctx.prefill_units_of(self.BLOCK_TOKENS)
        ops.separate_attention(a, queries.dtype, units=units, num_units=count, tensor_cores=True)

    def forward(self, x, ctx, rope=None, step=None):
        """``x`` [T, H] -> the output linear's partial sums."""
        m, T, dev = self.mixer, x.shape[0], x.device
        proj, _ = self.linear_in(x)
        expanded = self._expansion(x, ctx)
        # queries: the absorbed form fills whole rows, the expanded one needs the rotated part alone
        q_stride, q_rot_at = (m.row_width, m.kv_pad) if expanded is None else (m.row_width - m.kv_pad, 0)
        q_full = torch.empty((T, m.heads, max(q_stride, 8)), dtype=x.dtype, device=dev)
        pool = ctx.latent_cache(self.cache_layer_number)
        decode = ctx.is_decode_only()
        a = _lib.LatentArgs()
        a.proj, a.proj_ld, a.dkv_offset = proj.data_ptr(), proj.stride(0), self.dkv_offset
        a.gate_offset = self.gate_offset if m.gate == "head" or expanded is not None else -1  # (absorbed: values are gated behind the kernel)
        a.norm_weight = None if self.latent_norm is None else self.latent_norm.data_ptr()
        a.max_positions = 1
        if rope is not None:
            a.rope_cos, a.rope_sin, a.max_positions = rope[0].data_ptr(), rope[1].data_ptr(), rope[0].shape[0]
        a.token_to_pos = ctx.token_to_position_in_request.data_ptr()
        a.token_to_chunk_idx = ctx.token_to_chunk_idx.data_ptr()
        a.token_to_local_pos = ctx.token_to_local_position_within_kv_chunk.data_ptr()
        a.block_table = ctx.request_to_kv_chunk_ids_cudagraph_only.data_ptr()
        a.max_chunks_per_row = ctx.request_to_kv_chunk_ids_cudagraph_only.shape[1]
        a.pool, a.num_chunks, a.chunk_size = pool.data_ptr(), pool.shape[0], pool.shape[1]
        a.q_full, a.q_stride, a.q_rot_at = q_full.data_ptr(), q_stride, q_rot_at
        a.num_tokens, a.heads, a.dim, a.rot_dim, a.rot_dims = T, m.heads, m.dim, m.rot_dim, 0 if m.rot is None else m.rot.dims
        a.kv_rank, a.kv_pad, a.row_width = m.kv_rank, m.kv_pad, m.row_width
        a.window, a.scale, a.eps = m.window or 0, m.scale, self.config.layernorm_epsilon
        a.dtype, a.num_splits = ops.dtype_code(x.dtype), 1
        a.sinks = None if self.sinks is None else self.sinks.data_ptr()
        values = torch.empty((T, m.heads * m.vdim), dtype=x.dtype, device=dev)
        queries = proj
        if m.q_rank is not None:
            q_latent = torch.empty((T, m.q_rank), dtype=x.dtype, device=dev)
            a.q_latent_out, a.q_rank, a.q_latent_offset = q_latent.data_ptr(), m.q_rank, self.offsets["dq"]
            a.q_norm_weight = self.query_norm.data_ptr()
            queries = torch.empty((T, self.query_width), dtype=x.dtype, device=dev)
            a.q, a.q_ld = queries.data_ptr(), queries.stride(0)
        if expanded is not None:
            table, num_keys = expanded[:2]
            key_rows = torch.empty((num_keys, m.row_width), dtype=x.dtype, device=dev)
            ops.latent_append(a, pool)
            if m.q_rank is not None:
                ops.linear(q_latent, self.query_up, out=queries)
            a.num_rows, a.num_keys, a.max_row_tokens, a.vdim = table.shape[1] - 1, num_keys, ctx.max_seqlen_q, m.vdim
            a.value_gates = int(m.gate == "value")
            a.cu_tokens = ctx.cu_query_seq_lengths_cudagraph_only.data_ptr()
            a.cu_keys, a.key_start, a.key_rows = table[0].data_ptr(), table[1].data_ptr(), key_rows.data_ptr()
            a.key_end = table[2].data_ptr()
            ops.latent_gather(a, pool)
            key_values = ops.linear(key_rows, self.key_value_up, K=m.kv_rank)
            if self.prompts_as_grouped:
                self._attend_grouped(queries, key_values, expanded[2], proj, values, ctx)
                return self.linear_proj(values, defer_reduction=True)[0]
            a.key_values, a.out = key_values.data_ptr(), values.data_ptr()
            ops.latent_prompt_attention(a, pool)
            return self.linear_proj(values, defer_reduction=True)[0]
        latent_out = torch.empty((T, m.heads * m.kv_rank), dtype=x.dtype, device=dev)
        a.out = latent_out.data_ptr()
        if decode:
            a.kv_seq_lengths = ctx.kv_seq_lengths_cudagraph_only.data_ptr()
            if x.dtype == torch.bfloat16:
                a.num_splits = choose_latent_splits(T, m.heads, m.window, ctx.max_sequence_length,
                                                    ops.latent_decode_blocks(m.heads, m.kv_rank, m.row_width, pool.shape[1]))
        else:
            a.unit_tokens = self.UNIT_TOKENS
            units, a.num_units = ctx.prefill_units_of(a.unit_tokens)
            a.units = units.data_ptr()
        if m.q_rank is not None:
            ops.latent_append(a, pool)
            ops.linear(q_latent, self.query_up, out=queries)
        # absorbed queries: per head W_uk^T q
        ops.linear(queries, self.key_up, out=q_full.view(T, -1), batch=m.heads, x_batch=m.dim + m.rot_dim, y_batch=m.row_width, K=m.dim)
        if m.q_rank is None:
            ops.latent_append(a, pool)
        ops.latent_attention(a, pool)
        gates = proj[:, self.gate_offset:] if m.gate == "value" else None
        ops.linear(latent_out, self.value_up, out=values, batch=m.heads, x_batch=m.kv_rank, y_batch=m.vdim, K=m.kv_rank, gate=gates)
        return self.linear_proj(values, defer_reduction=True)[0]
