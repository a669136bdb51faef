"""Grouped-query attention with its parts as parameters: rotation, norms and biases in front of it, a window that keeps the first tokens, a bias
by distance, capped scores, a sink, two maps whose difference counts, and rows of another layer.

A mixer part: it reads its columns of a projection that `JoinedMixer` made and fills its columns of the output linear's input."""
from __future__ import annotations

import math

import torch

from .. import _lib, ops
from ..tensor_parallel.layers import _device
from .attention import choose_attention_splits
from .hybrid_config import GroupedAttentionConfig, HybridConfig

EXTRA = 2  # AttentionArgs.separate


class GroupedAttention(torch.nn.Module):
    def __init__(self, config: HybridConfig, mixer: GroupedAttentionConfig, layer_index: int):
        super().__init__()
        self.config, self.mixer, self.layer_number = config, mixer, layer_index + 1
        self.rows_of = self.layer_number if mixer.kv_from is None else mixer.kv_from + 1
        m, dt, dev = mixer, config.params_dtype, _device()
        own = m.kv_from is None
        # columns of the projection
        self.inputs = {"q": m.heads * m.maps * m.dim}
        if own:
            self.inputs["k"] = m.kv_heads * m.maps * m.dim
            if not m.values_from_keys:
                self.inputs["v"] = m.kv_heads * m.vdim
        if m.gate or m.head_gate:
            self.inputs["g"] = m.heads * (m.vdim if m.gate else 1)
        self.first_values = config.mixes_values_first(layer_index)
        self.out_width = m.heads * m.vdim

        def param(shape, dtype):
            return torch.nn.Parameter(torch.zeros(shape, dtype=dtype, device=dev), requires_grad=False)

        self.q_bias = param(self.inputs["q"], dt) if m.biases else None
        self.k_bias = param(self.inputs["k"], dt) if m.biases and own else None
        self.sinks = param(m.heads, torch.float32) if m.sink else None
        self.bias_rows = m.distance_bias.rows_by_distance() if m.distance_bias is not None else None
        self.distance_bias = param((m.heads, len(self.bias_rows)), torch.float32) if self.bias_rows is not None else None
        self.mix = param(1, dt) if m.value_mix and not self.first_values else None
        self.lambda_ = 0.0  # weight of the second map

    @property
    def tensor_cores(self) -> bool:
        return self.config.params_dtype == torch.bfloat16 and self.mixer.tensor_cores

    def prefill_unit_tokens(self) -> int:
        """Query tokens that share a block of 64 query rows (0: the attention kernel works token by token)."""
        return 64 // (self.mixer.heads // self.mixer.kv_heads) if self.tensor_cores else 0

    def checkpoint_tensors(self) -> dict:
        """Checkpoint name (below this part of the mixer) -> shape, without the input linear's weights."""
        m = self.mixer
        out = {}
        if m.biases:
            out["q.b"] = (self.inputs["q"],)
            if self.k_bias is not None:
                out["k.b"] = (self.inputs["k"],)
        if m.sink:
            out["sink"] = (m.heads,)
        if self.mix is not None:
            out["vmix"] = ()
        if m.distance_bias is not None:
            out["rel"] = (m.distance_bias.rows, m.heads)
        if m.diff is not None:
            out.update({k: (m.dim,) for k in ("lq1", "lk1", "lq2", "lk2")})
        return out

    def ignored_tensors(self) -> set:
        return {"vmix"} - set(self.checkpoint_tensors())

    def load(self, get) -> None:
        m = self.mixer
        if self.mix is not None:
            self.mix.data.copy_(get("vmix").reshape(1))
        for dst, name in ((self.q_bias, "q.b"), (self.k_bias, "k.b"), (self.sinks, "sink")):
            if dst is not None:
                dst.data.copy_(get(name))
        if self.distance_bias is not None:
            self.distance_bias.data.copy_(get("rel").float()[self.bias_rows].t())
        if m.diff is not None:
            dots = [float((get("lq" + i).double() * get("lk" + i).double()).sum()) for i in "12"]
            self.lambda_ = math.exp(dots[0]) - math.exp(dots[1]) + m.diff

    def forward(self, x, proj, column: int, out, out_column: int, scale: float, ctx, rope, step=None) -> None:
        """``proj`` [T, ...]: this part's columns from ``column`` on; ``out`` [T, ...]: its output, times ``scale``, from ``out_column`` on.
        ``step`` (shared by the layers of one forward) carries the first mixing layer's values on to the others."""
        m, T, es = self.mixer, proj.shape[0], proj.element_size()
        at, c = {}, column
        for name, n in self.inputs.items():
            at[name] = c
            c += n
        pool = ctx.token_rows(self.rows_of)
        values_at = m.kv_heads * m.maps * m.dim
        v_pool = pool[:, :, values_at:]
        r = _lib.RotateAppendArgs()
        r.proj, r.proj_ld, r.num_tokens, r.dtype = proj.data_ptr(), proj.stride(0), T, ops.dtype_code(proj.dtype)
        r.dim, r.vdim, r.rms, r.eps = m.dim, m.vdim, int(m.unit_queries_keys), self.config.layernorm_epsilon
        if m.rot is not None and m.rot.dims:
            r.rope_cos, r.rope_sin, r.max_positions = rope[0].data_ptr(), rope[1].data_ptr(), rope[0].shape[0]
            r.rot_dims, r.halves, r.token_to_pos = m.rot.dims, int(m.rot.halves), ctx.token_to_position_in_request.data_ptr()
        queries = None
        if r.rot_dims or m.unit_queries_keys or m.biases:
            queries = torch.empty((T, self.inputs["q"]), dtype=proj.dtype, device=proj.device)
            r.q_out, r.off_q, r.q_vecs = queries.data_ptr(), at["q"], m.heads * m.maps
            r.q_bias = None if self.q_bias is None else self.q_bias.data_ptr()
        if m.kv_from is None:
            r.k_pool, r.v_pool, r.pool_row_elems = pool.data_ptr(), v_pool.data_ptr(), pool.shape[2]
            r.chunk_idx, r.local_pos = ctx.token_to_chunk_idx.data_ptr(), ctx.token_to_local_position_within_kv_chunk.data_ptr()
            r.num_chunks, r.chunk_size = pool.shape[0], pool.shape[1]
            r.off_k, r.k_vecs, r.off_v, r.v_vecs = at["k"], m.kv_heads * m.maps, at.get("v", at["k"]), m.kv_heads
            r.k_bias = None if self.k_bias is None else self.k_bias.data_ptr()
            r.v_bias = r.k_bias if m.values_from_keys else None
            if self.first_values:
                step["first_values"] = torch.empty((T, m.kv_heads * m.vdim), dtype=proj.dtype, device=proj.device)
                r.v_first_out = step["first_values"].data_ptr()
            elif self.mix is not None:
                r.v_first_in, r.mix = step["first_values"].data_ptr(), self.mix.data_ptr()
        if r.q_vecs or r.k_vecs:
            ops.struct_kernel("rotate_append", r, pool)
        decode, tc = ctx.is_decode_only(), self.tensor_cores
        table = ctx.request_to_kv_chunk_ids_cudagraph_only
        a = _lib.AttentionArgs()
        a.separate, a.softmax_scale, a.window, a.keep_first = EXTRA, m.scale, m.window or 0, m.keep_first
        if queries is None:
            a.qkv, a.q_ld = proj.data_ptr() + at["q"] * es, proj.stride(0)
        else:
            a.qkv, a.q_ld = queries.data_ptr(), queries.stride(0)
        a.out, a.out_ld, a.out_scale = out.data_ptr() + out_column * es, out.stride(0), scale
        a.k_cache, a.v_cache, a.pool_row_elems = pool.data_ptr(), v_pool.data_ptr(), pool.shape[2]
        a.block_table, a.max_chunks_per_row = table.data_ptr(), table.shape[1]
        a.num_tokens, a.num_q_heads, a.num_kv_heads, a.head_dim, a.value_dim = T, m.heads, m.kv_heads, m.dim, m.vdim
        a.num_chunks, a.chunk_size, a.num_splits = pool.shape[0], pool.shape[1], 1
        a.softcap = m.softcap or 0.0
        a.sinks = None if self.sinks is None else self.sinks.data_ptr()
        if m.head_gate:
            a.gate, a.gate_ld = proj.data_ptr() + at["g"] * es, proj.stride(0)
        if self.distance_bias is not None:
            a.distance_bias, a.bias_len = self.distance_bias.data_ptr(), self.distance_bias.shape[1]
        if decode:
            a.kv_seq_lengths, a.row_order = ctx.kv_seq_lengths_cudagraph_only.data_ptr(), ctx.attention_row_order.data_ptr()
            if tc:
                longest = ctx.max_sequence_length if m.window is None else min(ctx.max_sequence_length, m.window + m.keep_first + 64)
                a.num_splits = choose_attention_splits(T, m.kv_heads, longest, pool.shape[1])
        else:
            a.kv_seq_lengths, a.row_of_token = ctx.token_kv_lengths.data_ptr(), ctx.token_to_block_table_row.data_ptr()
        a._anchor = pool
        maps_out = None
        if m.diff is not None:
            a.maps, a.lambda_, a.diff_scale, a.eps = 2, self.lambda_, 1.0 - m.diff, self.config.layernorm_epsilon
            if m.gate:
                a.gate, a.gate_ld = proj.data_ptr() + at["g"] * es, proj.stride(0)
            width = m.vdim if not tc else 64 if m.vdim <= 64 else 128
            maps_out = torch.empty(T * 2 * m.heads * a.num_splits * (width + 1), dtype=torch.float32, device=proj.device)
            a.workspace, a.workspace_bytes = maps_out.data_ptr(), 4 * maps_out.numel()
        if decode or not tc:
            ops.separate_attention(a, proj.dtype, tensor_cores=tc)
        else:
            units, count = ctx.prefill_units_of(self.prefill_unit_tokens())
            ops.separate_attention(a, proj.dtype, units=units, num_units=count, tensor_cores=True)
