"""Arguments of the short-convolution kernels, and the rows of a step that kernels with state per request need."""
from __future__ import annotations

import torch

from .. import _lib, ops


def short_conv_args(ctx, *, proj, filter_, state, channels: int, taps: int, out) -> _lib.ConvArgs:
    """What the short-convolution kernels need of a step: where every token's request starts and keeps its last inputs."""
    a = _lib.ConvArgs()
    a.proj, a.proj_ld, a.filter, a.channels, a.taps = proj.data_ptr(), proj.stride(0), filter_.data_ptr(), channels, taps
    a.state, a.state_slots = (None, 0) if state is None else (state.data_ptr(), state.shape[0])
    step_rows(a, ctx, proj.shape[0])
    a.out, a.dtype = out.data_ptr(), ops.dtype_code(proj.dtype)
    return a


def step_rows(a, ctx, num_tokens: int) -> None:
    """The step's rows in an argument struct: state slots, and (steps that are not one token per row) which tokens a row has."""
    a.state_in, a.state_out, a.num_tokens = ctx.state_read_slots.data_ptr(), ctx.state_write_slots.data_ptr(), num_tokens
    if ctx.is_decode_only():
        a.num_rows = num_tokens
    else:
        a.num_rows = ctx.padded_active_request_count
        a.cu_tokens = ctx.cu_query_seq_lengths_cudagraph_only.data_ptr()
        if hasattr(a, "row_of_token"):
            a.row_of_token = ctx.token_to_block_table_row.data_ptr()


def filter_of(taps: torch.Tensor) -> torch.Tensor:
    """[channels, taps] as a checkpoint holds it -> [taps, channels]."""
    return taps.transpose(0, 1).contiguous()
