"""RMSNorm / LayerNorm module over the fused add+norm kernel.

Stands where the reference uses ``WrappedTorchNorm`` (``megatron/core/transformer/torch_norm.py:38-51``)
or ``TENorm`` (``megatron/core/extensions/transformer_engine.py:204-238``): same constructor
(``config, hidden_size, eps``), same parameter names (``weight``, and ``bias`` for LayerNorm).
"""
from __future__ import annotations

import torch

from .. import ops
from .short_conv import short_conv_args


class B200Norm(torch.nn.Module):
    def __init__(self, config, hidden_size: int, eps: float = 1e-5, **_):
        super().__init__()
        dev = torch.device("cuda", torch.cuda.current_device()) if torch.cuda.is_available() else torch.device("cpu")
        self.eps = eps
        self.weight = torch.nn.Parameter(torch.ones(hidden_size, dtype=config.params_dtype, device=dev), requires_grad=False)
        if config.normalization == "LayerNorm":
            self.bias = torch.nn.Parameter(torch.zeros(hidden_size, dtype=config.params_dtype, device=dev), requires_grad=False)
        else:
            self.register_parameter("bias", None)

    accepts_gemm_partials = True  # add_and_norm takes the split-K partial sums of the linear before it

    @staticmethod
    def _op(quantize):
        return {None: ops.add_norm, False: ops.add_norm, "mxfp8": ops.add_norm_mxfp8,
                "blockwise": ops.add_norm_fp8_rowblock}[quantize]

    def forward(self, x, quantize=None):
        """Normalised rows; ``quantize`` ("mxfp8" | "blockwise") makes the output the FP8 input of a linear."""
        return self._op(quantize)(x, self.weight, beta=self.bias, eps=self.eps)[1]

    def add_and_norm(self, x, residual, bias=None, quantize=None):
        """(hidden, normed) with hidden = x (+bias) + residual: the bias-dropout-add of the
        reference (``fused_bias_dropout.py:11-57``, eval mode) fused with the norm that follows it
        and, with ``quantize``, with the FP8 quantisation of the next linear's input.  ``x`` may be the
        un-reduced split-K partial sums of the linear that produced it (`ops.GemmPartials`)."""
        if type(x).__name__ == "TpPending":  # partial outputs of the tensor-parallel ranks, summed by the kernel
            return ops.allreduce_add_norm(x, self.weight, bias=bias, residual=residual, beta=self.bias, eps=self.eps,
                                          want_hidden=True, quantize=quantize or None)
        if isinstance(x, ops.GemmPartials):
            return ops.add_norm_splitk(x, self.weight, bias=bias, residual=residual, beta=self.bias, eps=self.eps,
                                       want_hidden=True, quantize=quantize or None)
        return self._op(quantize)(x, self.weight, bias=bias, residual=residual, beta=self.bias, eps=self.eps, want_hidden=True)


class OutputNorm(torch.nn.Module):
    """Layer norm (a weight, no bias) of a sublayer's OUTPUT, added to a 32-bit residual stream by the same kernel:
    ``hidden += norm(f(x))``, where the sublayer read the stream itself.  The stream is fp32 ``[T, H]``; what the next
    sublayer reads is its copy in the activation type (the stream itself when that is fp32)."""

    accepts_gemm_partials = True

    def __init__(self, config, hidden_size: int, eps: float = 1e-5, **_):
        super().__init__()
        dev = torch.device("cuda", torch.cuda.current_device()) if torch.cuda.is_available() else torch.device("cpu")
        self.eps = eps
        self.weight = torch.nn.Parameter(torch.ones(hidden_size, dtype=config.params_dtype, device=dev), requires_grad=False)

    def start_stream(self, table, ids):
        """(fp32 stream, activations) of ``norm(table[ids])``."""
        hidden = torch.empty((ids.numel(), table.shape[1]), dtype=torch.float32, device=table.device)
        return hidden, ops.out_norm(table, self.weight, eps=self.eps, hidden=hidden, ids=ids)

    def add_to_stream(self, hidden, source):
        """hidden += norm(source) in place; ``source``: `ops.GemmPartials` of the sublayer's last linear."""
        return ops.out_norm(source, self.weight, eps=self.eps, hidden=hidden, accumulate=True)

    def of_rows(self, hidden, row_index=None):
        """norm of the stream's rows (all, or those picked by ``row_index``) in the activation type."""
        return ops.out_norm(hidden, self.weight, eps=self.eps, row_index=row_index)


class StreamNorm(torch.nn.Module):
    """Several 32-bit residual streams ``[T, streams, H]`` in place of one: what one sublayer left is written into all of them, and their blend
    (``blend``) is layer-normed for the next, in one kernel.  ``mix`` [from, to] and ``gain`` say what the sublayer behind this norm does to
    the streams (`left_by`).  ``plain`` without these weights: the streams' sum, and an ordinary residual sum."""

    def __init__(self, config, hidden_size: int, eps: float, streams: int, plain: bool = False):
        super().__init__()
        dev = torch.device("cuda", torch.cuda.current_device()) if torch.cuda.is_available() else torch.device("cpu")
        self.eps, self.streams, self.plain = eps, streams, plain

        def param(value, dtype):
            return torch.nn.Parameter(value.to(device=dev, dtype=dtype), requires_grad=False)

        self.weight, self.bias = param(torch.ones(hidden_size), config.params_dtype), param(torch.zeros(hidden_size), config.params_dtype)
        self.blend, self.gain = param(torch.ones(streams), torch.float32), param(torch.ones(streams), torch.float32)
        self.mix = param(torch.eye(streams), torch.float32)

    def checkpoint_tensors(self, norm: str, blends: str) -> dict:
        """Checkpoint tensor name -> shape, with the norm under ``norm`` and the streams' weights under ``blends``."""
        out = {norm: tuple(self.weight.shape), norm + ".b": tuple(self.weight.shape)}
        if not self.plain:
            out.update({blends + ".in": (self.streams,), blends + ".out": (self.streams,), blends + ".mix": (self.streams, self.streams)})
        return out

    def load(self, get, norm: str, blends: str) -> None:
        self.weight.data.copy_(get(norm))
        self.bias.data.copy_(get(norm + ".b"))
        if not self.plain:
            for dst, name in ((self.blend, ".in"), (self.gain, ".out"), (self.mix, ".mix")):
                dst.data.copy_(get(blends + name))

    def left_by(self, partials=None, bias=None, experts=None) -> "ops.PendingStreams":
        """What the sublayer behind this norm computed, for the next norm to write into the streams."""
        return ops.PendingStreams(partials=partials, bias=bias, experts=experts, mix=self.mix, gain=self.gain)

    def forward(self, hidden, pending, row_index=None):
        """Writes ``pending`` (a `PendingStreams`, or None) into ``hidden`` and returns the normed blend; with ``row_index`` (int64) only those
        rows are computed and ``hidden`` stays as it is."""
        rows = hidden.shape[0] if row_index is None else row_index.numel()
        out = torch.empty((rows, hidden.shape[2]), dtype=self.weight.dtype, device=hidden.device)
        ops.stream_norm(hidden, pending, blend=self.blend, gamma=self.weight, beta=self.bias, out=out, eps=self.eps, row_index=row_index)
        return out


class ParallelNorm(torch.nn.Module):
    """Everything a parallel block adds to the 32-bit residual stream and the RMS norms of the result, in one kernel.  ``outputs``
    norms of the same row (weights stored as the distance from ``config.norm_offset``) feed the branches that run side by side."""

    def __init__(self, config, hidden_size: int, eps: float, outputs: int = 2, out_scale: float = 1.0):
        super().__init__()
        dev = torch.device("cuda", torch.cuda.current_device()) if torch.cuda.is_available() else torch.device("cpu")
        self.eps, self.out_scale, self.gain = eps, out_scale, config.norm_offset
        self.weight = torch.nn.Parameter(torch.zeros((outputs, hidden_size), dtype=config.params_dtype, device=dev), requires_grad=False)

    def forward(self, hidden, pending, row_index=None):
        """Adds ``pending`` (a `PendingRows`, or None) to ``hidden`` [T, H] in place and returns the norms; with ``row_index`` (int64)
        only those rows are computed and ``hidden`` stays as it is."""
        rows = hidden.shape[0] if row_index is None else row_index.numel()
        out = [torch.empty((rows, hidden.shape[1]), dtype=self.weight.dtype, device=hidden.device) for _ in range(self.weight.shape[0])]
        ops.residual_norm(hidden, pending, list(self.weight), out, eps=self.eps, gain=self.gain, out_scale=self.out_scale, row_index=row_index)
        return out


class FilteredNorm(torch.nn.Module):
    """Everything a parallel block adds to the 32-bit residual stream, ONE RMS norm of the result, and in front of each branch a short causal
    filter of the normed rows over time, added to them: branch i reads u + filter_i(u).  The last taps - 1 normed rows are a request's
    state.  One kernel in decode steps; the filters are a kernel of their own in the others."""

    def __init__(self, config, hidden_size: int, eps: float, outputs: int, layer_number: int):
        super().__init__()
        dev = torch.device("cuda", torch.cuda.current_device()) if torch.cuda.is_available() else torch.device("cpu")
        self.eps, self.gain, self.layer_number = eps, config.norm_offset, layer_number

        def param(*shape):
            return torch.nn.Parameter(torch.zeros(shape, dtype=config.params_dtype, device=dev), requires_grad=False)

        self.weight, self.filters = param(hidden_size), param(outputs, config.input_taps, hidden_size)

    def forward(self, hidden, pending, ctx):
        """Adds ``pending`` (a `PendingRows`) to ``hidden`` [T, H] in place; what the branches read."""
        state = ctx.recurrent_state(self.layer_number, "input") if self.filters.shape[1] > 1 else None
        out = [torch.empty(hidden.shape, dtype=self.weight.dtype, device=hidden.device) for _ in range(self.filters.shape[0])]
        if ctx.is_decode_only():
            ops.residual_norm(hidden, pending, [self.weight], out, eps=self.eps, gain=self.gain, filters=list(self.filters), state=state,
                              state_slots=(ctx.state_read_slots, ctx.state_write_slots))
            return out
        normed = torch.empty(hidden.shape, dtype=self.weight.dtype, device=hidden.device)
        ops.residual_norm(hidden, pending, [self.weight], [normed], eps=self.eps, gain=self.gain)
        T, taps, width = hidden.shape[0], *self.filters.shape[1:]
        a = short_conv_args(ctx, proj=normed, filter_=self.filters[0], state=state, channels=width, taps=taps, out=out[0])
        if len(out) > 1:
            a.filter_2, a.out_2 = self.filters[1].data_ptr(), out[1].data_ptr()
        ops.struct_kernel("conv_add", a, normed)
        return out
