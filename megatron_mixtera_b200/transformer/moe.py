"""Mixture of experts: every token runs its `top` best experts - on its input times their sigmoid scores, beside a gated shared expert, or
(`SoftmaxRouting`, `ChosenSoftmaxRouting`) with softmax scores as weights of the outputs.  Tokens are sorted by expert on the device; the products of all experts are
one grouped GEMM."""
from __future__ import annotations

import torch

from .. import _lib, ops
from ..tensor_parallel.layers import _device
from .hybrid_config import ChosenSoftmaxRouting, HybridConfig, MoeConfig, SoftmaxRouting


def _padded(ff: int) -> int:
    """Whole blocks of 64 features: a 128-row tile of the up weights holds 64 gate rows and the matching up rows (16 in turn)."""
    return -(-ff // 64) * 64


def interleave_up(gate: torch.Tensor, up: torch.Tensor) -> torch.Tensor:
    """[ff, H] each -> [2 * padded ff, H], blocks of 16 gate rows and 16 up rows, missing rows zero."""
    ff, H = gate.shape
    pad = _padded(ff)
    out = torch.zeros((pad // 16, 2, 16, H), dtype=gate.dtype, device=gate.device)
    for i, w in enumerate((gate, up)):
        full = torch.zeros((pad, H), dtype=gate.dtype, device=gate.device)
        full[:ff] = w
        out[:, i] = full.view(pad // 16, 16, H)
    return out.view(2 * pad, H)


class ExpertOutputs:
    """What `MixtureOfExperts` hands to the kernel that adds it to the stream: expert outputs sorted by expert, where a token's rows
    lie among them, and the shared expert's rows with their gates; under softmax routing the rows' weights, and the input for the pairs of
    identity experts."""

    __slots__ = ("rows", "pairs", "offsets", "top", "experts", "shared_rows", "shared_gate", "weights", "identity", "input")

    def __init__(self, rows, pairs, offsets, top, experts, shared_rows=None, shared_gate=None, weights=None, identity=0, input=None):
        self.rows, self.pairs, self.offsets, self.top, self.experts = rows, pairs, offsets, top, experts
        self.shared_rows, self.shared_gate, self.weights, self.identity, self.input = shared_rows, shared_gate, weights, identity, input


class MixtureOfExperts(torch.nn.Module):
    def __init__(self, config: HybridConfig, moe: MoeConfig):
        super().__init__()
        self.config, self.moe = config, moe
        H = config.hidden_size

        def param(*shape):
            return torch.nn.Parameter(torch.zeros(shape, dtype=config.params_dtype, device=_device()), requires_grad=False)

        self.ff = _padded(moe.expert.ff)
        # router rows (identity experts' included), then the shared expert's gate
        self.columns = moe.experts + (moe.routing.identity if isinstance(moe.routing, SoftmaxRouting) else 0)
        self.shared_gated = moe.shared is not None and moe.routing is None
        self.router = param(-(-(self.columns + self.shared_gated) // 8) * 8, H)
        # added to the scores that choose (a bias on the logits, part of the score, where the chosen ones' softmax weighs)
        self.correction = param(self.columns) if moe.routing is not None else None
        self.correction_name = "router.b" if isinstance(moe.routing, ChosenSoftmaxRouting) else "correction"
        rows = 2 if moe.expert.gated else 1
        self.names = ("gate", "up", "down") if moe.expert.gated else ("up", "down")
        self.up, self.down = param(moe.experts, rows * self.ff, H), param(moe.experts, H, self.ff)
        self.shared_ff, self.shared_up, self.shared_down = 0, None, None
        if moe.shared is not None:
            self.shared_ff = _padded(moe.shared.ff)
            self.shared_up, self.shared_down = param(rows * self.shared_ff, H), param(H, self.shared_ff)

    def checkpoint_tensors(self) -> dict:
        H, c = self.config.hidden_size, self.moe
        out = {"router": (self.columns, H)}
        if c.routing is not None:
            out[self.correction_name] = (self.columns,)
        parts = [(f"e{e}", c.expert.ff) for e in range(c.experts)]
        if c.shared is not None:
            parts.append(("shared", c.shared.ff))
            if self.shared_gated:
                out["shared.sg"] = (1, H)
        for name, ff in parts:
            out.update({f"{name}.{k}": (H, ff) if k == "down" else (ff, H) for k in self.names})
        return out

    def load(self, get) -> None:
        c, dev = self.moe, self.router.device
        self.router.data[: self.columns].copy_(get("router"))
        if self.correction is not None:
            self.correction.data.copy_(get(self.correction_name))

        def put_up(dst, name, ff):
            if c.expert.gated:
                dst.copy_(interleave_up(get(f"{name}.gate").to(dev), get(f"{name}.up").to(dev)))
            else:
                dst[:ff].copy_(get(f"{name}.up"))

        for e in range(c.experts):
            put_up(self.up.data[e], f"e{e}", c.expert.ff)
            self.down.data[e, :, : c.expert.ff].copy_(get(f"e{e}.down"))
        if c.shared is not None:
            if self.shared_gated:
                self.router.data[c.experts].copy_(get("shared.sg")[0])
            put_up(self.shared_up.data, "shared", c.shared.ff)
            self.shared_down.data[:, : c.shared.ff].copy_(get("shared.down"))

    @staticmethod
    def tile_tokens(pairs: int, experts: int, simt: bool) -> int:
        """Tokens of a tile of the grouped products, by how many an expert gets on average."""
        if simt:
            return 64
        average = pairs / experts
        return 256 if average >= 768 else 128 if average >= 128 else 64 if average >= 40 else 32

    def forward(self, x) -> ExpertOutputs:
        c, (T, H), dev, dt = self.moe, x.shape, x.device, x.dtype
        pairs, simt = T * c.top, dt == torch.float32 or H % 8 != 0
        a = _lib.MoeArgs()
        a.num_tokens, a.width, a.experts, a.top, a.ff, a.shared_ff = T, H, c.experts, c.top, self.ff, self.shared_ff
        a.limit, a.alpha, a.simt, a.dtype = c.expert.limit or 0.0, c.expert.alpha, int(simt), ops.dtype_code(dt)
        a.relu2 = int(not c.expert.gated)
        identity = 0
        if isinstance(c.routing, SoftmaxRouting):
            r, identity = c.routing, c.routing.identity
            a.plain, a.identity, a.groups, a.keep_groups, a.weight_scale = 1, identity, r.groups, r.keep_groups, r.scale
        elif c.routing is not None:
            a.plain, a.groups, a.keep_groups, a.weight_scale = 2, 1, 1, 1.0
        if c.routing is not None:
            a.correction = self.correction.data_ptr()
        a.tile_tokens = self.tile_tokens(pairs, c.experts, simt)
        a.max_tiles = pairs // a.tile_tokens + min(c.experts, pairs)
        # bookkeeping in one block of 32-bit words: pairs | weights | row scales | shared gates | offsets | tiles | number of tiles
        sizes = (2 * pairs, pairs, pairs, T, c.experts + 1, 4 * a.max_tiles, 1)
        starts = [0]
        for n in sizes:
            starts.append(starts[-1] + -(-n // 4) * 4)  # 16-byte aligned
        words = torch.empty(starts[-1], dtype=torch.int32, device=dev)
        at = [words.data_ptr() + 4 * s for s in starts]
        a.pairs, a.pair_weight, a.row_scale, shared_gate, a.offsets, a.tiles, a.num_tiles = at[:7]
        a.counts = ops.moe_counters(dev, c.experts).data_ptr()
        a.x, a.up, a.down = x.data_ptr(), self.up.data_ptr(), self.down.data_ptr()
        x_sorted = torch.empty((pairs, H), dtype=dt, device=dev)
        inter, rows = torch.empty((pairs, self.ff), dtype=dt, device=dev), torch.empty((pairs, H), dtype=dt, device=dev)
        a.x_sorted, a.inter, a.y = x_sorted.data_ptr(), inter.data_ptr(), rows.data_ptr()
        shared_rows = shared_inter = None
        if c.shared is not None:
            shared_inter, shared_rows = torch.empty((T, self.shared_ff), dtype=dt, device=dev), torch.empty((T, H), dtype=dt, device=dev)
            a.shared_gate = shared_gate if self.shared_gated else None
            a.shared_up, a.shared_down = self.shared_up.data_ptr(), self.shared_down.data_ptr()
            a.shared_inter, a.shared_y, a.shared_limit = shared_inter.data_ptr(), shared_rows.data_ptr(), c.shared.limit or 0.0
        logits = ops.linear_partials(x, self.router)  # fp32 sums of exact products: the router's 32-bit logits
        a.router, a.router_splits = ops.partials_of(logits)
        a.router_ld = self.router.shape[0]
        for kernel in ("moe_route", "moe_gather", "moe_up", "moe_down"):
            ops.struct_kernel(kernel, a, x)
        gates = words[starts[3]: starts[3] + T].view(torch.float32) if self.shared_gated else None
        weights = words[starts[1]:] if c.routing is not None else None
        return ExpertOutputs(rows, words, words[starts[4]:], c.top, c.experts, shared_rows, gates, weights, identity, x if identity else None)
