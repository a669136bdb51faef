"""Hybrid decoder of parallel blocks: x += mixer(norm1(x)) + experts(norm2(x)), mixers that are windowed attention with short
convolutions, wkv time mixing or the gated delta rule, in any order; scaled embeddings and an output head of its own.

One kernel per block joins everything the block adds to the 32-bit stream with the two norms the next block starts with."""
from __future__ import annotations

from typing import Dict, Optional

import torch

from .. import ops
from ..tensor_parallel.layers import ColumnParallelLinear, VocabParallelEmbedding
from ..transformer.gated_delta import GatedDelta
from ..transformer.hybrid_config import GatedDeltaConfig, HybridConfig, ShortConvAttentionConfig, WkvConfig
from ..transformer.moe import MixtureOfExperts
from ..transformer.norm import ParallelNorm
from ..transformer.short_conv_attention import ShortConvAttention
from ..transformer.wkv import Wkv
from .hybrid_model import HybridDecoder

MIXERS = {ShortConvAttentionConfig: ShortConvAttention, WkvConfig: Wkv, GatedDeltaConfig: GatedDelta}


class ParallelLayer(torch.nn.Module):
    def __init__(self, config: HybridConfig, index: int):
        super().__init__()
        layer = config.layers[index]
        self.moe = MixtureOfExperts(config, layer.moe) if layer.moe is not None else None
        self.norm = ParallelNorm(config, config.hidden_size, config.layernorm_epsilon, outputs=1 if self.moe is None else 2)
        self.mixer = MIXERS[type(layer.mixer)](config, layer.mixer, index)

    def forward(self, hidden, pending: ops.PendingRows, ctx, step: dict) -> ops.PendingRows:
        """Adds what the layer before left to the stream and runs both branches.  (The mixer comes last: its output linear leaves
        partial sums that the next GEMM would overwrite.)"""
        normed = self.norm(hidden, pending)
        experts = self.moe(normed[1]) if self.moe is not None else None
        return ops.PendingRows(partials=self.mixer(normed[0], ctx, step), experts=experts)


class ParallelHybridModel(HybridDecoder):
    def __init__(self, config: HybridConfig, max_sequence_length: int):
        super().__init__(config, max_sequence_length)
        self.word_embeddings = VocabParallelEmbedding(config.vocab_size, config.hidden_size, config=config)
        self.layers = torch.nn.ModuleList(ParallelLayer(config, i) for i in range(config.num_layers))
        self.final_norm = ParallelNorm(config, config.hidden_size, config.layernorm_epsilon, outputs=1, out_scale=config.logit_scale)
        self.output_layer = ColumnParallelLinear(config.hidden_size, config.vocab_size, config=config, bias=False)

    def prefill_unit_tokens(self) -> list:
        """Tokens per work unit of the prompt attention kernel, one size per head grouping."""
        sizes = {layer.mixer.prefill_unit_tokens() for layer in self.layers if isinstance(layer.mixer, ShortConvAttention)} - {0}
        return sorted(sizes, reverse=True) or [0]

    # ------------------------------------------------------------------------------------------
    def forward_rows(self, input_ids, position_ids, inference_context, row_indices=None,
                     runtime_gather_output: Optional[bool] = None, streams: Optional[list] = None):
        """Logits ``[rows, vocab]`` of every token, or of the rows in ``row_indices`` (int64, on the device).  ``streams``
        (a list) receives a copy of the residual stream after every layer."""
        ids = input_ids.reshape(-1)
        hidden = torch.empty((ids.numel(), self.config.hidden_size), dtype=torch.float32, device=ids.device)
        pending = ops.PendingRows(table=self.word_embeddings.weight, ids=ids, table_scale=self.config.embedding_scale)
        step = {}
        for layer in self.layers:
            pending = layer(hidden, pending, inference_context, step)
            if streams is not None:
                ops.residual_norm(hidden, pending, [], [], eps=1.0)
                pending = None
                streams.append(hidden.clone())
        logits, _ = self.output_layer(self.final_norm(hidden, pending, row_indices)[0])
        return logits

    # ------------------------------------------------------------------------------------------
    def checkpoint_tensors(self) -> Dict[str, tuple]:
        c = self.config
        out = {"embed": (c.vocab_size, c.hidden_size), "head": (c.vocab_size, c.hidden_size), "final.norm": (c.hidden_size,)}
        for i, layer in enumerate(self.layers):
            out[f"l{i}.norm1"] = (c.hidden_size,)
            out.update({f"l{i}.mix.{k}": s for k, s in layer.mixer.checkpoint_tensors().items()})
            if layer.moe is not None:
                out[f"l{i}.norm2"] = (c.hidden_size,)
                out.update({f"l{i}.mlp.{k}": s for k, s in layer.moe.checkpoint_tensors().items()})
        return out

    def ignored_tensors(self) -> set:
        out = set()
        for i, layer in enumerate(self.layers):
            out |= {f"l{i}.mix.{k}" for k in getattr(layer.mixer, "ignored_tensors", set)()}
            if layer.moe is None:
                out.add(f"l{i}.norm2")
        return out

    def _load(self, tensors: Dict[str, torch.Tensor]) -> None:
        def get(prefix):
            return lambda name: tensors[prefix + name].to(self.config.params_dtype)

        top = get("")
        self.word_embeddings.weight.data.copy_(top("embed"))
        self.output_layer.weight.data.copy_(top("head"))
        self.final_norm.weight.data[0].copy_(top("final.norm"))
        for i, layer in enumerate(self.layers):
            layer.norm.weight.data[0].copy_(top(f"l{i}.norm1"))
            layer.mixer.load(get(f"l{i}.mix."))
            if layer.moe is not None:
                layer.norm.weight.data[1].copy_(top(f"l{i}.norm2"))
                layer.moe.load(get(f"l{i}.mlp."))

    def synthetic_tensor(self, name: str, shape: tuple, seed: int, std: float, device) -> torch.Tensor:
        """Layer norms are stored around zero here; only the heads' norms lie around one."""
        t = super().synthetic_tensor(name, shape, seed, std, device)
        return t - 1.0 if name.rsplit(".", 1)[-1] in ("norm1", "norm2") or name == "final.norm" else t
