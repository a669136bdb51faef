"""Hybrid decoder of parallel blocks on a 32-bit residual stream, with scaled embeddings and an output head of its own:
x += mixer(norm1(x)) + experts(norm2(x)), or (``input_taps``) x += mixer(filter1(norm(x))) + experts(filter2(norm(x))).  Mixers come in any
order: windowed attention with short convolutions, wkv time mixing, the gated delta rule, latent attention, grouped-query attention in its
forms, a gated scan.

One kernel per block joins everything the block adds to the stream with the norms the next block starts with."""
from __future__ import annotations

from typing import Dict, Optional

import torch

from .. import ops
from ..tensor_parallel.layers import ColumnParallelLinear, VocabParallelEmbedding
from ..transformer.gated_delta import GatedDelta
from ..transformer.hybrid_config import GatedDeltaConfig, HybridConfig, LatentAttentionConfig, ShortConvAttentionConfig, WkvConfig
from ..transformer.joined_mixer import PARTS, JoinedMixer
from ..transformer.latent_attention import LatentAttention
from ..transformer.moe import MixtureOfExperts
from ..transformer.norm import FilteredNorm, ParallelNorm
from ..transformer.rotary import rotary_tables
from ..transformer.short_conv_attention import ShortConvAttention
from ..transformer.short_conv import filter_of
from ..transformer.wkv import Wkv
from .hybrid_model import HybridDecoder

MIXERS = {ShortConvAttentionConfig: ShortConvAttention, WkvConfig: Wkv, GatedDeltaConfig: GatedDelta, LatentAttentionConfig: LatentAttention,
          **{c: JoinedMixer for c in PARTS}}


class ParallelLayer(torch.nn.Module):
    def __init__(self, config: HybridConfig, index: int):
        super().__init__()
        layer = config.layers[index]
        self.moe = MixtureOfExperts(config, layer.moe) if layer.moe is not None else None
        outputs = 1 if self.moe is None else 2
        self.filtered = config.input_taps > 0
        if self.filtered:
            self.norm = FilteredNorm(config, config.hidden_size, config.layernorm_epsilon, outputs, index + 1)
        else:
            self.norm = ParallelNorm(config, config.hidden_size, config.layernorm_epsilon, outputs=outputs)
        self.mixer = MIXERS[type(layer.mixer)](config, layer.mixer, index)

    def forward(self, hidden, pending: ops.PendingRows, ctx, rope, step: dict) -> ops.PendingRows:
        """Adds what the layer before left to the stream and runs both branches.  (The mixer comes last: its output linear leaves
        partial sums that the next GEMM would overwrite.)"""
        normed = self.norm(hidden, pending, ctx) if self.filtered else self.norm(hidden, pending)
        experts = self.moe(normed[1]) if self.moe is not None else None
        return ops.PendingRows(partials=self.mixer(normed[0], ctx, rope, step), experts=experts)


class ParallelHybridModel(HybridDecoder):
    def __init__(self, config: HybridConfig, max_sequence_length: int):
        super().__init__(config, max_sequence_length)
        self.word_embeddings = VocabParallelEmbedding(config.vocab_size, config.hidden_size, config=config)
        self.layers = torch.nn.ModuleList(ParallelLayer(config, i) for i in range(config.num_layers))
        self.final_norm = ParallelNorm(config, config.hidden_size, config.layernorm_epsilon, outputs=1, out_scale=config.logit_scale)
        self.output_layer = ColumnParallelLinear(config.hidden_size, config.vocab_size, config=config, bias=False)
        tables = {}
        self._rope = []  # per layer (joined mixers: per part)
        for layer in self.layers:
            rots = [getattr(m, "rot", None) for m in ([p.mixer for p in layer.mixer.parts] if isinstance(layer.mixer, JoinedMixer) else [layer.mixer.mixer])]
            for rot in rots:
                if rot is not None and rot not in tables:
                    tables[rot] = rotary_tables(rot, max_sequence_length, self.word_embeddings.weight.device)
            found = [tables.get(rot) for rot in rots]
            self._rope.append(found if isinstance(layer.mixer, JoinedMixer) else found[0])

    def prefill_unit_tokens(self) -> list:
        """Tokens per work unit of the prompt attention kernels, one size per head grouping."""
        sizes = set()
        for layer in self.layers:
            of_layer = getattr(layer.mixer, "prefill_unit_tokens", set)()
            sizes |= of_layer if isinstance(of_layer, set) else {of_layer}
        return sorted(sizes - {0}, reverse=True) or [0]

    # ------------------------------------------------------------------------------------------
    def forward_rows(self, input_ids, position_ids, inference_context, row_indices=None,
                     runtime_gather_output: Optional[bool] = None, streams: Optional[list] = None):
        """Logits ``[rows, vocab]`` of every token, or of the rows in ``row_indices`` (int64, on the device).  ``streams``
        (a list) receives a copy of the residual stream after every layer."""
        ids = input_ids.reshape(-1)
        hidden = torch.empty((ids.numel(), self.config.hidden_size), dtype=torch.float32, device=ids.device)
        pending = ops.PendingRows(table=self.word_embeddings.weight, ids=ids, table_scale=self.config.embedding_scale)
        step = {}
        for layer, rope in zip(self.layers, self._rope):
            pending = layer(hidden, pending, inference_context, rope, step)
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
            if layer.filtered:
                out.update({f"l{i}.canon{n + 1}": (c.hidden_size, c.input_taps) for n in range(layer.norm.filters.shape[0])})
            if layer.moe is not None:
                if not layer.filtered:
                    out[f"l{i}.norm2"] = (c.hidden_size,)
                out.update({f"l{i}.mlp.{k}": s for k, s in layer.moe.checkpoint_tensors().items()})
        return out

    def ignored_tensors(self) -> set:
        out = set()
        for i, layer in enumerate(self.layers):
            out |= {f"l{i}.mix.{k}" for k in getattr(layer.mixer, "ignored_tensors", set)()}
            if layer.moe is None:
                out.add(f"l{i}.canon2" if layer.filtered else f"l{i}.norm2")
        return out

    def _load(self, tensors: Dict[str, torch.Tensor]) -> None:
        def get(prefix):
            return lambda name: tensors[prefix + name].to(self.config.params_dtype)

        top = get("")
        self.word_embeddings.weight.data.copy_(top("embed"))
        self.output_layer.weight.data.copy_(top("head"))
        self.final_norm.weight.data[0].copy_(top("final.norm"))
        for i, layer in enumerate(self.layers):
            if layer.filtered:
                layer.norm.weight.data.copy_(top(f"l{i}.norm1"))
                for n in range(layer.norm.filters.shape[0]):
                    layer.norm.filters.data[n].copy_(filter_of(top(f"l{i}.canon{n + 1}")))
            else:
                layer.norm.weight.data[0].copy_(top(f"l{i}.norm1"))
            layer.mixer.load(get(f"l{i}.mix."))
            if layer.moe is not None:
                if not layer.filtered:
                    layer.norm.weight.data[1].copy_(top(f"l{i}.norm2"))
                layer.moe.load(get(f"l{i}.mlp."))

    def synthetic_tensor(self, name: str, shape: tuple, seed: int, std: float, device) -> torch.Tensor:
        """Layer norms lie around one after ``norm_offset`` is added; the heads' and latents' norms always do."""
        t = super().synthetic_tensor(name, shape, seed, std, device)
        return t - self.config.norm_offset if name.rsplit(".", 1)[-1] in ("norm1", "norm2") or name == "final.norm" else t
