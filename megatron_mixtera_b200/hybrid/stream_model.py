"""Hybrid decoder with several residual streams: every sublayer reads a blend of the streams through a layer norm and writes its output, and a mix
of the streams, back into all of them.  Mixers are grouped-query attention in its forms, or attention and a matrix memory side by side; the
feed-forward is dense or a mixture of experts; scaled embeddings, tied head.

One kernel per sublayer does what the sublayer before left to the streams and the norm in front of the next one."""
from __future__ import annotations

from typing import Dict, Optional

import torch

from .. import ops
from ..tensor_parallel.layers import ColumnParallelLinear, RowParallelLinear, VocabParallelEmbedding
from ..transformer.hybrid_config import HybridConfig
from ..transformer.joined_mixer import JoinedMixer
from ..transformer.mlp import MLP, MLPSubmodules
from ..transformer.moe import MixtureOfExperts
from ..transformer.norm import StreamNorm
from ..transformer.rotary import rotary_tables
from .hybrid_model import HybridDecoder


class StreamLayer(torch.nn.Module):
    def __init__(self, config: HybridConfig, index: int):
        super().__init__()
        layer, self.index = config.layers[index], index
        norm = dict(config=config, hidden_size=config.hidden_size, eps=config.layernorm_epsilon, streams=max(config.streams, 1),
                    plain=config.streams == 0)
        self.norm1 = StreamNorm(**norm)
        self.mixer = JoinedMixer(config, layer.mixer, index)
        self.norm2 = self.mlp = self.moe = None
        if layer.moe is not None:
            self.moe = MixtureOfExperts(config, layer.moe)
        elif layer.ffn_hidden_size is not None:
            self.mlp = MLP(config.for_layer(index), MLPSubmodules(linear_fc1=ColumnParallelLinear, linear_fc2=RowParallelLinear))
        if self.mlp is not None or self.moe is not None:
            self.norm2 = StreamNorm(**norm)

    def forward(self, hidden, pending: ops.PendingStreams, ctx, rope) -> ops.PendingStreams:
        x = self.norm1(hidden, pending)
        pending = self.norm1.left_by(partials=self.mixer(x, ctx, rope), bias=self.mixer.output_bias)
        if self.norm2 is None:
            return pending
        x = self.norm2(hidden, pending)
        if self.moe is not None:
            return self.norm2.left_by(experts=self.moe(x))
        return self.norm2.left_by(partials=self.mlp(x, defer_output_reduction=True)[0])

    def checkpoint_tensors(self) -> Dict[str, tuple]:
        p = f"l{self.index}."
        out = self.norm1.checkpoint_tensors(p + "norm1", p + "hc1")
        out.update({p + "mix." + k: s for k, s in self.mixer.checkpoint_tensors().items()})
        if self.norm2 is not None:
            out.update(self.norm2.checkpoint_tensors(p + "norm2", p + "hc2"))
        if self.moe is not None:
            out.update({p + "mlp." + k: s for k, s in self.moe.checkpoint_tensors().items()})
        elif self.mlp is not None:
            H, F = self.mlp.linear_fc2.weight.shape
            out.update({p + "mlp.gate": (F, H), p + "mlp.up": (F, H), p + "mlp.down": (H, F)})
        return out

    def load(self, get) -> None:
        p = f"l{self.index}."
        self.norm1.load(get, p + "norm1", p + "hc1")
        self.mixer.load(lambda k: get(p + "mix." + k))
        if self.norm2 is not None:
            self.norm2.load(get, p + "norm2", p + "hc2")
        if self.moe is not None:
            self.moe.load(lambda k: get(p + "mlp." + k))
        elif self.mlp is not None:
            self.mlp.load_gated(*(get(p + "mlp." + k) for k in ("gate", "up", "down")))


class StreamHybridModel(HybridDecoder):
    def __init__(self, config: HybridConfig, max_sequence_length: int):
        super().__init__(config, max_sequence_length)
        self.streams = max(config.streams, 1)
        self.word_embeddings = VocabParallelEmbedding(config.vocab_size, config.hidden_size, config=config)
        self.layers = torch.nn.ModuleList(StreamLayer(config, i) for i in range(config.num_layers))
        self.final_norm = StreamNorm(config, config.hidden_size, config.layernorm_epsilon, self.streams, plain=True)
        self.output_layer = ColumnParallelLinear(config.hidden_size, config.vocab_size, config=config, bias=False,
                                                 skip_weight_param_allocation=True)
        tables = {}
        self._rope = []  # per layer, per part of its mixer
        for layer in self.layers:
            rots = [getattr(p.mixer, "rot", None) for p in layer.mixer.parts]
            for rot in rots:
                if rot is not None and rot not in tables:
                    tables[rot] = rotary_tables(rot, max_sequence_length, self.word_embeddings.weight.device)
            self._rope.append([tables.get(rot) for rot in rots])

    def prefill_unit_tokens(self) -> list:
        """Tokens per work unit of the prompt attention kernel, one size per head grouping."""
        sizes = set().union(*(layer.mixer.prefill_unit_tokens() for layer in self.layers)) - {0}
        return sorted(sizes, reverse=True) or [0]

    # ------------------------------------------------------------------------------------------
    def forward_rows(self, input_ids, position_ids, inference_context, row_indices=None,
                     runtime_gather_output: Optional[bool] = None, streams: Optional[list] = None):
        """Logits ``[rows, vocab]`` of every token, or of the rows in ``row_indices`` (int64, on the device).  ``streams``
        (a list) receives the sum of the residual streams after every layer."""
        ids = input_ids.reshape(-1)
        hidden = torch.empty((ids.numel(), self.streams, self.config.hidden_size), dtype=torch.float32, device=ids.device)
        pending = ops.PendingStreams(table=self.word_embeddings.weight, ids=ids, table_scale=self.config.embedding_scale)
        for layer, rope in zip(self.layers, self._rope):
            pending = layer(hidden, pending, inference_context, rope)
            if streams is not None:
                ops.stream_norm(hidden, pending)
                pending = None
                streams.append(hidden.sum(dim=1))
        logits, _ = self.output_layer(self.final_norm(hidden, pending, row_indices), weight=self.word_embeddings.weight)
        return logits

    # ------------------------------------------------------------------------------------------
    def checkpoint_tensors(self) -> Dict[str, tuple]:
        c = self.config
        out = {"embed": (c.vocab_size, c.hidden_size), **self.final_norm.checkpoint_tensors("final.norm", "")}
        for layer in self.layers:
            out.update(layer.checkpoint_tensors())
        return out

    def ignored_tensors(self) -> set:
        return {f"l{layer.index}.{k}" for layer in self.layers if layer.norm2 is None
                for k in ("norm2", "norm2.b", "hc2.in", "hc2.out", "hc2.mix")}

    def _load(self, tensors: Dict[str, torch.Tensor]) -> None:
        dev, dtype = self.word_embeddings.weight.device, self.config.params_dtype

        def get(name):
            return tensors[name].to(device=dev, dtype=dtype)

        self.word_embeddings.weight.data.copy_(get("embed"))
        self.final_norm.load(get, "final.norm", "")
        for layer in self.layers:
            layer.load(get)

    def synthetic_tensor(self, name: str, shape: tuple, seed: int, std: float, device) -> torch.Tensor:
        """The streams' weights lie around an ordinary residual sum, forget gates keep."""
        t = super().synthetic_tensor(name, shape, seed, std, device)
        last = name.rsplit(".", 1)[-1]
        if ".hc" in name:
            t = t + {"in": 1.0 / self.streams, "out": 1.0, "mix": torch.eye(self.streams, device=t.device)}[last]
        return t + 4.0 if name.endswith(".f.b") else t
