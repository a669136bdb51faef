"""Hybrid decoders for the dynamic inference path, with the same calls as `GPTModel` (`forward`, `forward_rows`).

`HybridDecoder`: what they share - the context made for their layers, strict checkpoint loading, synthetic weights.
`HybridModel`: layers of latent attention or the generalized delta rule with norms on the sublayers' outputs, a 32-bit residual
stream and tied embeddings.  (`ParallelHybridModel` is in parallel_model.py.)"""
from __future__ import annotations

from typing import Dict, Optional

import torch

from ..gpt.gpt_model import DynamicForward
from ..inference.contexts.dynamic_context import DynamicInferenceContext
from ..synthetic import canonical_tensor
from ..tensor_parallel.layers import ColumnParallelLinear, RowParallelLinear, VocabParallelEmbedding
from ..transformer.delta_rule import GeneralDeltaRule
from ..transformer.hybrid_config import DeltaRuleConfig, HybridConfig, LatentAttentionConfig
from ..transformer.latent_attention import LatentAttention
from ..transformer.mlp import MLP, MLPSubmodules
from ..transformer.norm import OutputNorm
from ..transformer.rotary import rotary_tables

MIXERS = {LatentAttentionConfig: LatentAttention, DeltaRuleConfig: GeneralDeltaRule}


class HybridLayer(torch.nn.Module):
    """x += norm1(mixer(x)); x += norm2(mlp(x))."""

    def __init__(self, config: HybridConfig, index: int):
        super().__init__()
        layer = config.layers[index]
        kw = dict(config=config, hidden_size=config.hidden_size, eps=config.layernorm_epsilon)
        self.mixer = MIXERS[type(layer.mixer)](config, layer.mixer, index)
        self.mixer_norm = OutputNorm(**kw)
        self.mlp = self.mlp_norm = None
        if layer.ffn_hidden_size is not None:
            self.mlp = MLP(config.for_layer(index), MLPSubmodules(linear_fc1=ColumnParallelLinear, linear_fc2=RowParallelLinear))
            self.mlp_norm = OutputNorm(**kw)

    def forward(self, x, hidden, ctx, rope):
        """``hidden``: the fp32 stream, updated in place; ``x``: its copy in the activation type.  Returns the next copy."""
        x = self.mixer_norm.add_to_stream(hidden, self.mixer(x, ctx, rope))
        if self.mlp is not None:
            x = self.mlp_norm.add_to_stream(hidden, self.mlp(x, defer_output_reduction=True)[0])
        return x


class HybridDecoder(DynamicForward, torch.nn.Module):
    def __init__(self, config: HybridConfig, max_sequence_length: int):
        super().__init__()
        self.config, self.vocab_size, self.max_sequence_length = config, config.vocab_size, max_sequence_length

    def make_context(self, *, buffer_size_gb: Optional[float] = None, max_cached_tokens: Optional[int] = None,
                     chunk_size_tokens: int = 64, **kwargs) -> DynamicInferenceContext:
        """A context with the token rows and the state this model's layers keep.  The pool is given in GB, or as the number of
        tokens it must hold (in whole chunks; one more chunk takes the padding tokens' writes)."""
        c = self.config
        widths = [layer.mixer.cached_row_width() for layer in c.layers]
        states = [c.request_state(i) for i in range(c.num_layers)]
        if max_cached_tokens is not None:
            chunks = -(-max_cached_tokens // chunk_size_tokens) + 1
            nbytes = DynamicInferenceContext.latent_chunk_bytes(widths, chunk_size_tokens, c.params_dtype)
            buffer_size_gb = (chunks + 0.5) * nbytes / 1024**3
        return DynamicInferenceContext(
            params_dtype=c.params_dtype, num_layers=c.num_layers, kv_channels=0, num_attention_heads=0,
            max_sequence_length=self.max_sequence_length, buffer_size_gb=buffer_size_gb, cache_mla_latent=True,
            latent_row_widths=widths, state_shapes=states, chunk_size_tokens=chunk_size_tokens,
            tensor_model_parallel_size=1, **{"buffer_guaranteed_fraction": 0.0, **kwargs})

    # ------------------------------------------------------------------------------------------
    def checkpoint_tensors(self) -> Dict[str, tuple]:
        """Checkpoint tensor name -> shape of everything this model loads."""
        raise NotImplementedError

    def ignored_tensors(self) -> set:
        """Names that a checkpoint may hold although nothing reads them."""
        return set()

    def _load(self, tensors: Dict[str, torch.Tensor]) -> None:
        raise NotImplementedError

    def load_checkpoint(self, tensors: Dict[str, torch.Tensor]) -> None:
        """Load checkpoint tensors (any float type; converted to the model's)."""
        want = self.checkpoint_tensors()
        for name, shape in want.items():
            if name not in tensors:
                raise KeyError(f"checkpoint tensor {name!r} is missing")
            if tuple(tensors[name].shape) != tuple(shape):
                raise ValueError(f"checkpoint tensor {name!r} has shape {tuple(tensors[name].shape)}, expected {tuple(shape)}")
        unknown = sorted(set(tensors) - set(want) - self.ignored_tensors())
        if unknown:
            raise KeyError(f"checkpoint tensors this model does not use: {unknown[:4]}")
        self._load(tensors)

    def synthetic_tensor(self, name: str, shape: tuple, seed: int, std: float, device) -> torch.Tensor:
        """Seeded N(0, std) values (norm scales 1 + N(0, std))."""
        t = canonical_tensor(name, shape, seed=seed, std=std, dtype=torch.float32, device=device)
        return t + 1.0 if name.rsplit(".", 1)[-1] in ("norm", "norm1", "norm2") else t

    def init_synthetic_weights(self, seed: int = 0, std: float = 0.02, device=None) -> None:
        dev = self.word_embeddings.weight.device if device is None else device
        self.load_checkpoint({n: self.synthetic_tensor(n, s, seed, std, dev) for n, s in self.checkpoint_tensors().items()})


class HybridModel(HybridDecoder):
    def __init__(self, config: HybridConfig, max_sequence_length: int):
        super().__init__(config, max_sequence_length)
        kw = dict(config=config, hidden_size=config.hidden_size, eps=config.layernorm_epsilon)
        self.word_embeddings = VocabParallelEmbedding(config.vocab_size, config.hidden_size, config=config)
        self.embedding_norm = OutputNorm(**kw)
        self.layers = torch.nn.ModuleList(HybridLayer(config, i) for i in range(config.num_layers))
        self.final_norm = OutputNorm(**kw)
        self.output_layer = ColumnParallelLinear(config.hidden_size, config.vocab_size, config=config, bias=False,
                                                 skip_weight_param_allocation=True)
        tables = {}
        self._rope = []
        for layer in config.layers:
            rot = getattr(layer.mixer, "rot", None)
            if rot is not None and rot not in tables:
                tables[rot] = rotary_tables(rot, max_sequence_length, self.word_embeddings.weight.device)
            self._rope.append(tables.get(rot))

    # ------------------------------------------------------------------------------------------
    def prefill_unit_tokens(self) -> int:
        """Tokens per work unit of the prompt attention kernel (it cuts a unit into blocks of query rows itself)."""
        return 16

    # ------------------------------------------------------------------------------------------
    def forward_rows(self, input_ids, position_ids, inference_context, row_indices=None,
                     runtime_gather_output: Optional[bool] = None, streams: Optional[list] = None):
        """Logits ``[rows, vocab]`` of every token, or of the rows in ``row_indices`` (int64, on the device).  ``streams``
        (a list) receives a copy of the residual stream after every layer."""
        hidden, x = self.embedding_norm.start_stream(self.word_embeddings.weight, input_ids.reshape(-1))
        for layer, rope in zip(self.layers, self._rope):
            x = layer(x, hidden, inference_context, rope)
            if streams is not None:
                streams.append(hidden.clone())
        logits, _ = self.output_layer(self.final_norm.of_rows(hidden, row_indices), weight=self.word_embeddings.weight)
        return logits

    # ------------------------------------------------------------------------------------------
    def checkpoint_tensors(self) -> Dict[str, tuple]:
        c = self.config
        out = {"embed": (c.vocab_size, c.hidden_size), "embed.norm": (c.hidden_size,), "final.norm": (c.hidden_size,)}
        for i, layer in enumerate(self.layers):
            out[f"l{i}.norm1"] = (c.hidden_size,)
            out.update({f"l{i}.mix.{k}": s for k, s in layer.mixer.checkpoint_tensors().items()})
            if layer.mlp is not None:
                ffn = c.layers[i].ffn_hidden_size
                out.update({f"l{i}.norm2": (c.hidden_size,), f"l{i}.mlp.up": (ffn, c.hidden_size), f"l{i}.mlp.down": (c.hidden_size, ffn)})
        return out

    def _load(self, tensors: Dict[str, torch.Tensor]) -> None:
        def put(param, name):
            param.data.copy_(tensors[name])

        put(self.word_embeddings.weight, "embed")
        put(self.embedding_norm.weight, "embed.norm")
        put(self.final_norm.weight, "final.norm")
        for i, layer in enumerate(self.layers):
            put(layer.mixer_norm.weight, f"l{i}.norm1")
            layer.mixer.load(lambda k, p=f"l{i}.mix.": tensors[p + k].to(self.config.params_dtype))
            if layer.mlp is not None:
                put(layer.mlp_norm.weight, f"l{i}.norm2")
                put(layer.mlp.linear_fc1.weight, f"l{i}.mlp.up")
                put(layer.mlp.linear_fc2.weight, f"l{i}.mlp.down")
