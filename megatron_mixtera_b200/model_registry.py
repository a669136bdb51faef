"""Model classes by the ``architecture`` of a model folder (``config.json`` + ``model.safetensors``), and the serving stack
around a loaded model."""
from __future__ import annotations

import json
import os
from typing import Callable, Dict, Tuple

import torch

from . import checkpoint
from .transformer.hybrid_config import (ChosenSoftmaxRouting, DeltaRuleConfig, DistanceBias, ExpertConfig, GatedDeltaConfig, GatedScanConfig,
                                        GroupedAttentionConfig, HybridConfig, HybridLayerConfig, LatentAttentionConfig, MatrixMemoryConfig,
                                        MoeConfig, RotaryConfig, ShortConvAttentionConfig, SideBySideConfig, SoftmaxRouting, WkvConfig,
                                        YarnScaling)
from .transformer.transformer_config import TransformerConfig


# ---------------------------------------------------------------------------------------------------------------------
# Zinurax
# ---------------------------------------------------------------------------------------------------------------------
def _rotary(rot: dict, halves: bool = False) -> RotaryConfig:
    scaling = rot.get("scaling")
    return RotaryConfig(base=float(rot["base"]), dims=rot["dims"], halves=halves,
                        scaling=YarnScaling(**{k: float(scaling[k]) for k in ("factor", "original", "fast", "slow")}) if scaling else None)


def _latent_attention_config(m: dict) -> LatentAttentionConfig:
    return LatentAttentionConfig(
        heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], vdim=m["vdim"], kv_rank=m["kv_rank"], scale=float(m["scale"]),
        rot=_rotary(m["rot"]), window=(m.get("mask") or {}).get("size"), kv_from=m.get("kv_from"))


def zinurax_config(config: dict, shapes: Dict[str, tuple], dtype: torch.dtype) -> HybridConfig:
    """``config.json`` -> `HybridConfig`; ``shapes`` (checkpoint tensor -> shape) gives what the file leaves to the tensors."""
    layers = []
    for i, layer in enumerate(config["layers"]):
        m, mlp = layer["mixer"], layer.get("mlp")
        if layer["type"] == "latent_attention":
            mixer = _latent_attention_config(m)
        elif layer["type"] == "general_delta":
            mixer = DeltaRuleConfig(heads=m["heads"], dim=m["dim"], rank=shapes[f"l{i}.mix.w1"][0])
        else:
            raise ValueError(f"layer {i}: unknown mixer {layer['type']!r}")
        if mlp is not None and mlp["kind"] != "dense":
            raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
        layers.append(HybridLayerConfig(mixer=mixer, ffn_hidden_size=None if mlp is None else mlp["ff"]))
    return HybridConfig(vocab_size=config["vocab"], hidden_size=config["width"], layers=tuple(layers),
                        layernorm_epsilon=float(config["norm"]["eps"]), params_dtype=dtype)


def _build_zinurax(config: dict, shapes: Dict[str, tuple], dtype: torch.dtype, max_sequence_length: int):
    from .hybrid.hybrid_model import HybridModel

    return HybridModel(zinurax_config(config, shapes, dtype), max_sequence_length)


# ---------------------------------------------------------------------------------------------------------------------
# Fabivik
# ---------------------------------------------------------------------------------------------------------------------
def _expert(e: dict) -> ExpertConfig:
    return ExpertConfig(ff=e["ff"], limit=float(e["limit"]))


def fabivik_config(config: dict, shapes: Dict[str, tuple], dtype: torch.dtype) -> HybridConfig:
    """``config.json`` -> `HybridConfig`; ``shapes`` (checkpoint tensor -> shape) gives what the file leaves to the tensors."""
    layers = []
    for i, layer in enumerate(config["layers"]):
        m, mlp = layer["mixer"], layer.get("mlp")
        if layer["type"] == "attention":
            mixer = ShortConvAttentionConfig(
                heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], scale=float(m["scale"]), conv=m["conv"],
                window=(m.get("mask") or {}).get("size"), value_mix=bool(m.get("v_mix", False)))
        elif layer["type"] == "wkv":
            mixer = WkvConfig(heads=m["heads"], dim=m["dim"], rank=shapes[f"l{i}.mix.w1"][0])
        elif layer["type"] == "delta":
            mixer = GatedDeltaConfig(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], conv=m["conv"])
        else:
            raise ValueError(f"layer {i}: unknown mixer {layer['type']!r}")
        moe = None
        if mlp is not None:
            if mlp["kind"] != "moe":
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            moe = MoeConfig(experts=mlp["router"]["experts"], top=mlp["router"]["top"], expert=_expert(mlp["expert"]),
                            shared=_expert(mlp["shared"]) if mlp.get("shared") else None)
        layers.append(HybridLayerConfig(mixer=mixer, moe=moe))
    return HybridConfig(vocab_size=config["vocab"], hidden_size=config["width"], layers=tuple(layers), block="parallel",
                        layernorm_epsilon=float(config["norm"]["eps"]), params_dtype=dtype,
                        embedding_scale=float(config["embedding"]["scale"]), logit_scale=float(config["logit_scale"]))


def _build_fabivik(config: dict, shapes: Dict[str, tuple], dtype: torch.dtype, max_sequence_length: int):
    from .hybrid.parallel_model import ParallelHybridModel

    return ParallelHybridModel(fabivik_config(config, shapes, dtype), max_sequence_length)


# ---------------------------------------------------------------------------------------------------------------------
# Lukarax
# ---------------------------------------------------------------------------------------------------------------------
def _grouped(m: dict, **kwargs) -> GroupedAttentionConfig:
    mask = m.get("mask") or {}
    return GroupedAttentionConfig(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], scale=float(m["scale"]),
                                  window=mask.get("size"), keep_first=mask.get("keep_first") or 0, **kwargs)


def lukarax_config(config: dict, shapes: Dict[str, tuple], dtype: torch.dtype) -> HybridConfig:
    """``config.json`` -> `HybridConfig`; ``shapes`` (checkpoint tensor -> shape) gives what the file leaves to the tensors."""
    layers = []
    for i, layer in enumerate(config["layers"]):
        m, mlp = layer["mixer"], layer.get("mlp")
        if layer["type"] == "attention":
            mixer = _grouped(m, rot=_rotary(m["rot"]), diff=float(m["diff"]), gate=True, kv_from=m.get("kv_from"))
        elif layer["type"] == "attention_2":
            mixer = _grouped(m, rot=_rotary(m["rot"], halves=True), unit_queries_keys=True, values_from_keys=True, biases=True, sink=True,
                             softcap=float(m["softcap"]) if m.get("softcap") else None)
        elif layer["type"] == "parallel":
            left, right = m["left"], m["right"]
            bias = DistanceBias(rows=shapes[f"l{i}.mix.left.rel"][0], longest=float(left["bias_max"]))
            memory = MatrixMemoryConfig(heads=right["heads"], dim=right["dim"], vdim=right["vdim"], gate_cap=float(right["gate_cap"]))
            mixer = SideBySideConfig((("left", _grouped(left, distance_bias=bias), float(m["left_scale"])),
                                      ("right", memory, float(m["right_scale"]))))
        else:
            raise ValueError(f"layer {i}: unknown mixer {layer['type']!r}")
        ff = moe = None
        if mlp is not None and mlp["kind"] == "dense":
            ff = mlp["ff"]
        elif mlp is not None and mlp["kind"] == "moe":
            r = mlp["router"]
            groups = r.get("groups") or {"count": 1, "keep": 1}
            moe = MoeConfig(experts=r["experts"], top=r["top"], expert=ExpertConfig(ff=mlp["expert"]["ff"]),
                            routing=SoftmaxRouting(identity=r.get("identity") or 0, groups=groups["count"], keep_groups=groups["keep"],
                                                   scale=float(r["scale"])))
        elif mlp is not None:
            raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
        layers.append(HybridLayerConfig(mixer=mixer, ffn_hidden_size=ff, moe=moe))
    return HybridConfig(vocab_size=config["vocab"], hidden_size=config["width"], layers=tuple(layers), block="streams",
                        streams=config.get("streams") or 0, gated_linear_unit=True, activation="silu",
                        layernorm_epsilon=float(config["norm"]["eps"]), params_dtype=dtype,
                        embedding_scale=float(config["embedding"]["scale"]))


def _build_lukarax(config: dict, shapes: Dict[str, tuple], dtype: torch.dtype, max_sequence_length: int):
    from .hybrid.stream_model import StreamHybridModel

    return StreamHybridModel(lukarax_config(config, shapes, dtype), max_sequence_length)


# ---------------------------------------------------------------------------------------------------------------------
# Maginex
# ---------------------------------------------------------------------------------------------------------------------
def maginex_config(config: dict, shapes: Dict[str, tuple], dtype: torch.dtype) -> HybridConfig:
    """``config.json`` -> `HybridConfig`."""
    layers = []
    for i, layer in enumerate(config["layers"]):
        m, mlp = layer["mixer"], layer.get("mlp")
        if layer["type"] == "latent_attention":
            mixer = LatentAttentionConfig(heads=m["heads"], dim=m["dim"], rot_dim=0, vdim=m["vdim"], kv_rank=m["kv_rank"], q_rank=m["q_rank"],
                                          scale=float(m["scale"]), sink=True, gate="value")
        elif layer["type"] == "mingru":
            mixer = GatedScanConfig(width=m["width"])
        elif layer["type"] == "attention":
            mixer = _grouped(m, rot=_rotary(m["rot"], halves=True) if m.get("rot") else None, sink=True, head_gate=True,
                             value_mix=bool(m.get("v_mix", False)))
        else:
            raise ValueError(f"layer {i}: unknown mixer {layer['type']!r}")
        moe = None
        if mlp is not None:
            if mlp["kind"] != "moe":
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            shared = mlp.get("shared")
            moe = MoeConfig(experts=mlp["router"]["experts"], top=mlp["router"]["top"], expert=ExpertConfig(ff=mlp["expert"]["ff"], gated=False),
                            shared=ExpertConfig(ff=shared["ff"], gated=False) if shared else None, routing=ChosenSoftmaxRouting())
        layers.append(HybridLayerConfig(mixer=mixer, moe=moe))
    return HybridConfig(vocab_size=config["vocab"], hidden_size=config["width"], layers=tuple(layers), block="parallel",
                        layernorm_epsilon=float(config["norm"]["eps"]), params_dtype=dtype, norm_offset=0.0, input_taps=config["canon"]["taps"],
                        embedding_scale=float(config["embedding"]["scale"]))


def _build_maginex(config: dict, shapes: Dict[str, tuple], dtype: torch.dtype, max_sequence_length: int):
    from .hybrid.parallel_model import ParallelHybridModel

    return ParallelHybridModel(maginex_config(config, shapes, dtype), max_sequence_length)


# ---------------------------------------------------------------------------------------------------------------------
# GPTModel: config.json holds TransformerConfig fields under "transformer" and the model's own beside it
# ---------------------------------------------------------------------------------------------------------------------
def _build_gpt(config: dict, shapes: Dict[str, tuple], dtype: torch.dtype, max_sequence_length: int):
    from .gpt.gpt_model import GPTModel

    return GPTModel(TransformerConfig(params_dtype=dtype, **config["transformer"]), vocab_size=config["vocab_size"],
                    max_sequence_length=max_sequence_length,
                    position_embedding_type=config.get("position_embedding_type", "rope"),
                    rotary_base=config.get("rotary_base", 10000.0),
                    share_embeddings_and_output_weights=config.get("share_embeddings_and_output_weights", False))


Builder = Callable[[dict, Dict[str, tuple], torch.dtype, int], torch.nn.Module]
ARCHITECTURES: Dict[str, Builder] = {"Fabivik": _build_fabivik, "Lukarax": _build_lukarax, "Maginex": _build_maginex, "Zinurax": _build_zinurax,
                                     "GPTModel": _build_gpt}


def load_model(folder: str, *, dtype: torch.dtype = torch.bfloat16, max_sequence_length: int) -> torch.nn.Module:
    """The model of a folder, weights loaded, on the current device."""
    with open(os.path.join(folder, "config.json")) as f:
        config = json.load(f)
    name = config.get("architecture")
    if name not in ARCHITECTURES:
        raise ValueError(f"unknown architecture {name!r} (known: {', '.join(sorted(ARCHITECTURES))})")
    path = os.path.join(folder, "model.safetensors")
    model = ARCHITECTURES[name](config, checkpoint.tensor_shapes(path), dtype, max_sequence_length)
    tensors = checkpoint.load_safetensors(path)
    if hasattr(model, "load_checkpoint"):
        model.load_checkpoint(tensors)
    else:
        model.load_full_state_dict(tensors)
    return model


def make_context(model, *, max_cached_tokens: int, max_requests: int, max_step_tokens: int, chunk_size_tokens: int = 64, **kwargs):
    """A dynamic context whose pool holds ``max_cached_tokens`` (whole chunks), for ``max_requests`` live requests and steps of
    up to ``max_step_tokens`` tokens."""
    kwargs = dict(max_requests_override=max_requests, max_tokens_override=max_step_tokens, **kwargs)
    if hasattr(model, "make_context"):
        return model.make_context(max_cached_tokens=max_cached_tokens, chunk_size_tokens=chunk_size_tokens, **kwargs)
    from .inference.contexts.dynamic_context import DynamicInferenceContext

    c = model.config
    chunk_bytes = c.params_dtype.itemsize * 2 * c.num_layers * chunk_size_tokens * c.num_query_groups * c.kv_channels
    chunks = -(-max_cached_tokens // chunk_size_tokens) + 1
    return DynamicInferenceContext(
        params_dtype=c.params_dtype, num_layers=c.num_layers, kv_channels=c.kv_channels, num_attention_heads=c.num_query_groups,
        max_sequence_length=model.max_sequence_length, buffer_size_gb=(chunks + 0.5) * chunk_bytes / 1024**3,
        chunk_size_tokens=chunk_size_tokens, **{"buffer_guaranteed_fraction": 0.0, **kwargs})


def make_controller(model, context, tokenizer=None):
    """Wrapper and controller around a model and its context."""
    from .inference.model_inference_wrappers.gpt_inference_wrapper import GPTInferenceWrapper, InferenceWrapperConfig
    from .inference.text_generation_controllers.text_generation_controller import TextGenerationController

    cfg = InferenceWrapperConfig(hidden_size=model.config.hidden_size, params_dtype=model.config.params_dtype,
                                 padded_vocab_size=model.vocab_size)
    return TextGenerationController(GPTInferenceWrapper(model, cfg, context), tokenizer)


def serving_stack(folder: str, *, dtype: torch.dtype, max_cached_tokens: int, max_requests: int, max_sequence_length: int,
                  max_step_tokens: int, **context_kwargs) -> Tuple[torch.nn.Module, object, object]:
    """(model, context, controller) of a model folder."""
    model = load_model(folder, dtype=dtype, max_sequence_length=max_sequence_length)
    context = make_context(model, max_cached_tokens=max_cached_tokens, max_requests=max_requests, max_step_tokens=max_step_tokens,
                           **context_kwargs)
    return model, context, make_controller(model, context)
