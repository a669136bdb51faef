"""`bench.py --design fabivik`: prefill and decode throughput of the Fabivik design at sizes that resemble a real model's layers,
beside the framework's closest model (`GPTModel`: RMSNorm, rotary, grouped queries, SwiGLU, bf16) at equal width, layer count,
feed-forward weights per token, batch and context.  Same method as bench_zinurax.py: whole-model forwards, then every launch of one
step timed alone.  Synthetic weights and tokens; one GPU; one JSON line."""
from __future__ import annotations

import math

import torch

from bench_zinurax import FP32_FLOPS, PROMPT_LEN, PROMPTS, VOCAB, costs as zinurax_costs, measure

SIZES = {
    # attention heads / kv heads x dim / vdim, wkv heads x dim and decay rank, delta heads / kv heads x dim / vdim, experts
    "2k": dict(width=2048, layers=8, heads=16, kv_groups=8, dim=128, vdim=128, w_heads=32, w_dim=64, rank=64, d_heads=16, d_kv=8,
               d_dim=128, d_vdim=128, experts=32, top=4, ff=512, shared_ff=1024, gpt_ff=3072),
    "4k": dict(width=4096, layers=8, heads=32, kv_groups=8, dim=128, vdim=128, w_heads=64, w_dim=64, rank=128, d_heads=32, d_kv=16,
               d_dim=128, d_vdim=128, experts=64, top=8, ff=1024, shared_ff=2048, gpt_ff=10240),
    "4k_d64": dict(width=4096, layers=8, heads=64, kv_groups=8, dim=64, vdim=128, w_heads=32, w_dim=128, rank=96, d_heads=32, d_kv=32,
                   d_dim=64, d_vdim=64, experts=16, top=2, ff=4096, shared_ff=0, gpt_ff=8192),
}


def build_fabivik(s, max_len, tokens, requests, window):
    from megatron_mixtera_b200 import model_registry as R
    from megatron_mixtera_b200.hybrid.parallel_model import ParallelHybridModel
    from megatron_mixtera_b200.transformer import hybrid_config as C

    moe = C.MoeConfig(experts=s["experts"], top=s["top"], expert=C.ExpertConfig(s["ff"], 7.0),
                      shared=C.ExpertConfig(s["shared_ff"], 7.0) if s["shared_ff"] else None)
    attention = C.ShortConvAttentionConfig(heads=s["heads"], kv_heads=s["kv_groups"], dim=s["dim"], vdim=s["vdim"],
                                           scale=1.0 / math.sqrt(s["dim"]), conv=4, window=window, value_mix=True)
    wkv = C.WkvConfig(heads=s["w_heads"], dim=s["w_dim"], rank=s["rank"])
    delta = C.GatedDeltaConfig(heads=s["d_heads"], kv_heads=s["d_kv"], dim=s["d_dim"], vdim=s["d_vdim"], conv=4)
    layers = [C.HybridLayerConfig(mixer=(attention, wkv, attention, delta)[i % 4], moe=moe) for i in range(s["layers"])]
    model = ParallelHybridModel(C.HybridConfig(vocab_size=VOCAB, hidden_size=s["width"], layers=tuple(layers), block="parallel",
                                               embedding_scale=math.sqrt(s["width"])), max_len)
    model.init_synthetic_weights(seed=0)
    ctx = R.make_context(model, max_cached_tokens=tokens, max_requests=requests, max_step_tokens=max(PROMPTS * PROMPT_LEN, requests),
                         chunk_size_tokens=256)
    for b in ctx.latent_buffers:
        if b is not None:
            b.normal_(0.0, 0.5)
    return model, ctx, R.make_controller(model, ctx).inference_wrapped_model


def costs(s, T, visible_pairs, keys, design, decode, requests):
    """(bytes, flops, fp32 flops) per launch of the non-GEMM kernels."""
    if not design:
        return zinurax_costs(s, T, visible_pairs, keys, False, decode, requests)
    W, pairs = s["width"], T * s["top"]
    out = {"residual_norm": (T * W * (8.0 + 4 + 2 * s["top"] + (2 if s["shared_ff"] else 0) + 4), 0, 0)}
    H, G, d, v = s["heads"], s["kv_groups"], s["dim"], s["vdim"]
    channels = (H + G) * d + G * v
    out["conv_qkv"] = (4.0 * T * channels + (12.0 * requests * channels if decode else 0), 0, 0)
    io = 2.0 * T * H * (d + v)
    for k in ("paged_attention", "paged_prefill_attention"):
        out[k] = (2.0 * keys * G * (d + v) + io, 2.0 * visible_pairs * H * (d + v), 0)
    out["token_shift"] = (2.0 * T * W * 6, 0, 0)
    n, wd = s["w_heads"] * s["w_dim"], s["w_dim"]
    state = 8.0 * requests * n * wd
    out["recurrence_lora"] = (6.0 * T * s["rank"], 0, 0)
    out["wkv_decode"] = (state + 2.0 * T * n * 5 + 2.0 * n * s["rank"], 0, 6.0 * T * n * wd)
    out["wkv_scan"] = (state + T * n * (6.0 + 4 + 4), 0, 6.0 * T * n * wd)
    out["wkv_finish"] = (8.0 * T * n, 0, 0)
    dk, dv, nh = s["d_dim"], s["d_vdim"], s["d_heads"]
    dc = 2 * s["d_kv"] * dk + nh * dv
    state = 8.0 * requests * nh * dk * dv
    out["conv_silu"] = (4.0 * T * dc, 0, 0)
    out["delta_decode"] = (state + requests * dc * (2.0 + 12) + 4.0 * T * nh * dv, 0, 8.0 * T * nh * dk * dv)
    out["delta_scan"] = (state + 2.0 * T * dc + 4.0 * T * nh * dv, 0, 8.0 * T * nh * dk * dv)
    out["delta_finish"] = (8.0 * T * nh * dv, 0, 0)
    used, f, sf = min(s["experts"], pairs), s["ff"], s["shared_ff"]
    out["moe_route"] = (4.0 * T * (s["experts"] + 1), 0, 0)
    out["moe_gather"] = (2.0 * (T + pairs) * W, 0, 0)
    out["moe_up"] = (2.0 * (used * 2 * f * W + 2 * sf * W + (pairs + (T if sf else 0)) * W + pairs * f + T * sf), 4.0 * W * (pairs * f + T * sf), 0)
    out["moe_down"] = (2.0 * (used * f * W + sf * W + pairs * (f + W) + (T * (sf + W) if sf else 0)), 2.0 * W * (pairs * f + T * sf), 0)
    return out


def run(args, emit, peaks):
    from megatron_mixtera_b200 import build, ops

    build.build_torch_ops()
    hbm, tflops = peaks
    line = {"bench": "fabivik", "data": "synthetic", "dtype": "bf16", "n_gpus": 1, "window": args.design_window,
            "peaks": {"hbm_gbs": hbm, "bf16_tflops": tflops, "fp32_tflops_nominal": round(FP32_FLOPS / 1e12, 1)},
            "l2": "every sweep runs over all layers' own weights, cache and state", "sizes": {}}
    for name in (args.design_sizes.split(",") if args.design_sizes else SIZES):
        s = SIZES[name]
        line["sizes"][name] = {"shape": s}
        for kind in ("fabivik", "gpt"):
            line["sizes"][name][kind] = measure(kind, s, hbm, tflops, args.design_window, build=build_fabivik, costs=costs)
            torch.cuda.empty_cache()
    line["device_status"] = ops.device_status()
    line["gpu_launches"] = ops.launch_count
    emit(line)
