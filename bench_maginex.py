"""`bench.py --design maginex`: prefill and decode throughput of the Maginex design at sizes that resemble a real model's layers,
beside the framework's closest model (`GPTModel`: RMSNorm, rotary, grouped queries, SwiGLU, bf16) at equal width, layer count,
feed-forward weights per token, batch and context.  Same method as bench_zinurax.py: whole-model forwards, then every launch of one
step timed alone.  Synthetic weights and tokens; one GPU; one JSON line."""
from __future__ import annotations

import math

import torch

import bench_zinurax as Z
from bench_zinurax import FP32_FLOPS, PROMPT_LEN, PROMPTS, VOCAB, measure

SIZES = {
    # latent attention heads x dim / vdim over kv_rank, windowed attention heads / kv heads x dim, scan width, experts
    "2k": dict(width=2048, layers=8, heads=16, dim=128, kv_rank=512, q_rank=768, a_dim=128, rot=64, kv_groups=8, scan=3072, experts=32, top=4, ff=768,
               shared=1536, gpt_ff=3072),
    "4k": dict(width=4096, layers=8, heads=32, dim=128, kv_rank=512, q_rank=1536, a_dim=128, rot=64, kv_groups=8, scan=6144, experts=64, top=8,
               ff=1024, shared=2048, gpt_ff=6784),
    "4k_d64": dict(width=4096, layers=8, heads=64, dim=64, kv_rank=256, q_rank=1024, a_dim=64, rot=32, kv_groups=8, scan=4096, experts=16, top=2,
                   ff=4096, shared=4096, gpt_ff=8192),
}
TAPS = 4


def build_maginex(s, max_len, tokens, requests, window):
    from megatron_mixtera_b200 import model_registry as R
    from megatron_mixtera_b200.hybrid.parallel_model import ParallelHybridModel
    from megatron_mixtera_b200.transformer import hybrid_config as C

    d, a = s["dim"], s["a_dim"]
    latent = C.LatentAttentionConfig(heads=s["heads"], dim=d, rot_dim=0, vdim=d, kv_rank=s["kv_rank"], q_rank=s["q_rank"], scale=d ** -0.5,
                                     sink=True, gate="value")
    windowed = C.GroupedAttentionConfig(heads=s["heads"], kv_heads=s["kv_groups"], dim=a, vdim=a, scale=a ** -0.5, window=window, sink=True,
                                        rot=C.RotaryConfig(500000.0, s["rot"], halves=True), head_gate=True, value_mix=True)
    scan = C.GatedScanConfig(s["scan"])
    moe = C.MoeConfig(experts=s["experts"], top=s["top"], expert=C.ExpertConfig(s["ff"], gated=False),
                      shared=C.ExpertConfig(s["shared"], gated=False), routing=C.ChosenSoftmaxRouting())
    layers = [C.HybridLayerConfig(mixer=(scan, windowed, scan, latent)[i % 4], moe=moe) for i in range(s["layers"])]
    model = ParallelHybridModel(C.HybridConfig(vocab_size=VOCAB, hidden_size=s["width"], layers=tuple(layers), block="parallel", norm_offset=0.0,
                                               input_taps=TAPS, embedding_scale=math.sqrt(s["width"])), max_len)
    model.init_synthetic_weights(seed=0)
    ctx = R.make_context(model, max_cached_tokens=tokens, max_requests=requests, max_step_tokens=max(PROMPTS * PROMPT_LEN, requests),
                         chunk_size_tokens=256)
    for b in ctx.latent_buffers:
        if b is not None:
            b.normal_(0.0, 0.5)
    return model, ctx, R.make_controller(model, ctx).inference_wrapped_model


def label(name, args):
    """Kernels that serve several mechanisms, by the one a launch is for."""
    from megatron_mixtera_b200 import _lib, ops

    if name == "attention":
        a = _lib.AttentionArgs.from_buffer_copy(args[0].numpy().tobytes())
        if a.separate == 2:
            return ("latent_prompt" if a.value_gates else "window_decode" if args[2] == 1 else "window_prompt"), None
    if name == "hybrid":
        kernel = (Z.HYBRID + tuple(ops._STRUCT_KERNELS))[args[2]]
        if kernel == "residual_norm":
            a = _lib.ResidualNormArgs.from_buffer_copy(args[0].numpy().tobytes())
            return "residual_norm" + (" start" if a.table else " last" if a.row_index or not a.taps and a.rows <= 256 else ""), None
    return Z.label(name, args)


def costs(s, T, visible_pairs, keys, design, decode, requests):
    """(bytes, flops, fp32 flops) per launch of the non-GEMM kernels."""
    if not design:
        return Z.costs(s, T, visible_pairs, keys, False, decode, requests)
    W, H, G, d, a, pairs = s["width"], s["heads"], s["kv_groups"], s["dim"], s["a_dim"], T * s["top"]
    r, rank, n = -(-s["kv_rank"] // 32) * 32, s["kv_rank"], s["scan"]
    left = 4 * 2 + 4 + 2 * s["top"] + 2  # stream in and out, mixer's sums, expert rows, shared row
    filtered = (2 * 2 + 2 * 2 * (TAPS - 1)) if decode else 2
    out = {"residual_norm start": (T * W * (2.0 + 4 + filtered), 0, 0), "residual_norm": (T * W * float(left + filtered), 0, 0),
           "conv_add": (T * W * 6.0, 0, 0)}
    out["rotate_append"] = (2.0 * T * a * (2 * H + 5 * G), 0, 0)
    for k in ("decode", "prompt"):
        out["window_" + k] = (2.0 * keys * G * 2 * a + 4.0 * T * H * a, 4.0 * visible_pairs * H * a, 0)
    out["latent_append"] = (4.0 * T * (s["q_rank"] + rank), 0, 0)
    out["latent_attention"] = (2.0 * (keys * r + T * H * (r + rank)), 2.0 * visible_pairs * H * (r + rank), 0)
    out["latent_prompt"] = (2.0 * (keys * H * 2 * d + T * H * 3 * d), 4.0 * visible_pairs * H * d, 0)
    out["latent_gather"] = (4.0 * keys * r, 0, 0)
    out["gated_scan"] = (T * n * ((12.0 if decode else 6.0) + 2) + 8.0 * requests * n, 0, 0)
    used, f, g = min(s["experts"], pairs), s["ff"], s["shared"]
    out["moe_route"] = (4.0 * T * s["experts"], 0, 0)
    out["moe_gather"] = (2.0 * (T + pairs) * W, 0, 0)
    out["moe_up"] = (2.0 * (used * f * W + g * W + pairs * (W + f) + T * (W + g)), 2.0 * W * (pairs * f + T * g), 0)
    out["moe_down"] = (2.0 * (used * f * W + g * W + pairs * (W + f) + T * (W + g)), 2.0 * W * (pairs * f + T * g), 0)
    return out


def run(args, emit, peaks):
    from megatron_mixtera_b200 import build, ops

    build.build_torch_ops()
    hbm, tflops = peaks
    line = {"bench": "maginex", "data": "synthetic", "dtype": "bf16", "n_gpus": 1, "window": args.design_window,
            "peaks": {"hbm_gbs": hbm, "bf16_tflops": tflops, "fp32_tflops_nominal": round(FP32_FLOPS / 1e12, 1)},
            "l2": "every sweep runs over all layers' own weights, cache and state", "sizes": {}}
    for name in (args.design_sizes.split(",") if args.design_sizes else SIZES):
        s = SIZES[name]
        line["sizes"][name] = {"shape": s}
        for kind in ("maginex", "gpt"):
            line["sizes"][name][kind] = measure(kind, s, hbm, tflops, args.design_window, build=build_maginex, costs=costs, label=label)
            torch.cuda.empty_cache()
    line["device_status"] = ops.device_status()
    line["gpu_launches"] = ops.launch_count
    emit(line)
