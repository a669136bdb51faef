"""`bench.py --design lukarax`: prefill and decode throughput of the Lukarax design at sizes that resemble a real model's layers,
beside the framework's closest model (`GPTModel`: RMSNorm, rotary, grouped queries, SwiGLU, bf16) at equal width, layer count,
feed-forward weights per token, batch and context.  Same method as bench_zinurax.py: whole-model forwards, then every launch of one
step timed alone.  Synthetic weights and tokens; one GPU; one JSON line."""
from __future__ import annotations

import math

import torch

import bench_zinurax as Z
from bench_zinurax import FP32_FLOPS, PROMPT_LEN, PROMPTS, VOCAB, measure

SIZES = {
    # differential heads / kv heads x dim / vdim, biased and sink attention heads / kv heads x dim, memory heads x dim / vdim, experts
    "2k": dict(width=2048, layers=8, heads=16, kv_groups=8, d_dim=64, d_vdim=128, dim=128, m_heads=16, m_dim=128, m_vdim=128, experts=32,
               identity=2, groups=2, top=4, ff=512, gpt_ff=2048),
    "4k": dict(width=4096, layers=8, heads=32, kv_groups=8, d_dim=64, d_vdim=128, dim=128, m_heads=32, m_dim=128, m_vdim=128, experts=64,
               identity=8, groups=4, top=8, ff=1024, gpt_ff=8192),
    "4k_d64": dict(width=4096, layers=8, heads=64, kv_groups=8, d_dim=32, d_vdim=64, dim=64, m_heads=32, m_dim=64, m_vdim=64, experts=16,
                   identity=2, groups=2, top=2, ff=4096, gpt_ff=8192),
}
STREAMS, KEEP = 4, 4


def build_lukarax(s, max_len, tokens, requests, window):
    from megatron_mixtera_b200 import model_registry as R
    from megatron_mixtera_b200.hybrid.stream_model import StreamHybridModel
    from megatron_mixtera_b200.transformer import hybrid_config as C

    rot = C.RotaryConfig(500000.0, s["d_dim"])
    yarn = C.RotaryConfig(500000.0, s["dim"] // 2, C.YarnScaling(4.0, 2048, 32.0, 1.0), halves=True)
    common = dict(heads=s["heads"], kv_heads=s["kv_groups"])

    def differential(source):
        return C.GroupedAttentionConfig(**common, dim=s["d_dim"], vdim=s["d_vdim"], scale=s["d_dim"] ** -0.5, rot=rot, diff=0.3, gate=True, kv_from=source)

    biased = C.GroupedAttentionConfig(**common, dim=s["dim"], vdim=s["dim"], scale=s["dim"] ** -0.5, window=window, keep_first=KEEP,
                                      distance_bias=C.DistanceBias(32, 128))
    sink = C.GroupedAttentionConfig(**common, dim=s["dim"], vdim=s["dim"], scale=s["dim"] ** -0.5, window=window, rot=yarn, unit_queries_keys=True,
                                    values_from_keys=True, biases=True, softcap=20.0, sink=True)
    memory = C.MatrixMemoryConfig(heads=s["m_heads"], dim=s["m_dim"], vdim=s["m_vdim"], gate_cap=15.0)
    side = C.SideBySideConfig((("left", biased, 0.8), ("right", memory, 0.9)))
    moe = C.MoeConfig(experts=s["experts"], top=s["top"], expert=C.ExpertConfig(s["ff"]),
                      routing=C.SoftmaxRouting(s["identity"], s["groups"], s["groups"] // 2, 2.0))
    layers = []
    for i in range(s["layers"]):  # the first layer dense; every second differential layer reads its predecessor's rows
        mixer = (differential(None if i % 8 == 0 else i - 4), side, sink, side)[i % 4]
        layers.append(C.HybridLayerConfig(mixer=mixer, moe=moe) if i else C.HybridLayerConfig(mixer=mixer, ffn_hidden_size=s["gpt_ff"]))
    model = StreamHybridModel(C.HybridConfig(vocab_size=VOCAB, hidden_size=s["width"], layers=tuple(layers), block="streams", streams=STREAMS,
                                             gated_linear_unit=True, activation="silu", embedding_scale=math.sqrt(s["width"])), max_len)
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
            return ("differential" if a.maps == 2 else "biased" if a.distance_bias else "sink") + ("_decode" if args[2] == 1 else "_prompt"), None
    if name == "hybrid":
        kernel = (Z.HYBRID + tuple(ops._STRUCT_KERNELS))[args[2]]
        raw = args[0].numpy().tobytes()
        if kernel == "stream_norm":
            a = _lib.StreamNormArgs.from_buffer_copy(raw)
            return "stream_norm" + (" start" if a.table else " last" if a.row_index or not a.in_ else " experts" if a.expert_rows else ""), None
        if kernel == "rotate_append":
            a = _lib.RotateAppendArgs.from_buffer_copy(raw)
            return "append " + ("sink" if a.rms else "biased" if not a.q_vecs else "differential" if a.k_vecs else "queries"), None
        if kernel.startswith("recurrence_"):
            return "memory" + kernel[len("recurrence"):], None
    return Z.label(name, args)


def costs(s, T, visible_pairs, keys, design, decode, requests):
    """(bytes, flops, fp32 flops) per launch of the non-GEMM kernels."""
    if not design:
        return Z.costs(s, T, visible_pairs, keys, False, decode, requests)
    W, H, G, d, dd, dv, pairs = s["width"], s["heads"], s["kv_groups"], s["dim"], s["d_dim"], s["d_vdim"], T * s["top"]
    routed = pairs * s["experts"] // (s["experts"] + s["identity"])
    out = {"stream_norm start": (T * W * (2.0 + 4 * STREAMS + 2), 0, 0), "stream_norm": (T * W * (8.0 * STREAMS + 4 + 2), 0, 0),
           "stream_norm experts": (T * W * (8.0 * STREAMS + 2) + 2.0 * W * (routed + T), 0, 0)}
    out["append differential"] = (4.0 * T * (2 * H * dd + G * (2 * dd + dv)), 0, 0)
    out["append queries"] = (4.0 * T * 2 * H * dd, 0, 0)
    out["append biased"] = (4.0 * T * 2 * G * d, 0, 0)
    out["append sink"] = (2.0 * T * (2 * H * d + 3 * G * d), 0, 0)
    for k in ("decode", "prompt"):
        out["differential_" + k] = (2.0 * keys * G * (2 * dd + dv) + 2.0 * T * H * (2 * dd + 2 * dv), 4.0 * visible_pairs * H * (dd + dv), 0)
        out["biased_" + k] = out["sink_" + k] = (2.0 * keys * G * 2 * d + 4.0 * T * H * d, 4.0 * visible_pairs * H * d, 0)
    mh, mk, mv = s["m_heads"], s["m_dim"], s["m_vdim"]
    state = 8.0 * requests * mh * mk * (mv + 1)
    out["memory_decode"] = (state + 2.0 * T * mh * (2 * mk + 3 * mv), 0, 6.0 * T * mh * mk * (mv + 1))
    out["memory_gates"] = (T * mh * 24.0, 0, 0)
    out["memory_scan"] = (state + 2.0 * T * mh * (2 * mk + mv) + 4.0 * T * mh * mv, 0, 6.0 * T * mh * mk * (mv + 1))
    out["memory_finish"] = (8.0 * T * mh * mv, 0, 0)
    used, f = min(s["experts"], routed), s["ff"]
    out["moe_route"] = (4.0 * T * (s["experts"] + s["identity"]), 0, 0)
    out["moe_gather"] = (2.0 * (T + routed) * W, 0, 0)
    out["moe_up"] = (2.0 * (used * 2 * f * W + routed * (W + f)), 4.0 * W * routed * f, 0)
    out["moe_down"] = (2.0 * (used * f * W + routed * (f + W)), 2.0 * W * routed * f, 0)
    return out


def run(args, emit, peaks):
    from megatron_mixtera_b200 import build, ops

    build.build_torch_ops()
    hbm, tflops = peaks
    line = {"bench": "lukarax", "data": "synthetic", "dtype": "bf16", "n_gpus": 1, "window": args.design_window,
            "peaks": {"hbm_gbs": hbm, "bf16_tflops": tflops, "fp32_tflops_nominal": round(FP32_FLOPS / 1e12, 1)},
            "l2": "every sweep runs over all layers' own weights, cache and state", "sizes": {}}
    for name in (args.design_sizes.split(",") if args.design_sizes else SIZES):
        s = SIZES[name]
        line["sizes"][name] = {"shape": s}
        for kind in ("lukarax", "gpt"):
            line["sizes"][name][kind] = measure(kind, s, hbm, tflops, args.design_window, build=build_lukarax, costs=costs, label=label)
            torch.cuda.empty_cache()
    line["device_status"] = ops.device_status()
    line["gpu_launches"] = ops.launch_count
    emit(line)
