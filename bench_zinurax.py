"""`bench.py --design zinurax`: prefill and decode throughput of the Zinurax design at sizes that resemble a real model's
layers, beside the framework's closest model (`GPTModel`: RMSNorm, rotary, grouped queries, SwiGLU, bf16) at equal width, layer
count, feed-forward weights, batch and context.  Synthetic weights and tokens; one GPU; one JSON line.

  prefill  `prompts` prompts of `prompt_len` tokens in one step, whole-model forward, CUDA events
  decode   `requests` requests at `context` cached tokens, one token each, whole-model CUDA graph, CUDA events
  kernels  every launch of one such step, timed alone: all launches of one kind (one per layer, each on its own weights, cache
           and state) back to back in a CUDA graph, against the larger of bytes / measured copy bandwidth and FLOPs / measured
           matrix throughput (fp32 work: the nominal CUDA-core rate)
"""
from __future__ import annotations

import math

import torch

SIZES = {
    # width, layers, heads, kv_rank, rot_dim, head dim, delta heads x dim, decay rank, feed-forward
    "2k": dict(width=2048, layers=8, heads=16, kv_rank=512, rot_dim=64, dim=128, vdim=128, d_heads=32, d_dim=64, rank=64, ff=8192,
               kv_groups=8, gpt_ff=5504),
    "4k": dict(width=4096, layers=8, heads=32, kv_rank=512, rot_dim=64, dim=128, vdim=128, d_heads=64, d_dim=64, rank=128, ff=21504,
               kv_groups=8, gpt_ff=14336),
    "4k_d128": dict(width=4096, layers=8, heads=32, kv_rank=256, rot_dim=32, dim=64, vdim=64, d_heads=32, d_dim=128, rank=128, ff=16384,
                    kv_groups=8, gpt_ff=10880),
}
VOCAB = 32768
FP32_FLOPS = 148 * 128 * 2 * 1.965e9  # CUDA cores, nominal
REQUESTS, CONTEXT, PROMPTS, PROMPT_LEN = 64, 4096, 4, 2048


def build_zinurax(s, max_len, tokens, requests, window):
    from megatron_mixtera_b200 import model_registry as R
    from megatron_mixtera_b200.hybrid.hybrid_model import HybridModel
    from megatron_mixtera_b200.transformer import hybrid_config as C

    rot = C.RotaryConfig(10000.0, s["rot_dim"], C.YarnScaling(8.0, 4096, 32.0, 1.0))
    layers = []
    for i in range(s["layers"]):  # recurrent and attention layers in turn; every other attention layer reads its predecessor's rows
        if i % 2 == 0:
            mixer = C.DeltaRuleConfig(heads=s["d_heads"], dim=s["d_dim"], rank=s["rank"])
        else:
            mixer = C.LatentAttentionConfig(
                heads=s["heads"], dim=s["dim"], rot_dim=s["rot_dim"], vdim=s["vdim"], kv_rank=s["kv_rank"],
                scale=1.0 / math.sqrt(s["dim"] + s["rot_dim"]), rot=rot, window=window, kv_from=i - 2 if i % 4 == 3 else None)
        layers.append(C.HybridLayerConfig(mixer=mixer, ffn_hidden_size=s["ff"]))
    model = HybridModel(C.HybridConfig(vocab_size=VOCAB, hidden_size=s["width"], layers=tuple(layers)), max_len)
    model.init_synthetic_weights(seed=0)
    ctx = R.make_context(model, max_cached_tokens=tokens, max_requests=requests, max_step_tokens=max(PROMPTS * PROMPT_LEN, requests),
                         chunk_size_tokens=256)
    for b in ctx.latent_buffers:
        if b is not None:
            b.normal_(0.0, 0.5)
    return model, ctx, R.make_controller(model, ctx).inference_wrapped_model


def build_gpt(s, max_len, tokens, requests, window):
    from megatron_mixtera_b200 import model_registry as R
    from megatron_mixtera_b200.gpt.gpt_model import GPTModel
    from megatron_mixtera_b200.transformer.transformer_config import TransformerConfig

    cfg = TransformerConfig(num_layers=s["layers"], hidden_size=s["width"], num_attention_heads=s["width"] // 128,
                            num_query_groups=s["kv_groups"], kv_channels=128, ffn_hidden_size=s["gpt_ff"], normalization="RMSNorm",
                            gated_linear_unit=True, activation="silu", add_bias_linear=False)
    model = GPTModel(cfg, vocab_size=VOCAB, max_sequence_length=max_len, position_embedding_type="rope",
                     share_embeddings_and_output_weights=True)
    model.init_synthetic_weights(seed=0)
    ctx = R.make_context(model, max_cached_tokens=tokens, max_requests=requests, max_step_tokens=max(PROMPTS * PROMPT_LEN, requests),
                         chunk_size_tokens=256)
    ctx.memory_buffer.normal_(0.0, 0.5)
    return model, ctx, R.make_controller(model, ctx).inference_wrapped_model


# ---------------------------------------------------------------------------------------------------------------------
def elapsed_us(fn, reps):
    fn()
    torch.cuda.synchronize()
    best = math.inf
    for _ in range(reps):
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        fn()
        e1.record()
        torch.cuda.synchronize()
        best = min(best, e0.elapsed_time(e1) * 1e3)
    return best


def graphed(fn):
    fn()
    torch.cuda.synchronize()
    graph = torch.cuda.CUDAGraph()
    with torch.cuda.graph(graph):
        out = fn()
    return graph, out


class Recorder:
    """Every kernel launch of one forward, kept replayable: the temporaries its pointers refer to stay alive."""

    def __enter__(self):
        from megatron_mixtera_b200 import ops

        self.ops, self.launch, self.empty, self.calls, self.keep = ops, ops._launch, torch.empty, [], []

        def launch(name, *args):
            self.calls.append((name, args))
            return self.launch(name, *args)

        def empty(*a, **k):
            t = self.empty(*a, **k)
            self.keep.append(t)
            return t

        ops._launch, torch.empty = launch, empty
        return self

    def __exit__(self, *exc):
        self.ops._launch, torch.empty = self.launch, self.empty


HYBRID = ("out_norm", "latent_append", "latent_attention", "delta_decode", "delta_lora", "delta_scan", "delta_finish",
          "latent_gather", "latent_prompt_attention")


def label(name, args):
    from megatron_mixtera_b200 import _lib, ops

    if name == "linear":
        batch = args[9]
        return "gemm %dx%dx%d%s" % (args[5], args[6], args[7], " x%d heads" % batch if batch > 1 else ""), (args[5], args[6] * batch, args[7], batch)
    if name in ("gemm", "gemm_splitk"):
        M, N, K = args[-3:]
        return "gemm %dx%dx%d" % (M, N, K), (M, N, K, 1)
    if name == "gemm_bf16_swiglu":
        M, (N, K) = args[0].numel() // args[0].shape[-1], args[1].shape
        return "gemm %dx%dx%d +swiglu" % (M, N, K), (M, N, K, 1)
    if name == "hybrid":
        kernel = (HYBRID + tuple(ops._STRUCT_KERNELS))[args[2]]
        if kernel in ("recurrence_decode", "recurrence_scan", "recurrence_finish"):  # one kernel, two rules
            kernel = ("wkv", "delta")[_lib.RecurrenceArgs.from_buffer_copy(args[0].numpy().tobytes()).kind] + kernel[len("recurrence"):]
        return kernel, None
    if name == "attention":
        return ("rope_append", "paged_attention", "paged_prefill_attention")[args[2]], None
    return name, None


def costs(s, T, visible_pairs, keys, zinurax, decode, requests):
    """(bytes, flops, fp32 flops) per launch of the non-GEMM kernels."""
    W = s["width"]
    out = {"gather_rows": (4.0 * T * W, 0, 0), "add_norm": (8.0 * T * W, 0, 0), "out_norm": (4.0 * T * W * 3 + 2.0 * T * W, 0, 0)}
    if zinurax:
        R, H, r = s["kv_rank"] + s["rot_dim"], s["heads"], s["kv_rank"]
        out["latent_append"] = (2.0 * T * (H * s["rot_dim"] * 2 + 2 * R), 0, 0)
        out["latent_attention"] = (2.0 * (keys * R + T * H * (R + r)), 2.0 * visible_pairs * H * (R + r), 0)
        # expanded keys and values: (dim + rot_dim) and vdim products per pair; every key's vectors once
        e = s["dim"] + s["vdim"]
        out["latent_prompt_attention"] = (2.0 * (keys * (H * e + s["rot_dim"]) + T * H * (e + s["rot_dim"])),
                                          2.0 * visible_pairs * H * (e + s["rot_dim"]), 0)
        out["latent_gather"] = (4.0 * keys * R, 0, 0)
        n, d = s["d_heads"] * s["d_dim"], s["d_dim"]
        state = 8.0 * requests * s["d_heads"] * d * d
        vec = 2.0 * T * n * 6
        out["delta_decode"] = (state + vec + 2.0 * n * s["rank"], 0, 10.0 * T * n * d)
        out["delta_scan"] = (state + vec + 4.0 * T * n, 0, 10.0 * T * n * d)
        out["delta_finish"] = (T * n * (4.0 + 2 + 2), 0, 0)
        out["delta_lora"] = (4.0 * T * s["rank"], 0, 0)
    else:
        H, G = W // 128, s["kv_groups"]
        io = 2.0 * T * (2 * H + 2 * G) * 128
        for k in ("paged_attention", "paged_prefill_attention"):
            out[k] = (2.0 * keys * 2 * G * 128 + io, 4.0 * visible_pairs * H * 128, 0)
        out["rope_append"] = (2.0 * T * 2 * 2 * G * 128, 0, 0)
    return out


def kernel_table(rec, cost, hbm, tflops, label=label):
    groups = {}
    for name, args in rec.calls:
        key, shape = label(name, args)
        groups.setdefault(key, ([], shape))[0].append((name, args))
    table = {}
    for key, (calls, shape) in groups.items():
        times = max(1, 16 // len(calls))
        graph, _ = graphed(lambda: [rec.launch(n, *a) for _ in range(times) for n, a in calls])
        us = elapsed_us(graph.replay, 3) / (times * len(calls))
        if shape:
            M, N, K, b = shape
            nbytes, flops, f32 = 2.0 * (N * K + M * K * b + M * N), 2.0 * M * N * K, 0
        else:
            nbytes, flops, f32 = cost.get(key, (0, 0, 0))
        bounds = {"HBM": nbytes / hbm / 1e3, "tensor": flops / tflops / 1e6, "fp32": f32 / FP32_FLOPS * 1e6}
        bound = max(bounds, key=bounds.get)
        table[key] = {"launches": len(calls), "us": round(us, 2), "bound": bound, "roofline": round(bounds[bound] / us, 3)}
        del graph
    return table


def measure(kind, s, hbm, tflops, window, build=None, costs=costs, label=label):
    """``kind`` "gpt": the GPT model; anything else: the design that ``build`` makes, with ``costs`` for its kernels, told apart by
    ``label``."""
    requests, max_len = REQUESTS, CONTEXT + 64
    tokens = requests * (-(-max_len // 256) * 256) + PROMPTS * (PROMPT_LEN + 256)
    gpt = kind == "gpt"
    model, ctx, wrapper = (build_gpt if gpt else build or build_zinurax)(s, max_len, tokens, requests, window)
    out = {"parameters": sum(p.numel() for p in model.parameters())}
    with torch.inference_mode():
        # ---- prefill ----
        T = PROMPTS * PROMPT_LEN
        g = torch.Generator().manual_seed(0)
        ctx.schedule_tokens([(i, torch.randint(0, VOCAB, (PROMPT_LEN,), generator=g)) for i in range(PROMPTS)])
        ctx.initialize_attention_state()
        ids, pos = ctx.current_input_and_position_ids()
        last = torch.from_numpy(ctx.last_token_indices()).cuda()
        fwd = lambda: model.forward_rows(ids, pos, ctx, last, True)
        fwd()
        us = elapsed_us(fwd, 5)
        per_prompt = sum(p + 1 if gpt else min(p + 1, window) for p in range(PROMPT_LEN))
        with Recorder() as rec:
            fwd()
        cost = costs(s, T, PROMPTS * per_prompt, T, not gpt, False, PROMPTS)
        out["prefill"] = {"tokens": T, "ms": round(us / 1e3, 3), "tokens_per_s": round(T / us * 1e6),
                          "kernels": kernel_table(rec, cost, hbm, tflops, label)}
        del rec
        ctx.reset_attention_state()
        ctx.reset()
        # ---- decode: the requests' contexts exist in the bookkeeping only, their rows are the pool's noise ----
        for i in range(requests):
            ctx.schedule_tokens([(i, torch.zeros(CONTEXT - 1, dtype=torch.int64))])
            ctx.complete_step()
        ctx.schedule_tokens([(i, torch.randint(0, VOCAB, (1,), generator=g)) for i in range(requests)])
        ctx.initialize_attention_state()
        ids, pos = ctx.current_input_and_position_ids()
        fwd = lambda: model.forward_rows(ids, pos, ctx, None, True)
        graph, _ = graphed(fwd)
        us = elapsed_us(graph.replay, 20)
        with Recorder() as rec:
            fwd()
        keys = requests * (CONTEXT if gpt else min(CONTEXT, window))
        cost = costs(s, requests, keys, keys, not gpt, True, requests)
        out["decode"] = {"requests": requests, "context": CONTEXT, "us": round(us, 1), "tokens_per_s": round(requests / us * 1e6),
                         "kernels": kernel_table(rec, cost, hbm, tflops, label)}
        del rec, graph
    return out


def run(args, emit, peaks):
    from megatron_mixtera_b200 import build, ops

    build.build_torch_ops()
    hbm, tflops = peaks
    line = {"bench": "zinurax", "data": "synthetic", "dtype": "bf16", "n_gpus": 1, "window": args.design_window,
            "peaks": {"hbm_gbs": hbm, "bf16_tflops": tflops, "fp32_tflops_nominal": round(FP32_FLOPS / 1e12, 1)},
            "l2": "every sweep runs over all layers' own weights, cache and state", "sizes": {}}
    for name in (args.design_sizes.split(",") if args.design_sizes else SIZES):
        s = SIZES[name]
        line["sizes"][name] = {"shape": s}
        for kind in ("zinurax", "gpt"):
            line["sizes"][name][kind] = measure(kind, s, hbm, tflops, args.design_window)
            torch.cuda.empty_cache()
    line["device_status"] = ops.device_status()
    line["gpu_launches"] = ops.launch_count
    emit(line)

