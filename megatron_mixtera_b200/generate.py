"""Generate from a model folder (`config.json` + `model.safetensors`) with token ids in and token ids out.

    python -m megatron_mixtera_b200.generate --model DIR --prompt 11,250,4 --prompt 9,9 --num-tokens 16

One line per prompt, in order: the generated ids, comma-separated.  Prompts may also come from standard input, one per line.
"""
from __future__ import annotations

import argparse
import sys
import types


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="generate", description="Generate token ids from a model folder.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--prompt", action="append", default=[], help="comma-separated token ids; may be repeated (default: standard input)")
    ap.add_argument("--num-tokens", type=int, default=16, help="tokens to generate per prompt")
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    ap.add_argument("--top-k", type=int, default=1, help="1: greedy; 0: the whole vocabulary, or the nucleus of --top-p")
    ap.add_argument("--top-p", type=float, default=0.0)
    ap.add_argument("--temperature", type=float, default=1.0)
    ap.add_argument("--seed", type=int, default=0)
    ap.add_argument("--stop-token", type=int, default=-1, help="a request ends when it generates this id")
    ap.add_argument("--max-requests", type=int, default=64, help="requests decoded together")
    ap.add_argument("--cuda-graphs", type=int, default=4, help="graph sizes to capture for decode steps (0: none)")
    args = ap.parse_args(argv)

    import torch

    from . import build, model_registry
    from .inference.engines.dynamic_engine import DynamicInferenceEngine
    from .inference.sampling_params import SamplingParams

    texts = args.prompt or [line for line in sys.stdin.read().splitlines() if line.strip()]
    prompts = [[int(t) for t in p.replace(",", " ").split()] for p in texts]
    if not prompts or not all(prompts):
        ap.error("every prompt needs at least one token id")
    build.build_torch_ops()
    longest, total = max(map(len, prompts)) + args.num_tokens, sum(map(len, prompts))
    requests = min(args.max_requests, len(prompts))
    pages = requests * (-(-longest // 64) + 1)
    model, context, controller = model_registry.serving_stack(
        args.model, dtype=getattr(torch, args.dtype), max_cached_tokens=64 * (pages + -(-longest // 64)), max_requests=requests,
        max_sequence_length=longest, max_step_tokens=total + requests, num_cuda_graphs=args.cuda_graphs or None)
    if any(not 0 <= t < model.vocab_size for p in prompts for t in p):
        ap.error(f"token ids must lie in [0, {model.vocab_size})")
    model.config.enable_cuda_graph = args.cuda_graphs > 0
    controller.tokenizer = types.SimpleNamespace(vocab_size=model.vocab_size)
    controller.sampling_rng.manual_seed(args.seed)
    engine = DynamicInferenceEngine(controller, context, termination_id=args.stop_token, random_seed=args.seed,
                                    enable_cuda_graph=args.cuda_graphs > 0, overlap_host_and_device=args.cuda_graphs > 0)
    params = SamplingParams(top_k=args.top_k, top_p=args.top_p, temperature=args.temperature, num_tokens_to_generate=args.num_tokens)
    for r in sorted(engine.generate(prompts, params), key=lambda r: r.request_id):
        print(",".join(map(str, r.generated_tokens)), flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
