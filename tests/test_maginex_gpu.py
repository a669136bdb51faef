"""Maginex on the GPU against the plain oracle: whole prompts, portions, decoding, mixed batches, reuse of chunks and slots,
generation through the engine and the command lines."""
import json
import os
import subprocess
import types

import maginex_helpers as H
import numpy as np
import pytest
import torch

pytestmark = pytest.mark.gpu

LIMIT = {torch.float32: 1e-4, torch.bfloat16: 0.06}
DTYPES = [torch.float32, torch.bfloat16]


@pytest.fixture(scope="module")
def case():
    cache = {}

    def get(name, lengths, dtype, gain=1.0):
        settled = dtype == torch.bfloat16
        key = (name, tuple(lengths), settled, gain)
        if key not in cache:
            cfg = H.CONFIGS[name]
            w = H.weights(cfg, seed=3, gain=gain, settled=settled)
            reqs = [H.tokens(n, cfg["vocab"], 10 + i) for i, n in enumerate(lengths)]
            cache[key] = (cfg, w, reqs, [H.oracle_logits(r, cfg, w) for r in reqs])
        return cache[key]

    return get


def check(got, want, dtype):
    """32-bit: every position.  16-bit: nearly every one (the experts are settled there: a token whose last chosen expert won by less than
    rounding could take the other one)."""
    for i, g in got.items():
        e = H.position_errors(g, want[i][: g.shape[0]])
        over = float((e > LIMIT[dtype]).float().sum())
        if dtype == torch.float32:
            assert over == 0, (i, e.max())
        else:
            assert over <= max(1.0, 0.02 * e.numel()) and float(e.max()) < 3 * LIMIT[dtype] and float(e.median()) < LIMIT[dtype] / 2, (
                i, over, e.topk(min(8, e.numel())), e.median())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(H.CONFIGS))
def test_prompt_portions_and_decoding(case, name, dtype):
    """The same sequence whole, in portions of changing size (down to two tokens, across chunk and window edges), and token
    by token from the first one; slots and chunks are used again by every pass."""
    cfg, w, reqs, want = case(name, [161], dtype)
    _, ctx, ctl = H.build(cfg, w, dtype, max_cached_tokens=192)
    for schedule in ([161], [2, 62, 2, 3, 31, 33, 2, 1, 1, 17, 7], [1] * 161, [63] + [1] * 98):
        check(H.replay(ctl, [[(0, n)] for n in schedule], reqs), want, dtype)
    assert ctx.chunk_allocator.chunk_count_avail >= 3 and ctx.total_request_count == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "wide", "odd"])
def test_batches_of_unequal_requests(case, name, dtype):
    """Portions beside single tokens, requests sitting out and going on, more requests than slots over time."""
    cfg, w, reqs, want = case(name, [130, 3, 67, 1, 90, 40], dtype)
    _, ctx, ctl = H.build(cfg, w, dtype, max_cached_tokens=448)
    schedule = [[(0, 64), (1, 2)], [(2, 5), (0, 1), (1, 1)], [(3, 1), (0, 2), (2, 60)], [(0, 1), (2, 1), (4, 33)],
                [(2, 1), (4, 1)], [(5, 17), (0, 60)], [(4, 50), (0, 1), (5, 1)], [(4, 1), (5, 21)]]
    schedule += [[(4, 1), (0, 1), (5, 1)], [(4, 2)], [(4, 2)]]
    got = H.replay(ctl, schedule, reqs)
    assert all(len(got[i]) == len(reqs[i]) for i in got)
    check(got, want, dtype)
    assert ctx.total_request_count == 0 and len(ctx._free_state_slots) == ctx.num_state_slots


@pytest.mark.parametrize("dtype", DTYPES)
def test_result_does_not_depend_on_the_batch(case, dtype):
    cfg, w, reqs, _ = case("mixed", [130, 3, 67, 1, 90, 40], dtype)
    _, _, ctl = H.build(cfg, w, dtype)
    alone = H.replay(ctl, [[(0, 70)]] + [[(0, 1)]] * 60, reqs)[0].cpu().float()
    _, _, ctl = H.build(cfg, w, dtype)
    together = H.replay(ctl, [[(2, 30), (0, 70), (4, 9)]] + [[(4, 1), (0, 1)]] * 60, reqs)[0]
    e = H.position_errors(together, alone)
    assert float(e.max()) < LIMIT[dtype] / 2


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_with_peaked_attention(case, dtype):
    """Hundreds of decoded tokens: windows slide over decoded tokens, the recurrent state has long forgotten the prompt."""
    cfg, w, reqs, want = case("mixed", [420], dtype, gain=1.6)
    _, _, ctl = H.build(cfg, w, dtype)
    check(H.replay(ctl, [[(0, 20)]] + [[(0, 1)]] * 400, reqs), want, dtype)


def test_first_tokens_of_many_sequences(case):
    """What lies in front of a sequence is zero for its filters and its recurrence, whatever a slot's last owner left there."""
    cfg, w, reqs, want = case("mixed", [9, 8, 7, 6, 5, 4, 3, 2, 1], torch.float32)
    _, ctx, ctl = H.build(cfg, w, torch.float32, max_cached_tokens=256)
    for b in ctx.state_buffers:
        for t in b.values():
            t.fill_(float("nan"))
    schedule = []
    for group in ((0, 1, 2), (3, 4, 5), (6, 7, 8)):
        for t in range(len(reqs[group[0]])):
            schedule.append([(i, 1) for i in group if t < len(reqs[i])])
    check(H.replay(ctl, schedule, reqs), want, torch.float32)
    check(H.replay(ctl, [[(0, 9), (4, 5), (8, 1)], [(1, 8), (7, 2), (2, 7)], [(3, 2), (5, 4)], [(3, 4), (6, 3)]], reqs), want, torch.float32)


def test_residual_stream_after_every_layer(case):
    cfg, w, reqs, _ = case("mixed", [40], torch.float32)
    model, ctx, _ = H.build(cfg, w, torch.float32)
    ctx.schedule_tokens([(0, reqs[0])])
    ctx.initialize_attention_state()
    streams, plain = [], []
    with torch.inference_mode():
        model.forward_rows(*ctx.current_input_and_position_ids(), ctx, streams=streams)
    H.oracle_logits(reqs[0], cfg, w, plain)
    for s, p in zip(streams, plain, strict=True):
        assert float((s[:40].cpu() - p).norm() / p.norm()) < 1e-5


def greedy_oracle(cfg, w, prompt, n):
    toks, margins = list(prompt), []
    for _ in range(n):
        logits = H.oracle_logits(toks, cfg, w)[-1]
        top = torch.topk(logits, 2).values
        margins.append(float(top[0] - top[1]))
        toks.append(int(logits.argmax()))
    return toks[len(prompt):], min(margins)


@pytest.fixture(scope="module")
def greedy():
    cfg = H.CONFIGS["mixed"]
    w = H.weights(cfg, seed=3)
    prompts = [H.tokens(k, cfg["vocab"], 30 + k) for k in (50, 1, 64, 9, 130, 20, 33)]
    want = [greedy_oracle(cfg, w, p, 20) for p in prompts]
    assert min(m for _, m in want) > 1e-3  # no near-ties: the tokens are well defined in 32-bit arithmetic
    return cfg, w, prompts, [t for t, _ in want]


@pytest.mark.parametrize("graphs,overlap", [(None, False), (2, False), (2, True)])
def test_greedy_generation_through_the_engine(greedy, graphs, overlap):
    """The engine's own loop - queue, batching, pausing at chunk ends, sampling kernels - with and without CUDA graphs and
    the forward enqueued early, against greedy decoding with the oracle."""
    from megatron_mixtera_b200.inference.engines.dynamic_engine import DynamicInferenceEngine
    from megatron_mixtera_b200.inference.sampling_params import SamplingParams

    cfg, w, prompts, want = greedy
    _, ctx, ctl = H.build(cfg, w, torch.float32, max_cached_tokens=1024, cuda_graphs=graphs is not None, num_cuda_graphs=graphs)
    ctl.tokenizer = types.SimpleNamespace(vocab_size=cfg["vocab"])
    engine = DynamicInferenceEngine(ctl, ctx, termination_id=-1, random_seed=0, enable_cuda_graph=graphs is not None,
                                    overlap_host_and_device=overlap)
    for _ in range(2):  # a second round uses the same slots, chunks and graphs again
        done = engine.generate(prompts, SamplingParams(top_k=1, num_tokens_to_generate=20))
        assert len(done) == len(prompts)
        first = min(r.request_id for r in done)
        for r in done:
            assert r.generated_tokens == want[r.request_id - first], r.request_id - first
    if graphs:
        assert ctl.inference_wrapped_model.graph_replays > 0


@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_bf16_graph_replay_equals_eager(case, name):
    cfg, w, reqs, _ = case(name, [130, 3, 67, 1, 90, 40], torch.bfloat16)
    schedule = [[(0, 20), (2, 30)]] + [[(0, 1), (2, 1)]] * 30
    _, _, ctl = H.build(cfg, w, torch.bfloat16)
    eager = H.replay(ctl, schedule, reqs)
    _, _, ctl = H.build(cfg, w, torch.bfloat16, cuda_graphs=True, num_cuda_graphs=1)
    graph = H.replay(ctl, schedule, reqs)
    assert ctl.inference_wrapped_model.graph_replays == 30
    for i in eager:
        assert torch.equal(eager[i], graph[i])


def test_mixed_steps_under_cuda_graphs(case):
    """Prefill and mixed steps padded to a graph size: captured once, replayed on other requests."""
    from megatron_mixtera_b200.inference.engines.dynamic_engine import DynamicInferenceEngine
    from megatron_mixtera_b200.inference.sampling_params import SamplingParams

    cfg, w, _, _ = case("mixed", [130, 3, 67, 1, 90, 40], torch.float32)
    prompts = [H.tokens(n, cfg["vocab"], 70 + n) for n in (3, 9, 2, 11, 5, 1, 7, 4)]
    want = [greedy_oracle(cfg, w, p, 6)[0] for p in prompts]
    _, ctx, ctl = H.build(cfg, w, torch.float32, max_cached_tokens=2048, max_requests=16, cuda_graphs=True, num_cuda_graphs=2)
    ctl.tokenizer = types.SimpleNamespace(vocab_size=cfg["vocab"])
    engine = DynamicInferenceEngine(ctl, ctx, termination_id=-1, random_seed=0, enable_cuda_graph=True)
    for r0 in range(0, 8, 2):
        done = sorted(engine.generate(prompts[r0: r0 + 2], SamplingParams(top_k=1, num_tokens_to_generate=6)), key=lambda r: r.request_id)
        assert [r.generated_tokens for r in done] == want[r0: r0 + 2]
    assert ctl.inference_wrapped_model.non_decode_graph_replays > 1


def test_sampling(case):
    from megatron_mixtera_b200.inference.engines.dynamic_engine import DynamicInferenceEngine
    from megatron_mixtera_b200.inference.sampling_params import SamplingParams

    cfg, w, reqs, _ = case("mixed", [130, 3, 67, 1, 90, 40], torch.float32)
    for dtype in DTYPES:
        for params in (dict(top_k=5), dict(top_k=0, top_p=0.8)):
            _, ctx, ctl = H.build(cfg, w, dtype)
            ctl.tokenizer = types.SimpleNamespace(vocab_size=cfg["vocab"])
            engine = DynamicInferenceEngine(ctl, ctx, termination_id=-1, random_seed=0)
            done = engine.generate(reqs[:3], SamplingParams(num_tokens_to_generate=4, **params))
            assert all(0 <= t < cfg["vocab"] for r in done for t in r.generated_tokens)


def folder(tmp_path, cfg, w):
    from megatron_mixtera_b200 import checkpoint

    (tmp_path / "config.json").write_text(json.dumps(cfg))
    checkpoint.save_safetensors(str(tmp_path / "model.safetensors"), w)


def test_trace_replay_of_a_model_folder(case, tmp_path):
    """The command-line replay: model folder in, one logits file per step that wants some."""
    cfg, w, reqs, want = case("mixed", [130, 3, 67, 1, 90, 40], torch.float32)
    folder(tmp_path, cfg, w)
    out = tmp_path / "out"
    out.mkdir()
    lines = [{"step": 0, "entries": [{"id": "x", "tokens": reqs[0][:70], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "y", "tokens": reqs[1], "want": [2, 0]}, {"id": "x", "tokens": reqs[0][70:71], "want": [0]}],
              "end": ["x", "y"]}]
    exe = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "bin", "trace_run")
    run = subprocess.run([exe, "--model", str(tmp_path), "--dtype", "float32", "--out", str(out), "--max-tokens", "192"],
                         input="".join(json.dumps(x) + "\n" for x in lines), capture_output=True, text=True, timeout=600)
    assert run.returncode == 0, run.stderr
    assert [x for x in run.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1"]
    assert not (out / "0.f32").exists()
    got = torch.from_numpy(np.fromfile(out / "1.f32", dtype="<f4")).view(3, cfg["vocab"])
    assert H.error(got, torch.stack([want[1][2], want[1][0], want[0][70]])) < LIMIT[torch.float32]


def test_generate_command_line(greedy, tmp_path, capsys):
    """Token ids in, greedy token ids out, in the prompts' order and independent of how they are batched."""
    from megatron_mixtera_b200 import generate

    cfg, w, prompts, want = greedy
    folder(tmp_path, cfg, w)
    base = ["--model", str(tmp_path), "--dtype", "float32", "--num-tokens", "8"] + [x for p in prompts[:3] for x in ("--prompt", ",".join(map(str, p)))]
    for extra in ([], ["--cuda-graphs", "0", "--max-requests", "1"]):
        assert generate.main(base + extra) == 0
        lines = [[int(t) for t in x.split(",")] for x in capsys.readouterr().out.strip().splitlines()]
        assert lines == [t[:8] for t in want[:3]]
