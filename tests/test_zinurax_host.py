"""Zinurax without a GPU: configuration and checkpoint reading, rotation tables, the context's bookkeeping for latent rows,
state slots and steps of given tokens, and that mistakes of each mechanism would show in the numerics tests."""
import json
import math

import numpy as np
import pytest
import torch

import zinurax_helpers as H
from oracle import zinurax_oracle as Z


def make_context(max_requests=4, tokens=320, max_len=256, chunk=64, states=((2, 4, 4), None), widths=(0, 32), **kw):
    from megatron_mixtera_b200.inference.contexts.dynamic_context import DynamicInferenceContext as C

    nbytes = C.latent_chunk_bytes(widths, chunk, torch.float32)
    return C(params_dtype=torch.float32, num_layers=2, kv_channels=0, num_attention_heads=0, max_sequence_length=max_len,
             buffer_size_gb=(tokens // chunk + 1.5) * nbytes / 1024**3, buffer_guaranteed_fraction=0.0, chunk_size_tokens=chunk,
             max_requests_override=max_requests, max_tokens_override=512, tensor_model_parallel_size=1, cache_mla_latent=True,
             latent_row_widths=list(widths), state_shapes=list(states), device="cpu", debug_validate=True, **kw)


# ---------------------------------------------------------------------------------------------------------------------
# configuration, checkpoint
# ---------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", list(H.CONFIGS))
def test_config_and_checkpoint_names(name):
    from megatron_mixtera_b200 import model_registry as R
    from megatron_mixtera_b200.transformer.hybrid_config import DeltaRuleConfig, LatentAttentionConfig

    cfg, rank = H.CONFIGS[name]
    w = H.weights(cfg, rank)
    model = R.ARCHITECTURES["Zinurax"](cfg, {k: tuple(v.shape) for k, v in w.items()}, torch.bfloat16, 64)
    assert {k: tuple(s) for k, s in model.checkpoint_tensors().items()} == {k: tuple(v.shape) for k, v in w.items()}
    for mine, layer in zip(model.config.layers, cfg["layers"], strict=True):
        m = layer["mixer"]
        if layer["type"] == "latent_attention":
            assert isinstance(mine.mixer, LatentAttentionConfig)
            assert (mine.mixer.window, mine.mixer.kv_from, mine.mixer.scale) == (m["mask"]["size"], m.get("kv_from"), m["scale"])
            assert mine.mixer.row_width % 32 == 0 and mine.mixer.row_width >= m["kv_rank"] + m["rot_dim"]
        else:
            assert isinstance(mine.mixer, DeltaRuleConfig) and mine.mixer.rank == rank
        assert mine.ffn_hidden_size == (layer["mlp"] or {"ff": None})["ff"]
    if torch.cuda.is_available():
        return
    model.load_checkpoint(w)
    for i, layer in enumerate(cfg["layers"]):
        mix = model.layers[i].mixer
        if layer["type"] == "latent_attention":
            m = layer["mixer"]
            h, d = m["heads"] - 1, m["dim"] - 1  # absorbed form: [head][latent][dim]
            assert torch.equal(mix.key_up[h * m["kv_rank"]: (h + 1) * m["kv_rank"], d], w[f"l{i}.mix.uk"][h * m["dim"] + d])
            assert torch.equal(mix.linear_in.weight[mix.gate_offset: mix.in_width], w[f"l{i}.mix.g"])
        assert bool((mix.linear_in.weight[mix.in_width:] == 0).all())
    with pytest.raises(KeyError):
        model.load_checkpoint({k: v for k, v in w.items() if k != "final.norm"})
    with pytest.raises(KeyError):
        model.load_checkpoint({**w, "l9.mix.q": w["embed"]})
    with pytest.raises(ValueError):
        model.load_checkpoint({**w, "embed": w["embed"][:-1]})


def test_config_errors():
    from megatron_mixtera_b200 import model_registry as R

    cfg, rank = H.CONFIGS["mixed"]
    shapes = {k: tuple(v.shape) for k, v in H.weights(cfg, rank).items()}

    def broken(change):
        c = json.loads(json.dumps(cfg))
        change(c)
        with pytest.raises((ValueError, KeyError, NotImplementedError)):
            R.zinurax_config(c, shapes, torch.float32)

    broken(lambda c: c["layers"][0].update(type="other"))
    broken(lambda c: c["layers"][0]["mlp"].update(kind="other"))
    broken(lambda c: c["layers"][2]["mixer"].update(kv_from=0))    # a recurrent layer has no rows
    broken(lambda c: c["layers"][2]["mixer"].update(kv_from=2))    # itself
    broken(lambda c: c["layers"][2]["mixer"].update(kv_rank=64))   # rows of another shape
    with pytest.raises(ValueError):
        R.zinurax_config(cfg, shapes, torch.float16)


def test_unknown_architecture(tmp_path):
    from megatron_mixtera_b200 import model_registry as R

    (tmp_path / "config.json").write_text('{"architecture": "Nothing"}')
    with pytest.raises(ValueError):
        R.load_model(str(tmp_path), max_sequence_length=8)


def test_safetensors_round_trip(tmp_path):
    from megatron_mixtera_b200 import checkpoint as C

    t = {"a": torch.randn(3, 5).to(torch.bfloat16), "b.c": torch.arange(7, dtype=torch.int32), "d": torch.randn(2, 2, 2)}
    path = str(tmp_path / "m.safetensors")
    C.save_safetensors(path, t)
    got = C.load_safetensors(path)
    assert list(got) == list(t) and all(torch.equal(got[k], t[k]) and got[k].dtype == t[k].dtype for k in t)
    assert C.tensor_shapes(path) == {k: tuple(v.shape) for k, v in t.items()}


@pytest.mark.parametrize("scaling", [None, (4.0, 96, 8.0, 1.0), (8.0, 4096, 32.0, 1.0), (2.0, 16, 40.0, 30.0), (32.0, 100000, 2.0, 0.001)])
@pytest.mark.parametrize("base,dims", [(10000.0, 64), (500.0, 6), (1e6, 2)])
def test_rotary_tables(scaling, base, dims):
    """Against the oracle's rotation of unit vectors, including ramps that clamp at either end or collapse."""
    from megatron_mixtera_b200.transformer.hybrid_config import RotaryConfig, YarnScaling
    from megatron_mixtera_b200.transformer.rotary import rotary_tables

    rot = {"base": base, "dims": dims}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    cos, sin = rotary_tables(RotaryConfig(base, dims, YarnScaling(*scaling) if scaling else None), 300, "cpu")
    x = torch.zeros(300, dims, dtype=torch.float64)
    x[:, 0::2] = 1.0
    y = Z.rotate(x, torch.arange(300), rot)
    assert (cos - y[:, 0::2]).abs().max() < 1e-6 and (sin - y[:, 1::2]).abs().max() < 1e-6


# ---------------------------------------------------------------------------------------------------------------------
# bookkeeping
# ---------------------------------------------------------------------------------------------------------------------
def step(ctx, entries, finished=()):
    """One step; returns per entry (positions, (chunk, place) of its tokens, state read, state written)."""
    ctx.schedule_tokens(entries)
    ctx.initialize_attention_state()
    out, a = [], 0
    for k, (_, toks) in enumerate(entries):
        b = a + len(toks)
        out.append((ctx.token_to_position_in_request[a:b].tolist(),
                    list(zip(ctx.token_to_chunk_idx[a:b].tolist(), ctx.token_to_local_position_within_kv_chunk[a:b].tolist())),
                    int(ctx.state_read_slots[k]), int(ctx.state_write_slots[k])))
        assert ctx.token_to_input_ids[a:b].tolist() == list(toks)
        a = b
    ctx.complete_step(finished)
    return out


def test_steps_of_given_tokens():
    ctx = make_context(tokens=384)
    seen = {}

    def run(entries, finished=()):
        for (rid, toks), (pos, places, rd, wr) in zip(entries, step(ctx, entries, finished)):
            before = seen.setdefault(rid, [])
            assert pos == list(range(len(before), len(before) + len(toks)))
            # the state written last is what is read next; a new request reads none
            assert rd == (before[-1][1] if before else -1) and wr >= 0 and wr != rd
            if before:
                assert wr % ctx.num_state_slots == rd % ctx.num_state_slots
            before += [(p, wr) for p in places]
            for i, (place, _) in enumerate(before):  # a request's chunks are its own and stay where they are
                assert place[1] == i % 64 and place[0] == before[i // 64 * 64][0][0]
        live = {r: s for r, s in seen.items() if r not in finished}
        chunks = [c for s in live.values() for c in {p[0] for p, _ in s}]
        assert len(chunks) == len(set(chunks))
        for r in finished:
            del seen[r]

    run([(7, [1, 2, 3]), (8, list(range(70)))])
    run([(8, [5]), (9, [6] * 64)])
    run([(7, [4] * 61), (9, [1])])
    run([(10, [3])], finished=[10])
    run([(9, [2]), (7, [9, 9]), (8, [1])], finished=[9, 8])
    run([(11, [1] * 100), (7, [2]), (12, [5])])
    run([(12, [5])], finished=[7, 11, 12])
    assert ctx.total_request_count == 0 and ctx.chunk_allocator.chunk_count_avail == 6
    assert sorted(ctx._free_state_slots) == [0, 1, 2, 3]


def test_step_that_does_not_fit_changes_nothing():
    from megatron_mixtera_b200.inference.contexts import dynamic_context as D

    ctx = make_context(max_requests=4, tokens=320)
    step(ctx, [(0, [1] * 100), (1, [1] * 64), (2, [1]), (3, [1])])

    def state():
        return [a.clone() for a in ctx._request_arrays()] + [torch.tensor([ctx.total_request_count, ctx.chunk_allocator.chunk_count_avail])]

    before = state()
    for entries, err in (([(4, [1])], D.RequestOverflowError), ([(0, [1] * 157)], D.MaxSequenceLengthOverflowError),
                         ([(1, [1]), (2, [1] * 64)], D.ChunkOverflowError), ([(0, [1]), (0, [2])], ValueError), ([(0, [])], ValueError),
                         ([(0, [1] * 513)], D.TokenOverflowError)):
        with pytest.raises(err):
            ctx.schedule_tokens(entries)
        assert all(torch.equal(a, b) for a, b in zip(before, state()))
    step(ctx, [(0, [1] * 28)])
    with pytest.raises(KeyError):
        ctx.complete_step([99])


def test_state_slots_follow_requests_through_generation():
    """`update_requests` with finishing, pausing and compaction: every row keeps its slot, and reads what it last wrote."""
    ctx = make_context(max_requests=4, tokens=576, max_len=192)
    rng = np.random.default_rng(0)
    last, next_id, done = {}, 0, 0
    while done < 30:
        while next_id < 34 and ctx.total_request_count < 4:
            try:
                ctx.add_request(next_id, torch.arange(int(rng.integers(1, 66))), 40)
            except Exception:
                break
            next_id += 1
        for _ in range(2):  # initialising twice (a repeated forward) changes nothing
            ctx.initialize_attention_state()
        p, t = ctx.paused_request_count, ctx.total_request_count
        ids = ctx.request_ids[p:t].tolist()
        rd, wr = ctx.state_read_slots[: t - p].tolist(), ctx.state_write_slots[: t - p].tolist()
        for i, r, w in zip(ids, rd, wr):
            assert r == last.get(i, -1), (i, r, last.get(i))
            last[i] = w
        assert len(set(wr)) == len(wr) and not set(wr) & {s for j, s in last.items() if j not in ids}
        n = t - p
        mask = (rng.random(n) > 0.15).astype(np.int64)
        if n and not mask.any() and ctx.paused_request_count:
            mask[0] = 1
        for i, keep in zip(ids, mask):
            if not keep:
                del last[i]
                done += 1
        ctx.update_requests(mask, np.ones(n, dtype=np.int64))
    assert len(ctx._free_state_slots) + ctx.total_request_count == 4


def test_reset_gives_everything_back():
    ctx = make_context()
    ctx.add_request(0, torch.arange(10), 5)
    ctx.reset()
    assert sorted(ctx._free_state_slots) == [0, 1, 2, 3] and int(ctx.request_state_slots.max()) == -1
    step(ctx, [(3, [1, 2])])


def test_latent_geometry_arguments():
    from megatron_mixtera_b200.inference.contexts.dynamic_context import DynamicInferenceContext as C

    kw = dict(params_dtype=torch.bfloat16, num_layers=3, kv_channels=0, num_attention_heads=0, max_sequence_length=128,
              buffer_size_gb=0.001, buffer_guaranteed_fraction=0.0, chunk_size_tokens=64, tensor_model_parallel_size=1, device="cpu",
              cache_mla_latent=True, max_requests_override=4, max_tokens_override=64)
    ctx = C(kv_lora_rank=48, qk_pos_emb_head_dim=16, **kw)
    assert [b.shape[1:] for b in ctx.latent_buffers] == [(64, 64)] * 3 and ctx.chunk_size_bytes == 2 * 64 * 64 * 3
    ctx = C(latent_row_widths=[0, 96, 0], **kw)
    assert ctx.latent_buffers[0] is None and ctx.latent_cache(2).shape[1:] == (64, 96)
    for bad in (dict(), dict(latent_row_widths=[32])):
        with pytest.raises(ValueError):
            C(**bad, **kw)


# ---------------------------------------------------------------------------------------------------------------------
# the numerics tests can see each mechanism
# ---------------------------------------------------------------------------------------------------------------------
def planted(name, gain, change):
    """Error that a changed configuration, weight or oracle function makes on the tests' own inputs."""
    cfg, rank = H.CONFIGS[name]
    w = H.weights(cfg, rank, seed=3, gain=gain)
    toks = H.tokens(161, cfg["vocab"], 10)
    want = H.oracle_logits(toks, cfg, w)
    c2, w2 = json.loads(json.dumps(cfg)), dict(w)
    change(c2, w2)
    return H.error(H.oracle_logits(toks, c2, w2), want)


def _each(cfg, kind, fn):
    for i, layer in enumerate(cfg["layers"]):
        if layer["type"] == kind:
            fn(i, layer["mixer"])


PLANTS = {
    "window one longer": lambda c, w: _each(c, "latent_attention", lambda i, m: m["mask"].update(size=m["mask"]["size"] + 1)),
    "window one shorter": lambda c, w: _each(c, "latent_attention", lambda i, m: m["mask"].update(size=m["mask"]["size"] - 1)),
    "frequencies not scaled": lambda c, w: _each(c, "latent_attention", lambda i, m: m["rot"].pop("scaling")),
    "ramp of another length": lambda c, w: _each(c, "latent_attention", lambda i, m: m["rot"]["scaling"].update(slow=0.2)),
    "scores scaled otherwise": lambda c, w: _each(c, "latent_attention", lambda i, m: m.update(scale=m["scale"] * 1.2)),
    "no head gate": lambda c, w: _each(c, "latent_attention", lambda i, m: w.update({f"l{i}.mix.g": w[f"l{i}.mix.g"] * 0})),
    "no removal": lambda c, w: _each(c, "general_delta", lambda i, m: w.update({f"l{i}.mix.a.b": w[f"l{i}.mix.a.b"] - 40})),
    "no decay bias": lambda c, w: _each(c, "general_delta", lambda i, m: w.update({f"l{i}.mix.w0": w[f"l{i}.mix.w0"] * 0})),
    "decay from its bias alone": lambda c, w: _each(c, "general_delta", lambda i, m: w.update({f"l{i}.mix.w2": w[f"l{i}.mix.w2"] * 0})),
    "a feed-forward left out": lambda c, w: c["layers"][0].update(mlp=None),
    "epsilon a thousand times larger": lambda c, w: c["norm"].update(eps=1e-2),
}


@pytest.mark.parametrize("what", list(PLANTS))
def test_planted_mistakes_exceed_the_limits(what):
    limit = 1e-4 if "epsilon" in what else 0.08  # the 32-bit limit / the bf16 one of the GPU tests
    assert planted("mixed", 1.0, PLANTS[what]) > limit * 1.5


def test_lost_state_and_wrong_slot_exceed_the_limits():
    """A state that is dropped, or taken from another request, at a portion's edge."""
    cfg, rank = H.CONFIGS["mixed"]
    w = {k: v.double() for k, v in H.weights(cfg, rank, seed=3).items()}
    m = cfg["layers"][0]["mixer"]
    h = Z.layer_norm(w["embed"][torch.tensor(H.tokens(161, cfg["vocab"], 10))], w["embed.norm"], 1e-5)
    ins = Z.delta_inputs(h, w, "l0.mix", m)
    whole, _ = Z.delta_scan(*ins)
    cut = 64
    first, S = Z.delta_scan(*(x[:cut] for x in ins))
    good, _ = Z.delta_scan(*(x[cut:] for x in ins), state=S)
    assert (torch.cat([first, good]) - whole).abs().max() < 1e-9
    lost, _ = Z.delta_scan(*(x[cut:] for x in ins))
    scale = whole[cut:].square().mean().sqrt()
    assert (lost[0] - whole[cut]).square().mean().sqrt() / scale > 0.2
    assert (lost[-1] - whole[-1]).square().mean().sqrt() / scale > 1e-3  # some channels remember 97 tokens


def test_scaling_factor_of_the_rotation():
    freq, mag = Z.rope_frequencies({"base": 10000.0, "dims": 8, "scaling": {"factor": 4.0, "original": 1e9, "fast": 2.0, "slow": 1.0}})
    assert mag == pytest.approx(0.1 * math.log(4.0) + 1.0)
    assert freq == pytest.approx([10000.0 ** (-2 * i / 8) for i in range(4)])  # everything turns often over such a context
    freq, _ = Z.rope_frequencies({"base": 10000.0, "dims": 8, "scaling": {"factor": 4.0, "original": 1.0, "fast": 2.0, "slow": 1.0}})
    assert freq[1:] == pytest.approx([10000.0 ** (-2 * i / 8) / 4.0 for i in range(1, 4)])
