"""Fabivik without a GPU: configuration, checkpoint names and layouts, bookkeeping, and mistakes planted in the oracle, which must
exceed the limits of the GPU tests."""
import copy
import math

import fabivik_helpers as H
import pytest
import torch

from oracle import fabivik_oracle as F

LIMIT_BF16, LIMIT_F32 = 0.08, 1e-4  # of tests/test_fabivik_gpu.py


def build(name, dtype=torch.bfloat16, seed=1, **edit):
    from megatron_mixtera_b200 import model_registry as R

    cfg = H.CONFIGS[name]
    w = H.weights(cfg, seed=seed)
    return cfg, w, R.ARCHITECTURES["Fabivik"](cfg, {k: tuple(v.shape) for k, v in w.items()}, dtype, 256)


@pytest.mark.parametrize("seed", [0, 1])
@pytest.mark.parametrize("name", list(H.CONFIGS))
def test_checkpoint_names_and_config(name, seed):
    """Every tensor of a checkpoint is asked for under its name and shape, whether or not it holds the first layer's unused mix."""
    cfg, w, model = build(name, seed=seed)
    want = model.checkpoint_tensors()
    assert set(want) <= set(w) and set(w) - set(want) <= model.ignored_tensors()
    assert all(tuple(w[k].shape) == tuple(s) for k, s in want.items())
    model.load_checkpoint(w)
    c = model.config
    assert (c.hidden_size, c.vocab_size, c.num_layers) == (cfg["width"], cfg["vocab"], len(cfg["layers"]))
    assert (c.embedding_scale, c.logit_scale, c.layernorm_epsilon) == (cfg["embedding"]["scale"], cfg["logit_scale"], cfg["norm"]["eps"])
    for layer, spec in zip(c.layers, cfg["layers"]):
        assert (layer.moe is None) == (spec["mlp"] is None)
        if spec["mlp"]:
            assert (layer.moe.experts, layer.moe.top) == (spec["mlp"]["router"]["experts"], spec["mlp"]["router"]["top"])
            assert layer.moe.expert.limit == spec["mlp"]["expert"]["limit"] and (layer.moe.shared is None) == (spec["mlp"]["shared"] is None)


def test_loading_is_strict():
    _, w, model = build("mixed")
    for bad in ({**w, "l0.mix.extra": w["embed"]}, {k: v for k, v in w.items() if k != "l1.mix.u"}, {**w, "head": w["embed"][:-1]}):
        with pytest.raises((KeyError, ValueError)):
            model.load_checkpoint(bad)


def test_unknown_parts_are_refused():
    from megatron_mixtera_b200 import model_registry as R

    for path, value in ((("type",), "retention"), (("mlp", "kind"), "dense")):
        cfg = copy.deepcopy(H.CONFIGS["attention_only"])
        at = cfg["layers"][0]
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        with pytest.raises(ValueError):
            R.fabivik_config(cfg, {}, torch.float32)
    cfg = H.config([H.attention(), H.attention(kv_heads=3)])
    with pytest.raises(ValueError):  # values of different shapes cannot be mixed
        R.fabivik_config(cfg, {}, torch.float32)
    with pytest.raises(ValueError):
        R.fabivik_config(H.config([H.attention(conv=9)]), {}, torch.float32)


def test_expert_weight_layout():
    """Blocks of 16 gate rows and the 16 matching up rows, padded with zero rows; down columns of the padding are zero."""
    from megatron_mixtera_b200.transformer.moe import interleave_up

    gate, up = torch.randn(100, 8), torch.randn(100, 8)
    x = interleave_up(gate, up)
    assert x.shape == (256, 8)
    x = x.view(8, 2, 16, 8)
    for i, w in enumerate((gate, up)):
        assert torch.equal(x[:, i].reshape(128, 8)[:100], w) and float(x[:, i].reshape(128, 8)[100:].abs().max()) == 0.0
    _, w, model = build("wide")
    model.load_checkpoint(w)
    moe = model.layers[0].moe
    assert torch.equal(moe.down[3, :, :100], w["l0.mlp.e3.down"]) and float(moe.down[:, :, 100:].abs().max()) == 0.0
    assert torch.equal(moe.router[40], w["l0.mlp.shared.sg"][0]) and moe.router.shape[0] == 48


def test_tiles_cover_every_split_of_the_tokens():
    """The bound on the tile list holds however the pairs fall on the experts."""
    from megatron_mixtera_b200.transformer.moe import MixtureOfExperts

    for pairs, experts in ((1, 1), (7, 40), (64, 3), (5000, 8), (5000, 100), (65536, 64)):
        tile = MixtureOfExperts.tile_tokens(pairs, experts, False)
        bound = pairs // tile + min(experts, pairs)
        g = torch.Generator().manual_seed(pairs)
        for split in ([pairs] + [0] * (experts - 1), torch.bincount(torch.randint(0, experts, (pairs,), generator=g), minlength=experts).tolist(),
                      [1] * min(experts, pairs) + [0] * (experts - min(experts, pairs))):
            split[0] += pairs - sum(split)
            assert sum(-(-n // tile) for n in split) <= bound


def test_context_of_a_model():
    """Row widths and state parts of every layer; slots are handed out, swapped and given back for all parts together."""
    cfg, w, model = build("mixed")
    ctx = model.make_context(max_cached_tokens=512, max_requests_override=4, max_tokens_override=512, device="cpu", debug_validate=True)
    assert ctx.latent_row_widths == [2 * 64, 0, 2 * 64, 0, 4 * 32, 0]
    shapes = [{k: tuple(v.shape[1:]) for k, v in b.items()} for b in ctx.state_buffers]
    assert shapes == [{"conv": (3, 6 * 24 + 2 * 64)}, {"state": (3, 40, 40), "shift": (160,)}, {"conv": (3, 2 * 24 + 2 * 64)},
                      {"state": (6, 48, 32), "conv": (3, 2 * 3 * 32 + 6 * 48)}, {"conv": (2, 4 * 16 * 3)}, {"state": (2, 64, 64), "shift": (160,)}]
    assert ctx.recurrent_state(2, "state").dtype == torch.float32 and ctx.recurrent_state(2, "shift").dtype == torch.bfloat16
    assert ctx.recurrent_state(2, "conv") is None
    ctx.set_prefill_q_block(*model.prefill_unit_tokens())
    seen = set()
    for step, (entries, gone) in enumerate([([(0, [1] * 70), (1, [2])], []), ([(1, [3])], [1]), ([(2, [4] * 5), (0, [1])], [0]), ([(2, [4])], [2])]):
        ctx.schedule_tokens(entries)
        ctx.initialize_attention_state()
        n = len(entries)
        read, write = ctx.state_read_slots[:n].tolist(), ctx.state_write_slots[:n].tolist()
        assert not set(write) & {r for r in read if r >= 0} and len(set(write)) == n
        seen |= set(write)
        ctx.complete_step(gone)
    assert sorted(ctx._free_state_slots) == list(range(ctx.num_state_slots))


def test_models_without_state_or_rows():
    """No convolution memory, or nothing cached: the context still counts and numbers its slots."""
    for layers in ([H.attention(conv=1)], [H.wkv()], [H.delta(conv=1)]):
        from megatron_mixtera_b200 import model_registry as R

        cfg = H.config(layers)
        w = H.weights(cfg)
        model = R.ARCHITECTURES["Fabivik"](cfg, {k: tuple(v.shape) for k, v in w.items()}, torch.float32, 128)
        ctx = model.make_context(max_cached_tokens=256, max_requests_override=4, max_tokens_override=128, device="cpu", debug_validate=True)
        ctx.schedule_tokens([(0, [1, 2, 3])])
        ctx.initialize_attention_state()
        assert int(ctx.state_write_slots[0]) >= 0
        ctx.complete_step([0])
        assert ctx.chunk_allocator.chunk_count_avail == 4


def test_work_lists_of_several_block_sizes():
    """Layers that group their heads differently read lists cut for their own blocks."""
    _, _, model = build("mixed")
    assert model.prefill_unit_tokens() == [64, 21]
    ctx = model.make_context(max_cached_tokens=512, max_requests_override=4, max_tokens_override=512, device="cpu")
    ctx.set_prefill_q_block(*model.prefill_unit_tokens())
    ctx.schedule_tokens([(0, [1] * 50), (1, [2]), (2, [3] * 64)])
    ctx.initialize_attention_state()
    for qb, want in ((64, [(0, 0, 50), (1, 50, 1), (2, 51, 64)]),
                     (21, [(0, 0, 21), (0, 21, 21), (0, 42, 8), (1, 50, 1), (2, 51, 21), (2, 72, 21), (2, 93, 21), (2, 114, 1)])):
        units, n = ctx.prefill_units_of(qb)
        assert [tuple(u[:3]) for u in units[:n].tolist()] == want


# ---------------------------------------------------------------------------------------------------------------------
def planted():
    """name -> a function that puts one mistake into the oracle."""
    def set_(name, fn):
        return lambda mp: mp.setattr(F, name, fn)

    attend, short_conv, expert, mixture, wkv_scan, delta_inputs, wkv_inputs = (
        F.attend, F.short_conv, F.expert, F.mixture, F.wkv_scan, F.delta_inputs, F.wkv_inputs)

    def grouped_wrong(q, k, v, scale, size):
        g = q.shape[1] // k.shape[1]
        return attend(q, k.repeat(1, g, 1), v.repeat(1, g, 1), scale, size)

    def output_weighted(h, w, p, m):
        return sum_experts(h, w, p, m, lambda s, x, q, lim: s * expert(x, w, q, lim))

    def renormalised(h, w, p, m):
        return sum_experts(h, w, p, m, lambda s, x, q, lim: expert(s * x, w, q, lim), renorm=True)

    def sum_experts(h, w, p, m, apply, renorm=False):
        score = torch.sigmoid(h @ w[p + ".router"].T)
        out = torch.zeros_like(h)
        for t in range(h.shape[0]):
            top = torch.topk(score[t], m["router"]["top"])
            total = top.values.sum() if renorm else 1.0
            for s, e in zip(top.values, top.indices.tolist()):
                out[t] += apply(s / total, h[t], f"{p}.e{e}", m["expert"]["limit"])
        if m.get("shared"):
            out = out + torch.sigmoid(h @ w[p + ".shared.sg"].T) * expert(h, w, p + ".shared", m["shared"]["limit"])
        return out

    def ungated(h, w, p, m):
        return mixture(h, w, p, {**m, "shared": None}) + (expert(h, w, p + ".shared", m["shared"]["limit"]) if m.get("shared") else 0)

    def swapped_taps(u, taps):
        return short_conv(u, taps.flip(1))

    def late_decay(q, k, v, beta, decay, state=None):  # writes before it forgets
        T, Hd, d = q.shape
        S, out = torch.zeros(Hd, d, v.shape[2], dtype=q.dtype), torch.empty_like(v)
        for t in range(T):
            u = beta[t][:, None] * (v[t] - torch.einsum("hij,hi->hj", S, k[t]))
            S = decay[t][:, None, None] * (S + k[t][:, :, None] * u[:, None, :])
            out[t] = torch.einsum("hij,hi->hj", S, q[t])
        return out, S

    return {
        "window one short": set_("visible", lambda n, size: (a := torch.arange(n)[:, None] - torch.arange(n)[None]) * 0 + ((a >= 0) & (a < (size or n + 2) - 1) | (a == 0)) > 0),
        "window one long": set_("visible", lambda n, size: (a := torch.arange(n)[:, None] - torch.arange(n)[None]) * 0 + ((a >= 0) & (a < (size or n) + 1)) > 0),
        "head groups interleaved": set_("attend", grouped_wrong),
        "no convolution memory": set_("short_conv", lambda u, taps: u * taps[:, -1]),
        "taps reversed": set_("short_conv", swapped_taps),
        "no token shift": set_("shifted", lambda h: h),
        "shift without zeros at the start": set_("shifted", lambda h: torch.cat([h[:1], h[:-1]])),
        "no bonus": set_("wkv_scan", lambda r, k, v, decay, bonus, state=None: wkv_scan(r, k, v, decay, torch.ones_like(bonus))),
        "delta decays after the write": set_("delta_scan", late_decay),
        "delta query not scaled": set_("delta_inputs", lambda h, w, p, m: (lambda q, *r: (q * 3.0, *r))(*delta_inputs(h, w, p, m))),
        "delta step size one": set_("delta_inputs", lambda h, w, p, m: (lambda q, k, v, b, g: (q, k, v, torch.ones_like(b), g))(*delta_inputs(h, w, p, m))),
        "weight on the expert's output": set_("mixture", output_weighted),
        "weights renormalised": set_("mixture", renormalised),
        "shared expert not gated": set_("mixture", ungated),
        "no limit": set_("expert", lambda x, w, p, limit: expert(x, w, p, 1e9)),
        "norm without the one": set_("layer_norm", lambda x, weight, eps: F.unit_rms(x, eps) * (weight + 0.8)),
    }


@pytest.mark.parametrize("mistake", list(planted()))
def test_planted_mistakes_exceed_the_limits(mistake, monkeypatch):
    """A mistake in one mechanism moves the 32-bit logits far beyond the GPU tests' limit everywhere, and the 16-bit ones beyond what
    those tests let pass.  (Two are invisible in some places: a query's scale before a norm, the first token's shift.)"""
    cfg = H.CONFIGS["mixed"]
    w = H.weights(cfg, seed=3)
    toks = H.tokens(90, cfg["vocab"], 10)
    want = H.oracle_logits(toks, cfg, w)
    planted()[mistake](monkeypatch)
    e = H.position_errors(H.oracle_logits(toks, cfg, w), want)
    if mistake == "delta query not scaled":  # the head norm divides it out, but for eps
        assert float(e.max()) > LIMIT_F32 / 10
    elif mistake == "shift without zeros at the start":
        assert float(e[0]) > 10 * LIMIT_F32
    else:
        assert float(e.max()) > 100 * LIMIT_F32
        assert float((e > LIMIT_BF16).float().mean()) > 0.06 or float(e.median()) > LIMIT_BF16 / 2, (e.max(), e.median())


def test_oracle_portions():
    """The oracle's own recurrences carry a state: two halves give what the whole gives."""
    cfg = H.CONFIGS["mixed"]
    w = {k: v.double() for k, v in H.weights(cfg, seed=3).items()}
    h = torch.randn(30, cfg["width"], dtype=torch.float64, generator=torch.Generator().manual_seed(0))
    r, k, v, d, _ = F.wkv_inputs(h, w, "l1.mix", cfg["layers"][1]["mixer"])
    whole, last = F.wkv_scan(r, k, v, d, w["l1.mix.u"])
    a, S = F.wkv_scan(r[:11], k[:11], v[:11], d[:11], w["l1.mix.u"])
    b, S = F.wkv_scan(r[11:], k[11:], v[11:], d[11:], w["l1.mix.u"], S)
    assert torch.allclose(torch.cat([a, b]), whole) and torch.allclose(S, last)
    x = F.delta_inputs(h, w, "l3.mix", cfg["layers"][3]["mixer"])
    whole, last = F.delta_scan(*x)
    a, S = F.delta_scan(*(y[:11] for y in x))
    b, S = F.delta_scan(*(y[11:] for y in x), S)
    assert torch.allclose(torch.cat([a, b]), whole) and torch.allclose(S, last)
    assert math.isfinite(float(last.abs().max()))
