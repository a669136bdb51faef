"""Maginex without a GPU: configuration, checkpoint names and layouts, bookkeeping, and mistakes planted in the oracle, which must
exceed the limits of the GPU tests."""
import copy
import math

import maginex_helpers as H
import pytest
import torch

from oracle import maginex_oracle as M

LIMIT_BF16, LIMIT_F32 = 0.06, 1e-4  # of tests/test_maginex_gpu.py


def build(name, dtype=torch.bfloat16, seed=1):
    from megatron_mixtera_b200 import model_registry as R

    cfg = H.CONFIGS[name] if isinstance(name, str) else name
    w = H.weights(cfg, seed=seed)
    return cfg, w, R.ARCHITECTURES["Maginex"](cfg, {k: tuple(v.shape) for k, v in w.items()}, dtype, 256)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", list(H.CONFIGS))
def test_checkpoint_names_and_config(name, dtype):
    """Every tensor of a checkpoint is asked for under its name and shape; every constant arrives where it is used."""
    cfg, w, model = build(name, dtype)
    want = model.checkpoint_tensors()
    mixing = [i for i, x in enumerate(cfg["layers"]) if x["mixer"].get("v_mix")]
    unused = {f"l{i}.mix.vmix" for i in mixing[:1]}
    assert set(want) == set(w) - unused and all(tuple(w[k].shape) == tuple(s) for k, s in want.items())
    model.load_checkpoint(w)
    model.load_checkpoint({k: v for k, v in w.items() if k not in unused})
    c = model.config
    assert (c.hidden_size, c.vocab_size, c.num_layers, c.input_taps) == (cfg["width"], cfg["vocab"], len(cfg["layers"]), cfg["canon"]["taps"])
    assert (c.embedding_scale, c.layernorm_epsilon, c.norm_offset, c.logit_scale) == (cfg["embedding"]["scale"], cfg["norm"]["eps"], 0.0, 1.0)
    for i, (layer, spec) in enumerate(zip(c.layers, cfg["layers"])):
        m, mlp, a = spec["mixer"], spec["mlp"], layer.mixer
        assert (layer.moe is not None) == (mlp is not None)
        if mlp is not None:
            assert (layer.moe.experts, layer.moe.top, layer.moe.expert.ff, layer.moe.expert.gated) == (
                mlp["router"]["experts"], mlp["router"]["top"], mlp["expert"]["ff"], False)
            assert (layer.moe.shared.ff if layer.moe.shared else None) == (mlp["shared"]["ff"] if mlp["shared"] else None)
        if spec["type"] == "latent_attention":
            assert (a.heads, a.dim, a.rot_dim, a.vdim, a.kv_rank, a.q_rank, a.scale, a.sink, a.gate, a.window) == (
                m["heads"], m["dim"], 0, m["vdim"], m["kv_rank"], m["q_rank"], m["scale"], True, "value", None)
        elif spec["type"] == "mingru":
            assert a.width == m["width"]
        else:
            assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.window, a.rot.dims, a.rot.base, a.rot.halves, a.rot.scaling) == (
                m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"], (m.get("mask") or {}).get("size"), m["rot"]["dims"], m["rot"]["base"], True, None)
            assert (a.sink, a.head_gate, a.gate, a.value_mix, a.keep_first, a.softcap) == (True, True, False, m["v_mix"], 0, None)
            assert model.layers[i].mixer.parts[0].first_values == (mixing[:1] == [i])


def test_loading_is_strict_but_ignores_what_nothing_reads():
    cfg, w, model = build("mixed")
    for bad in ({**w, "l0.mix.extra": w["embed"]}, {k: v for k, v in w.items() if k != "l2.mix.z.b"}, {**w, "embed": w["embed"][:-1]},
                {k: v for k, v in w.items() if k != "l3.mix.vmix"}, {**w, "l0.norm2": w["l0.norm1"]}):
        with pytest.raises((KeyError, ValueError)):
            model.load_checkpoint(bad)
    assert cfg["layers"][4]["mlp"] is None
    model.load_checkpoint({**w, "l4.canon2": w["l4.canon1"], "l5.mix.vmix": w["l3.mix.vmix"]})  # (no feed-forward; values that are not mixed)


def test_unknown_or_impossible_parts_are_refused():
    from megatron_mixtera_b200 import model_registry as R

    def config(edit):
        cfg = copy.deepcopy(H.CONFIGS["mixed"])
        edit(cfg)
        return R.maginex_config(cfg, {}, torch.float32)

    def setter(i, *path, value):
        def edit(cfg):
            at = cfg["layers"][i]
            for k in path[:-1]:
                at = at[k]
            at[path[-1]] = value
        return edit

    config(lambda cfg: None)
    for bad in (setter(0, "type", value="retention"), setter(1, "mlp", "kind", value="dense"), setter(0, "mixer", "kv_heads", value=4),
                setter(0, "mixer", "rot", value={"base": 100.0, "dims": 34}), setter(0, "mixer", "rot", value={"base": 100.0, "dims": 5}),
                setter(1, "mlp", "router", "top", value=7), setter(3, "mixer", "vdim", value=32), setter(0, "mixer", "mask", value={"size": 0}),
                lambda cfg: cfg.update(canon={"taps": 9})):
        with pytest.raises(ValueError):
            config(bad)


def test_parts_that_do_not_go_together_are_refused():
    from megatron_mixtera_b200.transformer import hybrid_config as C

    shared = C.ExpertConfig(8, gated=False)
    for bad in (lambda: C.LatentAttentionConfig(2, 8, 4, 8, 16, 1.0, q_rank=8), lambda: C.LatentAttentionConfig(2, 8, 0, 8, 16, 1.0, gate="column"),
                lambda: C.ExpertConfig(8, limit=1.0, gated=False), lambda: C.MoeConfig(4, 2, C.ExpertConfig(8), shared=shared, routing=C.ChosenSoftmaxRouting()),
                lambda: C.MoeConfig(4, 2, C.ExpertConfig(8), shared=C.ExpertConfig(8), routing=C.SoftmaxRouting()),
                lambda: C.GroupedAttentionConfig(2, 1, 8, 8, 1.0, diff=0.1, gate=True, head_gate=True),
                lambda: C.GroupedAttentionConfig(2, 1, 8, 8, 1.0, value_mix=True, kv_from=0),
                lambda: C.HybridConfig(8, 8, (C.HybridLayerConfig(C.GatedScanConfig(8)),), block="streams", input_taps=4),
                lambda: C.HybridConfig(8, 8, (C.HybridLayerConfig(C.GatedScanConfig(8), moe=C.MoeConfig(2, 1, shared, shared=shared, routing=C.ChosenSoftmaxRouting())),),
                                       block="streams")):
        with pytest.raises(ValueError):
            bad()


def test_fused_linears():
    """What is read as vectors starts at multiples of 8; what lies between and behind is zero; filters are kept tap by tap."""
    cfg, w, model = build("odd")
    model.load_checkpoint(w)
    mix = model.layers[0].mixer
    assert mix.offsets == {"dq": 0, "dkv": 24, "g": 48} and mix.linear_in.weight.shape[0] == 88
    W = mix.linear_in.weight
    for name, n in (("dq", 19), ("dkv", 21), ("g", 39)):
        assert torch.equal(W[mix.offsets[name]: mix.offsets[name] + n], w[f"l0.mix.{name}"])
    assert all(float(W[a:b].abs().max()) == 0.0 for a, b in ((19, 24), (45, 48), (87, 88)))
    assert torch.equal(mix.key_up.view(3, 21, 11)[1], w["l0.mix.uk"].view(3, 11, 21)[1].t()) and torch.equal(mix.value_up, w["l0.mix.uv"])
    W = model.layers[2].mixer.linear_in.weight
    assert torch.equal(W[60:120], w["l2.mix.k"]) and torch.equal(W[153:156], w["l2.mix.g"]) and W.shape[0] == 160 and float(W[156:].abs().max()) == 0.0
    assert torch.equal(model.layers[1].norm.filters[1], w["l1.canon2"].t()) and model.layers[3].norm.filters.shape[0] == 1
    moe = model.layers[1].moe
    assert moe.up.shape == (5, 64, 101) and torch.equal(moe.up[3, :9], w["l1.mlp.e3.up"]) and float(moe.up[:, 9:].abs().max()) == 0.0
    assert moe.shared_up is None and moe.router.shape[0] == 8 and torch.equal(moe.correction, w["l1.mlp.router.b"])
    assert torch.equal(model.layers[0].moe.shared_down[:, :13], w["l0.mlp.shared.down"])


def test_context_of_a_model():
    """Row widths and state parts of every layer; slots are handed out, swapped and given back for all parts together."""
    cfg, w, model = build("mixed")
    ctx = model.make_context(max_cached_tokens=512, max_requests_override=4, max_tokens_override=512, device="cpu", debug_validate=True)
    assert ctx.latent_row_widths == [2 * 56, 64, 0, 2 * 56, 0, 2 * 48, 96, 2 * 56]
    shapes = [{k: tuple(v.shape[1:]) for k, v in b.items()} for b in ctx.state_buffers]
    inputs = {"input": (2, 160)}
    assert shapes == [inputs, inputs, {"state": (72,), **inputs}, inputs, {"state": (104,), **inputs}, inputs, inputs, inputs]
    assert ctx.recurrent_state(3, "state").dtype == torch.float32 and ctx.recurrent_state(3, "input").dtype == torch.bfloat16
    ctx.set_prefill_q_block(*model.prefill_unit_tokens())
    for entries, gone in (([(0, [1] * 70), (1, [2])], []), ([(1, [3])], [1]), ([(2, [4] * 5), (0, [1])], [0]), ([(2, [4])], [2])):
        ctx.schedule_tokens(entries)
        ctx.initialize_attention_state()
        n = len(entries)
        read, write = ctx.state_read_slots[:n].tolist(), ctx.state_write_slots[:n].tolist()
        assert not set(write) & {r for r in read if r >= 0} and len(set(write)) == n
        ctx.complete_step(gone)
    assert sorted(ctx._free_state_slots) == list(range(ctx.num_state_slots))


def test_models_without_state_or_rows():
    """A filter of one tap keeps nothing, a model may cache nothing: the context still counts and numbers its slots."""
    for layers, taps in (([H.windowed()], 1), ([H.mingru()], 4), ([H.latent()], 1)):
        cfg, w, model = build(H.config(layers, taps=taps), torch.float32)
        ctx = model.make_context(max_cached_tokens=256, max_requests_override=4, max_tokens_override=128, device="cpu", debug_validate=True)
        ctx.schedule_tokens([(0, [1, 2, 3])])
        ctx.initialize_attention_state()
        assert int(ctx.state_write_slots[0]) >= 0
        ctx.complete_step([0])
        assert ctx.chunk_allocator.chunk_count_avail == 4


def test_work_lists_of_several_block_sizes():
    assert build("mixed")[2].prefill_unit_tokens() == [64, 32, 21, 16, 12]
    assert build("odd")[2].prefill_unit_tokens() == [16] and build("mixed", torch.float32)[2].prefill_unit_tokens() == [16]
    assert build("scans")[2].prefill_unit_tokens() == [0]


def test_expanded_keys_in_whole_chunks():
    """Rows of expanded keys start at whole chunks, the block table walks them in order, and the table says where a row's keys end."""
    _, _, model = build("latents")
    ctx = model.make_context(max_cached_tokens=1024, max_requests_override=4, max_tokens_override=512, device="cpu")
    ctx.set_prefill_q_block(*model.prefill_unit_tokens())
    ctx.schedule_tokens([(0, [1] * 130), (1, [2] * 5)])
    ctx.initialize_attention_state()
    plain, total = ctx.expanded_keys(None)
    assert total == 135 and plain[0].tolist() == [0, 130, 135]
    table, total, blocks = ctx.expanded_keys(None, 64)
    assert total == 256 and table.tolist() == [[0, 192, 256], [0, 0, 0], [130, 5, 0]] and blocks.tolist() == [[0, 1, 2], [3, 3, 3]]
    ctx.complete_step()
    ctx.schedule_tokens([(1, [2] * 60), (0, [1] * 100)])
    ctx.initialize_attention_state()
    table, total, blocks = ctx.expanded_keys(None, 64)
    order = [65, 230] if table[2, 0] == 65 else [230, 65]
    assert table[2, :2].tolist() == order and total == 64 * (2 + 4) and blocks.shape == (2, 4)
    assert sorted(set(blocks.flatten().tolist())) == list(range(6)) and table[0, -1] == total
    ctx.complete_step()
    ctx.schedule_tokens([(0, [1] * 2)])  # (a long past and few queries: not worth it)
    ctx.initialize_attention_state()
    assert ctx.expanded_keys(None, 64) is None


# ---------------------------------------------------------------------------------------------------------------------
def planted():
    """name -> a function that puts one mistake into the oracle."""
    def set_(name, fn):
        return lambda mp: mp.setattr(M, name, fn)

    attend, visible, rotate, rms, filt, choose, scan, latent, attention, experts, mingru, ff = (
        M.attend, M.visible, M.rotate_halves, M.rms_norm, M.causal_filter, M.choose, M.gated_scan, M.latent_attention, M.attention, M.experts, M.mingru,
        M.squared_relu_ff)

    def grouped_wrong(q, k, v, scale, size, sink):
        g = q.shape[1] // k.shape[1]
        return attend(q, k.repeat(1, g, 1), v.repeat(1, g, 1), scale, size, sink)

    def pairs_next(x, base, dims):
        out, freq = x.clone(), torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=x.dtype)
        a = torch.arange(x.shape[0], dtype=x.dtype)[:, None] * freq
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        out[..., 0:dims:2], out[..., 1:dims:2] = x[..., 0:dims:2] * c - x[..., 1:dims:2] * s, x[..., 1:dims:2] * c + x[..., 0:dims:2] * s
        return out

    def with_weights(fn, **change):
        """The mechanism with some of its tensors changed."""
        def wrapped(h, w, p, *a):
            return fn(h, {**w, **{p + n: f(w[p + n]) for n, f in change.items() if p + n in w}}, p, *a)
        return wrapped

    def gate_per_head(h, w, p, m, eps):
        g = w[p + "g"].view(m["heads"], m["vdim"], -1)
        return latent(h, {**w, p + "g": g[:, :1].expand_as(g).reshape(w[p + "g"].shape)}, p, m, eps)

    def first_mixed_too(h, w, p, m, carried):
        if m.get("v_mix") and "first" not in carried:
            attention(h, w, p, m, carried)
            carried["first"] = carried["first"] * 0.5
        return attention(h, w, p, m, carried)

    def first_not_carried(h, w, p, m, carried):
        return attention(h, w, p, {**m, "v_mix": False}, carried)

    def lose_state(z, c, state=None):  # a state that starts anew every 64 tokens
        return torch.cat([scan(z[i: i + 64], c[i: i + 64]) for i in range(0, len(z), 64)])

    def lose_inputs(h, taps):  # filters that start anew every 64 tokens
        return torch.cat([filt(h[i: i + 64], taps) for i in range(0, len(h), 64)])

    def weights_of_all(z, top):
        chosen, _ = choose(z, top)
        return chosen, torch.softmax(z, -1).gather(1, chosen)

    def bias_in_choice_only(x, w, p, mlp):
        def pick(z, top):
            chosen, _ = choose(z, top)
            return chosen, torch.softmax((z - w[p + "router.b"]).gather(1, chosen), -1)
        M.choose = pick
        try:
            return experts(x, w, p, mlp)
        finally:
            M.choose = choose

    return {
        "window one short": set_("visible", lambda n, s: visible(n, s if s is None else max(s - 1, 1))),
        "window one long": set_("visible", lambda n, s: visible(n, s if s is None else s + 1)),
        "no window": set_("visible", lambda n, s: visible(n, None)),
        "window on latents": set_("attend", lambda q, k, v, sc, size, sink: attend(q, k, v, sc, 64 if size is None else size, sink)),
        "head groups interleaved": set_("attend", grouped_wrong),
        "no sink": set_("attend", lambda q, k, v, sc, size, sink: attend(q, k, v, sc, size, sink - 1e4)),
        "sink scaled": set_("attend", lambda q, k, v, sc, size, sink: attend(q, k, v, sc, size, sink * sc)),
        "sink counted twice": set_("attend", lambda q, k, v, sc, size, sink: attend(q, k, v, sc, size, sink + math.log(2))),
        "scale from the size": set_("attend", lambda q, k, v, sc, size, sink: attend(q, k, v, q.shape[-1] ** -0.5, size, sink)),
        "neighbours rotate": set_("rotate_halves", pairs_next),
        "rotation turns all": set_("rotate_halves", lambda x, b, d: rotate(x, b, x.shape[-1])),
        "rotation one position late": set_("rotate_halves", lambda x, b, d: rotate(torch.cat([x[:1], x]), b, d)[1:] if x.shape[1] == 2 else rotate(x, b, d)),
        "values not mixed": set_("mixed_values", lambda v, first, share: v),
        "shares of the mixing swapped": set_("mixed_values", lambda v, first, share: v if first is None else share * v + (1 - share) * first),
        "first layer's values mixed": set_("attention", first_mixed_too),
        "values of the layer before": set_("attention", first_not_carried),
        "no head gate": set_("attention", with_weights(attention, g=lambda t: t * 0)),
        "no value gate": set_("latent_attention", with_weights(latent, g=lambda t: t * 0)),
        "value gate per head": set_("latent_attention", gate_per_head),
        "no query norm weight": set_("latent_attention", with_weights(latent, **{"dq.norm": torch.ones_like})),
        "no latent norm weight": set_("latent_attention", with_weights(latent, **{"dkv.norm": torch.ones_like})),
        "norm with one added": set_("rms_norm", lambda x, w, eps: rms(x, w + 1, eps)),
        "norm without the root": set_("rms_norm", lambda x, w, eps: x / ((x * x).mean(-1, keepdim=True) + eps) * w),
        "no filters": set_("causal_filter", lambda h, t: h * 0),
        "filter backwards": set_("causal_filter", lambda h, t: filt(h, t.flip(-1))),
        "filter one tap short": set_("causal_filter", lambda h, t: filt(h, torch.cat([t[:, :1] * 0, t[:, 1:]], 1))),
        "filter instead of sum": set_("mixed_with_past", lambda h, t: filt(h, t)),
        "filters lose their inputs": set_("causal_filter", lose_inputs),
        "state lost": set_("gated_scan", lose_state),
        "update gate the other way": set_("gated_scan", lambda z, c, s=None: scan(1 - z, c, s)),
        "candidate plain": set_("candidate_of", lambda u: u),
        "candidate sigmoid": set_("candidate_of", torch.sigmoid),
        "candidate without its half": set_("candidate_of", lambda u: torch.where(u >= 0, u, torch.sigmoid(u))),
        "no update bias": set_("mingru", with_weights(mingru, **{"z.b": torch.zeros_like})),
        "no input bias": set_("mingru", with_weights(mingru, **{"x.b": torch.zeros_like})),
        "sigmoid instead of silu": set_("silu", torch.sigmoid),
        "relu not squared": set_("squared_relu_ff", lambda x, w, p: torch.relu(x @ w[p + ".up"].T) @ w[p + ".down"].T),
        "no shared expert": set_("squared_relu_ff", lambda x, w, p: ff(x, w, p) * (0.0 if p.endswith("shared") else 1.0)),
        "softmax over all experts": set_("choose", weights_of_all),
        "experts weigh the same": set_("choose", lambda z, top: (choose(z, top)[0], torch.full((z.shape[0], top), 1.0 / top, dtype=z.dtype))),
        "router bias in the choice only": set_("experts", bias_in_choice_only),
        "one expert fewer": set_("choose", lambda z, top: choose(z, max(top - 1, 1))),
    }


SUBTLE = {"window one short", "window one long", "first layer's values mixed", "one expert fewer", "norm without the root", "no input bias",
          "rotation turns all", "window on latents", "sink counted twice", "no query norm weight", "softmax over all experts"}


@pytest.mark.parametrize("mistake", list(planted()))
def test_planted_mistakes_exceed_the_limits(mistake, monkeypatch):
    """A mistake in one mechanism moves the 32-bit logits far beyond the GPU tests' limit, and nearly all of them the 16-bit ones too."""
    cfg = H.CONFIGS["mixed"]
    toks = H.tokens(130, cfg["vocab"], 10)
    base = {s: H.weights(cfg, seed=3, gain=1.6, settled=s) for s in (False, True)}
    want = {s: H.oracle_logits(toks, cfg, w) for s, w in base.items()}
    planted()[mistake](monkeypatch)
    e32, e16 = (H.position_errors(H.oracle_logits(toks, cfg, base[s]), want[s]) for s in (False, True))
    assert float(e32.max()) > 100 * LIMIT_F32, float(e32.max())
    if mistake not in SUBTLE:
        assert float((e16 > LIMIT_BF16).float().mean()) > 0.03 or float(e16.max()) > 3 * LIMIT_BF16, e16.topk(8)


def test_oracle_portions():
    """The oracle's own recurrence carries a state: two halves give what the whole gives; maps of tokens compose."""
    g = torch.Generator().manual_seed(0)
    z, c = torch.rand(30, 5, dtype=torch.float64, generator=g), torch.randn(30, 5, dtype=torch.float64, generator=g)
    whole = M.gated_scan(z, c)
    a = M.gated_scan(z[:11], c[:11])
    assert torch.allclose(torch.cat([a, M.gated_scan(z[11:], c[11:], a[-1])]), whole)
    keep, add = torch.ones(5, dtype=torch.float64), torch.zeros(5, dtype=torch.float64)
    for t in range(30):
        keep, add = (1 - z[t]) * keep, (1 - z[t]) * add + z[t] * c[t]
    assert torch.allclose(keep * 3.0 + add, M.gated_scan(z, c, torch.full((5,), 3.0, dtype=torch.float64))[-1])
