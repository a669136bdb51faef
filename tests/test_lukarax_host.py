"""Lukarax without a GPU: configuration, checkpoint names and layouts, bookkeeping, and mistakes planted in the oracle, which must
exceed the limits of the GPU tests."""
import copy
import math

import lukarax_helpers as H
import pytest
import torch

from oracle import lukarax_oracle as L

LIMIT_BF16, LIMIT_F32 = 0.08, 1e-4  # of tests/test_lukarax_gpu.py


def build(name, dtype=torch.bfloat16, seed=1):
    from megatron_mixtera_b200 import model_registry as R

    cfg = H.CONFIGS[name] if isinstance(name, str) else name
    w = H.weights(cfg, seed=seed)
    return cfg, w, R.ARCHITECTURES["Lukarax"](cfg, {k: tuple(v.shape) for k, v in w.items()}, dtype, 256)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", list(H.CONFIGS))
def test_checkpoint_names_and_config(name, dtype):
    """Every tensor of a checkpoint is asked for under its name and shape; every constant arrives where it is used."""
    cfg, w, model = build(name, dtype)
    want = model.checkpoint_tensors()
    assert set(want) == set(w) and all(tuple(w[k].shape) == tuple(s) for k, s in want.items())
    model.load_checkpoint(w)
    c = model.config
    assert (c.hidden_size, c.vocab_size, c.num_layers, c.streams) == (cfg["width"], cfg["vocab"], len(cfg["layers"]), cfg["streams"])
    assert (c.embedding_scale, c.layernorm_epsilon) == (cfg["embedding"]["scale"], cfg["norm"]["eps"])
    for i, (layer, spec) in enumerate(zip(c.layers, cfg["layers"])):
        m, mlp = spec["mixer"], spec["mlp"]
        assert (layer.moe is not None) == (mlp is not None and mlp["kind"] == "moe")
        assert layer.ffn_hidden_size == (mlp["ff"] if mlp and mlp["kind"] == "dense" else None)
        if layer.moe is not None:
            r, q = layer.moe.routing, mlp["router"]
            assert (layer.moe.experts, layer.moe.top, r.identity, r.groups, r.keep_groups, r.scale, layer.moe.expert.ff) == (
                q["experts"], q["top"], q["identity"], q["groups"]["count"], q["groups"]["keep"], q["scale"], mlp["expert"]["ff"])
        if spec["type"] == "attention":
            a = layer.mixer
            assert (a.diff, a.maps, a.gate, a.rot.dims, a.rot.base, a.rot.halves, a.kv_from, a.scale) == (
                m["diff"], 2, True, m["rot"]["dims"], m["rot"]["base"], False, m.get("kv_from"), m["scale"])
            part = model.layers[i].mixer.parts[0]
            wd = {k: v.double() for k, v in w.items()}
            assert abs(part.lambda_ - float(L.differential_lambda(wd, f"l{i}.mix", m))) < 1e-12
        elif spec["type"] == "attention_2":
            a = layer.mixer
            assert (a.window, a.softcap, a.sink, a.values_from_keys, a.rot.halves, a.rot.scaling.factor, a.keep_first) == (
                m["mask"]["size"], m["softcap"], True, True, True, m["rot"]["scaling"]["factor"], 0)
        else:
            (_, a, left), (_, r, right) = layer.mixer.parts
            assert (left, right, a.window, a.keep_first, r.gate_cap, r.dim, r.vdim) == (
                m["left_scale"], m["right_scale"], m["left"]["mask"]["size"], m["left"]["mask"]["keep_first"], m["right"]["gate_cap"],
                m["right"]["dim"], m["right"]["vdim"])
            assert (a.distance_bias.rows, a.distance_bias.longest) == (spec["bias_rows"], m["left"]["bias_max"])


def test_loading_is_strict_but_ignores_what_a_missing_feed_forward_leaves():
    cfg, w, model = build("mixed")
    for bad in ({**w, "l0.mix.extra": w["embed"]}, {k: v for k, v in w.items() if k != "l1.mix.right.f.b"}, {**w, "embed": w["embed"][:-1]},
                {**w, "l3.mix.k": w["l0.mix.k"]}):  # (rows of another layer: no keys of its own)
        with pytest.raises((KeyError, ValueError)):
            model.load_checkpoint(bad)
    assert cfg["layers"][4]["mlp"] is None
    model.load_checkpoint({**w, "l4.norm2": w["l0.norm2"], "l4.norm2.b": w["l0.norm2.b"]})


def test_unknown_or_impossible_parts_are_refused():
    from megatron_mixtera_b200 import model_registry as R

    def config(edit):
        cfg = copy.deepcopy(H.CONFIGS["mixed"])
        edit(cfg)
        w = H.weights(H.CONFIGS["mixed"])
        return R.lukarax_config(cfg, {k: tuple(v.shape) for k, v in w.items()}, torch.float32)

    def setter(i, *path, value):
        def edit(cfg):
            at = cfg["layers"][i]
            for k in path[:-1]:
                at = at[k]
            at[path[-1]] = value
        return edit

    config(lambda cfg: None)
    for bad in (setter(0, "type", value="retention"), setter(1, "mlp", "kind", value="sparse"), setter(3, "mixer", "kv_from", value=1),
                setter(3, "mixer", "kv_from", value=3), setter(3, "mixer", "dim", value=32), setter(0, "mixer", "kv_heads", value=4),
                setter(1, "mlp", "router", "groups", value={"count": 3, "keep": 1}), setter(1, "mlp", "router", "top", value=5),
                setter(0, "mixer", "rot", value={"base": 100.0, "dims": 26}), lambda cfg: cfg.update(streams=17)):
        with pytest.raises(ValueError):
            config(bad)


def test_without_streams_the_residual_is_plain():
    """No streams in the configuration: no blend weights in the checkpoint, and the ordinary residual sum."""
    cfg = copy.deepcopy(H.CONFIGS["maps"])
    w = {k: v for k, v in H.weights({**cfg, "streams": 1}).items() if ".hc" not in k}
    del cfg["streams"]
    from megatron_mixtera_b200 import model_registry as R

    model = R.ARCHITECTURES["Lukarax"](cfg, {k: tuple(v.shape) for k, v in w.items()}, torch.float32, 64)
    model.load_checkpoint(w)
    n = model.layers[0].norm1
    assert model.streams == 1 and (float(n.blend), float(n.gain), float(n.mix)) == (1.0, 1.0, 1.0)


@pytest.mark.parametrize("rows,longest", [(32, 128), (12, 70), (2, 4), (6, 9.5), (64, 500), (8, 30.0), (32, 240)])
def test_rows_of_the_distance_bias(rows, longest):
    """One row per distance at first, then logarithmic ones; the table ends where the last row starts."""
    from megatron_mixtera_b200.transformer.hybrid_config import DistanceBias

    got = DistanceBias(rows, longest).rows_by_distance()
    assert got == [L.bucket(d, rows, longest) for d in range(len(got))] and got[-1] == rows - 1 and rows - 1 not in got[:-1]
    assert got[: rows // 2] == list(range(rows // 2))
    assert all(L.bucket(d, rows, longest) == rows - 1 for d in range(len(got), len(got) + 1000))


def test_rotation_tables_of_halves():
    """The tables are those of the pairs, whichever dimensions a pair joins; the ramp's ends and the factor follow the scaling."""
    from megatron_mixtera_b200.transformer.hybrid_config import RotaryConfig, YarnScaling
    from megatron_mixtera_b200.transformer.rotary import rotary_tables

    spec = H.sink()["mixer"]["rot"]
    freq, factor = L.frequencies(spec)
    for halves in (False, True):
        c, s = rotary_tables(RotaryConfig(spec["base"], spec["dims"], YarnScaling(**spec["scaling"]), halves), 50, "cpu")
        angle = torch.arange(50, dtype=torch.float64)[:, None] * torch.tensor(freq, dtype=torch.float64)
        assert float((c - torch.cos(angle) * factor).abs().max()) < 1e-6 and float((s - torch.sin(angle) * factor).abs().max()) < 1e-6
    assert factor > 1 and len(set(f / b for f, b in zip(freq, L.frequencies({**spec, "scaling": None})[0]))) > 2


def test_fused_linears():
    """Parts side by side: input rows and output columns of every part start at multiples of 8, what lies between is zero."""
    cfg, w, model = build("odd")
    model.load_checkpoint(w)
    mixer = model.layers[2].mixer
    left, right = mixer.parts
    assert mixer.columns == [0, 64] and left.inputs == {"q": 36, "k": 12, "v": 11} and mixer.out_columns == [0, 40]
    W = mixer.linear_in.weight
    assert torch.equal(W[36:48], w["l2.mix.left.k"]) and torch.equal(W[64: 64 + 60], w["l2.mix.right.q"]) and float(W[59:64].abs().max()) == 0.0
    O = mixer.linear_proj.weight
    assert torch.equal(O[:, 40:73], w["l2.mix.right.o"]) and float(O[:, 33:40].abs().max()) == 0.0 and O.shape[1] == 80
    assert torch.equal(right.weight_gates[3:6], w["l2.mix.right.f"]) and right.weight_gates.shape[0] == 8


def test_context_of_a_model():
    """Row widths and state parts of every layer; slots are handed out, swapped and given back for all parts together."""
    cfg, w, model = build("mixed")
    ctx = model.make_context(max_cached_tokens=512, max_requests_override=4, max_tokens_override=512, device="cpu", debug_validate=True)
    assert ctx.latent_row_widths == [2 * (48 + 40), 2 * 56, 2 * 64, 0, 2 * 56, 48, 0]
    shapes = [b and {k: tuple(v.shape[1:]) for k, v in b.items()} for b in ctx.state_buffers]
    memory = {"state": (3, 41, 32), "top": (3,)}
    assert shapes == [None, memory, None, None, memory, None, None]
    assert all(t.dtype == torch.float32 for t in ctx.state_buffers[1].values())
    ctx.set_prefill_q_block(*model.prefill_unit_tokens())
    for entries, gone in (([(0, [1] * 70), (1, [2])], []), ([(1, [3])], [1]), ([(2, [4] * 5), (0, [1])], [0]), ([(2, [4])], [2])):
        ctx.schedule_tokens(entries)
        ctx.initialize_attention_state()
        n = len(entries)
        read, write = ctx.state_read_slots[:n].tolist(), ctx.state_write_slots[:n].tolist()
        assert not set(write) & {r for r in read if r >= 0} and len(set(write)) == n
        ctx.complete_step(gone)
    assert sorted(ctx._free_state_slots) == list(range(ctx.num_state_slots))


def test_work_lists_of_several_block_sizes():
    _, _, model = build("mixed")
    assert model.prefill_unit_tokens() == [32, 21, 16]
    assert build("odd")[2].prefill_unit_tokens() == [0] and build("mixed", torch.float32)[2].prefill_unit_tokens() == [0]


# ---------------------------------------------------------------------------------------------------------------------
def planted():
    """name -> a function that puts one mistake into the oracle."""
    def set_(name, fn):
        return lambda mp: mp.setattr(L, name, fn)

    (attend, visible, rotate, bucket, frequencies, route, unit_rms, memory_scan, memory_inputs, combine, lam, diff_keys, sink_attention, streams_in,
     streams_out) = (L.attend, L.visible, L.rotate, L.bucket, L.frequencies, L.route, L.unit_rms, L.memory_scan, L.memory_inputs, L.differential_combine,
                     L.differential_lambda, L.differential_keys, L.sink_attention, L.streams_in, L.streams_out)

    def mask_edit(**change):
        return lambda n, m: visible(n, m and {**m, **{k: f(m[k]) for k, f in change.items() if k in m}})

    def attend_with(**change):
        def fn(q, k, v, scale, mask, **kw):
            return attend(q, k, v, scale, mask, **{**kw, **{n: f(kw[n]) for n, f in change.items() if kw.get(n) is not None}})
        return fn

    def grouped_wrong(q, k, v, scale, mask, **kw):
        g = q.shape[1] // k.shape[1]
        return attend(q, k.repeat(1, g, 1), v.repeat(1, g, 1), scale, mask, **kw)

    def cap_after_bias(q, k, v, scale, mask, *, softcap=None, **kw):
        return attend(q, k, v, scale, mask, **kw) if softcap is None else attend(q * 1.0, k, v, scale, mask, **kw)

    def no_floor(q, k, v, i, f, state=None):  # divided by the normaliser however small
        T, Hn, d = q.shape
        S, n, top, out = torch.zeros(Hn, d, v.shape[2], dtype=q.dtype), torch.zeros(Hn, d, dtype=q.dtype), torch.zeros(Hn, dtype=q.dtype), torch.empty_like(v)
        for t in range(T):
            new = torch.maximum(f[t] + top, i[t])
            keep, write = torch.exp(f[t] + top - new), torch.exp(i[t] - new)
            S = keep[:, None, None] * S + write[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
            n = keep[:, None] * n + write[:, None] * k[t]
            top = new
            out[t] = torch.einsum("hij,hi->hj", S, q[t]) / ((n * q[t]).sum(-1).abs() + 1e-6)[:, None]
        return out, None

    def no_normaliser(q, k, v, i, f, state=None):
        T, Hn, d = q.shape
        S, top, out = torch.zeros(Hn, d, v.shape[2], dtype=q.dtype), torch.zeros(Hn, dtype=q.dtype), torch.empty_like(v)
        for t in range(T):
            new = torch.maximum(f[t] + top, i[t])
            S = torch.exp(f[t] + top - new)[:, None, None] * S + torch.exp(i[t] - new)[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
            top = new
            out[t] = torch.einsum("hij,hi->hj", S, q[t]) * 1e-3
        return out, None

    def routed(change):
        return lambda z, c, r: change(z, c, r)

    def open_groups(z, c, r):
        return route(z, c, {**r, "groups": None})

    def weights_with_correction(z, c, r):
        chosen, _ = route(z, c, r)
        s = (torch.softmax(z, -1) + c)[chosen]
        return chosen, s / (s.sum() + 1e-20) * r["scale"]

    def not_renormalised(z, c, r):
        chosen, _ = route(z, c, r)
        return chosen, torch.softmax(z, -1)[chosen] * r["scale"]

    def sigmoid_scores(z, c, r):
        chosen, _ = route(z, c, r)
        s = torch.sigmoid(z)[chosen]
        return chosen, s / s.sum() * r["scale"]

    def closed_as_zero(z, c, r):
        s = torch.softmax(z, -1)
        g = r["groups"]
        of_group = (s + c).view(g["count"], -1)
        best = torch.topk(of_group.amax(-1), g["keep"]).indices
        open_ = torch.zeros(g["count"], 1)
        open_[best] = 1
        chosen = torch.topk((of_group * open_).reshape(-1), r["top"]).indices
        return chosen.tolist(), s[chosen] / s[chosen].sum() * r["scale"]

    def values_after_rotation(h, w, p, m, eps):
        T, Hq, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
        q, k = (unit_rms(rotate((h @ w[p + n].T + w[p + n + ".b"]).view(T, c, d), m["rot"], True), eps) for n, c in ((".q", Hq), (".k", G)))
        return attend(q, k, k, m["scale"], m["mask"], softcap=m["softcap"], sink=w[p + ".sink"]).reshape(T, -1) @ w[p + ".o"].T + w[p + ".o.b"]

    return {
        "window one short": set_("visible", mask_edit(size=lambda s: max(s - 1, 1))),
        "window one long": set_("visible", mask_edit(size=lambda s: s + 1)),
        "first tokens not kept": set_("visible", mask_edit(keep_first=lambda k: 0)),
        "one first token too many": set_("visible", mask_edit(keep_first=lambda k: k + 1)),
        "head groups interleaved": set_("attend", grouped_wrong),
        "no distance bias": set_("attend", attend_with(bias=lambda b: 0 * b)),
        "bias off by one distance": set_("bucket", lambda n, rows, longest: bucket(n + 1, rows, longest)),
        "bias classes linear": set_("bucket", lambda n, rows, longest: min(n, rows - 1)),
        "no cap": set_("attend", cap_after_bias),
        "no sink": set_("attend", attend_with(sink=lambda s: s - 1e4)),
        "sink capped": set_("attend", attend_with(sink=lambda s: 1.5 * torch.tanh(s / 1.5))),
        "pairs the other way": set_("rotate", lambda x, rot, halves: rotate(x, rot, not halves)),
        "no rotation scaling": set_("frequencies", lambda rot: frequencies({**rot, "scaling": None})),
        "no rotation factor": set_("frequencies", lambda rot: (frequencies(rot)[0], 1.0)),
        "norm before rotation's factor": set_("unit_rms", lambda x, eps: x if x.dim() == 3 and x.shape[1] in (2, 8) and x.shape[2] == 32 else unit_rms(x, eps)),
        "values after rotation": set_("sink_attention", values_after_rotation),
        "maps added": set_("differential_combine", lambda a1, a2, lam_, diff, eps: combine(a1, -a2, lam_, diff, eps)),
        "no head norm": set_("differential_combine", lambda a1, a2, lam_, diff, eps: (a1 - lam_ * a2) * (1.0 - diff)),
        "no factor behind the head norm": set_("differential_combine", lambda a1, a2, lam_, diff, eps: combine(a1, a2, lam_, 0.0, eps)),
        "lambda without its constant": set_("differential_lambda", lambda w, p, m: lam(w, p, m) - m["diff"]),
        "maps swapped in the keys": set_("differential_keys", lambda h, w, p, m: (lambda k, v: (k.flip(2), v))(*diff_keys(h, w, p, m))),
        "no floor under the normaliser": set_("memory_scan", no_floor),
        "no normaliser": set_("memory_scan", no_normaliser),
        "query not scaled": set_("memory_inputs", lambda h, w, p, m: (lambda q, *r: (q * m["dim"] ** 0.5, *r))(*memory_inputs(h, w, p, m))),
        "gates not capped": set_("memory_inputs", lambda h, w, p, m: memory_inputs(h, w, p, {**m, "gate_cap": 1e6})),
        "forget gate plain": set_("log_sigmoid", lambda x: torch.log(torch.clamp(torch.sigmoid(x) * 0.97, min=1e-30))),
        "groups open": set_("route", routed(open_groups)), "closed groups count zero": set_("route", routed(closed_as_zero)),
        "weights with the correction": set_("route", routed(weights_with_correction)), "weights not renormalised": set_("route", routed(not_renormalised)),
        "sigmoid scores": set_("route", routed(sigmoid_scores)),
        "identity experts dropped": set_("route", lambda z, c, r: (lambda e, a: ([x for x in e if x < r["experts"]], a[[i for i, x in enumerate(e) if x < r["experts"]]]))(*route(z, c, r))),
        "one stream read": set_("streams_in", lambda x, w, p: x[0]),
        "mix transposed": set_("streams_out", lambda x, y, w, p: torch.einsum("ts,snw->tnw", w[p + ".mix"], x) + w[p + ".out"][:, None, None] * y),
        "output into one stream": set_("streams_out", lambda x, y, w, p: streams_out(x, y * 0, w, p) + torch.cat([y[None], 0 * x[1:]])),
        "norm without its bias": set_("layer_norm", lambda x, weight, bias, eps: L.unit_rms(x - x.mean(-1, keepdim=True), eps) * weight),
        "norm without the mean": set_("layer_norm", lambda x, weight, bias, eps: L.unit_rms(x, eps) * weight + bias),
    }


SUBTLE = {"one first token too many", "sink capped", "norm without the mean", "no rotation factor", "query not scaled", "gates not capped", "closed groups count zero"}
BEHIND_A_NORM = {"no floor under the normaliser", "no normaliser", "query not scaled"}  # the head's norm divides them out, but for its eps


@pytest.mark.parametrize("mistake", list(planted()))
def test_planted_mistakes_exceed_the_limits(mistake, monkeypatch):
    """A mistake in one mechanism moves the 32-bit logits far beyond the GPU tests' limit, and nearly all of them the 16-bit ones too."""
    cfg = {**H.CONFIGS["mixed"], "norm": {"eps": 0.3}} if mistake in BEHIND_A_NORM else H.CONFIGS["mixed"]
    toks = H.tokens(130, cfg["vocab"], 10)
    base = {s: H.weights(cfg, seed=3, gain=1.6, settled=s) for s in (False, True)}
    want = {s: H.oracle_logits(toks, cfg, w) for s, w in base.items()}
    planted()[mistake](monkeypatch)
    e32, e16 = (H.position_errors(H.oracle_logits(toks, cfg, base[s]), want[s]) for s in (False, True))
    assert float(e32.max()) > 100 * LIMIT_F32, float(e32.max())
    if mistake not in SUBTLE:
        assert float((e16 > LIMIT_BF16).float().mean()) > 0.03 or float(e16.max()) > 4 * LIMIT_BF16, e16.topk(8)


def test_oracle_portions():
    """The oracle's own recurrence carries a state: two halves give what the whole gives."""
    cfg = H.CONFIGS["mixed"]
    w = {k: v.double() for k, v in H.weights(cfg, seed=3).items()}
    h = torch.randn(30, cfg["width"], dtype=torch.float64, generator=torch.Generator().manual_seed(0))
    x = L.memory_inputs(h, w, "l1.mix.right", cfg["layers"][1]["mixer"]["right"])
    whole, last = L.memory_scan(*x)
    a, S = L.memory_scan(*(y[:11] for y in x))
    b, S = L.memory_scan(*(y[11:] for y in x), S)
    assert torch.allclose(torch.cat([a, b]), whole) and all(torch.allclose(p, q) for p, q in zip(S, last))
    assert all(math.isfinite(float(p.abs().max())) for p in last)


def test_oracle_maximum_cancels():
    """With the divisor on the normaliser's side the running maximum leaves no trace: the plain sums give the same."""
    g = torch.Generator().manual_seed(0)
    T, Hn, d, dv = 20, 2, 8, 5
    q, k, v = (torch.randn(T, Hn, n, generator=g, dtype=torch.float64) for n in (d, d, dv))
    i, f = torch.randn(T, Hn, generator=g, dtype=torch.float64) + 2.0, -torch.rand(T, Hn, generator=g, dtype=torch.float64)
    got, _ = L.memory_scan(q, k, v, i, f)
    b = f.cumsum(0)
    for t in range(T):
        weight = torch.exp(b[t] - b[: t + 1] + i[: t + 1])
        nq = torch.einsum("sh,shd,hd->h", weight, k[: t + 1], q[t])
        o = torch.einsum("sh,shd,hd,shv->hv", weight, k[: t + 1], q[t], v[: t + 1])
        below = torch.maximum(nq.abs(), torch.ones(Hn, dtype=torch.float64))
        assert float((got[t] - o / below[:, None]).abs().max() / (o / below[:, None]).abs().max()) < 1e-5
