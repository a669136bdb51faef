"""Each mechanism of the Lukarax design alone on the GPU, against the plain oracle's function for it."""
import math

import lukarax_helpers as H
import pytest
import torch

from oracle import lukarax_oracle as L

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]
LIMIT = {torch.float32: 2e-5, torch.bfloat16: 0.04}
SCHEDULES = {
    "whole": [[(0, 150)], [(1, 70)], [(2, 1)]],
    "portions": [[(0, n)] for n in (2, 62, 2, 3, 1, 31, 33, 2, 1, 13)] + [[(1, 64)], [(1, 6)], [(2, 1)]],
    "tokens": [[(0, 1)]] * 150 + [[(1, 1)]] * 70 + [[(2, 1)]],
    "batch": [[(0, 64), (1, 2)], [(1, 3), (2, 1), (0, 1)], [(0, 1), (1, 1)], [(1, 20), (0, 2)], [(0, 60)], [(1, 1), (0, 2)], [(0, 20), (1, 43)]],
}


def bf(t):
    return t.to(torch.bfloat16).float()


def rows(n, width, seed):
    return bf(torch.randn(n, width, generator=torch.Generator().manual_seed(seed)))


def close(got, want, dtype, factor=1.0):
    """Every row within the limit; in 16 bits a row in which large terms cancel may be off by a few times its share."""
    want = want.float()
    e = (got.float().cpu() - want).square().mean(-1).sqrt() / want.square().mean().sqrt()
    limit = LIMIT[dtype] * factor
    if dtype == torch.float32:
        return float(e.max()) < limit
    return float(e.max()) < 4 * limit and float((e > limit).float().sum()) <= 0.02 * e.numel()


def model_of(layers, dtype, width=96, seed=0, edit=None, gain=1.0, eps=1e-5, **kw):
    cfg = H.config(layers if isinstance(layers, list) else [layers], width=width, eps=eps)
    w = H.weights(cfg, seed=seed, gain=gain)
    if edit is not None:
        edit(w)
    model, ctx, _ = H.build(cfg, w, dtype, **kw)
    return cfg, w, model, ctx


MIXERS = {
    "maps": H.differential(mlp=None), "maps, many heads": H.differential(heads=16, kv_heads=1, dim=64, vdim=64, rot=64, mlp=None),
    "maps, wide": H.differential(heads=4, kv_heads=2, dim=64, vdim=128, rot=32, mlp=None),
    "maps, wider than a tile": H.differential(heads=4, kv_heads=2, dim=128, vdim=128, rot=128, mlp=None),
    "maps, dim 96": H.differential(heads=5, kv_heads=5, dim=96, vdim=48, rot=8, diff=0.8, mlp=None),
    "maps, no rotation": H.differential(heads=2, kv_heads=1, dim=16, vdim=24, rot=0, mlp=None),
    "maps, odd": H.differential(heads=3, kv_heads=1, dim=10, vdim=7, rot=6, mlp=None),
    "maps, large": H.differential(heads=2, kv_heads=1, dim=160, vdim=200, rot=64, mlp=None),
    "sink": H.sink(mlp=None), "sink, one token": H.sink(size=1, mlp=None), "sink, page": H.sink(heads=3, kv_heads=1, dim=64, rot=64, size=64, mlp=None),
    "sink, wide": H.sink(heads=16, kv_heads=1, dim=128, rot=32, size=100, softcap=40.0, mlp=None),
    "sink, partial rotation": H.sink(heads=2, kv_heads=2, dim=80, rot=48, size=90, scaling=(8.0, 64, 4.0, 1.0), mlp=None),
    "sink, odd": H.sink(heads=2, kv_heads=2, dim=11, rot=6, size=40, mlp=None), "sink, large": H.sink(heads=2, kv_heads=1, dim=200, rot=200, size=90, mlp=None),
    "side by side": H.parallel(mlp=None), "side by side, wide": H.parallel(heads=8, kv_heads=1, dim=128, vdim=128, size=64, keep=64, rows=32, longest=100,
                                                                            m_heads=2, m_dim=128, m_vdim=128, mlp=None),
    "side by side, kept beyond the window": H.parallel(size=5, keep=70, rows=8, longest=30, m_heads=1, m_dim=64, m_vdim=72, mlp=None),
    "side by side, nothing kept": H.parallel(size=33, keep=0, rows=64, longest=500, m_heads=5, m_dim=16, m_vdim=300, mlp=None),
    "side by side, one class": H.parallel(rows=2, longest=3, size=90, keep=1, m_dim=256, m_heads=1, m_vdim=64, mlp=None),
    "side by side, odd": H.parallel(heads=3, kv_heads=3, dim=9, vdim=10, size=19, keep=2, rows=6, longest=11.0, m_heads=3, m_dim=20, m_vdim=11, mlp=None),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which", list(MIXERS))
def test_mixers(which, dtype):
    """Whole prompts, portions, single tokens and unequal batches give the same rows; pages and slots are used again all the time."""
    cfg, w, model, ctx = model_of(MIXERS[which], dtype, gain=1.5)
    hs = [rows(n, 96, 5 + i) for i, n in enumerate((150, 70, 1))]
    want = [H.mixer_oracle(h, cfg, w, 0) for h in hs]
    for name, schedule in SCHEDULES.items():
        got = H.run_mixer(model, ctx, 0, hs, schedule)
        assert all(close(g, x, dtype) for g, x in zip(got, want)), (name, [H.rel(g, x) for g, x in zip(got, want)])
    assert ctx.total_request_count == 0 and ctx.chunk_allocator.chunk_count_avail == ctx.chunk_allocator.chunk_count_total - 1
    assert ctx.state_shapes is None or len(ctx._free_state_slots) == ctx.num_state_slots


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim", [24, 128])
def test_rows_of_another_layer(dim, dtype):
    """Own queries, lambda and gate over the keys and values another layer cached."""
    layers = [H.differential(dim=dim, mlp=None), H.sink(mlp=None), H.differential(dim=dim, kv_from=0, diff=0.2, mlp=None)]
    cfg, w, model, ctx = model_of(layers, dtype)
    assert ctx.latent_row_widths[2] == 0
    hs = [rows(n, 96, 5 + i) for i, n in enumerate((150, 70, 1))]
    want = [H.mixer_oracle(h, cfg, w, 2) for h in hs]
    for name, schedule in SCHEDULES.items():
        got = H.run_mixer(model, ctx, 2, hs, schedule)
        assert all(close(g, x, dtype) for g, x in zip(got, want)), name


def standing_out(layer, p, heads, kv_rows, dim, asks, shown, W=96, seed=1, small=0.2):
    """Weights in which a token of ``asks`` asks for a token of ``shown`` with every head and map, and little else matters."""
    g = torch.Generator().manual_seed(seed)
    cfg = H.config([layer], width=W)
    w = H.weights(cfg, seed=seed)
    s = torch.randn(dim, generator=g) / math.sqrt(dim)
    q = torch.randn(heads * dim, W, generator=g) * small / math.sqrt(W) + torch.outer(s.repeat(heads), asks)
    k = torch.randn(kv_rows * dim, W, generator=g) * small / math.sqrt(W) + torch.outer(s.repeat(kv_rows), shown)
    w[p + "q"], w[p + "k"] = q.to(torch.bfloat16), k.to(torch.bfloat16)
    return cfg, w


def stand_out_rows(T, W, key, places):
    axis = torch.eye(W)
    h = rows(T, W, 9)
    h[:, :2] *= 0.02
    h[key] = bf(h[key] * 0.1 + 8 * axis[1])
    for p in places:
        h[p] = bf(h[p] * 0.1 + 8 * axis[0])
    return h


def run_schedules(cfg, w, dtype, h, key, places, want, factor=2.0):
    T = h.shape[0]
    model, ctx, _ = H.build(cfg, w, dtype)
    ctx.token_rows(1).fill_(30.0)  # nothing may be read from slots that hold no token of the request
    for schedule in ([T], [key + 1, 1, T - key - 2] if key + 2 < T else [T], [64] * 4 + [T - 256], [key + 1] + [1] * (T - key - 1), [2] * (T // 2)):
        got = H.run_mixer(model, ctx, 0, [h], [[(0, n)] for n in schedule if n])[0]
        assert H.rel(got[places], want[places]) < factor * LIMIT[dtype], schedule[:4]
        assert H.rel(got, want) < factor * LIMIT[dtype], schedule[:4]
        ctx.token_rows(1).fill_(30.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size,keep,key", [(96, 0, 63), (96, 3, 64), (64, 2, 100), (65, 0, 0), (65, 1, 0), (40, 4, 3), (40, 4, 4), (2, 0, 127), (130, 70, 69),
                                           (40, 70, 70), (1, 64, 63)])
def test_one_key_stands_out_under_a_window_that_keeps_the_first(size, keep, key, dtype):
    """Queries just inside the window, and everywhere if the key is one of the kept, answer with its value; the others do not."""
    W, T, heads, dim = 96, 260, 2, 64
    axis = torch.eye(W)
    layer = H.parallel(heads=heads, kv_heads=1, dim=dim, vdim=32, size=size, keep=keep, right=0.0, left=1.0, mlp=None)
    layer["mixer"]["left"]["scale"] = 0.4
    cfg, w = standing_out(layer, "l0.mix.left.", heads, 1, dim, axis[0], axis[1])
    w["l0.mix.left.rel"] *= 0.3
    places = sorted({p for p in (key, key + 1, key + 2, key + size - 2, key + size - 1, key + size, key + size + 1, key + 63, key + 64, T - 1) if key < p < T})
    h = stand_out_rows(T, W, key, places)
    want = H.mixer_oracle(h, cfg, w, 0)
    wd = {k: v.double() for k, v in w.items()}
    value = (h.double()[key] @ wd["l0.mix.left.v"].T).repeat(heads) @ wd["l0.mix.left.o"].T
    for p in places:  # (what the case claims)
        near = float((want[p] - value).norm() / value.norm())
        assert (near < 0.2) == (p - key < size or key < keep), (p, near)
    run_schedules(cfg, w, dtype, h, key, places, want)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size,key", [(96, 63), (64, 100), (65, 0), (2, 127), (130, 30)])
def test_one_key_stands_out_beside_a_sink(size, key, dtype):
    W, T, heads, dim = 96, 260, 2, 64
    axis = torch.eye(W)
    layer = H.sink(heads=heads, kv_heads=1, dim=dim, rot=16, size=size, softcap=14.0, mlp=None)
    layer["mixer"]["scale"] = 0.25
    cfg, w = standing_out(layer, "l0.mix.", heads, 1, dim, axis[0], axis[1], small=0.5)
    w["l0.mix.q.b"] *= 0.05
    w["l0.mix.k.b"] *= 0.05
    places = sorted({p for p in (key, key + 1, key + size - 2, key + size - 1, key + size, key + size + 1, T - 1) if key < p < T})
    h = stand_out_rows(T, W, key, places)
    want = H.mixer_oracle(h, cfg, w, 0)
    wd = {k: v.double() for k, v in w.items()}
    value = (h.double()[key] @ wd["l0.mix.k"].T + wd["l0.mix.k.b"]).repeat(heads)
    got = [float(torch.dot(want[p] - wd["l0.mix.o.b"], value @ wd["l0.mix.o"].T) / (value @ wd["l0.mix.o"].T).square().sum()) for p in places]
    assert all((g > 0.5) == (p - key < size) for p, g in zip(places, got)), got
    run_schedules(cfg, w, dtype, h, key, places, want)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("key", [0, 63, 64, 130])
def test_one_key_stands_out_for_both_maps(key, dtype):
    """The first map finds the key, the second looks at everything: the difference shows both."""
    W, T, heads, dim = 96, 260, 2, 40
    axis = torch.eye(W)
    layer = H.differential(heads=heads, kv_heads=1, dim=dim, vdim=32, rot=8, mlp=None)
    layer["mixer"]["scale"] = 0.6
    cfg, w = standing_out(layer, "l0.mix.", heads * 2, 2, dim, axis[0], axis[1])
    w["l0.mix.q"].view(heads, 2, dim, W)[:, 1] *= 0.02
    places = [p for p in (key + 1, key + 2, key + 63, key + 64, T - 1) if p < T]
    h = stand_out_rows(T, W, key, places)
    want = H.mixer_oracle(h, cfg, w, 0)
    run_schedules(cfg, w, dtype, h, key, places, want)


@pytest.mark.parametrize("dtype", DTYPES)
def test_sink_alone_and_capped_scores(dtype):
    """Sinks that take nearly everything or nothing; scores far beyond the cap; the output's bias stays."""
    layer = H.sink(heads=4, kv_heads=2, dim=32, size=50, softcap=3.0, mlp=None)
    layer["mixer"]["scale"] = 5.0

    def edit(w):
        w["l0.mix.sink"] = torch.tensor([30.0, -30.0, 3.0, 4.5]).to(torch.bfloat16)

    cfg, w, model, ctx = model_of(layer, dtype, edit=edit)
    h = rows(150, 96, 2)
    want = H.mixer_oracle(h, cfg, w, 0)
    for schedule in ([150], [1] * 150, [7, 63, 2, 78]):
        assert close(H.run_mixer(model, ctx, 0, [h], [[(0, n)] for n in schedule])[0], want, dtype)


@pytest.mark.parametrize("which", ["maps", "maps, wider than a tile", "sink, wide", "side by side, wide"])
def test_decode_attention_split_over_the_context(which):
    """Long rows: several splits of one context, rows shorter than a split beside them."""
    import copy

    layer = copy.deepcopy(MIXERS[which])
    part = layer["mixer"].get("left", layer["mixer"])
    if "mask" in part:
        part["mask"]["size"] = 3000
        if "keep_first" in part["mask"]:
            part["mask"]["keep_first"] = 100
    cfg, w, model, ctx = model_of(layer, torch.bfloat16, max_cached_tokens=9000, max_sequence_length=4096, max_step_tokens=4096)
    hs = [rows(n, 96, 3 + i) for i, n in enumerate((3500, 40))]
    want = [tail_oracle(h, cfg, w, 20) for h in hs]
    got = H.run_mixer(model, ctx, 0, hs, [[(0, 3490)], [(1, 30)]] + [[(0, 1), (1, 1)]] * 10)
    assert max(H.rel(g[-20:], x) for g, x in zip(got, want)) < LIMIT[torch.bfloat16]


def tail_oracle(h, cfg, w, n):
    return H.mixer_oracle(h, cfg, w, 0)[-n:]


# ---------------------------------------------------------------------------------------------------------------------
MEMORIES = [dict(m_heads=3, m_dim=32, m_vdim=40), dict(m_heads=2, m_dim=64, m_vdim=64), dict(m_heads=2, m_dim=128, m_vdim=100), dict(m_heads=9, m_dim=12, m_vdim=5),
            dict(m_heads=1, m_dim=256, m_vdim=64)]


@pytest.mark.parametrize("which", range(len(MEMORIES)))
def test_memory_state_after_a_portion(which):
    """The matrix, its normaliser and the maximum themselves; another request's slot is left alone."""
    cfg, w, model, ctx = model_of(H.parallel(**MEMORIES[which], mlp=None), torch.float32)
    h = rows(37, 96, 1)
    m = cfg["layers"][0]["mixer"]["right"]
    wd = {k: v.double() for k, v in w.items()}
    _, (S, n, top) = L.memory_scan(*L.memory_inputs(h.double(), wd, "l0.mix.right", m))
    for schedule in ([37], [1] * 37, [2, 30, 5]):
        H.run_mixer(model, ctx, 0, [torch.cat([h, h])], [[(0, k)] for k in schedule])
        side = int(ctx.request_state_side[0]) * ctx.num_state_slots + int(ctx.request_state_slots[0])
        got, got_top = ctx.recurrent_state(1, "state")[side].cpu(), ctx.recurrent_state(1, "top")[side].cpu()
        assert float((got[:, :-1] - S.transpose(1, 2)).abs().max() / S.abs().max()) < 1e-5
        assert float((got[:, -1] - n).abs().max() / n.abs().max()) < 1e-5 and float((got_top - top).abs().max()) < 1e-5
        ctx.reset()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", ["long memory", "forgets at once", "input gates closed", "input gates open", "normaliser near zero"])
def test_memory_extremes(case, dtype):
    """The maximum follows its floor, the input gates or the forget gates; the divisor is e^-maximum or the normaliser (an eps of the size of
    the outputs keeps the norm behind them from hiding it)."""
    f, i = {"long memory": (9.0, 0.0), "forgets at once": (-9.0, 0.0), "input gates closed": (3.0, -9.0), "input gates open": (3.0, 9.0),
            "normaliser near zero": (5.0, -2.0)}[case]

    def edit(w):
        w["l0.mix.right.f.b"].fill_(f)
        w["l0.mix.right.i.b"].fill_(i)
        if case == "normaliser near zero":
            w["l0.mix.right.q"] *= 0.05

    cfg, w, model, ctx = model_of(H.parallel(left=0.0, right=1.0, m_dim=48, m_vdim=64, mlp=None), dtype, edit=edit, eps=0.2)
    hs = [rows(n, 96, 5 + k) for k, n in enumerate((150, 70, 1))]
    want = [H.mixer_oracle(h, cfg, w, 0) for h in hs]
    for name, schedule in SCHEDULES.items():
        got = H.run_mixer(model, ctx, 0, hs, schedule)
        assert all(close(g, x, dtype, 1.5) for g, x in zip(got, want)), (name, [H.rel(g, x) for g, x in zip(got, want)])


def test_memory_reaches_far_back():
    """One token writes, hundreds of closed input gates later it is read back, in prompts longer than a gate kernel's block and in decoding."""
    W, T = 96, 1500

    def edit(w):
        for k in ("i", "f"):
            w["l0.mix.right." + k] *= 0.0
        w["l0.mix.right.i"][:, 1] = 4.0
        w["l0.mix.right.i.b"].fill_(-8.0)
        w["l0.mix.right.f.b"].fill_(8.5)

    cfg, w, model, ctx = model_of(H.parallel(left=0.0, right=1.0, m_dim=64, m_vdim=32, mlp=None), torch.float32, edit=edit, max_cached_tokens=2048,
                                  max_sequence_length=2048, max_step_tokens=2048)
    h = rows(T, W, 9)
    h[:, 1] = 0.0
    h[40, 1] = 8.0
    want = H.mixer_oracle(h, cfg, w, 0)
    g = h.clone()
    g[40, 1] = 0.0
    assert H.rel(H.mixer_oracle(g, cfg, w, 0)[-5:], want[-5:]) > 0.3  # (the token is remembered)
    # (a query at right angles to the remembered key reads rounding, which the norm behind it blows up: not in 32-bit arithmetic)
    single = L.matrix_memory(h, {k: v.float() for k, v in w.items()}, "l0.mix.right", cfg["layers"][0]["mixer"]["right"], 1e-5)
    sure = (single - want).square().mean(-1).sqrt() < 1e-5 * want.square().mean().sqrt()
    assert float(sure.float().mean()) > 0.9
    for schedule in ([T], [1400, 60] + [1] * 40, [30, 9, 2, 1, 1025, 433]):
        got = H.run_mixer(model, ctx, 0, [h], [[(0, n)] for n in schedule])[0]
        assert H.rel(got[sure], want[sure]) < 1e-4, schedule[:3]


# ---------------------------------------------------------------------------------------------------------------------
def add_up(model, index, x, base):
    """base + the mixture of layer ``index`` for the rows ``x`` (one stream, mixed with 1 and 1)."""
    from megatron_mixtera_b200 import ops

    one = torch.ones(1, device="cuda")
    with torch.inference_mode():
        hidden = base.cuda()[:, None].contiguous()
        experts = model.layers[index].moe(x.cuda().to(model.config.params_dtype))
        ops.stream_norm(hidden, ops.PendingStreams(experts=experts, mix=one.view(1, 1), gain=one))
    return hidden[:, 0].cpu()


def sure_of(x, w, r):
    """Tokens whose choice no rounding can change: experts, and groups."""
    keep = []
    for t, z in enumerate(x.double() @ w["l0.mlp.router"].T):
        choice = torch.softmax(z, -1) + w["l0.mlp.correction"]
        chosen, _ = L.route(z, w["l0.mlp.correction"], r)
        g = r["groups"]
        best = choice.view(g["count"], -1).amax(-1).sort(descending=True).values
        gaps = [best[g["keep"] - 1] - best[g["keep"]]] if g["keep"] < g["count"] else []
        size = choice.numel() // g["count"]
        open_ = {e // size for e in torch.topk(choice.view(g["count"], -1).amax(-1), g["keep"]).indices.tolist() for e in range(e * size, (e + 1) * size)}
        rest = [float(c) for e, c in enumerate(choice) if e // size in open_ and e not in chosen]
        if rest:
            gaps.append(min(float(choice[e]) for e in chosen) - max(rest))
        if all(g_ > 1e-6 for g_ in gaps):
            keep.append(t)
    return keep


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens", [1, 7, 64, 300, 2000])
@pytest.mark.parametrize("case", range(7))
def test_experts(case, tokens, dtype):
    """Routing inside groups, identity experts, the sort, the grouped products and the weighted sum, over one to many tokens per expert."""
    mlp = (H.experts(), H.experts(40, 5, 100, 8, (6, 2), 2.5), H.experts(3, 3, 64, 0, (1, 1)), H.experts(1, 1, 8, 0, (1, 1)), H.experts(125, 1, 24, 3, (16, 1)),
           H.experts(9, 10, 70, 1, (2, 2)), H.experts(2, 3, 40, 6, (4, 3)))[case]
    width = 100 if case == 2 else 96
    cfg, w0, model, _ = model_of(H.sink(mlp=mlp), dtype, width=width)
    w = {k: v.double() for k, v in w0.items()}
    x, base = rows(tokens, width, 4), torch.randn(tokens, width, generator=torch.Generator().manual_seed(8))
    got = add_up(model, 0, x, base)
    check = list(range(tokens)) if tokens <= 64 else list(range(0, tokens, tokens // 50))
    sure = [check[i] for i in sure_of(x[check], w, mlp["router"])]
    assert len(sure) >= len(check) - 1
    want = base[sure].double() + L.mixture(x[sure].double(), w, "l0.mlp", mlp)
    assert H.rel(got[sure], want) < LIMIT[dtype] / 4
    from megatron_mixtera_b200 import ops

    assert int(ops.moe_counters(torch.device("cuda", 0), mlp["router"]["experts"])[: 4 * (mlp["router"]["experts"] + 1)].max()) == 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_choice_and_weights_differ(dtype):
    """The correction decides who is chosen - also with choice scores below zero, where a closed group is still closed - and is no part
    of the weights; one group of identity experts alone, one expert for all tokens."""
    mlp = H.experts(6, 2, 64, 2, (4, 1), 1.3)

    def edit(w):
        w["l0.mlp.router"] *= 0.2
        w["l0.mlp.correction"] = torch.tensor([-3.0, -3.0, -2.0, -2.5, -4.0, -4.0, -2.25, -2.2]).to(torch.bfloat16)

    cfg, w0, model, _ = model_of(H.sink(mlp=mlp), dtype, edit=edit)
    w = {k: v.double() for k, v in w0.items()}
    x = rows(300, 96, 4)
    chosen = {tuple(sorted(L.route(z, w["l0.mlp.correction"], mlp["router"])[0])) for z in x.double() @ w["l0.mlp.router"].T}
    assert chosen == {(2, 3)}  # (the best group by its largest choice score)
    assert H.rel(add_up(model, 0, x, torch.zeros(300, 96))[::9], L.mixture(x[::9].double(), w, "l0.mlp", mlp)) < LIMIT[dtype] / 4
    w0["l0.mlp.correction"][6:] = 5.0  # identity experts only: nothing is left to multiply
    model.load_checkpoint(w0)
    want = x * 1.3
    assert H.rel(add_up(model, 0, x, torch.zeros(300, 96)), want) < (1e-6 if dtype == torch.float32 else 1e-6)


@pytest.mark.parametrize("tile", [32, 64, 128, 256])
def test_expert_tiles(tile, monkeypatch):
    from megatron_mixtera_b200.transformer.moe import MixtureOfExperts

    mlp = H.experts(5, 2, 72, 1, (2, 2))
    cfg, w0, model, _ = model_of(H.sink(mlp=mlp), torch.bfloat16, width=200)
    w = {k: v.double() for k, v in w0.items()}
    monkeypatch.setattr(MixtureOfExperts, "tile_tokens", staticmethod(lambda *a: tile))
    for tokens in (1, 31, 700):
        x = rows(tokens, 200, 4)
        got = add_up(model, 0, x, torch.zeros(tokens, 200))
        pick = list(range(0, tokens, max(1, tokens // 40)))
        pick = [pick[i] for i in sure_of(x[pick], w, mlp["router"])]
        assert H.rel(got[pick], L.mixture(x[pick].double(), w, "l0.mlp", mlp)) < LIMIT[torch.bfloat16] / 4


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,ff", [(96, 72), (160, 64), (160, 192), (100, 37), (256, 1000)])
def test_dense_feed_forward(width, ff, dtype):
    from megatron_mixtera_b200 import ops

    cfg, w0, model, _ = model_of(H.sink(mlp=H.dense(ff)), dtype, width=width)
    w = {k: v.double() for k, v in w0.items()}
    one = torch.ones(1, device="cuda")
    for tokens in (1, 65, 700):
        x = rows(tokens, width, 4)
        hidden = torch.zeros((tokens, 1, width), device="cuda")
        with torch.inference_mode():
            y = model.layers[0].mlp(x.cuda().to(dtype), defer_output_reduction=True)[0]
            ops.stream_norm(hidden, ops.PendingStreams(partials=y, mix=one.view(1, 1), gain=one))
        assert H.rel(hidden[:, 0], L.gated(x.double(), w, "l0.mlp.".rstrip("."))) < LIMIT[dtype] / 2
    model.load_checkpoint(w0)  # (rows that were rearranged for the fused kernel load again)
    with torch.inference_mode():
        again = model.layers[0].mlp(x.cuda().to(dtype))[0].float().cpu()
    assert H.rel(again, L.gated(x.double(), w, "l0.mlp")) < LIMIT[dtype] / 2


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,streams", [(32, 1), (100, 2), (101, 3), (160, 4), (1028, 5), (2056, 4), (4100, 8), (8192, 4), (64, 16)])
def test_streams_and_norm(width, streams, dtype):
    """Embedding start, a sublayer's output with a bias written into all streams, the blend's layer norm, picked rows, the plain sum."""
    from megatron_mixtera_b200 import ops

    g = torch.Generator().manual_seed(0)
    T, V, K, S = 9, 20, 64, streams
    table, gamma, beta, bias = (bf(torch.randn(*s, generator=g)) for s in ((V, width), (width,), (width,), (width,)))
    ids = torch.randint(0, V, (T,), generator=g)
    mix, gain, blend = torch.randn(S, S, generator=g) / math.sqrt(S), torch.randn(S, generator=g), torch.randn(S, generator=g) + 0.5
    dev = [t.cuda().to(dtype) for t in (table, gamma, beta, bias)]
    d32 = [t.cuda().contiguous() for t in (mix, gain, blend)]
    hidden = torch.empty((T, S, width), dtype=torch.float32, device="cuda")
    out = torch.empty((T, width), dtype=dtype, device="cuda")
    kw = dict(gamma=dev[1], beta=dev[2], eps=1e-3)
    ops.stream_norm(hidden, ops.PendingStreams(table=dev[0], ids=ids.cuda(), table_scale=3.7), blend=d32[2], out=out, **kw)
    x = (table[ids] * 3.7).double()[None].repeat(S, 1, 1)
    w = {"p.in": blend.double(), "p.out": gain.double(), "p.mix": mix.double()}

    def norm(u):
        return L.layer_norm(u, gamma.double(), beta.double(), 1e-3)

    assert float((hidden.cpu().transpose(0, 1) - x).abs().max()) < 1e-5
    tol = 2e-5 if dtype == torch.float32 else 4e-2
    assert float((out.float().cpu() - norm(L.streams_in(x, w, "p"))).abs().max()) < tol
    x = torch.randn(S, T, width, generator=g).double()  # streams that differ
    hidden.copy_(x.transpose(0, 1))
    a, b = bf(torch.randn(T, K, generator=g)), bf(torch.randn(width, K, generator=g) / 8)
    pending = lambda: ops.PendingStreams(partials=ops.linear_partials(a.cuda().to(dtype), b.cuda().to(dtype)), bias=dev[3], mix=d32[0], gain=d32[1])  # noqa: E731
    pick = torch.tensor([8, 0, 3])
    picked = torch.empty((3, width), dtype=dtype, device="cuda")
    ops.stream_norm(hidden, pending(), out=picked, row_index=pick.cuda(), **kw)
    y = L.streams_out(x, a.double() @ b.double().T + bias.double(), w, "p")
    assert float((hidden.cpu().transpose(0, 1) - x).abs().max()) < 1e-6  # (picked rows leave the streams as they are)
    assert float((picked.float().cpu() - norm(y.sum(0)[pick])).abs().max()) < tol
    ops.stream_norm(hidden, pending(), blend=d32[2], out=out, **kw)
    assert float((hidden.cpu().transpose(0, 1) - y).abs().max()) < 2e-4
    assert float((out.float().cpu() - norm(L.streams_in(y, w, "p"))).abs().max()) < 2 * tol


def test_wrong_arguments_are_refused():
    """The host checks turn impossible sizes into errors before anything is launched."""
    from megatron_mixtera_b200 import _lib, ops

    x = torch.zeros(8, device="cuda")
    for name, args in (("stream_norm", _lib.StreamNormArgs()), ("rotate_append", _lib.RotateAppendArgs()), ("recurrence_gates", _lib.RecurrenceArgs()),
                       ("swiglu", _lib.SwigluArgs()), ("moe_route", _lib.MoeArgs(plain=1))):
        with pytest.raises(ops.B200Error):
            ops.struct_kernel(name, args, x)
    hidden = torch.zeros((2, 17, 8), device="cuda")
    with pytest.raises(ops.B200Error):  # more streams than the kernel holds
        ops.stream_norm(hidden, ops.PendingStreams(mix=torch.zeros((17, 17), device="cuda"), gain=torch.zeros(17, device="cuda")))
