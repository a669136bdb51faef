"""Each mechanism of the Fabivik design alone on the GPU, against the plain oracle's function for it."""
import math

import fabivik_helpers as H
import pytest
import torch

from oracle import fabivik_oracle as F

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]
LIMIT = {torch.float32: 2e-5, torch.bfloat16: 0.04}
SCHEDULES = {
    "whole": [[(0, 150)], [(1, 70)], [(2, 1)]],
    "portions": [[(0, n)] for n in (2, 62, 2, 3, 1, 31, 33, 2, 1, 13)] + [[(1, 64)], [(1, 6)], [(2, 1)]],
    "tokens": [[(0, 1)]] * 150 + [[(1, 1)]] * 70 + [[(2, 1)]],
    "batch": [[(0, 64), (1, 2)], [(1, 3), (2, 1), (0, 1)], [(0, 1), (1, 1)], [(1, 20), (0, 2)], [(0, 60)], [(1, 1), (0, 2)], [(0, 20), (1, 43)]],
}


def close(got, want, dtype, factor=1.0):
    """Every row within the limit; in 16 bits a row in which large terms cancel may be off by a few times its share."""
    want = want.float()
    e = (got.float().cpu() - want).square().mean(-1).sqrt() / want.square().mean().sqrt()
    limit = LIMIT[dtype] * factor
    if dtype == torch.float32:
        return float(e.max()) < limit
    return float(e.max()) < 4 * limit and float((e > limit).float().sum()) <= 0.02 * e.numel()


def bf(t):
    return t.to(torch.bfloat16).float()


def rows(n, width, seed):
    return bf(torch.randn(n, width, generator=torch.Generator().manual_seed(seed)))


def one_layer(layer, dtype, width=96, eps=1e-5, seed=0, **kw):
    cfg = H.config([layer] if isinstance(layer, dict) else layer, width=width, eps=eps)
    w = H.weights(cfg, seed=seed)
    model, ctx, _ = H.build(cfg, w, dtype, **kw)
    return cfg, w, {k: v.double() for k, v in w.items()}, model, ctx


MIXERS = {
    "wkv": (H.wkv(mlp=None), H.wkv(heads=2, dim=64, rank=16, mlp=None), H.wkv(heads=1, dim=12, rank=5, mlp=None),
            H.wkv(heads=2, dim=128, rank=40, mlp=None), H.wkv(heads=1, dim=256, rank=8, mlp=None)),
    "delta": (H.delta(mlp=None), H.delta(heads=2, kv_heads=2, dim=64, vdim=64, conv=2, mlp=None),
              H.delta(heads=4, kv_heads=1, dim=128, vdim=72, conv=6, mlp=None), H.delta(heads=3, kv_heads=1, dim=20, vdim=11, conv=1, mlp=None),
              H.delta(heads=1, kv_heads=1, dim=256, vdim=300, conv=8, mlp=None)),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind,which", [(k, i) for k in MIXERS for i in range(5)])
def test_recurrent_mixers(kind, which, dtype):
    """Whole prompts, portions, single tokens and unequal batches give the same rows; slots are used again all the time."""
    layer = MIXERS[kind][which]
    cfg, _, w, model, ctx = one_layer(layer, dtype)
    hs = [rows(n, 96, 5 + i) for i, n in enumerate((150, 70, 1))]
    fn = F.wkv if kind == "wkv" else F.gated_delta
    want = [fn(h.double(), w, "l0.mix", layer["mixer"], 1e-5) for h in hs]
    for name, schedule in SCHEDULES.items():
        got = H.run_mixer(model, ctx, 0, hs, schedule)
        assert all(close(g, x, dtype) for g, x in zip(got, want)), name
    assert len(ctx._free_state_slots) == ctx.num_state_slots


@pytest.mark.parametrize("kind", list(MIXERS))
def test_recurrent_state_after_a_portion(kind):
    """The state itself, and that a padding row or another request's slot is left alone."""
    layer = MIXERS[kind][0]
    cfg, _, w, model, ctx = one_layer(layer, torch.float32)
    h = rows(37, 96, 1)
    H.run_mixer(model, ctx, 0, [torch.cat([h, h])], [[(0, 37)]])
    side = int(ctx.request_state_side[0]) * ctx.num_state_slots + int(ctx.request_state_slots[0])
    buffers = ctx.recurrent_state(1)
    scan = F.wkv_scan(*F.wkv_inputs(h.double(), w, "l0.mix", layer["mixer"])[:4], w["l0.mix.u"]) if kind == "wkv" else \
        F.delta_scan(*F.delta_inputs(h.double(), w, "l0.mix", layer["mixer"]))
    S = scan[1].transpose(1, 2).float()
    assert float((buffers["state"][side].cpu() - S).abs().max() / S.abs().max()) < 1e-5
    if kind == "wkv":
        assert torch.equal(buffers["shift"][side].cpu(), h[-1])
    else:
        u = torch.cat([h.double() @ w["l0.mix." + k].T for k in "qkv"], dim=1)[-3:].float()
        assert float((buffers["conv"][side].cpu() - u).abs().max()) < 1e-4
    others = [i for i in range(2 * ctx.num_state_slots) if i != side]
    assert all(float(b[others].abs().max()) == 0.0 for b in buffers.values())


ATTENTIONS = [H.attention(mlp=None), H.attention(heads=3, kv_heads=3, dim=64, vdim=64, size=64, conv=2, v_mix=False, mlp=None),
              H.attention(heads=4, kv_heads=1, dim=128, vdim=128, size=100, v_mix=False, mlp=None),
              H.attention(heads=16, kv_heads=1, dim=72, vdim=16, size=5, conv=7, v_mix=False, mlp=None),
              H.attention(heads=5, kv_heads=1, dim=16, vdim=128, size=None, v_mix=False, mlp=None),
              H.attention(heads=2, kv_heads=2, dim=11, vdim=7, size=40, conv=1, v_mix=False, mlp=None),
              H.attention(heads=2, kv_heads=1, dim=200, vdim=256, size=90, conv=3, v_mix=False, mlp=None)]


def attention_oracle(h, w, layer, index=0, first=None):
    p, m = f"l{index}.mix", layer["mixer"]
    v = F.attention_values(h, w, p, m)
    if first is not None:
        v = (1 - w[p + ".vmix"]) * v + w[p + ".vmix"] * first
    return F.attention(h, w, p, m, 1e-5, v)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which", range(len(ATTENTIONS)))
def test_attention(which, dtype):
    layer = ATTENTIONS[which]
    cfg, _, w, model, ctx = one_layer(layer, dtype)
    hs = [rows(n, 96, 5 + i) for i, n in enumerate((150, 70, 1))]
    want = [attention_oracle(h.double(), w, layer) for h in hs]
    for name, schedule in SCHEDULES.items():
        got = H.run_mixer(model, ctx, 0, hs, schedule)
        assert all(close(g, x, dtype) for g, x in zip(got, want)), name


@pytest.mark.parametrize("dtype", DTYPES)
def test_value_mixing(dtype):
    """The second mixing layer blends in the first one's values, with a layer that does not mix in between."""
    layers = [H.attention(mlp=None), H.attention(heads=4, kv_heads=4, dim=16, vdim=8, v_mix=False, mlp=None), H.attention(heads=2, mlp=None)]
    cfg, _, w, model, ctx = one_layer(layers, dtype)
    hs = [rows(n, 96, 5 + i) for i, n in enumerate((150, 70, 1))]
    want = [attention_oracle(h.double(), w, layers[2], 2, F.attention_values(h.double(), w, "l0.mix", layers[0]["mixer"])) for h in hs]
    plain = [attention_oracle(h.double(), w, layers[2], 2) for h in hs]
    for schedule in SCHEDULES.values():
        got = H.run_mixer(model, ctx, 2, hs, schedule)
        assert all(close(g, x, dtype) for g, x in zip(got, want))
    assert min(H.rel(a, b) for a, b in zip(plain, want)) > 0.1  # (mixing matters)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size,key", [(96, 63), (96, 64), (64, 100), (65, 0), (1, 40), (2, 127), (None, 3), (130, 30)])
def test_one_key_stands_out(size, key, dtype):
    """One key that outweighs hundreds of others: queries just inside the window answer with its value, those just outside do not, in a
    prompt, in portions cut beside it, and decoded; every other pool slot a page holds is poisoned."""
    heads, dim, W, T = 2, 64, 96, 260
    layer = H.attention(heads=heads, kv_heads=1, dim=dim, vdim=32, size=size, v_mix=False, scale=2.0 / math.sqrt(dim), mlp=None)
    cfg = H.config([layer], width=W)
    w = H.weights(cfg, seed=1)
    g = torch.Generator().manual_seed(2)
    axis = torch.eye(W)
    asks, shown, s = axis[0] * 8, axis[1] * 8, torch.randn(dim, generator=g)
    small = 0.2 / math.sqrt(W)
    w["l0.mix.q"] = (torch.randn(heads * dim, W, generator=g) * small + torch.outer(s.repeat(heads), axis[0])).to(torch.bfloat16)
    w["l0.mix.k"] = (torch.randn(dim, W, generator=g) * small + torch.outer(s, axis[1])).to(torch.bfloat16)
    for k in ("q", "k"):  # positions stay sharp: the newest input outweighs the older ones
        w[f"l0.mix.{k}.conv"] *= 0.05
        w[f"l0.mix.{k}.conv"][:, -1] = 1.0
        w[f"l0.mix.{k}.norm"] = torch.full((dim,), 1.5).to(torch.bfloat16)
    h = rows(T, W, 9)
    h[:, :2] *= 0.02
    h[key] = bf(h[key] * 0.1 + shown)
    reach = size if size is not None else T
    places = sorted({p for p in (key, key + 1, key + 2, key + reach - 2, key + reach - 1, key + reach, key + reach + 1, key + 63, key + 64, T - 1)
                     if key < p < T})
    for p in places:
        h[p] = bf(h[p] * 0.1 + asks)
    wd = {k: v.double() for k, v in w.items()}
    want = attention_oracle(h.double(), wd, layer)
    value = F.attention_values(h.double(), wd, "l0.mix", layer["mixer"])[key, 0].repeat(heads) @ wd["l0.mix.o"].T
    for p in places:  # (what the case claims)
        near = float((want[p] - value).norm() / value.norm())
        assert (near < 0.2) == (p - key < reach), (p, near)
    model, ctx, _ = H.build(cfg, w, dtype)
    ctx.token_rows(1).fill_(30.0)  # nothing may be read from slots that hold no token of the request
    for schedule in ([T], [key + 1, 1, T - key - 2] if key + 2 < T else [T], [64] * 4 + [4], [key + 1] + [1] * (T - key - 1), [2] * (T // 2)):
        got = H.run_mixer(model, ctx, 0, [h], [[(0, n)] for n in schedule if n])[0]
        assert H.rel(got[places], want[places]) < 2 * LIMIT[dtype], schedule[:4]
        assert H.rel(got, want) < 2 * LIMIT[dtype], schedule[:4]
        ctx.token_rows(1).fill_(30.0)


def test_decode_attention_split_over_the_context():
    """Long rows: several splits of one window, rows shorter than a split beside them."""
    layer = H.attention(heads=4, kv_heads=2, dim=128, vdim=128, size=3000, v_mix=False, mlp=None)
    cfg, _, w, model, ctx = one_layer(layer, torch.bfloat16, max_cached_tokens=9000, max_sequence_length=4096, max_step_tokens=4096)
    from megatron_mixtera_b200.transformer.attention import choose_attention_splits

    assert choose_attention_splits(2, 2, 3064, 64) > 1
    hs = [rows(n, 96, 3 + i) for i, n in enumerate((3500, 40))]
    want = [attention_oracle(h.double(), w, layer) for h in hs]
    got = H.run_mixer(model, ctx, 0, hs, [[(0, 3490)], [(1, 30)]] + [[(0, 1), (1, 1)]] * 10)
    assert max(H.rel(g, x) for g, x in zip(got, want)) < LIMIT[torch.bfloat16]


def add_up(model, index, x, out):
    """out + the mixture of layer ``index`` for the rows ``x``."""
    from megatron_mixtera_b200 import ops

    with torch.inference_mode():
        hidden = out.cuda()
        ops.residual_norm(hidden, ops.PendingRows(experts=model.layers[index].moe(x.cuda().to(model.config.params_dtype))), [], [], eps=1.0)
    return hidden.cpu()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens", [1, 7, 64, 300, 2000])
@pytest.mark.parametrize("case", range(6))
def test_experts(case, tokens, dtype):
    """Routing, the sort, the grouped products and the sum, over one to many tokens per expert and tile."""
    mlp = (H.experts(), H.experts(40, 5, 100, 2.0, 130), H.experts(3, 3, 64, 0.5, 64), H.experts(1, 1, 8, 1.0, None), H.experts(130, 1, 24, 3.0, 16),
           H.experts(9, 9, 70, 1.0, None))[case]
    width = 100 if case == 2 else 96
    cfg, _, w, model, _ = one_layer(H.wkv(mlp=mlp), dtype, width=width)
    x, base = rows(tokens, width, 4), torch.randn(tokens, width, generator=torch.Generator().manual_seed(8))
    got = add_up(model, 0, x, base)
    check = list(range(tokens)) if tokens <= 64 else list(range(0, tokens, tokens // 50))
    score = torch.sigmoid(x.double() @ w["l0.mlp.router"].T).sort(-1, descending=True).values
    top = mlp["router"]["top"]
    sure = [t for t in check if top == score.shape[1] or score[t, top - 1] - score[t, top] > 1e-6]
    want = base[sure].double() + F.mixture(x[sure].double(), w, "l0.mlp", mlp)
    assert H.rel(got[sure], want) < LIMIT[dtype] / 4
    from megatron_mixtera_b200 import ops

    assert int(ops.moe_counters(torch.device("cuda", 0), mlp["router"]["experts"])[: 4 * (mlp["router"]["experts"] + 1)].max()) == 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_experts_all_tokens_at_one(dtype):
    """Every token chooses the same experts (the others get none), scores of zero and one included; limits bite on both sides."""
    mlp = H.experts(6, 2, 64, 0.3, 64, 0.2)
    cfg, w0, w, model, _ = one_layer(H.wkv(mlp=mlp), dtype)
    x = rows(500, 96, 4)
    x[:, 0] = 6.0
    for r in range(6):
        w0["l0.mlp.router"][r] *= 0.02
        w0["l0.mlp.router"][r, 0] = (-20.0, 3.0, -3.0, 20.0, -1.0, 0.0)[r]
    model.load_checkpoint(w0)
    w = {k: v.double() for k, v in w0.items()}
    got = add_up(model, 0, x, torch.zeros(500, 96))
    assert H.rel(got[::9], F.mixture(x[::9].double(), w, "l0.mlp", mlp)) < LIMIT[dtype] / 4


@pytest.mark.parametrize("tile", [32, 64, 128, 256])
def test_expert_tiles(tile, monkeypatch):
    from megatron_mixtera_b200.transformer.moe import MixtureOfExperts

    mlp = H.experts(5, 2, 72, 1.0, 200)
    cfg, _, w, model, _ = one_layer(H.wkv(mlp=mlp), torch.bfloat16, width=200)
    monkeypatch.setattr(MixtureOfExperts, "tile_tokens", staticmethod(lambda *a: tile))
    for tokens in (1, 31, 700):
        x = rows(tokens, 200, 4)
        got = add_up(model, 0, x, torch.zeros(tokens, 200))
        pick = list(range(0, tokens, max(1, tokens // 40)))
        assert H.rel(got[pick], F.mixture(x[pick].double(), w, "l0.mlp", mlp)) < LIMIT[torch.bfloat16] / 4


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [32, 100, 101, 160, 1028, 2056, 4100, 8200])
def test_residual_stream_and_norms(width, dtype):
    """Embedding start, partial sums, two norms of one row, picked rows, the scale of the output."""
    from megatron_mixtera_b200 import ops

    g = torch.Generator().manual_seed(0)
    T, V = 9, 20
    table = bf(torch.randn(V, width, generator=g))
    gam = [bf(0.3 * torch.randn(width, generator=g)) for _ in range(2)]
    ids = torch.randint(0, V, (T,), generator=g)
    hidden = torch.empty((T, width), dtype=torch.float32, device="cuda")
    dev = [t.cuda().to(dtype) for t in (table, *gam)]
    out = [torch.empty((T, width), dtype=dtype, device="cuda") for _ in range(2)]
    ops.residual_norm(hidden, ops.PendingRows(table=dev[0], ids=ids.cuda(), table_scale=3.7), dev[1:], out, eps=1e-3)
    x = table[ids] * 3.7
    assert float((hidden.cpu() - x).abs().max()) < 1e-5
    tol = 1e-5 if dtype == torch.float32 else 2e-2
    for o, w in zip(out, gam):
        assert float((o.float().cpu() - F.layer_norm(x.double(), w.double(), 1e-3)).abs().max()) < tol
    K = 64
    a, b = bf(torch.randn(T, K, generator=g)), bf(torch.randn(width, K, generator=g))
    pick = torch.tensor([8, 0, 3])
    picked = torch.empty((3, width), dtype=dtype, device="cuda")
    pend = lambda: ops.PendingRows(partials=ops.linear_partials(a.cuda().to(dtype), b.cuda().to(dtype)))  # noqa: E731
    ops.residual_norm(hidden, pend(), dev[1:2], [picked], eps=1e-3, out_scale=0.5, row_index=pick.cuda())
    assert float((hidden.cpu() - x).abs().max()) < 1e-5  # (picked rows leave the stream as it is)
    y = x.double() + a.double() @ b.double().T
    assert float((picked.float().cpu() - 0.5 * F.layer_norm(y[pick], gam[0].double(), 1e-3)).abs().max()) < tol
    ops.residual_norm(hidden, pend(), [], [], eps=1.0)
    assert float((hidden.cpu() - y).abs().max()) < 1e-4


def test_wrong_arguments_are_refused():
    """The host checks turn impossible sizes into errors before anything is launched."""
    from megatron_mixtera_b200 import _lib, ops

    x = torch.zeros(8, device="cuda")
    for name, args in (("residual_norm", _lib.ResidualNormArgs()), ("conv_qkv", _lib.ConvArgs()), ("token_shift", _lib.ShiftArgs()),
                       ("recurrence_scan", _lib.RecurrenceArgs()), ("moe_up", _lib.MoeArgs())):
        with pytest.raises(ops.B200Error):
            ops.struct_kernel(name, args, x)
