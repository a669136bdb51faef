"""Each mechanism of the Maginex design alone on the GPU, against the plain oracle's function for it."""
import math

import maginex_helpers as H
import pytest
import torch

from oracle import maginex_oracle as M

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]
LIMIT = {torch.float32: 2e-5, torch.bfloat16: 0.03}
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


def model_of(layers, dtype, width=96, seed=0, edit=None, gain=1.0, eps=1e-5, taps=4, **kw):
    cfg = H.config(layers if isinstance(layers, list) else [layers], width=width, eps=eps, taps=taps)
    w = H.weights(cfg, seed=seed, gain=gain)
    if edit is not None:
        edit(w)
    model, ctx, _ = H.build(cfg, w, dtype, **kw)
    return cfg, w, model, ctx


MIXERS = {
    "latent": H.latent(mlp=None), "latent, one head": H.latent(heads=1, dim=16, vdim=8, kv_rank=16, q_rank=8, mlp=None),
    "latent, 16 heads": H.latent(heads=16, dim=32, vdim=64, kv_rank=112, q_rank=48, mlp=None),
    "latent, 24 heads": H.latent(heads=24, dim=64, vdim=64, kv_rank=96, q_rank=128, mlp=None),
    "latent, 64 heads": H.latent(heads=64, dim=16, vdim=16, kv_rank=256, q_rank=64, mlp=None),
    "latent, 40 heads, wide values": H.latent(heads=40, dim=8, vdim=128, kv_rank=80, q_rank=24, mlp=None),
    "latent, rank 512": H.latent(heads=8, dim=128, vdim=128, kv_rank=512, q_rank=192, mlp=None),
    "latent, beyond the kernels": H.latent(heads=3, dim=136, vdim=160, kv_rank=600, q_rank=40, mlp=None),
    "latent, odd": H.latent(heads=3, dim=11, vdim=13, kv_rank=21, q_rank=19, mlp=None),
    "latent, odd values": H.latent(heads=2, dim=24, vdim=10, kv_rank=32, q_rank=16, mlp=None),
    "window": H.windowed(v_mix=False, mlp=None), "window, one token": H.windowed(size=1, v_mix=False, mlp=None),
    "window, page": H.windowed(heads=3, kv_heads=1, dim=64, vdim=64, rot=64, size=64, v_mix=False, mlp=None),
    "window, wide": H.windowed(heads=16, kv_heads=1, dim=128, vdim=128, rot=32, size=100, v_mix=False, mlp=None),
    "window, dim 96": H.windowed(heads=4, kv_heads=2, dim=96, vdim=40, rot=48, size=41, v_mix=False, mlp=None),
    "window, narrow keys": H.windowed(heads=4, kv_heads=4, dim=16, vdim=128, rot=16, size=90, v_mix=False, mlp=None),
    "no window": H.windowed(heads=5, kv_heads=5, dim=48, vdim=72, rot=24, size=None, v_mix=False, mlp=None),
    "no rotation": H.windowed(heads=2, kv_heads=1, rot=0, size=70, v_mix=False, mlp=None),
    "window, odd": H.windowed(heads=3, kv_heads=3, dim=11, vdim=7, rot=6, size=19, v_mix=False, mlp=None),
    "window, large": H.windowed(heads=2, kv_heads=1, dim=200, vdim=136, rot=200, size=90, v_mix=False, mlp=None),
    "scan": H.mingru(mlp=None), "scan, wide": H.mingru(1040, mlp=None), "scan, odd": H.mingru(45, mlp=None), "scan, narrow": H.mingru(2, mlp=None),
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
    assert len(ctx._free_state_slots) == ctx.num_state_slots


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kw", [dict(), dict(dim=20, vdim=11, rot=6, kv_heads=3, heads=3), dict(dim=128, vdim=128, rot=64, heads=8, kv_heads=1)])
def test_mixed_values(kw, dtype):
    """The first layer's values go into the others' caches, weighed by their own number; what the first one holds of it is not used."""
    layers = [H.mingru(mlp=None), H.windowed(mlp=None, **kw), H.windowed(mlp=None, v_mix=False, **kw), H.windowed(mlp=None, size=70, **kw)]
    cfg, w, model, ctx = model_of(layers, dtype)
    assert [model.layers[i].mixer.parts[0].first_values for i in (1, 2, 3)] == [True, False, False]
    hs = [rows(n, 96, 5 + i) for i, n in enumerate((150, 70, 1))]
    for index in (1, 3):
        want = [H.mixer_oracle(h, cfg, w, index) for h in hs]
        for name, schedule in SCHEDULES.items():
            got = H.run_mixer(model, ctx, index, hs, schedule)
            assert all(close(g, x, dtype) for g, x in zip(got, want)), (index, name)
    w["l3.mix.vmix"] = torch.tensor(0.0).to(torch.bfloat16)
    assert H.rel(H.mixer_oracle(hs[0], cfg, w, 3), want[0]) > 0.1  # (the case shows the mixing)


def stand_out_rows(T, W, key, places):
    """Rows in which ``key`` shows axis 1 and ``places`` ask along axis 0, and the others hardly do either."""
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
@pytest.mark.parametrize("size,key", [(96, 63), (96, 64), (64, 100), (65, 0), (2, 127), (130, 30), (1, 64), (40, 191)])
def test_one_key_stands_out_under_a_window(size, key, dtype):
    """Queries just inside the window answer with the key's value, those just outside do not: prompts, portions and decoding."""
    W, T, heads, dim = 96, 260, 2, 64
    axis, g = torch.eye(W), torch.Generator().manual_seed(1)
    cfg = H.config([H.windowed(heads=heads, kv_heads=1, dim=dim, vdim=32, rot=16, size=size, v_mix=False, mlp=None)], width=W)
    cfg["layers"][0]["mixer"]["scale"] = 0.4
    w = H.weights(cfg, seed=1)
    s = torch.randn(dim, generator=g) / math.sqrt(dim)
    s[:16] = 0.0  # (what turns takes no part)
    w["l0.mix.q"] = (torch.randn(heads * dim, W, generator=g) * 0.2 / math.sqrt(W) + torch.outer(s.repeat(heads), axis[0])).to(torch.bfloat16)
    w["l0.mix.k"] = (torch.randn(dim, W, generator=g) * 0.2 / math.sqrt(W) + torch.outer(s, axis[1])).to(torch.bfloat16)
    places = sorted({p for p in (key, key + 1, key + 2, key + size - 2, key + size - 1, key + size, key + size + 1, key + 63, key + 64, T - 1) if key < p < T})
    h = stand_out_rows(T, W, key, places)
    want = H.mixer_oracle(h, cfg, w, 0)
    wd = {k: v.double() for k, v in w.items()}
    gate = torch.sigmoid(h.double() @ wd["l0.mix.g"].T)
    for p in places:  # (what the case claims)
        value = ((h.double()[key] @ wd["l0.mix.v"].T)[None] * gate[p][:, None]).reshape(-1) @ wd["l0.mix.o"].T
        near = float((want[p] - value).norm() / value.norm())
        assert (near < 0.3) == (p - key < size), (p, near)
    run_schedules(cfg, w, dtype, h, key, places, want)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads", [2, 20])
@pytest.mark.parametrize("key", [0, 63, 64, 130])
def test_one_latent_stands_out_among_all(key, heads, dtype):
    """A token far back, at page borders and at the sequence's start outweighs hundreds of others."""
    W, T, dim, rank = 96, 260, 64, 32
    axis, g = torch.eye(W), torch.Generator().manual_seed(1)
    cfg = H.config([H.latent(heads=heads, dim=dim, vdim=32, kv_rank=rank, q_rank=24, mlp=None)], width=W)
    cfg["layers"][0]["mixer"]["scale"] = 0.05
    w = H.weights(cfg, seed=1)
    # the query latent's first entry grows with axis 0 and the key latent's first with axis 1; the heads match the two
    w["l0.mix.dq"][0], w["l0.mix.dkv"][0] = axis[0] * 4, axis[1] * 4
    w["l0.mix.uq"] = (w["l0.mix.uq"].float() * 0.2).to(torch.bfloat16)
    w["l0.mix.uk"] = (w["l0.mix.uk"].float() * 0.2).to(torch.bfloat16)
    w["l0.mix.uq"][:, 0] = 0.5
    w["l0.mix.uk"][:, 0] = 0.5
    places = sorted({p for p in (key + 1, key + 2, key + 63, key + 64, T - 1) if key < p < T})
    h = stand_out_rows(T, W, key, places)
    want = H.mixer_oracle(h, cfg, w, 0)
    wd = {k: v.double() for k, v in w.items()}
    c = M.rms_norm(h.double() @ wd["l0.mix.dkv"].T, wd["l0.mix.dkv.norm"], 1e-5)
    for p in places:
        value = (c[key] @ wd["l0.mix.uv"].T * torch.sigmoid(h.double()[p] @ wd["l0.mix.g"].T)) @ wd["l0.mix.o"].T
        assert float((want[p] - value).norm() / value.norm()) < 0.3, p
    run_schedules(cfg, w, dtype, h, key, places, want)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("layer", [H.latent(heads=4, mlp=None), H.latent(heads=20, dim=16, vdim=16, mlp=None), H.windowed(heads=4, v_mix=False, size=50, mlp=None),
                                   H.windowed(heads=4, dim=20, vdim=9, v_mix=False, size=None, mlp=None)])
def test_sinks_at_their_extremes(layer, dtype):
    """Sinks that take nearly everything or nothing, unscaled and counted once: at the first token too, where they stand beside one key."""
    heads = layer["mixer"]["heads"]

    def edit(w):
        w["l0.mix.sink"] = torch.tensor([30.0, -30.0, 3.0, 200.0] * (heads // 4)).to(torch.bfloat16)

    cfg, w, model, ctx = model_of(layer, dtype, edit=edit)
    h = rows(150, 96, 2)
    want = H.mixer_oracle(h, cfg, w, 0)
    for schedule in ([150], [1] * 150, [7, 63, 2, 78]):
        assert close(H.run_mixer(model, ctx, 0, [h], [[(0, n)] for n in schedule])[0], want, dtype)


@pytest.mark.parametrize("which", ["latent", "latent, 24 heads", "latent, 64 heads", "latent, rank 512", "window, wide", "no window"])
def test_decode_attention_split_over_the_context(which):
    """Long rows: several splits of one context (a sink counts once in all of them), rows shorter than a split beside them."""
    import copy

    layer = copy.deepcopy(MIXERS[which])
    if "mask" in layer["mixer"]:
        layer["mixer"]["mask"]["size"] = 3000
    cfg, w, model, ctx = model_of(layer, torch.bfloat16, max_cached_tokens=9000, max_sequence_length=4096, max_step_tokens=4096,
                                  edit=lambda w: w["l0.mix.sink"].add_(5.0))
    hs = [rows(n, 96, 3 + i) for i, n in enumerate((3500, 40))]
    want = [H.mixer_oracle(h, cfg, w, 0)[-20:] for h in hs]
    got = H.run_mixer(model, ctx, 0, hs, [[(0, 3490)], [(1, 30)]] + [[(0, 1), (1, 1)]] * 10)
    assert max(H.rel(g[-20:], x) for g, x in zip(got, want)) < LIMIT[torch.bfloat16]


@pytest.mark.parametrize("expand", [True, False])
@pytest.mark.parametrize("heads,dim,vdim", [(5, 64, 64), (6, 128, 128), (16, 96, 48), (3, 24, 128), (70, 16, 16)])
def test_both_prompt_forms_of_latent_attention(heads, dim, vdim, expand):
    """Expanded keys and values, in whole chunks of every row, and the absorbed form, on steps of several rows with and without a past."""
    cfg, w, model, ctx = model_of(H.latent(heads=heads, dim=dim, vdim=vdim, kv_rank=64, q_rank=40, mlp=None), torch.bfloat16, max_step_tokens=1024,
                                  max_cached_tokens=2048)
    mixer = model.layers[0].mixer
    mixer.expand_prompts = expand
    assert mixer.prompts_as_grouped
    hs = [rows(n, 96, 5 + i) for i, n in enumerate((300, 130, 64))]
    want = [H.mixer_oracle(h, cfg, w, 0) for h in hs]
    ctx.token_rows(1).fill_(float("nan"))  # (rows that no token wrote stay unread)
    for schedule in ([[(0, 300), (1, 130), (2, 64)]], [[(0, 100), (1, 65)], [(2, 63), (0, 200)], [(1, 65), (2, 1)]], [[(2, 64)], [(0, 10)], [(0, 290), (1, 130)]]):
        got = H.run_mixer(model, ctx, 0, hs, schedule)
        assert all(close(g, x, torch.bfloat16) for g, x in zip(got, want)), [H.rel(g, x) for g, x in zip(got, want)]
        ctx.token_rows(1).fill_(float("nan"))


# ---------------------------------------------------------------------------------------------------------------------
def recurrence(w, m):
    wd = {k: v.double() for k, v in w.items()}

    def states(h):
        z = torch.sigmoid(h.double() @ wd["l0.mix.z"].T + wd["l0.mix.z.b"])
        return M.gated_scan(z, M.candidate_of(h.double() @ wd["l0.mix.x"].T + wd["l0.mix.x.b"]))
    return states


@pytest.mark.parametrize("width", [72, 45, 512, 1])
def test_state_after_a_portion(width):
    """The state itself, in 32 bits; another request's slot is left alone."""
    cfg, w, model, ctx = model_of(H.mingru(width, mlp=None), torch.float32)
    h = rows(300, 96, 1)
    want = recurrence(w, cfg["layers"][0]["mixer"])(h)
    for schedule, n in (([37], 37), ([1] * 37, 37), ([2, 30, 5], 37), ([256], 256), ([255, 2, 1, 42], 300), ([257, 1], 258)):
        ctx.recurrent_state(1, "state").fill_(7.0)
        H.run_mixer(model, ctx, 0, [torch.cat([h[:n], h])], [[(0, k)] for k in schedule])
        side = int(ctx.request_state_side[0]) * ctx.num_state_slots + int(ctx.request_state_slots[0])
        got = ctx.recurrent_state(1, "state").cpu()
        assert float((got[side] - want[n - 1]).abs().max() / want[n - 1].abs().max()) < 1e-5
        mine = {side, (side + ctx.num_state_slots) % (2 * ctx.num_state_slots)}
        assert all(float(got[i].min()) == 7.0 == float(got[i].max()) for i in range(got.shape[0]) if i not in mine)
        ctx.reset()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("bias", [-90.0, -9.0, 0.0, 9.0, 90.0])
def test_update_gates_at_their_extremes(bias, dtype):
    """Gates that never open, hardly open, always stand open: nothing overflows, and what is kept is kept."""
    cfg, w, model, ctx = model_of(H.mingru(mlp=None), dtype, edit=lambda w: w["l0.mix.z.b"].fill_(bias))
    hs = [rows(n, 96, 5 + k) for k, n in enumerate((150, 70, 1))]
    want = [H.mixer_oracle(h, cfg, w, 0) for h in hs]
    for name, schedule in SCHEDULES.items():
        got = H.run_mixer(model, ctx, 0, hs, schedule)
        if bias == -90.0:
            assert all(bool(torch.isfinite(g).all()) and float(g.abs().max()) < 1e-6 for g in got)
        else:
            assert all(close(g, x, dtype, 1.5) for g, x in zip(got, want)), (name, [H.rel(g, x) for g, x in zip(got, want)])


@pytest.mark.parametrize("dtype", DTYPES)
def test_candidates_on_both_sides_of_zero(dtype):
    """u + 1/2 above zero and sigmoid(u) below it, also far from it."""
    def edit(w):
        w["l0.mix.x.b"] = torch.tensor([-100.0, -20.0, -3.0, -1e-3, 0.0, 1e-3, 3.0, 50.0] * 9).to(torch.bfloat16)

    cfg, w, model, ctx = model_of(H.mingru(72, mlp=None), dtype, edit=edit)
    h = rows(100, 96, 3)
    want = H.mixer_oracle(h, cfg, w, 0)
    for schedule in ([100], [1] * 100, [33, 2, 65]):
        assert close(H.run_mixer(model, ctx, 0, [h], [[(0, n)] for n in schedule])[0], want, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_scan_reaches_far_back(dtype):
    """One token writes, more than a thousand closed gates later its trace is still there: over tiles of a prompt, portions and decoding."""
    W, T = 96, 1500

    def edit(w):
        w["l0.mix.z"].zero_()
        w["l0.mix.z"][:, 1] = 4.0
        w["l0.mix.z.b"].fill_(-14.0)

    cfg, w, model, ctx = model_of(H.mingru(64, mlp=None), dtype, edit=edit, max_cached_tokens=2048, max_sequence_length=2048, max_step_tokens=2048)
    h = rows(T, W, 9)
    h[:, 1] = 0.0
    h[40, 1] = 8.0
    want = H.mixer_oracle(h, cfg, w, 0)
    other = h.clone()
    other[40, 1] = 0.0
    assert H.rel(H.mixer_oracle(other, cfg, w, 0)[-5:], want[-5:]) > 0.3  # (the token is remembered)
    for schedule in ([T], [1400, 60] + [1] * 40, [30, 9, 2, 1, 1025, 433]):
        got = H.run_mixer(model, ctx, 0, [h], [[(0, n)] for n in schedule])[0]
        assert H.rel(got[41:], want[41:]) < LIMIT[dtype], schedule[:3]


# ---------------------------------------------------------------------------------------------------------------------
def run_norm(model, ctx, hs, schedule):
    """Feed rows as what a layer before left (embedding rows) through layer 0's norm and filters."""
    from megatron_mixtera_b200 import ops

    dt, norm = model.config.params_dtype, model.layers[0].norm
    at, got = [0] * len(hs), [[[] for _ in hs] for _ in range(norm.filters.shape[0])]
    for part in schedule:
        ctx.schedule_tokens([(i, [0] * n) for i, n in part])
        ctx.initialize_attention_state()
        T = ctx.padded_active_token_count
        table = torch.zeros((T, model.config.hidden_size), dtype=dt, device="cuda")
        row = 0
        for i, n in part:
            table[row: row + n] = hs[i][at[i]: at[i] + n].to("cuda", dt)
            at[i] += n
            row += n
        hidden = torch.empty((T, model.config.hidden_size), dtype=torch.float32, device="cuda")
        with torch.inference_mode():
            outs = norm(hidden, ops.PendingRows(table=table, ids=torch.arange(T, device="cuda"), table_scale=2.0), ctx)
        assert float((hidden - 2.0 * table.float()).abs().max()) == 0.0
        row = 0
        for i, n in part:
            for k, o in enumerate(outs):
                got[k][i].append(o[row: row + n].float().cpu())
            row += n
        ctx.complete_step([i for i, _ in part if at[i] == len(hs[i])])
    return [[torch.cat(g) for g in of] for of in got]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,taps,mlp", [(96, 4, True), (96, 4, False), (160, 1, True), (101, 2, True), (64, 3, True), (1028, 5, True), (2056, 8, False),
                                            (4100, 4, True), (6000, 7, True), (32, 6, True)])
def test_filters_in_front_of_the_sublayers(width, taps, mlp, dtype):
    """One norm, two filters over time of its rows: prompts, portions shorter than a filter, single tokens, rows side by side."""
    layer = H.mingru(8, mlp=H.experts(1, 1, 8, 0) if mlp else None)
    cfg, w, model, ctx = model_of(layer, dtype, width=width, taps=taps, eps=1e-3)
    hs = [rows(n, width, 5 + i) for i, n in enumerate((150, 70, 1))]
    wd = {k: v.double() for k, v in w.items()}
    normed = [M.rms_norm(2.0 * h.double(), wd["l0.norm1"], 1e-3) for h in hs]
    tol = 2e-5 if dtype == torch.float32 else 0.05
    for name, schedule in SCHEDULES.items():
        for b in ctx.state_buffers:
            for t in b.values():
                t.fill_(float("nan"))
        got = run_norm(model, ctx, hs, schedule)
        assert len(got) == 1 + mlp
        for k, of in enumerate(got):
            for g, u in zip(of, normed):
                want = M.mixed_with_past(u, wd[f"l0.canon{k + 1}"])
                assert float((g - want).abs().max()) < tol * float(want.abs().max()), (name, k)
                assert H.rel(g, want) < (1e-5 if dtype == torch.float32 else 0.01)


def test_filters_do_not_depend_on_the_cut():
    """The normed rows are kept as they were stored: a prompt, its portions and its tokens one by one give the same bits but for the order of sums."""
    cfg, w, model, ctx = model_of(H.mingru(8, mlp=H.experts(1, 1, 8, 0)), torch.bfloat16, width=512)
    h = [rows(40, 512, 3)]
    whole = run_norm(model, ctx, h, [[(0, 40)]])
    for schedule in ([[(0, 1)]] * 40, [[(0, 2)]] * 20, [[(0, 37)], [(0, 3)]]):
        got = run_norm(model, ctx, h, schedule)
        for a, b in zip(got, whole):
            d = (a[0] - b[0]).abs()
            assert float((d > 0).float().mean()) < 0.02 and float((d / b[0].abs().clamp(min=0.1)).max()) < 0.01


# ---------------------------------------------------------------------------------------------------------------------
def add_up(model, x, base):
    """base + the mixture of layer 0 for the rows ``x``."""
    from megatron_mixtera_b200 import ops

    with torch.inference_mode():
        hidden = base.cuda().contiguous()
        ops.residual_norm(hidden, ops.PendingRows(experts=model.layers[0].moe(x.cuda().to(model.config.params_dtype))), [], [], eps=1.0)
    return hidden.cpu()


def sure_of(x, w, top):
    """Tokens whose choice no rounding can change."""
    z = (x.double() @ w["l0.mlp.router"].T + w["l0.mlp.router.b"]).sort(dim=-1, descending=True).values
    if top == z.shape[1]:
        return list(range(x.shape[0]))
    return (z[:, top - 1] - z[:, top] > 1e-5).nonzero()[:, 0].tolist()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens", [1, 7, 64, 300, 2000])
@pytest.mark.parametrize("case", range(8))
def test_experts(case, tokens, dtype):
    """Choice, weights, the sort, the grouped products with squared ReLU and the weighted sum, over one to many tokens per expert."""
    mlp = (H.experts(), H.experts(40, 5, 100, 64), H.experts(3, 3, 64, 0), H.experts(1, 1, 8, 24), H.experts(125, 1, 24, 200), H.experts(9, 8, 70, 0),
           H.experts(2, 1, 128, 128), H.experts(200, 12, 16, 40))[case]
    width = 100 if case == 2 else 96
    cfg, w0, model, _ = model_of(H.mingru(8, mlp=mlp), dtype, width=width)
    w = {k: v.double() for k, v in w0.items()}
    x, base = rows(tokens, width, 4), torch.randn(tokens, width, generator=torch.Generator().manual_seed(8))
    got = add_up(model, x, base)
    check = list(range(tokens)) if tokens <= 64 else list(range(0, tokens, tokens // 50))
    sure = [check[i] for i in sure_of(x[check], w, mlp["router"]["top"])]
    assert len(sure) >= len(check) - 1
    want = base[sure].double() + M.experts(x[sure].double(), w, "l0.mlp.", mlp)
    assert H.rel(got[sure], want) < LIMIT[dtype] / 3
    from megatron_mixtera_b200 import ops

    assert int(ops.moe_counters(torch.device("cuda", 0), mlp["router"]["experts"])[: 4 * (mlp["router"]["experts"] + 1)].max()) == 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_router_bias_counts_in_choice_and_weights(dtype):
    """Large and negative logits, a bias that decides, and weights that are the softmax over the chosen logits, bias included."""
    mlp = H.experts(6, 2, 64, 0)

    def edit(w):
        w["l0.mlp.router"] *= 0.1
        w["l0.mlp.router.b"] = torch.tensor([-300.0, -200.0, -201.5, -400.0, -1000.0, -203.0]).to(torch.bfloat16)

    cfg, w0, model, _ = model_of(H.mingru(8, mlp=mlp), dtype, edit=edit)
    w = {k: v.double() for k, v in w0.items()}
    x = rows(300, 96, 4)
    chosen, weight = M.choose(x.double() @ w["l0.mlp.router"].T + w["l0.mlp.router.b"], 2)
    assert set(map(tuple, chosen.sort(-1).values.tolist())) <= {(1, 2), (1, 5)} and 0.55 < float(weight[:, 0].mean()) < 0.95
    want = M.experts(x.double(), w, "l0.mlp.", mlp)
    assert H.rel(add_up(model, x, torch.zeros(300, 96)), want) < LIMIT[dtype] / 3


@pytest.mark.parametrize("tile", [32, 64, 128, 256])
def test_expert_tiles(tile, monkeypatch):
    from megatron_mixtera_b200.transformer.moe import MixtureOfExperts

    mlp = H.experts(5, 2, 72, 136)
    cfg, w0, model, _ = model_of(H.mingru(8, mlp=mlp), torch.bfloat16, width=200)
    w = {k: v.double() for k, v in w0.items()}
    monkeypatch.setattr(MixtureOfExperts, "tile_tokens", staticmethod(lambda *a: tile))
    for tokens in (1, 31, 700):
        x = rows(tokens, 200, 4)
        got = add_up(model, x, torch.zeros(tokens, 200))
        pick = list(range(0, tokens, max(1, tokens // 40)))
        pick = [pick[i] for i in sure_of(x[pick], w, 2)]
        assert H.rel(got[pick], M.experts(x[pick].double(), w, "l0.mlp.", mlp)) < LIMIT[torch.bfloat16] / 3


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M_,N,K,batch", [(1, 64, 64, 1), (33, 128, 48, 3), (64, 40, 128, 5), (130, 24, 16, 2), (300, 256, 64, 1), (5, 13, 21, 3)])
def test_gated_linear(M_, N, K, batch, dtype):
    """Outputs of per-head products times sigmoid of their own gates, wherever the gates lie in a wider matrix."""
    from megatron_mixtera_b200 import ops

    g = torch.Generator().manual_seed(0)
    x, wt, gate = (bf(torch.randn(*s, generator=g)) for s in ((M_, batch * K), (batch * N, K), (M_, 16 + batch * N)))
    out = torch.zeros((M_, batch * N), dtype=dtype, device="cuda")
    gates = gate.cuda().to(dtype)[:, 16:]
    ops.linear(x.cuda().to(dtype), wt.cuda().to(dtype), out=out, batch=batch, x_batch=K, y_batch=N, K=K, gate=gates)
    want = torch.einsum("mbk,bnk->mbn", x.view(M_, batch, K).double(), wt.view(batch, N, K).double()).reshape(M_, -1) * torch.sigmoid(gate[:, 16:].double())
    assert H.rel(out, want) < (1e-5 if dtype == torch.float32 else 0.01)


def test_wrong_arguments_are_refused():
    """The host checks turn impossible sizes into errors before anything is launched."""
    from megatron_mixtera_b200 import _lib, ops

    x = torch.zeros(8, device="cuda")
    p = x.data_ptr()
    for name, args in (("conv_add", _lib.ConvArgs()), ("gated_scan", _lib.GatedScanArgs()),
                       ("gated_scan", _lib.GatedScanArgs(proj=p, z_bias=p, u_bias=p, state=p, state_in=p, state_out=p, out=p, state_slots=1, width=8, num_tokens=1,
                                                         num_rows=1, proj_ld=8, out_ld=8, off_z=0, off_u=8, off_g=0)),
                       ("residual_norm", _lib.ResidualNormArgs(hidden=p, rows=1, source_rows=1, width=8, taps=9)),
                       ("moe_route", _lib.MoeArgs(plain=2, relu2=1))):
        with pytest.raises(ops.B200Error):
            ops.struct_kernel(name, args, x)
    with pytest.raises(ops.B200Error):  # a gate of another type
        ops.linear(torch.zeros((2, 8), device="cuda"), torch.zeros((8, 8), device="cuda"), gate=torch.zeros((2, 8), device="cuda", dtype=torch.bfloat16))
