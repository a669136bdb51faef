"""Small Maginex configurations, random weights and the loops that compare the framework with the plain oracle."""
import math

import torch
from hybrid_helpers import build, error, replay, tokens  # noqa: F401  (re-exported)

from oracle import maginex_oracle as M


def experts(n=6, top=3, ff=40, shared=56):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": n, "top": top}, "shared": {"ff": shared} if shared else None}


def latent(heads=5, dim=24, vdim=40, kv_rank=48, q_rank=56, scale=1.3, mlp=experts()):
    return {"type": "latent_attention", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
                                                             "scale": scale / math.sqrt(dim)}}


def mingru(width=72, mlp=experts()):
    return {"type": "mingru", "mlp": mlp, "mixer": {"width": width}}


def windowed(heads=6, kv_heads=2, dim=32, vdim=24, rot=16, base=9000.0, size=23, v_mix=True, scale=1.2, mlp=experts()):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale / math.sqrt(dim), "rot": {"base": base, "dims": rot},
         "v_mix": v_mix}
    if size is not None:
        m["mask"] = {"size": size}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def config(layers, width=160, vocab=301, eps=1e-5, scale=3.0, taps=4):
    return {"architecture": "Maginex", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width, "canon": {"taps": taps},
            "embedding": {"scale": scale}}


CONFIGS = {
    # every mixer, with and without experts and shared experts, values mixed in two later layers, several windows and head groupings
    "mixed": config([windowed(), latent(), mingru(), windowed(size=70, heads=2, mlp=experts(9, 2, 72, 0)), mingru(104, mlp=None),
                     windowed(dim=24, rot=24, size=None, heads=4, v_mix=False), latent(heads=16, dim=32, vdim=16, kv_rank=96, q_rank=40),
                     windowed(heads=10, rot=4, size=1)], taps=3),
    # real head sizes, groups of heads that do not divide 64, more heads than the small decode kernel takes, many experts
    "wide": config([latent(heads=24, dim=64, vdim=64, kv_rank=128, q_rank=96, mlp=experts(30, 5, 100, 200)),
                    windowed(heads=16, kv_heads=1, dim=128, vdim=128, rot=128, size=150), latent(heads=3, dim=128, vdim=128, kv_rank=256, q_rank=192),
                    mingru(512), windowed(heads=3, kv_heads=1, dim=64, vdim=128, rot=32, size=64, v_mix=False),
                    windowed(heads=4, kv_heads=1, dim=96, vdim=128, rot=48, size=65)], width=192, taps=5),
    # nothing is a multiple of 8, and hardly anything even
    "odd": config([latent(heads=3, dim=11, vdim=13, kv_rank=21, q_rank=19, mlp=experts(7, 2, 21, 13)), mingru(45, mlp=experts(5, 5, 9, 0)),
                   windowed(heads=3, kv_heads=3, dim=20, vdim=11, rot=12, size=19), latent(heads=1, dim=7, vdim=9, kv_rank=5, q_rank=3, mlp=None),
                   windowed(heads=9, kv_heads=3, dim=10, vdim=11, rot=6, size=64)], width=101, vocab=77, taps=2),
    # a filter of one tap, windows of one and two tokens, one expert, the smallest heads
    "tiny": config([windowed(heads=1, kv_heads=1, dim=8, vdim=8, rot=2, size=1, mlp=experts(1, 1, 8, 8)),
                    latent(heads=1, dim=8, vdim=8, kv_rank=8, q_rank=8, mlp=experts(3, 1, 8, 0)), mingru(8, mlp=experts(2, 2, 8, 16)),
                    windowed(heads=2, kv_heads=1, dim=8, vdim=8, rot=8, size=2, mlp=None)], width=32, vocab=40, taps=1),
    # sizes beyond the tensor-core kernels, the longest filter
    "large": config([latent(heads=2, dim=160, vdim=200, kv_rank=544, q_rank=264), windowed(heads=2, kv_heads=1, dim=200, vdim=144, rot=64, size=90),
                     latent(heads=40, dim=8, vdim=8, kv_rank=16, q_rank=24), mingru(1000),
                     windowed(heads=20, kv_heads=1, dim=24, vdim=144, rot=8, size=40, v_mix=True)], width=128, taps=8),
    # one kind of mixer alone
    "scans": config([mingru(), mingru(200, mlp=None), mingru(64)], width=96),
    "latents": config([latent(), latent(heads=8, dim=16, vdim=32, kv_rank=80, q_rank=24, mlp=None)], width=96, taps=2),
    "windows": config([windowed(size=64), windowed(size=65, heads=4, kv_heads=2), windowed(size=500, heads=8, kv_heads=2)], width=96),
}


def weights(cfg, seed=0, gain=1.0, settled=False):
    """Random weights as a checkpoint holds them (bf16 values).  Linears keep the scale of their input; ``gain`` sharpens attention (through
    the queries); update gates spread the channels between short and long memory.  ``settled``: which experts are chosen is beyond the doubt
    of 16-bit rounding (the weights still differ from token to token)."""
    g = torch.Generator().manual_seed(seed)

    def mat(n, k, s=1.0):
        return torch.randn(n, k, generator=g) * (s / math.sqrt(k))

    def vec(n, mean=1.0, std=0.2):
        return mean + std * torch.randn(n, generator=g)

    W, out = cfg["width"], {}
    out["embed"], out["head"], out["final.norm"] = torch.randn(cfg["vocab"], W, generator=g) / math.sqrt(W) * 2.0, mat(cfg["vocab"], W), vec(W)
    mixing = [i for i, x in enumerate(cfg["layers"]) if x["mixer"].get("v_mix")]
    for i, layer in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.mix.", layer["mixer"], layer["mlp"]
        out[f"l{i}.norm1"] = vec(W)
        for n in (1, 2) if mlp is not None else (1,):
            out[f"l{i}.canon{n}"] = torch.randn(W, cfg["canon"]["taps"], generator=g) * 0.4
        if layer["type"] == "latent_attention":
            H = m["heads"]
            out.update({p + "dq": mat(m["q_rank"], W), p + "dq.norm": vec(m["q_rank"]), p + "uq": mat(H * m["dim"], m["q_rank"], gain),
                        p + "dkv": mat(m["kv_rank"], W), p + "dkv.norm": vec(m["kv_rank"]), p + "uk": mat(H * m["dim"], m["kv_rank"]),
                        p + "uv": mat(H * m["vdim"], m["kv_rank"]), p + "sink": vec(H, 1.0, 1.0), p + "g": mat(H * m["vdim"], W, 1.5),
                        p + "o": mat(W, H * m["vdim"])})
        elif layer["type"] == "mingru":
            n = m["width"]
            out.update({p + "z": mat(n, W, 1.5), p + "z.b": vec(n, -1.5, 1.5), p + "x": mat(n, W, 1.5), p + "x.b": vec(n, 0.0, 0.5),
                        p + "g": mat(n, W, 1.5), p + "o": mat(W, n)})
        else:
            H, G = m["heads"], m["kv_heads"]
            out.update({p + "q": mat(H * m["dim"], W, gain), p + "k": mat(G * m["dim"], W), p + "v": mat(G * m["vdim"], W),
                        p + "sink": vec(H, 1.0, 1.0), p + "g": mat(H, W, 1.5), p + "o": mat(W, H * m["vdim"])})
            if m.get("v_mix"):
                out[p + "vmix"] = torch.tensor(0.35 if i != mixing[0] else 0.9)
        if mlp is None:
            continue
        p, n = f"l{i}.mlp.", mlp["router"]["experts"]
        out[p + "router"], out[p + "router.b"] = mat(n, W, 1.5), vec(n, 0.0, 0.4)
        if settled:
            out[p + "router"] *= 0.15
            rank = torch.randperm(n, generator=g)
            out[p + "router.b"] = 0.2 * rank + torch.where(rank >= n - mlp["router"]["top"], 4.0, 0.0)
        for name, ff in [(f"e{e}", mlp["expert"]["ff"]) for e in range(n)] + ([("shared", mlp["shared"]["ff"])] if mlp["shared"] else []):
            out[p + name + ".up"], out[p + name + ".down"] = mat(ff, W), mat(W, ff)
    return {k: v.to(torch.bfloat16) for k, v in out.items()}


def oracle_logits(toks, cfg, w, streams=None):
    with torch.inference_mode():
        return M.forward(cfg, {k: v.double() for k, v in w.items()}, toks, streams).float()


def position_errors(got, want):
    """rms(difference) / rms(logits) of every position, the mean over the vocabulary taken off."""
    d = got.float().cpu() - want
    d = d - d.mean(-1, keepdim=True)
    return d.square().mean(-1).sqrt() / (want - want.mean(-1, keepdim=True)).square().mean().sqrt()


def mixer_oracle(h, cfg, w, index):
    """What the mixer of layer ``index`` makes of the rows ``h`` (the first layer that mixes values saw the same rows)."""
    w, h, carried = {n: t.double() for n, t in w.items()}, h.double(), {}
    first = next((i for i, x in enumerate(cfg["layers"]) if x["mixer"].get("v_mix")), None)
    layer, p = cfg["layers"][index], f"l{index}.mix."
    if layer["type"] == "latent_attention":
        return M.latent_attention(h, w, p, layer["mixer"], float(cfg["norm"]["eps"]))
    if layer["type"] == "mingru":
        return M.mingru(h, w, p)
    if first is not None and first < index:
        M.attention(h, w, f"l{first}.mix.", cfg["layers"][first]["mixer"], carried)
    return M.attention(h, w, p, layer["mixer"], carried)


def run_mixer(model, ctx, index, hs, schedule):
    """Feed rows (``hs``: per request [T, width]) to the mixer of layer ``index`` under ``schedule`` = [[(request, count), ...], ...];
    returns its output per request.  What the layer keeps between steps is the context's."""
    from megatron_mixtera_b200 import ops

    dt, dev = model.config.params_dtype, torch.device("cuda")
    first = [j for j in range(index) if model.config.mixes_values_first(j)]
    at, got = [0] * len(hs), [[] for _ in hs]
    for part in schedule:
        ctx.schedule_tokens([(i, [0] * n) for i, n in part])
        ctx.initialize_attention_state()
        x = torch.zeros((ctx.padded_active_token_count, model.config.hidden_size), dtype=dt, device=dev)
        row = 0
        for i, n in part:
            x[row: row + n] = hs[i][at[i]: at[i] + n].to(dev, dt)
            at[i] += n
            row += n
        with torch.inference_mode():
            out, step = torch.zeros(x.shape, dtype=torch.float32, device=dev), {}
            for j in first + [index]:
                y = model.layers[j].mixer(x, ctx, model._rope[j], step)
            ops.residual_norm(out, ops.PendingRows(partials=y), [], [], eps=1.0)
        row = 0
        for i, n in part:
            got[i].append(out[row: row + n].cpu())
            row += n
        ctx.complete_step([i for i, _ in part if at[i] == len(hs[i])])
    return [torch.cat(g) if g else None for g in got]


def rel(got, want):
    """Largest row error relative to the rows' rms."""
    want = want.float()
    return float(((got.float().cpu() - want).square().mean(-1).sqrt() / want.square().mean().sqrt()).max())
