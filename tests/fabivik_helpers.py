"""Small Fabivik configurations, random weights and the loops that compare the framework with the plain oracle."""
import math

import torch
from hybrid_helpers import build, error, replay, tokens  # noqa: F401  (re-exported)

from oracle import fabivik_oracle as F


def experts(n=5, top=2, ff=40, limit=1.5, shared_ff=72, shared_limit=0.8):
    return {"kind": "moe", "router": {"experts": n, "top": top}, "expert": {"ff": ff, "limit": limit},
            "shared": None if shared_ff is None else {"ff": shared_ff, "limit": shared_limit}}


def attention(heads=6, kv_heads=2, dim=24, vdim=40, size=33, conv=4, scale=None, v_mix=True, mlp=experts()):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "v_mix": v_mix,
         "scale": scale if scale is not None else 1.3 / math.sqrt(dim), "mask": {"size": size} if size else None}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def wkv(heads=3, dim=40, rank=24, mlp=experts()):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim}, "mlp": mlp, "rank": rank}


def delta(heads=6, kv_heads=3, dim=32, vdim=48, conv=4, mlp=experts()):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": mlp}


def config(layers, width=160, vocab=301, eps=1e-5, scale=7.0, logit_scale=0.6):
    return {"architecture": "Fabivik", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width,
            "embedding": {"scale": scale}, "logit_scale": logit_scale}


CONFIGS = {
    # every mixer, a layer without feed-forward, two windows and two head groupings over mixed values, one layer outside the mixing
    "mixed": config([attention(size=33), wkv(), attention(heads=2, size=70, mlp=None), delta(),
                     attention(heads=4, kv_heads=4, dim=16, vdim=16, size=20, v_mix=False, conv=3), wkv(heads=2, dim=64, rank=16)]),
    # wide heads, a value size of its own, eight taps, many experts of which some get no token, feed-forwards that need padding
    "wide": config([delta(heads=2, kv_heads=1, dim=128, vdim=256, conv=8, mlp=experts(40, 5, 100, 2.0, 130)),
                    attention(heads=16, kv_heads=1, dim=128, vdim=64, size=150, conv=8), wkv(heads=1, dim=128, rank=64),
                    attention(heads=3, kv_heads=1, dim=72, vdim=128, size=64, v_mix=False, mlp=experts(3, 3))], width=192),
    # nothing is a multiple of 8
    "odd": config([attention(heads=3, kv_heads=3, dim=12, vdim=10, size=19, conv=2), delta(heads=3, kv_heads=1, dim=20, vdim=11, conv=3,
                   mlp=experts(7, 2, 21, 1.0, 33)), wkv(heads=3, dim=12, rank=5),
                   attention(heads=6, kv_heads=3, dim=9, vdim=10, size=50, mlp=experts(4, 1, 13, shared_ff=None))], width=100, vocab=77),
    # a window of one token, no convolution at all, one expert, the smallest heads
    "tiny": config([attention(heads=1, kv_heads=1, dim=8, vdim=8, size=1, conv=1, mlp=experts(1, 1, 8, shared_ff=8)),
                    delta(heads=1, kv_heads=1, dim=8, vdim=8, conv=1, mlp=experts(2, 2, 64)), wkv(heads=1, dim=8, rank=8, mlp=None),
                    attention(heads=2, kv_heads=1, dim=8, vdim=8, size=200, conv=2, mlp=experts(3, 1, 8))], width=32, vocab=40),
    # heads beyond the tensor-core kernels, no window
    "large_heads": config([attention(heads=2, kv_heads=1, dim=192, vdim=256, size=None), delta(heads=1, kv_heads=1, dim=256, vdim=32),
                           wkv(heads=1, dim=256, rank=32)], width=128),
    "wkv_only": config([wkv(), wkv(heads=4, dim=32)], width=96),
    "delta_only": config([delta(), delta(heads=2, kv_heads=2, dim=64, vdim=64)], width=96),
    "attention_only": config([attention(size=64), attention(size=65, heads=8), attention(size=None, v_mix=False)], width=96),
}


def weights(cfg, seed=0, gain=1.0):
    """Random weights as a checkpoint holds them (bf16 values).  Linears keep the scale of their input; ``gain`` sharpens attention
    (through the norms of queries and keys); decays spread the heads between short and long memory."""
    g = torch.Generator().manual_seed(seed)

    def mat(n, k, s=1.0):
        return torch.randn(n, k, generator=g) * (s / math.sqrt(k))

    def vec(n, mean=1.0, std=0.2):
        return mean + std * torch.randn(n, generator=g)

    W, out, mixing = cfg["width"], {}, 0
    out["embed"], out["head"] = torch.randn(cfg["vocab"], W, generator=g) / cfg["embedding"]["scale"], mat(cfg["vocab"], W)
    out["final.norm"] = vec(W, 0.0)
    for i, layer in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.mix.", layer["mixer"], layer["mlp"]
        out[f"l{i}.norm1"] = vec(W, 0.0)
        H, d = m["heads"], m["dim"]
        if layer["type"] == "wkv":
            n, rank = H * d, layer["rank"]
            for k in "rkvg":
                out[p + k] = mat(n, W)
            for k in "rkvgw":
                out[p + "mu." + k] = torch.rand(W, generator=g)
            out[p + "w1"], out[p + "w2"], out[p + "w0"] = mat(rank, W), mat(n, rank), vec(n, -3.0, 2.0)
            out[p + "u"], out[p + "norm"], out[p + "o"] = vec(n, 0.5, 0.5).view(H, d), vec(n), mat(W, n)
        else:
            G, dv = m["kv_heads"], m["vdim"]
            kv = {"attention": (H, G, G), "delta": (G, G, H)}[layer["type"]]
            for k, heads, size in zip("qkv", kv, (d, d, dv)):
                out[p + k] = mat(heads * size, W)
                taps = torch.randn(heads * size, m["conv"], generator=g) * 0.4
                taps[:, -1] += 1.0
                out[p + k + ".conv"] = taps
            out[p + "o"] = mat(W, H * dv)
            if layer["type"] == "attention":
                out[p + "q.norm"], out[p + "k.norm"] = vec(d, gain), vec(d, gain)
                if m["v_mix"]:
                    if mixing or seed % 2:  # (the first such layer's value is unused; a checkpoint may hold it all the same)
                        out[p + "vmix"] = torch.tensor(0.3)
                    mixing += 1
            else:
                out[p + "g"], out[p + "b"], out[p + "a"] = mat(H * dv, W), mat(H, W, 2.0), mat(H, W)
                out[p + "A_log"], out[p + "dt_bias"], out[p + "norm"] = vec(H, 0.0, 0.7), vec(H, -2.5, 1.5), vec(dv)
        if mlp is not None:
            out[f"l{i}.norm2"] = vec(W, 0.0)
            p = f"l{i}.mlp."
            out[p + "router"] = mat(mlp["router"]["experts"], W, 1.5)
            parts = [(f"e{e}", mlp["expert"]["ff"]) for e in range(mlp["router"]["experts"])]
            if mlp["shared"]:
                parts.append(("shared", mlp["shared"]["ff"]))
                out[p + "shared.sg"] = mat(1, W)
            for name, ff in parts:
                out[p + name + ".gate"], out[p + name + ".up"], out[p + name + ".down"] = mat(ff, W, 2.0), mat(ff, W), mat(W, ff)
    return {k: v.to(torch.bfloat16) for k, v in out.items()}


def oracle_logits(toks, cfg, w):
    return F.forward(toks, cfg, w).float()


def position_errors(got, want):
    """rms(difference) / rms(logits) of every position, the mean over the vocabulary taken off."""
    d = got.float().cpu() - want
    d = d - d.mean(-1, keepdim=True)
    return d.square().mean(-1).sqrt() / (want - want.mean(-1, keepdim=True)).square().mean().sqrt()


def run_mixer(model, ctx, index, hs, schedule):
    """Feed rows (``hs``: per request [T, width]) to the mixer of layer ``index`` under ``schedule`` = [[(request, count), ...], ...];
    returns its output per request.  What the layer keeps between steps is the context's."""
    from megatron_mixtera_b200 import ops

    dt, dev = model.config.params_dtype, torch.device("cuda")
    at = [0] * len(hs)
    got = [[] for _ in hs]
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
            out = torch.zeros(x.shape, dtype=torch.float32, device=dev)
            step = {}
            for j in range(index + 1):
                mixer = model.layers[j].mixer
                if j == index or getattr(mixer, "first_values", False):
                    y = mixer(x, ctx, step=step)
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
