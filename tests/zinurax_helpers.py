"""Small Zinurax configurations, random weights and the loops that compare the framework with the plain oracle."""
import math

import torch
from hybrid_helpers import build, error, replay, tokens  # noqa: F401  (re-exported)

from oracle import zinurax_oracle as Z


def latent(heads=5, dim=24, rot_dim=16, vdim=40, kv_rank=96, size=33, scale=None, base=5000.0, yarn=True, kv_from=None, ff=112):
    rot = {"base": base, "dims": rot_dim}
    if yarn:
        rot["scaling"] = {"factor": 4.0, "original": 96, "fast": 8.0, "slow": 1.0}
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "rot": rot, "mask": {"size": size},
         "scale": scale if scale is not None else 1.0 / math.sqrt(dim + rot_dim)}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def delta(heads=3, dim=48, ff=112):
    return {"type": "general_delta", "mixer": {"heads": heads, "dim": dim}, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(layers, width=160, vocab=301, eps=1e-5):
    return {"architecture": "Zinurax", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


CONFIGS = {
    # mixed order, a layer without feed-forward, two windows over one set of cached rows, sizes that TMA can address
    "mixed": (config([delta(), latent(), latent(heads=3, dim=16, size=70, kv_from=1, ff=None), delta(heads=2, dim=64, ff=72)]), 24),
    # many heads, a latent that needs padding, a window shorter than any tile, no frequency scaling; one wide recurrent head
    "many_heads": (config([latent(heads=20, dim=8, rot_dim=24, vdim=16, kv_rank=72, size=7, yarn=False), delta(heads=1, dim=128)],
                          width=136, vocab=260), 8),
    # nothing is a multiple of 8
    "odd": (config([latent(heads=3, dim=12, rot_dim=6, vdim=10, kv_rank=36, size=19), delta(heads=3, dim=20, ff=30),
                    latent(heads=7, dim=10, rot_dim=6, vdim=11, kv_rank=36, size=50, kv_from=0, ff=21)], width=100, vocab=77), 5),
    # a window of one token, a head of one channel pair, the smallest recurrent head
    "tiny": (config([latent(heads=1, dim=8, rot_dim=2, vdim=8, kv_rank=8, size=1), delta(heads=1, dim=8),
                     latent(heads=2, dim=8, rot_dim=2, vdim=8, kv_rank=16, size=200)], width=32, vocab=40), 3),
    # the widest latent of the tensor-core kernel, more heads than a block of query rows, the widest recurrent head
    "wide": (config([latent(heads=72, dim=16, rot_dim=64, vdim=8, kv_rank=512, size=150), delta(heads=1, dim=256)], width=128), 16),
    # recurrent layers only / attention only
    "delta_only": (config([delta(), delta(heads=2, dim=32)], width=96), 9),
    "latent_only": (config([latent(size=64), latent(heads=2, kv_from=0, size=65)], width=96), 0),
}


def weights(cfg, rank, seed=0, gain=1.0):
    """Random weights as a checkpoint holds them (bf16 values).  Linears keep the scale of their input (times ``gain`` for
    the queries: peaked attention); the decay's bias spreads the heads between short and long memory."""
    g = torch.Generator().manual_seed(seed)

    def mat(n, k, s=1.0):
        return torch.randn(n, k, generator=g) * (s / math.sqrt(k))

    def vec(n, mean=1.0, std=0.2):
        return mean + std * torch.randn(n, generator=g)

    W, out = cfg["width"], {}
    out["embed"] = torch.randn(cfg["vocab"], W, generator=g)
    out["embed.norm"], out["final.norm"] = vec(W), vec(W)
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", layer["mixer"]
        out[f"l{i}.norm1"] = vec(W)
        H, d = m["heads"], m["dim"]
        if layer["type"] == "latent_attention":
            out[p + "q"] = mat(H * (d + m["rot_dim"]), W, 2.0 * gain)
            if "kv_from" not in m:
                out[p + "dkv"] = mat(m["kv_rank"] + m["rot_dim"], W)
                out[p + "dkv.norm"] = vec(m["kv_rank"])
            out[p + "uk"], out[p + "uv"] = mat(H * d, m["kv_rank"]), mat(H * m["vdim"], m["kv_rank"])
            out[p + "g"], out[p + "o"] = mat(H, W), mat(W, H * m["vdim"])
        else:
            n = H * d
            for k in ("r", "k", "v", "g", "a"):
                out[p + k] = mat(n, W)
            out[p + "a.b"], out[p + "w0"] = vec(n, 0.0, 1.0), vec(n, -2.0, 2.0)
            out[p + "w1"], out[p + "w2"] = mat(rank, W), mat(n, rank)
            out[p + "norm"], out[p + "o"] = vec(n), mat(W, n)
        if layer["mlp"] is not None:
            ff = layer["mlp"]["ff"]
            out[f"l{i}.norm2"], out[f"l{i}.mlp.up"], out[f"l{i}.mlp.down"] = vec(W), mat(ff, W), mat(W, ff)
    return {k: v.to(torch.bfloat16) for k, v in out.items()}


def oracle_logits(toks, cfg, w):
    return Z.forward(toks, cfg, w).float()
