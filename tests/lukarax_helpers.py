"""Small Lukarax configurations, random weights and the loops that compare the framework with the plain oracle."""
import math

import torch
from hybrid_helpers import build, error, replay, tokens  # noqa: F401  (re-exported)

from oracle import lukarax_oracle as L


def dense(ff=72):
    return {"kind": "dense", "ff": ff}


def experts(n=6, top=3, ff=40, identity=2, groups=(4, 2), scale=1.7):
    return {"kind": "moe", "expert": {"ff": ff},
            "router": {"experts": n, "identity": identity, "top": top, "scale": scale, "groups": {"count": groups[0], "keep": groups[1]}}}


def differential(heads=6, kv_heads=2, dim=24, vdim=40, rot=16, diff=0.4, kv_from=None, base=7000.0, mlp=experts()):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": 1.4 / math.sqrt(dim), "diff": diff,
         "rot": {"base": base, "dims": rot}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


def sink(heads=8, kv_heads=2, dim=32, rot=16, size=23, softcap=9.0, scaling=(3.0, 512, 16.0, 1.5), mlp=experts()):
    return {"type": "attention_2", "mlp": mlp, "mixer": {
        "heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": 0.9 / math.sqrt(dim) * 4, "mask": {"size": size}, "softcap": softcap,
        "rot": {"base": 5000.0, "dims": rot, "scaling": dict(zip(("factor", "original", "fast", "slow"), scaling))}}}


def parallel(heads=4, kv_heads=2, dim=32, vdim=24, size=41, keep=3, rows=12, longest=70, m_heads=3, m_dim=32, m_vdim=40, cap=9.0,
             left=0.6, right=1.2, mlp=experts()):
    return {"type": "parallel", "mlp": mlp, "bias_rows": rows, "mixer": {
        "left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": 1.2 / math.sqrt(dim), "bias_max": longest,
                 "mask": {"size": size, "keep_first": keep}}, "left_scale": left,
        "right": {"heads": m_heads, "dim": m_dim, "vdim": m_vdim, "gate_cap": cap}, "right_scale": right}}


def config(layers, width=160, vocab=301, eps=1e-5, scale=3.0, streams=3):
    return {"architecture": "Lukarax", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width, "streams": streams,
            "embedding": {"scale": scale}}


CONFIGS = {
    # every mixer, both feed-forwards and none, rows read from another layer (twice), several windows and head groupings
    "mixed": config([differential(mlp=dense()), parallel(), sink(), differential(kv_from=0, diff=0.25), parallel(size=70, keep=66, mlp=None),
                     differential(heads=2, kv_heads=1, dim=16, vdim=16, rot=16, mlp=dense(40)), differential(heads=2, kv_heads=1, dim=16, vdim=16, rot=16, kv_from=5)]),
    # wide heads, value sizes of their own, groups of heads that do not divide 64, many experts in many groups, two streams
    "wide": config([parallel(heads=16, kv_heads=1, dim=128, vdim=64, size=150, keep=1, rows=32, longest=300, m_heads=2, m_dim=128, m_vdim=128,
                             mlp=experts(30, 5, 100, 6, (6, 3))),
                    differential(heads=3, kv_heads=1, dim=80, vdim=128, rot=80, mlp=dense(192)),
                    differential(heads=8, kv_heads=2, dim=64, vdim=128, rot=32), differential(heads=10, kv_heads=1, dim=64, vdim=64, rot=64),
                    sink(heads=6, kv_heads=2, dim=128, rot=128, size=64)], width=192, streams=2),
    # nothing is a multiple of 8
    "odd": config([sink(heads=3, kv_heads=3, dim=20, rot=12, size=19, mlp=experts(7, 2, 21, 0, (1, 1))),
                   differential(heads=3, kv_heads=3, dim=10, vdim=13, rot=6, mlp=dense(37)), parallel(heads=3, kv_heads=1, dim=12, vdim=11, size=30,
                   keep=5, rows=6, longest=9.5, m_heads=3, m_dim=20, m_vdim=11, mlp=experts(4, 3, 13, 1, (5, 4)))], width=100, vocab=77, streams=5),
    # windows of one token, one stream, one expert beside one identity expert, the smallest heads
    "tiny": config([differential(heads=1, kv_heads=1, dim=8, vdim=8, rot=8, mlp=experts(1, 1, 8, 1, (1, 1))),
                    parallel(heads=1, kv_heads=1, dim=8, vdim=8, size=1, keep=0, rows=2, longest=4, m_heads=1, m_dim=8, m_vdim=8, mlp=dense(8)),
                    sink(heads=2, kv_heads=1, dim=8, rot=8, size=1, mlp=experts(3, 1, 8, 0, (3, 1)))], width=32, vocab=40, streams=1),
    # heads beyond the tensor-core kernels, no window beside the kept tokens' one
    "large_heads": config([differential(heads=2, kv_heads=1, dim=144, vdim=256, rot=64), sink(heads=2, kv_heads=1, dim=200, rot=96, size=90),
                           parallel(heads=2, kv_heads=1, dim=192, vdim=136, m_heads=1, m_dim=256, m_vdim=32)], width=128, streams=4),
    "memory": config([parallel(m_heads=4, m_dim=64, m_vdim=64, left=0.1, right=1.5), parallel(m_heads=2, m_dim=16, m_vdim=96, left=0.05, right=1.0)],
                     width=96),
    "sinks": config([sink(size=64), sink(size=65, heads=4, kv_heads=4, softcap=30.0), sink(size=500)], width=96),
    "maps": config([differential(), differential(heads=4, kv_heads=4, dim=48, vdim=64, rot=24), differential(kv_from=0)], width=96),
}


def weights(cfg, seed=0, gain=1.0, settled=False):
    """Random weights as a checkpoint holds them (bf16 values).  Linears keep the scale of their input; ``gain`` sharpens attention (through the
    queries); forget gates spread the heads between short and long memory; the streams differ from one another.  ``settled``: which
    experts are chosen is beyond the doubt of 16-bit rounding (the weights still differ from token to token)."""
    g = torch.Generator().manual_seed(seed)

    def mat(n, k, s=1.0):
        return torch.randn(n, k, generator=g) * (s / math.sqrt(k))

    def vec(n, mean=1.0, std=0.2):
        return mean + std * torch.randn(n, generator=g)

    W, S, out = cfg["width"], cfg["streams"], {}
    out["embed"] = torch.randn(cfg["vocab"], W, generator=g) / math.sqrt(W) * 2.0

    def norm(name):
        out[name], out[name + ".b"] = vec(W), vec(W, 0.0, 0.1)

    def blends(p):
        out[p + ".in"], out[p + ".out"] = vec(S, 1.0 / S, 0.3), vec(S, 0.8, 0.3)
        out[p + ".mix"] = 0.9 * torch.eye(S) + 0.1 * torch.randn(S, S, generator=g)

    norm("final.norm")
    for i, layer in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.mix.", layer["mixer"], layer["mlp"]
        norm(f"l{i}.norm1")
        blends(f"l{i}.hc1")
        if layer["type"] == "attention":
            H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            out[p + "q"] = mat(H * 2 * d, W, gain)
            if "kv_from" not in m:
                out[p + "k"], out[p + "v"] = mat(G * 2 * d, W), mat(G * dv, W)
            for k in ("lq1", "lk1", "lq2", "lk2"):
                out[p + k] = vec(d, 0.0, 0.7 / d ** 0.25)
            out[p + "g"], out[p + "o"] = mat(H * dv, W), mat(W, H * dv)
        elif layer["type"] == "attention_2":
            H, G, d = m["heads"], m["kv_heads"], m["dim"]
            out[p + "q"], out[p + "q.b"], out[p + "k"], out[p + "k.b"] = mat(H * d, W), vec(H * d, 0.0, 0.3), mat(G * d, W), vec(G * d, 0.0, 0.3)
            out[p + "sink"], out[p + "o"], out[p + "o.b"] = vec(H, 1.0, 1.0), mat(W, H * d), vec(W, 0.0, 0.2)
        else:
            a, r = m["left"], m["right"]
            for k, n in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"])):
                out[p + "left." + k] = mat(n, W, gain if k == "q" else 1.0)
            out[p + "left.rel"], out[p + "left.o"] = vec(layer["bias_rows"] * a["heads"], 0.0, 1.0).view(-1, a["heads"]), mat(W, a["heads"] * a["vdim"])
            h, n = r["heads"], r["heads"] * r["vdim"]
            out.update({p + "right.q": mat(h * r["dim"], W), p + "right.k": mat(h * r["dim"], W), p + "right.v": mat(n, W), p + "right.g": mat(n, W),
                        p + "right.o": mat(W, n), p + "right.norm": vec(n), p + "right.i": mat(h, W, 1.5), p + "right.i.b": vec(h, -0.5, 0.5),
                        p + "right.f": mat(h, W, 1.5), p + "right.f.b": vec(h, 2.5, 1.5)})
        if mlp is None:
            continue
        norm(f"l{i}.norm2")
        blends(f"l{i}.hc2")
        p = f"l{i}.mlp."
        if mlp["kind"] == "dense":
            parts = [("", mlp["ff"])]
        else:
            r = mlp["router"]
            columns = r["experts"] + r["identity"]
            out[p + "router"], out[p + "correction"] = mat(columns, W, 1.5), vec(columns, -0.1, 0.1)
            if settled:
                out[p + "router"] *= 0.3
                out[p + "correction"] = 0.5 * torch.randperm(columns, generator=g) - 1.0
                if r["identity"] and r["top"] > 1:
                    out[p + "correction"][-1] = 0.5 * columns
            parts = [(f"e{e}.", mlp["expert"]["ff"]) for e in range(r["experts"])]
        for name, ff in parts:
            out[p + name + "gate"], out[p + name + "up"], out[p + name + "down"] = mat(ff, W, 2.0), mat(ff, W), mat(W, ff)
    return {k: v.to(torch.bfloat16) for k, v in out.items()}


def oracle_logits(toks, cfg, w):
    with torch.inference_mode():
        return L.forward(toks, cfg, w).float()


def position_errors(got, want):
    """rms(difference) / rms(logits) of every position, the mean over the vocabulary taken off."""
    d = got.float().cpu() - want
    d = d - d.mean(-1, keepdim=True)
    return d.square().mean(-1).sqrt() / (want - want.mean(-1, keepdim=True)).square().mean().sqrt()


def mixer_oracle(h, cfg, w, index):
    """What the mixer of layer ``index`` makes of the rows ``h`` (a layer that reads another's rows: that layer saw the same rows)."""
    w = {n: t.double() for n, t in w.items()}
    h, eps = h.double(), float(cfg["norm"]["eps"])
    layer, p = cfg["layers"][index], f"l{index}.mix"
    m = layer["mixer"]
    if layer["type"] == "attention":
        src = m.get("kv_from", index)
        return L.differential_attention(h, w, p, m, eps, L.differential_keys(h, w, f"l{src}.mix", cfg["layers"][src]["mixer"]))
    if layer["type"] == "attention_2":
        return L.sink_attention(h, w, p, m, eps)
    return (m["left_scale"] * L.biased_attention(h, w, p + ".left", m["left"])
            + m["right_scale"] * L.matrix_memory(h, w, p + ".right", m["right"], eps))


def run_mixer(model, ctx, index, hs, schedule):
    """Feed rows (``hs``: per request [T, width]) to the mixer of layer ``index`` under ``schedule`` = [[(request, count), ...], ...];
    returns its output per request.  What the layer keeps between steps is the context's."""
    from megatron_mixtera_b200 import ops

    dt, dev = model.config.params_dtype, torch.device("cuda")
    mixer = model.layers[index].mixer
    source = getattr(model.config.layers[index].mixer, "kv_from", None)
    one = torch.ones(1, device=dev)
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
            out = torch.zeros((x.shape[0], 1, x.shape[1]), dtype=torch.float32, device=dev)
            if source is not None:
                model.layers[source].mixer(x, ctx, model._rope[source])
            y = mixer(x, ctx, model._rope[index])
            ops.stream_norm(out, ops.PendingStreams(partials=y, bias=mixer.output_bias, mix=one.view(1, 1), gain=one))
        row = 0
        for i, n in part:
            got[i].append(out[row: row + n, 0].cpu())
            row += n
        ctx.complete_step([i for i, _ in part if at[i] == len(hs[i])])
    return [torch.cat(g) if g else None for g in got]


def rel(got, want):
    """Largest row error relative to the rows' rms."""
    want = want.float()
    return float(((got.float().cpu() - want).square().mean(-1).sqrt() / want.square().mean().sqrt()).max())
