"""Plain CPU oracle of the Lukarax design.  TEST INFRASTRUCTURE ONLY.

One slow function per mechanism, whole sequences only: no cache, no state between calls, no batching.
It shares no code with the shipped package.  Weights come as a dict of float tensors named as in a checkpoint, the
configuration as the dict of its ``config.json``.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

Tensor = torch.Tensor
Weights = Dict[str, Tensor]


def layer_norm(x: Tensor, weight: Tensor, bias: Tensor, eps: float) -> Tensor:
    d = x - x.mean(dim=-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(dim=-1, keepdim=True) + eps) * weight + bias


def unit_rms(x: Tensor, eps: float) -> Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def silu(x: Tensor) -> Tensor:
    return x * torch.sigmoid(x)


def log_sigmoid(x: Tensor) -> Tensor:
    return torch.clamp(x, max=0) - torch.log1p(torch.exp(-x.abs()))


# ---------------------------------------------------------------------------------------------------------------------
# Rotation
# ---------------------------------------------------------------------------------------------------------------------
def frequencies(rot: dict) -> tuple:
    """(frequency of every pair, factor on cos and sin)."""
    dims, base, sc = rot["dims"], float(rot["base"]), rot.get("scaling")
    freq = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not sc:
        return freq, 1.0

    def where(turns):
        return dims * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

    lo, hi = max(math.floor(where(sc["fast"])), 0), min(math.ceil(where(sc["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freq):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / sc["factor"] * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x: Tensor, rot: dict, halves: bool) -> Tensor:
    """x [T, vectors, dim] at positions 0, 1, ...: the first ``dims`` dimensions turn, in pairs (2i, 2i + 1) or, ``halves``,
    (i, i + dims / 2)."""
    freq, factor = frequencies(rot)
    dims, out = rot["dims"], x.clone()
    angle = torch.arange(x.shape[0], dtype=x.dtype)[:, None] * torch.tensor(freq, dtype=x.dtype)[None, :]
    c, s = (torch.cos(angle) * factor)[:, None, :], (torch.sin(angle) * factor)[:, None, :]
    iu = torch.arange(dims // 2) if halves else torch.arange(0, dims, 2)
    iv = iu + dims // 2 if halves else iu + 1
    u, v = x[..., iu], x[..., iv]
    out[..., iu], out[..., iv] = u * c - v * s, v * c + u * s
    return out


# ---------------------------------------------------------------------------------------------------------------------
# Attention
# ---------------------------------------------------------------------------------------------------------------------
def visible(n: int, mask: Optional[dict]) -> Tensor:
    """[query, key]: causal; with a size, that many newest tokens (the token itself included) and the ``keep_first`` first."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    ok = j <= i
    if mask and mask.get("size") is not None:
        ok = ok & ((i - j < mask["size"]) | (j < mask.get("keep_first", 0)))
    return ok


def bucket(n: int, rows: int, longest: float) -> int:
    """Row of a distance bias table: one per distance up to half the rows, logarithmic beyond."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(longest / half) * (rows - half)))


def distance_bias(n: int, table: Tensor, longest: float) -> Tensor:
    """[heads, query, key] (zero for keys after the query)."""
    row = torch.tensor([bucket(d, table.shape[0], longest) for d in range(n)])
    by_distance = table[row]  # [distance, head]
    age = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    return by_distance[age.clamp(min=0)].permute(2, 0, 1) * (age >= 0)


def attend(q: Tensor, k: Tensor, v: Tensor, scale: float, mask: Optional[dict], *, bias: Optional[Tensor] = None,
           softcap: Optional[float] = None, sink: Optional[Tensor] = None) -> Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, dv]; query heads in consecutive groups.  ``sink`` [H] joins the denominator."""
    group = q.shape[1] // k.shape[1]
    k, v = k.repeat_interleave(group, dim=1), v.repeat_interleave(group, dim=1)
    score = torch.einsum("qhd,khd->hqk", q, k) * scale
    if softcap:
        score = softcap * torch.tanh(score / softcap)
    if bias is not None:
        score = score + bias
    score = score.masked_fill(~visible(q.shape[0], mask), -math.inf)
    if sink is None:
        weight = torch.softmax(score, dim=-1)
    else:
        top = torch.maximum(score.amax(dim=-1, keepdim=True), sink[:, None, None])
        e = torch.exp(score - top)
        weight = e / (e.sum(dim=-1, keepdim=True) + torch.exp(sink[:, None, None] - top))
    return torch.einsum("hqk,khv->qhv", weight, v)


def differential_keys(h: Tensor, w: Weights, p: str, m: dict) -> tuple:
    """(keys [T, kv_heads, 2 maps, dim] after rotation, values [T, kv_heads, vdim])."""
    T, G, d = h.shape[0], m["kv_heads"], m["dim"]
    k = rotate((h @ w[p + ".k"].T).view(T, G * 2, d), m["rot"], False)
    return k.view(T, G, 2, d), (h @ w[p + ".v"].T).view(T, G, m["vdim"])


def differential_lambda(w: Weights, p: str, m: dict) -> Tensor:
    return torch.exp((w[p + ".lq1"] * w[p + ".lk1"]).sum()) - torch.exp((w[p + ".lq2"] * w[p + ".lk2"]).sum()) + m["diff"]


def differential_combine(a1: Tensor, a2: Tensor, lam: Tensor, diff: float, eps: float) -> Tensor:
    return unit_rms(a1 - lam * a2, eps) * (1.0 - diff)


def differential_attention(h: Tensor, w: Weights, p: str, m: dict, eps: float, kv: tuple) -> Tensor:
    """``kv``: keys and values, this layer's own or another's."""
    T, H, d = h.shape[0], m["heads"], m["dim"]
    q = rotate((h @ w[p + ".q"].T).view(T, H * 2, d), m["rot"], False).view(T, H, 2, d)
    k, v = kv
    a1, a2 = (attend(q[:, :, i], k[:, :, i], v, m["scale"], m.get("mask")) for i in range(2))
    o = differential_combine(a1, a2, differential_lambda(w, p, m), m["diff"], eps)
    return (o.reshape(T, -1) * torch.sigmoid(h @ w[p + ".g"].T)) @ w[p + ".o"].T


def biased_attention(h: Tensor, w: Weights, p: str, m: dict) -> Tensor:
    """No rotation; a learned bias by distance; a window that keeps the first tokens."""
    T = h.shape[0]
    q, k, v = ((h @ w[p + "." + s].T).view(T, n, d) for s, n, d in (
        ("q", m["heads"], m["dim"]), ("k", m["kv_heads"], m["dim"]), ("v", m["kv_heads"], m["vdim"])))
    o = attend(q, k, v, m["scale"], m.get("mask"), bias=distance_bias(T, w[p + ".rel"], m["bias_max"]))
    return o.reshape(T, -1) @ w[p + ".o"].T


def sink_attention(h: Tensor, w: Weights, p: str, m: dict, eps: float) -> Tensor:
    """Values are the projected keys; queries and keys are rotated, then normed; capped scores; a sink per head."""
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = (h @ w[p + ".q"].T + w[p + ".q.b"]).view(T, H, d)
    v = (h @ w[p + ".k"].T + w[p + ".k.b"]).view(T, G, d)
    q, k = (unit_rms(rotate(x, m["rot"], True), eps) for x in (q, v))
    o = attend(q, k, v, m["scale"], m.get("mask"), softcap=m.get("softcap"), sink=w[p + ".sink"])
    return o.reshape(T, -1) @ w[p + ".o"].T + w[p + ".o.b"]


# ---------------------------------------------------------------------------------------------------------------------
# Matrix memory
# ---------------------------------------------------------------------------------------------------------------------
def memory_inputs(h: Tensor, w: Weights, p: str, m: dict) -> tuple:
    """(q, k) [T, heads, dim], v [T, heads, vdim], (log input gate, log forget gate) [T, heads]."""
    T, H, d, cap = h.shape[0], m["heads"], m["dim"], m["gate_cap"]
    q, k = ((h @ w[p + "." + s].T).view(T, H, d) for s in "qk")
    i, f = (cap * torch.tanh((h @ w[p + "." + s].T + w[p + "." + s + ".b"]) / cap) for s in "if")
    return q * d ** -0.5, k, (h @ w[p + ".v"].T).view(T, H, m["vdim"]), i, log_sigmoid(f)


def memory_scan(q: Tensor, k: Tensor, v: Tensor, i: Tensor, f: Tensor, state: Optional[tuple] = None) -> tuple:
    """Token by token, scaled by a running maximum; returns (o [T, heads, vdim], (S, n, maximum))."""
    T, H, d = q.shape
    S, n, top = state if state is not None else (torch.zeros(H, d, v.shape[2], dtype=q.dtype), torch.zeros(H, d, dtype=q.dtype),
                                                 torch.zeros(H, dtype=q.dtype))
    out = torch.empty_like(v)
    for t in range(T):
        new = torch.maximum(f[t] + top, i[t])
        keep, write = torch.exp(f[t] + top - new), torch.exp(i[t] - new)
        S = keep[:, None, None] * S + write[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + write[:, None] * k[t]
        top = new
        below = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-top)) + 1e-6
        out[t] = torch.einsum("hij,hi->hj", S, q[t]) / below[:, None]
    return out, (S, n, top)


def matrix_memory(h: Tensor, w: Weights, p: str, m: dict, eps: float) -> Tensor:
    o, _ = memory_scan(*memory_inputs(h, w, p, m))
    o = unit_rms(o, eps).reshape(h.shape[0], -1) * w[p + ".norm"]
    return (o * torch.sigmoid(h @ w[p + ".g"].T)) @ w[p + ".o"].T


# ---------------------------------------------------------------------------------------------------------------------
# Feed-forward
# ---------------------------------------------------------------------------------------------------------------------
def gated(x: Tensor, w: Weights, p: str) -> Tensor:
    return (silu(x @ w[p + ".gate"].T) * (x @ w[p + ".up"].T)) @ w[p + ".down"].T


def route(z: Tensor, correction: Tensor, r: dict) -> tuple:
    """One token's logits -> (chosen experts, their weights)."""
    s = torch.softmax(z, dim=-1)
    choice = s + correction
    groups = r.get("groups")
    if groups:
        of_group = choice.view(groups["count"], -1)
        best = torch.topk(of_group.amax(dim=-1), groups["keep"]).indices
        closed = torch.ones(groups["count"], dtype=torch.bool)
        closed[best] = False
        choice = of_group.masked_fill(closed[:, None], -math.inf).reshape(-1)
    chosen = torch.topk(choice, r["top"]).indices
    weight = s[chosen]
    return chosen.tolist(), weight / (weight.sum() + 1e-20) * r["scale"]


def mixture(h: Tensor, w: Weights, p: str, m: dict) -> Tensor:
    out, tokens_of = torch.zeros_like(h), {}
    for t, z in enumerate(h @ w[p + ".router"].T):
        for e, a in zip(*route(z, w[p + ".correction"], m["router"])):
            tokens_of.setdefault(e, []).append((t, a))
    for e, pairs in tokens_of.items():
        t, a = [t for t, _ in pairs], torch.stack([a for _, a in pairs])
        out[t] += a[:, None] * (gated(h[t], w, f"{p}.e{e}") if e < m["router"]["experts"] else h[t])
    return out


def feed_forward(h: Tensor, w: Weights, p: str, m: dict) -> Tensor:
    return gated(h, w, p) if m["kind"] == "dense" else mixture(h, w, p, m)


# ---------------------------------------------------------------------------------------------------------------------
# Streams
# ---------------------------------------------------------------------------------------------------------------------
def streams_in(x: Tensor, w: Weights, p: str) -> Tensor:
    """x [streams, T, width] -> what the sublayer reads."""
    return torch.einsum("s,stw->tw", w[p + ".in"], x)


def streams_out(x: Tensor, y: Tensor, w: Weights, p: str) -> Tensor:
    return torch.einsum("st,snw->tnw", w[p + ".mix"], x) + w[p + ".out"][:, None, None] * y


def forward(tokens: List[int], cfg: dict, weights: Weights, *, dtype=torch.float64, layers_out: Optional[list] = None) -> Tensor:
    """Logits [T, vocab] of one sequence; ``layers_out`` collects the sum of the streams after every layer."""
    w = {n: t.to(dtype) if t.is_floating_point() else t for n, t in weights.items()}
    eps = float(cfg["norm"]["eps"])

    def norm(x, name):
        return layer_norm(x, w[name], w[name + ".b"], eps)

    x = w["embed"][torch.as_tensor(tokens, dtype=torch.int64)] * cfg["embedding"]["scale"]
    x = x[None].repeat(cfg["streams"], 1, 1)
    kv = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix", layer["mixer"]
        h = norm(streams_in(x, w, f"l{i}.hc1"), f"l{i}.norm1")
        if layer["type"] == "attention":
            source = m.get("kv_from")
            if source is None:
                kv[i] = differential_keys(h, w, p, m)
            y = differential_attention(h, w, p, m, eps, kv[i if source is None else source])
        elif layer["type"] == "attention_2":
            y = sink_attention(h, w, p, m, eps)
        elif layer["type"] == "parallel":
            y = (m["left_scale"] * biased_attention(h, w, p + ".left", m["left"])
                 + m["right_scale"] * matrix_memory(h, w, p + ".right", m["right"], eps))
        else:
            raise ValueError(layer["type"])
        x = streams_out(x, y, w, f"l{i}.hc1")
        if layer.get("mlp") is not None:
            h = norm(streams_in(x, w, f"l{i}.hc2"), f"l{i}.norm2")
            x = streams_out(x, feed_forward(h, w, f"l{i}.mlp", layer["mlp"]), w, f"l{i}.hc2")
        if layers_out is not None:
            layers_out.append(x.sum(dim=0))
    return norm(x.sum(dim=0), "final.norm") @ w["embed"].T
