"""Plain CPU oracle of the Maginex design.  TEST INFRASTRUCTURE ONLY.

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


def rms_norm(x: Tensor, weight: Tensor, eps: float) -> Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * weight


def silu(x: Tensor) -> Tensor:
    return x * torch.sigmoid(x)


def causal_filter(h: Tensor, taps: Tensor) -> Tensor:
    """h [T, C], taps [C, n]: y_t = sum over ages a of taps[:, n - 1 - a] h_(t - a), nothing before the start."""
    n, y = taps.shape[1], torch.zeros_like(h)
    for age in range(min(n, h.shape[0])):
        y[age:] += taps[:, n - 1 - age] * h[: h.shape[0] - age]
    return y


def mixed_with_past(h: Tensor, taps: Tensor) -> Tensor:
    """What a sublayer reads."""
    return h + causal_filter(h, taps)


# ---------------------------------------------------------------------------------------------------------------------
# Attention
# ---------------------------------------------------------------------------------------------------------------------
def rotate_halves(x: Tensor, base: float, dims: int) -> Tensor:
    """x [T, heads, dim] at positions 0, 1, ...: dimensions i and i + dims / 2 turn together, those from dims on stay."""
    half, out = dims // 2, x.clone()
    freq = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=x.dtype)
    angle = torch.arange(x.shape[0], dtype=x.dtype)[:, None] * freq
    c, s = torch.cos(angle)[:, None, :], torch.sin(angle)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    out[..., :half], out[..., half:dims] = u * c - v * s, v * c + u * s
    return out


def visible(n: int, size: Optional[int]) -> Tensor:
    """[query, key]: causal, and with a size only that many newest tokens (the token itself included)."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    return (j <= i) if size is None else (j <= i) & (i - j < size)


def attend(q: Tensor, k: Tensor, v: Tensor, scale: float, size: Optional[int], sink: Tensor) -> Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, dv], query heads in consecutive groups; ``sink`` [H] counts in the denominator only."""
    group = q.shape[1] // k.shape[1]
    k, v = k.repeat_interleave(group, dim=1), v.repeat_interleave(group, dim=1)
    score = (torch.einsum("qhd,khd->hqk", q, k) * scale).masked_fill(~visible(q.shape[0], size), -math.inf)
    top = torch.maximum(score.amax(dim=-1, keepdim=True), sink[:, None, None])
    e = torch.exp(score - top)
    weight = e / (e.sum(dim=-1, keepdim=True) + torch.exp(sink[:, None, None] - top))
    return torch.einsum("hqk,khv->qhv", weight, v)


def latent_attention(h: Tensor, w: Weights, p: str, m: dict, eps: float) -> Tensor:
    T, H = h.shape[0], m["heads"]
    c_q = rms_norm(h @ w[p + "dq"].T, w[p + "dq.norm"], eps)
    q = (c_q @ w[p + "uq"].T).view(T, H, m["dim"])
    c = rms_norm(h @ w[p + "dkv"].T, w[p + "dkv.norm"], eps)
    k, v = (c @ w[p + "uk"].T).view(T, H, m["dim"]), (c @ w[p + "uv"].T).view(T, H, m["vdim"])
    o = attend(q, k, v, m["scale"], None, w[p + "sink"]).reshape(T, -1)
    return (o * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def mixed_values(v: Tensor, first: Optional[Tensor], share: Tensor) -> Tensor:
    return v if first is None else (1 - share) * v + share * first


def attention(h: Tensor, w: Weights, p: str, m: dict, carried: dict) -> Tensor:
    """``carried["first"]``: the values of the first layer that mixes them."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q, k = (h @ w[p + "q"].T).view(T, H, m["dim"]), (h @ w[p + "k"].T).view(T, G, m["dim"])
    v = (h @ w[p + "v"].T).view(T, G, m["vdim"])
    rot = m.get("rot")
    if rot and rot["dims"]:
        q, k = (rotate_halves(x, float(rot["base"]), rot["dims"]) for x in (q, k))
    if m.get("v_mix"):
        first = carried.get("first")
        if first is None:
            carried["first"] = v
        else:
            v = mixed_values(v, first, w[p + "vmix"])
    o = attend(q, k, v, m["scale"], (m.get("mask") or {}).get("size"), w[p + "sink"])
    return (o * torch.sigmoid(h @ w[p + "g"].T)[:, :, None]).reshape(T, -1) @ w[p + "o"].T


# ---------------------------------------------------------------------------------------------------------------------
# Gated recurrence
# ---------------------------------------------------------------------------------------------------------------------
def gated_scan(z: Tensor, candidate: Tensor, state: Optional[Tensor] = None) -> Tensor:
    """S_t = (1 - z_t) S_(t-1) + z_t candidate_t, element by element; all S."""
    s, out = torch.zeros_like(z[0]) if state is None else state, []
    for t in range(z.shape[0]):
        s = (1 - z[t]) * s + z[t] * candidate[t]
        out.append(s)
    return torch.stack(out)


def candidate_of(u: Tensor) -> Tensor:
    return torch.where(u >= 0, u + 0.5, torch.sigmoid(u))


def mingru(h: Tensor, w: Weights, p: str) -> Tensor:
    z = torch.sigmoid(h @ w[p + "z"].T + w[p + "z.b"])
    s = gated_scan(z, candidate_of(h @ w[p + "x"].T + w[p + "x.b"]))
    return (s * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


# ---------------------------------------------------------------------------------------------------------------------
# Feed-forward
# ---------------------------------------------------------------------------------------------------------------------
def squared_relu_ff(x: Tensor, w: Weights, p: str) -> Tensor:
    return torch.relu(x @ w[p + ".up"].T).square() @ w[p + ".down"].T


def choose(logits: Tensor, top: int) -> tuple:
    """(experts of the ``top`` largest logits, the softmax over those alone)."""
    order = torch.sort(logits, dim=-1, descending=True, stable=True)
    return order.indices[:, :top], torch.softmax(order.values[:, :top], dim=-1)


def experts(x: Tensor, w: Weights, p: str, mlp: dict) -> Tensor:
    chosen, weight = choose(x @ w[p + "router"].T + w[p + "router.b"], mlp["router"]["top"])
    out = squared_relu_ff(x, w, p + "shared") if mlp.get("shared") else torch.zeros_like(x)
    for e in range(mlp["router"]["experts"]):
        t, k = (chosen == e).nonzero(as_tuple=True)
        if t.numel():
            out[t] += weight[t, k][:, None] * squared_relu_ff(x[t], w, p + f"e{e}")
    return out


# ---------------------------------------------------------------------------------------------------------------------
# Model
# ---------------------------------------------------------------------------------------------------------------------
def forward(config: dict, w: Weights, ids: List[int], streams: Optional[list] = None) -> Tensor:
    """Logits [T, vocab] of one sequence; ``streams`` receives the residual stream after every layer."""
    eps, carried = float(config["norm"]["eps"]), {}
    x = w["embed"][torch.as_tensor(ids)] * float(config["embedding"]["scale"])
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        h = rms_norm(x, w[p + "norm1"], eps)
        a, m = mixed_with_past(h, w[p + "canon1"]), layer["mixer"]
        if layer["type"] == "latent_attention":
            y = latent_attention(a, w, p + "mix.", m, eps)
        elif layer["type"] == "mingru":
            y = mingru(a, w, p + "mix.")
        else:
            y = attention(a, w, p + "mix.", m, carried)
        if layer.get("mlp"):
            y = y + experts(mixed_with_past(h, w[p + "canon2"]), w, p + "mlp.", layer["mlp"])
        x = x + y
        if streams is not None:
            streams.append(x.clone())
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T
