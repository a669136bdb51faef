"""Plain CPU oracle of the Fabivik design.  TEST INFRASTRUCTURE ONLY.

One slow function per mechanism, whole sequences only: no cache, no state between calls, no batching, experts one token at a
time.  It shares no code with the shipped package.  Weights come as a dict of float tensors named as in a checkpoint, the
configuration as the dict of its ``config.json``.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

Tensor = torch.Tensor
Weights = Dict[str, Tensor]


def unit_rms(x: Tensor, eps: float) -> Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def layer_norm(x: Tensor, weight: Tensor, eps: float) -> Tensor:
    """RMS norm whose stored weight is the distance from one."""
    return unit_rms(x, eps) * (1.0 + weight)


def short_conv(u: Tensor, taps: Tensor) -> Tensor:
    """Causal convolution over time per channel; ``taps`` [channels, n], the last column meets the current token."""
    n = taps.shape[1]
    out = torch.zeros_like(u)
    for j in range(n):
        back = n - 1 - j
        if back < u.shape[0]:
            out[back:] += taps[:, j] * u[: u.shape[0] - back]
    return out


def silu(x: Tensor) -> Tensor:
    return x * torch.sigmoid(x)


def visible(n: int, size: Optional[int]) -> Tensor:
    """[query, key] mask of a causal window of ``size`` tokens (the token itself included)."""
    age = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    ok = age >= 0
    return ok if size is None else ok & (age < size)


# ---------------------------------------------------------------------------------------------------------------------
# Attention
# ---------------------------------------------------------------------------------------------------------------------
def attention_values(h: Tensor, w: Weights, p: str, m: dict) -> Tensor:
    return short_conv(h @ w[p + ".v"].T, w[p + ".v.conv"]).view(h.shape[0], m["kv_heads"], m["vdim"])


def attend(q: Tensor, k: Tensor, v: Tensor, scale: float, size: Optional[int]) -> Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, dv]: ordinary softmax over the visible keys, query heads in consecutive groups."""
    group = q.shape[1] // k.shape[1]
    k, v = k.repeat_interleave(group, dim=1), v.repeat_interleave(group, dim=1)
    score = torch.einsum("qhd,khd->hqk", q, k) * scale
    score = score.masked_fill(~visible(q.shape[0], size), -math.inf)
    return torch.einsum("hqk,khv->qhv", torch.softmax(score, dim=-1), v)


def attention(h: Tensor, w: Weights, p: str, m: dict, eps: float, v: Tensor) -> Tensor:
    """``v``: this layer's values after mixing."""
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = short_conv(h @ w[p + ".q"].T, w[p + ".q.conv"]).view(T, H, d)
    k = short_conv(h @ w[p + ".k"].T, w[p + ".k.conv"]).view(T, G, d)
    q, k = unit_rms(q, eps) * w[p + ".q.norm"], unit_rms(k, eps) * w[p + ".k.norm"]
    o = attend(q, k, v, m["scale"], (m.get("mask") or {}).get("size"))
    return o.reshape(T, H * m["vdim"]) @ w[p + ".o"].T


# ---------------------------------------------------------------------------------------------------------------------
# wkv
# ---------------------------------------------------------------------------------------------------------------------
def shifted(h: Tensor) -> Tensor:
    """The previous token's row, zeros for the first token."""
    return torch.cat([torch.zeros_like(h[:1]), h[:-1]])


def wkv_inputs(h: Tensor, w: Weights, p: str, m: dict) -> tuple:
    """(r, k, v, decay), each [T, heads, dim], and the output gate [T, heads * dim]."""
    prev = shifted(h)
    mix = {s: h + (prev - h) * w[p + ".mu." + s] for s in "rkvgw"}
    shape = (h.shape[0], m["heads"], m["dim"])
    r, k, v = ((mix[s] @ w[p + "." + s].T).view(shape) for s in "rkv")
    log_rate = torch.tanh(mix["w"] @ w[p + ".w1"].T) @ w[p + ".w2"].T + w[p + ".w0"]
    return r, k, v, torch.exp(-torch.exp(log_rate)).view(shape), silu(mix["g"] @ w[p + ".g"].T)


def wkv_scan(r: Tensor, k: Tensor, v: Tensor, decay: Tensor, bonus: Tensor, state: Optional[Tensor] = None) -> tuple:
    """Token by token: o = (S + diag(bonus) k v^T)^T r, then S <- diag(decay) S + k v^T.  Returns (o, last S)."""
    T, H, d = r.shape
    S = torch.zeros(H, d, v.shape[2], dtype=r.dtype) if state is None else state.clone()
    out = torch.empty_like(v)
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hij,hi->hj", S + bonus[:, :, None] * kv, r[t])
        S = decay[t][:, :, None] * S + kv
    return out, S


def wkv(h: Tensor, w: Weights, p: str, m: dict, eps: float) -> Tensor:
    r, k, v, decay, gate = wkv_inputs(h, w, p, m)
    o, _ = wkv_scan(r, k, v, decay, w[p + ".u"])
    return (unit_rms(o, eps).reshape(h.shape[0], -1) * w[p + ".norm"] * gate) @ w[p + ".o"].T


# ---------------------------------------------------------------------------------------------------------------------
# Gated delta rule
# ---------------------------------------------------------------------------------------------------------------------
def unit_vector(x: Tensor) -> Tensor:
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


def softplus(x: Tensor) -> Tensor:
    return torch.log1p(torch.exp(-x.abs())) + torch.clamp(x, min=0)


def delta_inputs(h: Tensor, w: Weights, p: str, m: dict) -> tuple:
    """(q, k) [T, heads, dim], v [T, heads, vdim], (step size, decay) [T, heads]."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q, k, v = (silu(short_conv(h @ w[p + "." + s].T, w[p + "." + s + ".conv"])) for s in "qkv")
    q, k = (unit_vector(x.view(T, G, m["dim"])).repeat_interleave(H // G, dim=1) for x in (q, k))
    beta = torch.sigmoid(h @ w[p + ".b"].T)
    decay = torch.exp(-torch.exp(w[p + ".A_log"]) * softplus(h @ w[p + ".a"].T + w[p + ".dt_bias"]))
    return q * m["dim"] ** -0.5, k, v.view(T, H, m["vdim"]), beta, decay


def delta_scan(q: Tensor, k: Tensor, v: Tensor, beta: Tensor, decay: Tensor, state: Optional[Tensor] = None) -> tuple:
    """Token by token: S <- decay S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q.  Returns (o, last S)."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype) if state is None else state.clone()
    out = torch.empty_like(v)
    for t in range(T):
        S = decay[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hij,hi->hj", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hij,hi->hj", S, q[t])
    return out, S


def gated_delta(h: Tensor, w: Weights, p: str, m: dict, eps: float) -> Tensor:
    o, _ = delta_scan(*delta_inputs(h, w, p, m))
    o = unit_rms(o, eps) * w[p + ".norm"]
    return (o.reshape(h.shape[0], -1) * silu(h @ w[p + ".g"].T)) @ w[p + ".o"].T


# ---------------------------------------------------------------------------------------------------------------------
# Feed-forward
# ---------------------------------------------------------------------------------------------------------------------
def expert(x: Tensor, w: Weights, p: str, limit: float) -> Tensor:
    g = torch.clamp(x @ w[p + ".gate"].T, max=limit)
    u = torch.clamp(x @ w[p + ".up"].T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[p + ".down"].T


def mixture(h: Tensor, w: Weights, p: str, m: dict) -> Tensor:
    score = torch.sigmoid(h @ w[p + ".router"].T)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in torch.topk(score[t], m["router"]["top"]).indices.tolist():
            out[t] += expert(score[t, e] * h[t], w, f"{p}.e{e}", m["expert"]["limit"])
    if m.get("shared"):
        out = out + torch.sigmoid(h @ w[p + ".shared.sg"].T) * expert(h, w, p + ".shared", m["shared"]["limit"])
    return out


def forward(tokens: List[int], cfg: dict, weights: Weights, *, dtype=torch.float64, layers_out: Optional[list] = None) -> Tensor:
    """Logits [T, vocab] of one sequence; ``layers_out`` collects the residual stream after every layer."""
    w = {n: t.to(dtype) if t.is_floating_point() else t for n, t in weights.items()}
    eps = float(cfg["norm"]["eps"])
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.int64)] * cfg["embedding"]["scale"]
    v_first = None
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix", layer["mixer"]
        h = layer_norm(x, w[f"l{i}.norm1"], eps)
        if layer["type"] == "attention":
            v = attention_values(h, w, p, m)
            if m.get("v_mix"):
                if v_first is None:
                    v_first = v
                else:
                    v = (1.0 - w[p + ".vmix"]) * v + w[p + ".vmix"] * v_first
            y = attention(h, w, p, m, eps, v)
        elif layer["type"] == "wkv":
            y = wkv(h, w, p, m, eps)
        elif layer["type"] == "delta":
            y = gated_delta(h, w, p, m, eps)
        else:
            raise ValueError(layer["type"])
        if layer.get("mlp") is not None:
            y = y + mixture(layer_norm(x, w[f"l{i}.norm2"], eps), w, f"l{i}.mlp", layer["mlp"])
        x = x + y
        if layers_out is not None:
            layers_out.append(x.clone())
    return layer_norm(x, w["final.norm"], eps) @ w["head"].T * cfg["logit_scale"]
