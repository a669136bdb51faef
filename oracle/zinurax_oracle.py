"""Plain CPU oracle of the Zinurax design.  TEST INFRASTRUCTURE ONLY.

One slow function per mechanism, whole sequences only: no cache, no state between calls, no batching, keys and values
spelled out per head.  It shares no code with the shipped package.  Weights come as a dict of float tensors named as in a
checkpoint, the configuration as the dict of its ``config.json``.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

Tensor = torch.Tensor


def layer_norm(x: Tensor, weight: Tensor, eps: float) -> Tensor:
    centred = x - x.mean(dim=-1, keepdim=True)
    return centred / torch.sqrt((centred * centred).mean(dim=-1, keepdim=True) + eps) * weight


def rms_norm(x: Tensor, weight: Optional[Tensor], eps: float) -> Tensor:
    y = x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)
    return y if weight is None else y * weight


def rope_frequencies(rot: dict) -> tuple:
    """(frequency per pair, factor on cos and sin) of a rotation, YaRN-scaled when ``rot`` says so."""
    dims, base = int(rot["dims"]), float(rot["base"])
    plain = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return plain, 1.0
    factor, original = float(sc["factor"]), float(sc["original"])

    def pair_of(turns):  # (real-valued) dimension index that makes `turns` turns over the original context
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    low = max(math.floor(pair_of(float(sc["fast"]))), 0)
    high = min(math.ceil(pair_of(float(sc["slow"]))), dims - 1)
    out = []
    for i, f in enumerate(plain):
        ramp = min(max((i - low) / max(high - low, 0.001), 0.0), 1.0)
        out.append(f / factor * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(factor) + 1.0


def rotate(x: Tensor, positions: Tensor, rot: dict) -> Tensor:
    """Rotate the pairs (2i, 2i+1) of the first ``rot.dims`` entries of the last axis; ``x`` is [T, ..., n]."""
    freq, mag = rope_frequencies(rot)
    dims = int(rot["dims"])
    ang = positions.to(x.dtype)[:, None] * torch.tensor(freq, dtype=x.dtype)[None, :]
    shape = [x.shape[0]] + [1] * (x.dim() - 2) + [dims // 2]
    cos, sin = (torch.cos(ang) * mag).view(shape), (torch.sin(ang) * mag).view(shape)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2] = u * cos - v * sin
    out[..., 1:dims:2] = v * cos + u * sin
    return out


def visible(n: int, size: Optional[int]) -> Tensor:
    """[query, key] mask of a causal window of ``size`` tokens (the token itself included)."""
    age = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    ok = age >= 0
    return ok if size is None else ok & (age < size)


def latent_of(h: Tensor, w: Dict[str, Tensor], p: str, m: dict, eps: float) -> tuple:
    """(latent c [T, kv_rank], rotated shared key part [T, rot_dim]) of a layer that has a down projection."""
    d = h @ w[p + ".dkv"].T
    c = rms_norm(d[:, : m["kv_rank"]], w[p + ".dkv.norm"], eps)
    return c, rotate(d[:, m["kv_rank"]:], torch.arange(h.shape[0]), m["rot"])


def latent_attention(h: Tensor, w: Dict[str, Tensor], p: str, m: dict, c: Tensor, k_rot: Tensor) -> Tensor:
    T, H, d, r, dv = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    q = (h @ w[p + ".q"].T).view(T, H, d + r)
    q_rot = rotate(q[..., d:].contiguous(), torch.arange(T), m["rot"])
    k = (c @ w[p + ".uk"].T).view(T, H, d)
    v = (c @ w[p + ".uv"].T).view(T, H, dv)
    score = (torch.einsum("qhd,khd->hqk", q[..., :d], k) + torch.einsum("qhr,kr->hqk", q_rot, k_rot)) * m["scale"]
    score = score.masked_fill(~visible(T, (m.get("mask") or {}).get("size")), -math.inf)
    out = torch.einsum("hqk,khv->qhv", torch.softmax(score, dim=-1), v)
    out = out * torch.sigmoid(h @ w[p + ".g"].T)[:, :, None]
    return out.reshape(T, H * dv) @ w[p + ".o"].T


def delta_inputs(h: Tensor, w: Dict[str, Tensor], p: str, m: dict) -> tuple:
    """(r, k, v, decay, removal rate, unit key), each [T, heads, dim]."""
    shape = (h.shape[0], m["heads"], m["dim"])
    r, k, v = ((h @ w[p + "." + n].T).view(shape) for n in "rkv")
    z = torch.tanh(h @ w[p + ".w1"].T) @ w[p + ".w2"].T + w[p + ".w0"]
    decay = torch.exp(-math.exp(-0.5) * torch.sigmoid(z)).view(shape)
    a = torch.sigmoid(h @ w[p + ".a"].T + w[p + ".a.b"]).view(shape)
    u = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
    return r, k, v, decay, a, u


def delta_scan(r: Tensor, k: Tensor, v: Tensor, decay: Tensor, a: Tensor, u: Tensor, state: Optional[Tensor] = None) -> tuple:
    """Token by token: S' = diag(decay) S - (a u)(u^T S) + k v^T, o = S'^T r.  Returns (o [T, heads, dim], last S)."""
    T, H, d = r.shape
    S = torch.zeros(H, d, d, dtype=r.dtype) if state is None else state.clone()
    out = torch.empty_like(r)
    for t in range(T):
        seen = torch.einsum("hi,hij->hj", u[t], S)
        S = decay[t][:, :, None] * S - (a[t] * u[t])[:, :, None] * seen[:, None, :] + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hij,hi->hj", S, r[t])
    return out, S


def general_delta(h: Tensor, w: Dict[str, Tensor], p: str, m: dict, eps: float) -> Tensor:
    o, _ = delta_scan(*delta_inputs(h, w, p, m))
    o = rms_norm(o, None, eps).reshape(h.shape[0], -1) * w[p + ".norm"]
    return (o * torch.sigmoid(h @ w[p + ".g"].T)) @ w[p + ".o"].T


def dense_mlp(h: Tensor, w: Dict[str, Tensor], p: str) -> Tensor:
    return torch.relu(h @ w[p + ".up"].T).square() @ w[p + ".down"].T


def forward(tokens: List[int], cfg: dict, weights: Dict[str, Tensor], *, dtype=torch.float64,
            layers_out: Optional[list] = None) -> Tensor:
    """Logits [T, vocab] of one sequence; ``layers_out`` collects the residual stream after every layer."""
    w = {n: t.to(dtype) if t.is_floating_point() else t for n, t in weights.items()}
    eps = float(cfg["norm"]["eps"])
    x = layer_norm(w["embed"][torch.as_tensor(tokens, dtype=torch.int64)], w["embed.norm"], eps)
    latents = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix", layer["mixer"]
        if layer["type"] == "latent_attention":
            src = m.get("kv_from")
            if src is None:
                latents[i] = latent_of(x, w, p, m, eps)
            y = latent_attention(x, w, p, m, *latents[i if src is None else src])
        elif layer["type"] == "general_delta":
            y = general_delta(x, w, p, m, eps)
        else:
            raise ValueError(layer["type"])
        x = x + layer_norm(y, w[f"l{i}.norm1"], eps)
        if layer.get("mlp") is not None:
            x = x + layer_norm(dense_mlp(x, w, f"l{i}.mlp"), w[f"l{i}.norm2"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return layer_norm(x, w["final.norm"], eps) @ w["embed"].T
