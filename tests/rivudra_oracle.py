"""Plain, slow implementation of the Rivudra design, used as the oracle of its tests.

Every mechanism is one function on whole sequences (no cache, no batching, no kernels), computed in
the dtype of its inputs; the tests call it in float64.  Nothing here is shared with the product path.

Notation: T tokens, D width, H query heads over G key/value heads, E experts.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

SIGMOID_SLOPE = 1.702


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps), scaled by (1 + w)."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * (1 + w)


def rotate_interleaved(x: torch.Tensor, positions: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """x [T, heads, dim]: the pairs (2i, 2i + 1) of the first ``dims`` dimensions turned by
    p * base^(-2i / dims)."""
    out = x.clone()
    for i in range(dims // 2):
        angle = positions.to(torch.float64) * float(base) ** (-2.0 * i / dims)
        c, s = torch.cos(angle).to(x.dtype)[:, None], torch.sin(angle).to(x.dtype)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def visible(num_tokens: int, window: int) -> torch.Tensor:
    """[T, T] bool: which keys j a position i sees (0 <= i - j < window)."""
    i = torch.arange(num_tokens)[:, None]
    j = torch.arange(num_tokens)[None, :]
    return (i >= j) & (i - j < window)


def softmax_one_off(scores: torch.Tensor, mask: torch.Tensor) -> torch.Tensor:
    """exp(s_j) / (1 + sum_j exp(s_j)) over the visible keys: a key of score 0 without a value."""
    s = scores.masked_fill(~mask, -math.inf)
    m = s.amax(-1, keepdim=True).clamp_min(0)
    e = torch.exp(s - m)
    return e / (torch.exp(-m) + e.sum(-1, keepdim=True))


def attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, window: int) -> torch.Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, dv] (rotated already) -> [T, H * dv]."""
    t, h = q.shape[:2]
    per = h // k.shape[1]
    mask = visible(t, window)
    heads = []
    for n in range(h):
        p = softmax_one_off((q[:, n] @ k[:, n // per].T) * scale, mask)
        heads.append(p @ v[:, n // per])
    return torch.cat(heads, -1)


def mixer(h: torch.Tensor, w: Dict[str, torch.Tensor], p: dict) -> torch.Tensor:
    t = h.shape[0]
    pos = torch.arange(t)
    q = (h @ w["q"].T).view(t, p["heads"], p["dim"])
    k = (h @ w["k"].T).view(t, p["kv_heads"], p["dim"])
    v = (h @ w["v"].T).view(t, p["kv_heads"], p["vdim"])
    q = rotate_interleaved(q, pos, p["rot"]["dims"], p["rot"]["base"])
    k = rotate_interleaved(k, pos, p["rot"]["dims"], p["rot"]["base"])
    o = attention(q, k, v, p["scale"], p["mask"]["size"])
    return (o * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


def clamped_glu(gate: torch.Tensor, up: torch.Tensor, limit: float) -> torch.Tensor:
    g = gate.clamp(max=limit)
    u = up.clamp(-limit, limit)
    return g * torch.sigmoid(SIGMOID_SLOPE * g) * (u + 1)


def expert(h: torch.Tensor, w: Dict[str, torch.Tensor], limit: float) -> torch.Tensor:
    return clamped_glu(h @ w["gate"].T, h @ w["up"].T, limit) @ w["down"].T


def route(logits: torch.Tensor, top: int, groups: int, keep: int, scale: float) -> torch.Tensor:
    """Weights [T, E] of a token's experts, zero for those it does not use."""
    t, e = logits.shape
    s = torch.softmax(logits, -1)
    out = torch.zeros_like(s)
    size = e // groups
    for i in range(t):
        best = [float(s[i, g * size:(g + 1) * size].max()) for g in range(groups)]
        kept = sorted(range(groups), key=lambda g: -best[g])[:keep]
        allowed = [x for x in range(e) if x // size in kept]
        chosen = sorted(allowed, key=lambda x: -float(s[i, x]))[:top]
        total = sum(s[i, x] for x in chosen) + 1e-20
        for x in chosen:
            out[i, x] = s[i, x] / total * scale
    return out


def moe(h: torch.Tensor, w: Dict[str, torch.Tensor], p: dict) -> torch.Tensor:
    r = p["router"]
    weights = route(h @ w["router"].T, r["top"], r["groups"]["count"], r["groups"]["keep"], r["scale"])
    y = torch.zeros_like(h)
    for e in range(r["experts"]):
        y = y + weights[:, e:e + 1] * expert(h, _sub(w, f"e{e}."), p["expert"]["limit"])
    if p.get("shared"):
        y = y + expert(h, _sub(w, "shared."), p["shared"]["limit"])
    return y


def _sub(w: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def forward(tokens, weights: Dict[str, torch.Tensor], cfg: dict, dtype=torch.float64,
            layers_out: Optional[List[torch.Tensor]] = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence; ``layers_out`` collects the residual stream after every layer."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        lw = _sub(w, f"l{i}.")
        h = rms_norm(x, lw["norm1"], eps)
        y = mixer(h, _sub(lw, "mix."), layer["mixer"])
        if layer["mlp"] is not None:
            y = y + moe(h, _sub(lw, "mlp."), layer["mlp"])
        x = x + y
        if layers_out is not None:
            layers_out.append(x)
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T
