"""Plain, slow implementation of the Dalavik design, used as the oracle of its tests.

Every mechanism is one function on whole sequences (no cache, no batching, no kernels), computed in the
dtype of its inputs; the tests call it in float64.  Nothing here is shared with the product path.

Notation: T tokens, D width, H query heads over G key/value heads.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch


# ------------------------------------------------------------------ elementwise pieces
def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def group_norm(x: torch.Tensor, w: torch.Tensor, groups: int, eps: float) -> torch.Tensor:
    """Each of the equal consecutive parts of a row by its own root mean square, then the whole times w."""
    n = x.shape[-1] // groups
    return torch.cat([rms(x[..., g * n: (g + 1) * n], eps) for g in range(groups)], -1) * w


def rotate_pairs(x: torch.Tensor, positions: torch.Tensor, base: float) -> torch.Tensor:
    """x [T, heads, r]: the pairs (2i, 2i + 1) turned by p * base^(-2i / r)."""
    r = x.shape[-1]
    out = x.clone()
    for i in range(r // 2):
        angle = positions.to(torch.float64) * float(base) ** (-2.0 * i / r)
        c, s = torch.cos(angle).to(x.dtype)[:, None], torch.sin(angle).to(x.dtype)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


# ------------------------------------------------------------------ latent attention
def latent_rows(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float):
    """What a token leaves in the cache: (normed latent [T, rank], rotated key part [T, rot])."""
    a = h @ w["dkv"].T
    rank = m["kv_rank"]
    c = rms(a[:, :rank], eps) * w["dkv.norm"]
    pos = torch.arange(h.shape[0])
    return c, rotate_pairs(a[:, None, rank:], pos, m["rot"]["base"])[:, 0]


def latent_queries(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    """Queries through a latent, [T, H, dim + rot], the last part rotated."""
    d = m["dim"]
    q = (rms(h @ w["dq"].T, eps) * w["dq.norm"]) @ w["uq"].T
    q = q.reshape(h.shape[0], m["heads"], d + m["rot_dim"])
    return torch.cat([q[..., :d], rotate_pairs(q[..., d:], torch.arange(h.shape[0]), m["rot"]["base"])], -1)


def latent_attention(h, w, m: dict, eps: float, rows) -> torch.Tensor:
    """``rows``: the cache rows of this layer, or of the layer whose cache it reads."""
    t, n, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    c, kr = rows
    q = latent_queries(h, w, m, eps)
    k = (c @ w["uk"].T).reshape(t, n, d)
    v = (c @ w["uv"].T).reshape(t, n, e)
    hidden = torch.arange(t)[None, :] > torch.arange(t)[:, None]
    out = []
    for a in range(n):
        s = (q[:, a, :d] @ k[:, a].T + q[:, a, d:] @ kr.T) * m["scale"]
        out.append(torch.softmax(s.masked_fill(hidden, -math.inf), -1) @ v[:, a])
    return torch.cat(out, -1) @ w["o"].T


# ------------------------------------------------------------------ attention with mixed scores
def query_temperature(positions: torch.Tensor, coef: float, every: int) -> torch.Tensor:
    return 1 + coef * torch.log(torch.floor((positions + 1) / every) + 1)


def cap(s: torch.Tensor, limit: float) -> torch.Tensor:
    return limit * torch.tanh(s / limit)


def distance_bias(t: int, r1: torch.Tensor, r2: torch.Tensor) -> torch.Tensor:
    """[H, T, T]: r1 ln(1 + r2 (i - j)) for keys j <= i, zero elsewhere."""
    d = (torch.arange(t)[:, None] - torch.arange(t)[None, :]).clamp(min=0).to(r1.dtype)
    return r1[:, None, None] * torch.log(1 + r2[:, None, None] * d)


def mix_heads(s: torch.Tensor, talk: torch.Tensor) -> torch.Tensor:
    """s [H, T, T] -> the same, head h holding sum_g talk[h, g] s_g."""
    return torch.einsum("hg,gij->hij", talk, s)


def sink_softmax(s: torch.Tensor, sink: Optional[torch.Tensor]) -> torch.Tensor:
    """Over the last axis of s [H, T, T], the denominator also counting exp(sink_h)."""
    if sink is None:
        return torch.softmax(s, -1)
    extra = sink[:, None, None].expand(-1, s.shape[1], 1)
    return torch.softmax(torch.cat([s, extra], -1), -1)[..., :-1]


def mixed_attend(q, k, v, scale: float, softcap: Optional[float], r1, r2, talk, sink) -> torch.Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, e] -> [T, H * e]."""
    t, n = q.shape[:2]
    per = n // k.shape[1]
    s = torch.stack([q[:, a] @ k[:, a // per].T * scale for a in range(n)])
    if softcap:
        s = cap(s, softcap)
    if r1 is not None:
        s = s - distance_bias(t, r1, r2)
    if talk is not None:
        s = mix_heads(s, talk)
    hidden = torch.arange(t)[None, :] > torch.arange(t)[:, None]
    p = sink_softmax(s.masked_fill(hidden, -math.inf), sink)
    return torch.cat([p[a] @ v[:, a // per] for a in range(n)], -1)


def normed_queries_keys(q, k, qw, kw, eps: float, temp: Optional[dict], positions: torch.Tensor):
    """q [T, H, d], k [T, G, d]: every head by its root mean square and the weight; queries by their temperature."""
    q, k = rms(q, eps) * qw, rms(k, eps) * kw
    if temp:
        q = q * query_temperature(positions, temp["coef"], temp["every"]).to(q.dtype)[:, None, None]
    return q, k


def attention(h, w, m: dict, eps: float) -> torch.Tensor:
    t, n, g = h.shape[0], m["heads"], m["kv_heads"]
    q = (h @ w["q"].T + w["q.b"]).reshape(t, n, m["dim"])
    k = (h @ w["k"].T + w["k.b"]).reshape(t, g, m["dim"])
    v = (h @ w["v"].T + w["v.b"]).reshape(t, g, m["vdim"])
    q, k = normed_queries_keys(q, k, w["q.norm"], w["k.norm"], eps, m.get("q_temp"), torch.arange(t))
    return mixed_attend(q, k, v, m["scale"], m.get("softcap"), w["r1"], w["r2"], w["talk"], w["sink"]) @ w["o"].T


# ------------------------------------------------------------------ the rest of a layer
def feed_forward(x, w) -> torch.Tensor:
    return (torch.clamp(x @ w["gate"].T, min=0) * (x @ w["up"].T)) @ w["down"].T


def token_side(x, w, e, eps: float) -> torch.Tensor:
    """What the per-layer token row ``e`` adds to x."""
    y = (gelu_tanh(x @ w["gate"].T) * e) @ w["proj"].T
    return rms(y, eps) * w["norm"]


def part(w: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def forward(tokens: List[int], w: Dict[str, torch.Tensor], cfg: dict, layers_out: Optional[list] = None,
            dtype=torch.float64) -> torch.Tensor:
    """Logits [T, vocab]; ``layers_out`` takes the residual after every layer."""
    w = {k: v.to(dtype) for k, v in w.items()}
    ids = torch.tensor(tokens)
    eps, groups = cfg["norm"]["eps"], cfg["norm"]["groups"]
    x = w["embed"][ids]
    cached = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        mix = part(w, p + "mix.")
        if layer["type"] == "latent_attention":
            j = m.get("kv_from")
            cached[i] = latent_rows(x, mix, m, eps) if j is None else cached[j]
            y = latent_attention(x, mix, m, eps, cached[i])
        else:
            y = attention(x, mix, m, eps)
        x = x + group_norm(y, w[p + "norm1"], groups, eps)
        if layer["mlp"] is not None:
            x = x + group_norm(feed_forward(x, part(w, p + "mlp.")), w[p + "norm2"], groups, eps)
        if cfg.get("token_side"):
            n = cfg["token_side"]["dim"]
            x = x + token_side(x, part(w, p + "side."), w["side.embed"][ids][:, i * n: (i + 1) * n], eps)
        if layers_out is not None:
            layers_out.append(x)
    return group_norm(x, w["final.norm"], groups, eps) @ w["embed"].T
