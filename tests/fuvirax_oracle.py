"""Plain, slow implementation of the Fuvirax design, used as the oracle of its tests.

Every mechanism is one function on whole sequences (no cache, no batching, no kernels), computed in the
dtype of its inputs; the tests call it in float64.  Nothing here is shared with the product path.

Notation: T tokens, D width, N streams, H heads over G query/key heads, d and e the row and column
sizes of a head's state (or key and value sizes).
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

UNIT_EPS = 1e-6


# ------------------------------------------------------------------ elementwise pieces
def sigmoid(z: torch.Tensor) -> torch.Tensor:
    return 1 / (1 + torch.exp(-z))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * sigmoid(z)


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def xielu(z: torch.Tensor, p: torch.Tensor, q: torch.Tensor) -> torch.Tensor:
    neg = torch.clamp(z, max=0)
    return torch.where(z > 0, softplus(p) * z * z, (0.5 + softplus(q)) * (torch.expm1(neg) - neg)) + z / 2


def layer_norm(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor, eps: float) -> torch.Tensor:
    c = x - x.mean(-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(-1, keepdim=True) + eps) * w + b


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + UNIT_EPS)


def token_shift(h: torch.Tensor, mu: torch.Tensor) -> torch.Tensor:
    """(1 - mu) h_t + mu h_(t-1), with h_(-1) = 0."""
    out = h.clone()
    for t in range(h.shape[0]):
        before = h[t - 1] if t else torch.zeros_like(h[0])
        out[t] = h[t] + (before - h[t]) * mu
    return out


def rotate_halves(x: torch.Tensor, positions: torch.Tensor, base: float) -> torch.Tensor:
    """x [T, heads, r]: the pairs (i, i + r/2) turned by p * base^(-2i / r)."""
    r = x.shape[-1]
    out = x.clone()
    for i in range(r // 2):
        angle = positions.to(torch.float64) * float(base) ** (-2.0 * i / r)
        c, s = torch.cos(angle).to(x.dtype)[:, None], torch.sin(angle).to(x.dtype)[:, None]
        u, v = x[..., i], x[..., i + r // 2]
        out[..., i] = u * c - v * s
        out[..., i + r // 2] = v * c + u * s
    return out


# ------------------------------------------------------------------ mixers
def latent_core(q: torch.Tensor, down: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    """Queries q [T, H * (dim + rot)] over latents down [T, rank + rot] -> heads [T, H * vdim]."""
    t, heads, d, r, e, rank = q.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(t)
    q = q.view(t, heads, d + r)
    q_rot = rotate_halves(q[..., d:], pos, m["rot"]["base"])
    c = rms(down[:, :rank], eps) * w["dkv.norm"]
    k_rot = rotate_halves(down[:, None, rank:], pos, m["rot"]["base"])[:, 0]
    k = (c @ w["uk"].T).view(t, heads, d)
    v = (c @ w["uv"].T).view(t, heads, e)
    hidden = torch.triu(torch.ones(t, t, dtype=torch.bool), diagonal=1)
    out = []
    for n in range(heads):
        s = (q[:, n, :d] @ k[:, n].T + q_rot[:, n] @ k_rot.T) * m["scale"]
        out.append(torch.softmax(s.masked_fill(hidden, -math.inf), -1) @ v[:, n])
    return torch.cat(out, -1)


def latent_attention(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    return latent_core(h @ w["q"].T, h @ w["dkv"].T, w, m, eps) @ w["o"].T


def gated_linear_scan(q: torch.Tensor, f: torch.Tensor, v: torch.Tensor) -> torch.Tensor:
    """q, f [T, H, d], v [T, H, e]:  S <- diag(f) S + (1 - f) v^T,  o = S^T q  (per head, S = 0 before)."""
    t, heads, d = q.shape
    s = q.new_zeros(heads, d, v.shape[-1])
    out = []
    for i in range(t):
        s = f[i, :, :, None] * s + (1 - f[i])[:, :, None] * v[i, :, None, :]
        out.append((s * q[i, :, :, None]).sum(1))
    return torch.stack(out)


def hgrn2(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    t, heads, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = silu(h @ w["q"].T).view(t, heads, d)
    v = (h @ w["v"].T).view(t, heads, e)
    low = w["lower"]
    f = (low + (1 - low) * sigmoid(h @ w["f"].T + w["f.b"])).view(t, heads, d)
    o = rms(gated_linear_scan(q, f, v), eps) * w["norm"]
    return o.reshape(t, heads * e) @ w["o"].T


def short_conv(x: torch.Tensor, taps: torch.Tensor) -> torch.Tensor:
    """x [T, C], taps [C, K] (the last one meets the current token), zeros before the start, then silu."""
    t, k = x.shape[0], taps.shape[1]
    y = torch.zeros_like(x)
    for i in range(t):
        for j in range(k):
            src = i - (k - 1) + j
            if src >= 0:
                y[i] += taps[:, j] * x[src]
    return silu(y)


def delta_scan(q, k, v, g, beta) -> torch.Tensor:
    """q, k, g [T, H, d], v [T, H, e], beta [T, H]:
    S <- diag(g) S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q."""
    t, heads, d = q.shape
    s = q.new_zeros(heads, d, v.shape[-1])
    out = []
    for i in range(t):
        s = g[i, :, :, None] * s
        u = beta[i, :, None] * (v[i] - (s * k[i, :, :, None]).sum(1))
        s = s + k[i, :, :, None] * u[:, None, :]
        out.append((s * q[i, :, :, None]).sum(1))
    return torch.stack(out)


def channel_delta(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    t, heads, groups, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = short_conv(h @ w["q"].T, w["q.conv"]).view(t, groups, d)
    k = short_conv(h @ w["k"].T, w["k.conv"]).view(t, groups, d)
    v = short_conv(h @ w["v"].T, w["v.conv"]).view(t, heads, e)
    per = heads // groups
    q = (unit(q) * d ** -0.5).repeat_interleave(per, dim=1)
    k = unit(k).repeat_interleave(per, dim=1)
    beta = sigmoid(h @ w["b"].T)
    rate = softplus(h @ w["a1"].T @ w["a2"].T + w["dt_bias"]).view(t, heads, d)
    g = torch.exp(-torch.exp(w["A_log"])[None, :, None] * rate)
    o = rms(delta_scan(q, k, v, g, beta), eps) * w["norm"]
    gate = sigmoid(h @ w["g1"].T @ w["g2"].T).view(t, heads, e)
    return (o * gate).reshape(t, heads * e) @ w["o"].T


MIXERS = {"latent_attention": latent_attention, "hgrn2": hgrn2, "channel_delta": channel_delta}


# ------------------------------------------------------------------ the model
def dense(h: torch.Tensor, w: Dict[str, torch.Tensor]) -> torch.Tensor:
    return xielu(h @ w["up"].T, w["act"][0], w["act"][1]) @ w["down"].T


def hyper_connect(x: torch.Tensor, w_in, w_mix, w_out, sublayer) -> torch.Tensor:
    """x [N, T, D]: u = sum_s in_s x_s, then x_t <- sum_s mix[s, t] x_s + out_t * sublayer(u)."""
    u = sum(w_in[s] * x[s] for s in range(x.shape[0]))
    y = sublayer(u)
    return torch.stack([sum(w_mix[s, t] * x[s] for s in range(x.shape[0])) + w_out[t] * y
                        for t in range(x.shape[0])])


def layer_order(cfg: dict) -> List[int]:
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return list(range(n))
    body = list(range(loop["start"], loop["stop"]))
    return list(range(loop["start"])) + body * loop["times"] + list(range(loop["stop"], n))


def _sub(w: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def forward(tokens, weights: Dict[str, torch.Tensor], cfg: dict, dtype=torch.float64,
            layers_out: Optional[List[torch.Tensor]] = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence; ``layers_out`` collects the sum of the streams after every
    layer run."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps, streams = cfg["norm"]["eps"], cfg["streams"]
    x = w["embed"][torch.as_tensor(tokens)].expand(streams, -1, -1)
    for i in layer_order(cfg):
        layer, lw = cfg["layers"][i], _sub(w, f"l{i}.")

        def mix(u):
            h = token_shift(layer_norm(u, lw["norm1"], lw["norm1.b"], eps), lw["shift"])
            return MIXERS[layer["type"]](h, _sub(lw, "mix."), layer["mixer"], eps) * lw["ls1"]

        def feed(u):
            return dense(layer_norm(u, lw["norm2"], lw["norm2.b"], eps), _sub(lw, "mlp.")) * lw["ls2"]

        x = hyper_connect(x, lw["hc1.in"], lw["hc1.mix"], lw["hc1.out"], mix)
        if layer["mlp"] is not None:
            x = hyper_connect(x, lw["hc2.in"], lw["hc2.mix"], lw["hc2.out"], feed)
        if layers_out is not None:
            layers_out.append(x.sum(0))
    return layer_norm(x.sum(0), w["final.norm"], w["final.norm.b"], eps) @ w["embed"].T * cfg["logit_scale"]
