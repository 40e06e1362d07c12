"""Plain, slow implementation of the Gatosun design, used as the oracle of its tests.

Every mechanism is one function on whole sequences (no cache, no batching, no kernels), computed in the
dtype of its inputs; the tests call it in float64.  Nothing here is shared with the product path.

Notation: T tokens, D width, H query heads over G key/value heads, d and e the row and column sizes of a
head's state (or key and value sizes).
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch


# ------------------------------------------------------------------ elementwise pieces
def sigmoid(z: torch.Tensor) -> torch.Tensor:
    return 1 / (1 + torch.exp(-z))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * sigmoid(z)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def relu_squared(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0) ** 2


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rotate_halves(x: torch.Tensor, positions: torch.Tensor, r: int, base: float) -> torch.Tensor:
    """x [T, heads, d]: among the first r dimensions the pairs (i, i + r/2) turned by p * base^(-2i / r)."""
    out = x.clone()
    for i in range(r // 2):
        angle = positions.to(torch.float64) * float(base) ** (-2.0 * i / r)
        c, s = torch.cos(angle).to(x.dtype)[:, None], torch.sin(angle).to(x.dtype)[:, None]
        u, v = x[..., i], x[..., i + r // 2]
        out[..., i] = u * c - v * s
        out[..., i + r // 2] = v * c + u * s
    return out


# ------------------------------------------------------------------ attention
def attend(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, window: int = 0) -> torch.Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, e]: softmax over the keys j <= i (and i - j < window) -> [T, H * e]."""
    t, heads = q.shape[:2]
    per = heads // k.shape[1]
    i, j = torch.arange(t)[:, None], torch.arange(t)[None, :]
    hidden = j > i
    if window:
        hidden = hidden | (i - j >= window)
    out = []
    for n in range(heads):
        s = q[:, n] @ k[:, n // per].T * scale
        out.append(torch.softmax(s.masked_fill(hidden, -math.inf), -1) @ v[:, n // per])
    return torch.cat(out, -1)


def mix_values(v: torch.Tensor, first: Optional[torch.Tensor], lam) -> torch.Tensor:
    return v if first is None else (1 - lam) * v + lam * first


def attention_heads(q, k, v, w, m: dict, eps: float, v_first=None) -> torch.Tensor:
    """Projections q [T, H d], k [T, G d], v [T, G e] -> heads [T, H e]: norm over whole projections, rotation,
    values mixed with those of the first such layer."""
    t, pos = q.shape[0], torch.arange(q.shape[0])
    q = (rms(q, eps) * w["q.norm"]).view(t, m["heads"], m["dim"])
    k = (rms(k, eps) * w["k.norm"]).view(t, m["kv_heads"], m["dim"])
    r = m["rot"]
    v = mix_values(v, v_first, w.get("vmix"))
    return attend(rotate_halves(q, pos, r["dims"], r["base"]), rotate_halves(k, pos, r["dims"], r["base"]),
                  v.view(t, m["kv_heads"], m["vdim"]), m["scale"])


def unit_heads(q, k, v, m: dict, eps: float) -> torch.Tensor:
    """Projections -> heads: rotation, then every head divided by its root mean square, sliding window."""
    t, pos, r = q.shape[0], torch.arange(q.shape[0]), m["rot"]
    q = rms(rotate_halves(q.view(t, m["heads"], m["dim"]), pos, r["dims"], r["base"]), eps)
    k = rms(rotate_halves(k.view(t, m["kv_heads"], m["dim"]), pos, r["dims"], r["base"]), eps)
    return attend(q, k, v.view(t, m["kv_heads"], m["vdim"]), m["scale"], m["mask"]["size"])


# ------------------------------------------------------------------ recurrent layers
def decay_scan(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, g: torch.Tensor) -> torch.Tensor:
    """q, k, g [T, H, d], v [T, H, e]:  S <- diag(g) S + k v^T,  o = S^T q  (S = 0 before the first token)."""
    t, heads, d = q.shape
    s = q.new_zeros(heads, d, v.shape[-1])
    out = []
    for i in range(t):
        s = g[i, :, :, None] * s + k[i, :, :, None] * v[i, :, None, :]
        out.append((s * q[i, :, :, None]).sum(1))
    return torch.stack(out)


def bonus_scan(r, k, v, g, u) -> torch.Tensor:
    """As above, but the result is read before the update and the current token counts with weight u [H, d]:
    o = (S + diag(u) k v^T)^T r,  then  S <- diag(g) S + k v^T."""
    t, heads, d = r.shape
    s = r.new_zeros(heads, d, v.shape[-1])
    out = []
    for i in range(t):
        kv = k[i, :, :, None] * v[i, :, None, :]
        out.append(((s + u[:, :, None] * kv) * r[i, :, :, None]).sum(1))
        s = g[i, :, :, None] * s + kv
    return torch.stack(out)


def token_mix(h: torch.Tensor, mu: torch.Tensor) -> torch.Tensor:
    """h_t + (h_(t-1) - h_t) mu, with h_(-1) = 0."""
    out = h.clone()
    for t in range(h.shape[0]):
        before = h[t - 1] if t else torch.zeros_like(h[0])
        out[t] = h[t] + (before - h[t]) * mu
    return out


def time_mix(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    """Heads of the time mixing, normed and gated, before the output projection."""
    t, heads, d = h.shape[0], m["heads"], m["dim"]
    x = {s: token_mix(h, w["mu." + s]) for s in "rkvgw"}
    r, k, v = ((x[s] @ w[s].T).view(t, heads, d) for s in "rkv")
    gate = silu(x["g"] @ w["g"].T)
    decay = torch.exp(-torch.exp(torch.tanh(x["w"] @ w["w1"].T) @ w["w2"].T + w["w0"])).view(t, heads, d)
    o = rms(bonus_scan(r, k, v, decay, w["u"]), eps).reshape(t, heads * d)
    return o * w["norm"] * gate


def gla_heads(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    t, heads, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].T).view(t, heads, d) * d ** -0.5
    k, v = (h @ w["k"].T).view(t, heads, d), (h @ w["v"].T).view(t, heads, e)
    alpha = sigmoid(h @ w["a1"].T @ w["a2"].T + w["a2.b"]) ** (1 / m["tau"])
    o = rms(decay_scan(q, k, v, alpha.view(t, heads, d)), eps) * w["norm"]
    return o.reshape(t, heads * e) * silu(h @ w["g"].T)


# ------------------------------------------------------------------ mixers
def attention(h, w, m, eps, shared) -> torch.Tensor:
    q, k, v = (h @ w[s].T + w[s + ".b"] for s in "qkv")
    first = None
    if m.get("v_mix"):
        first = shared.get("v")
        shared.setdefault("v", v)
    return attention_heads(q, k, v, w, m, eps, first) @ w["o"].T + w["o.b"]


def parallel(h, w, m, eps, shared) -> torch.Tensor:
    lw, rw = _sub(w, "left."), _sub(w, "right.")
    left = unit_heads(*(h @ lw[s].T for s in "qkv"), m["left"], eps) @ lw["o"].T
    right = time_mix(h, rw, m["right"], eps) @ rw["o"].T
    return m["left_scale"] * left + m["right_scale"] * right


def gla(h, w, m, eps, shared) -> torch.Tensor:
    return gla_heads(h, w, m, eps) @ w["o"].T


MIXERS = {"attention": attention, "parallel": parallel, "gla": gla}


# ------------------------------------------------------------------ feed-forwards
def dense(h: torch.Tensor, w: Dict[str, torch.Tensor]) -> torch.Tensor:
    return (gelu_tanh(h @ w["gate"].T + w["gate.b"]) * (h @ w["up"].T + w["up.b"])) @ w["down"].T + w["down.b"]


def route(z: torch.Tensor, correction: torch.Tensor, r: dict):
    """Logits [T, E] -> (chosen experts, their scores) per token."""
    s = sigmoid(z)
    choice = s + correction
    n, keep = r["groups"]["count"], r["groups"]["keep"]
    size = z.shape[1] // n
    out = []
    for t in range(z.shape[0]):
        c = choice[t]
        score = [float(sum(sorted(c[g * size:(g + 1) * size].tolist(), reverse=True)[:2])) for g in range(n)]
        best = sorted(range(n), key=lambda g: -score[g])[:keep]
        open_ = [e for g in best for e in range(g * size, (g + 1) * size)]
        ids = sorted(open_, key=lambda e: -float(c[e]))[: r["top"]]
        out.append((ids, s[t, ids]))
    return out


def expert(h: torch.Tensor, w: Dict[str, torch.Tensor], prefix: str) -> torch.Tensor:
    return relu_squared(h @ w[prefix + ".up"].T) @ w[prefix + ".down"].T


def moe(h: torch.Tensor, w: Dict[str, torch.Tensor], f: dict) -> torch.Tensor:
    out = expert(h, w, "shared") if f.get("shared") else torch.zeros_like(h)
    for t, (ids, scores) in enumerate(route(h @ w["router"].T, w["correction"], f["router"])):
        for e, s in zip(ids, scores):
            out[t] = out[t] + s * expert(h[t], w, f"e{e}")
    return out


# ------------------------------------------------------------------ the model
def _sub(w: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def forward(tokens, weights: Dict[str, torch.Tensor], cfg: dict, dtype=torch.float64,
            layers_out: Optional[List[torch.Tensor]] = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence; ``layers_out`` collects the residual after every layer."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    x = w["embed"][torch.as_tensor(tokens)]
    shared: Dict[str, torch.Tensor] = {}
    for i, layer in enumerate(cfg["layers"]):
        lw = _sub(w, f"l{i}.")
        x = x + m * MIXERS[layer["type"]](rms(x, eps) * lw["norm1"], _sub(lw, "mix."), layer["mixer"], eps, shared)
        f = layer["mlp"]
        if f is not None:
            h, fw = rms(x, eps) * lw["norm2"], _sub(lw, "mlp.")
            x = x + m * (dense(h, fw) if f["kind"] == "dense" else moe(h, fw, f))
        if layers_out is not None:
            layers_out.append(x)
    return rms(x, eps) * w["final.norm"] @ w["head"].T
