"""Layers whose memory of a sequence is a state of fixed size: a matrix S per head, fp32.

    S <- diag(g) S;  S <- S + k u^T;  o = S^T q

with u = v (gated linear attention: keys 1 - g; decayed linear attention: keys of their own; time mixing: o
from the S before the token, the token itself with a weight of its own) or u = beta (v - S^T k) (delta rule).
A layer run's state
lives in slots (``ctx.states``), one per running sequence; a step carries it over all tokens of a portion
and stores it again, so prompt portions of any cut, single tokens and mixtures of both are one kernel call
(``ops.recurrent_scan``).  A sequence that starts at position 0 starts from zero whatever its slot holds.

Everything that enters the recurrence besides the projections and convolutions is fp32.
"""
from __future__ import annotations

from typing import Dict, Optional

import torch
from torch import nn

from .. import ops
from .metadata import AttentionMetadata, get_forward_context


def _pad4(n: int) -> int:
    return (n + 3) // 4 * 4


class _Recurrent(nn.Module):
    def __init__(self, num_heads: int, head_dim: int, v_head_dim: int, eps: float, dtype, device) -> None:
        super().__init__()
        self.num_heads, self.head_dim, self.v_dim, self.eps, self.dtype = num_heads, head_dim, v_head_dim, eps, dtype
        self.out_norm = self._param(v_head_dim, fill=1.0, dtype=dtype, device=device)

    @staticmethod
    def _param(*shape, fill=0.0, dtype=torch.float32, device=None) -> nn.Parameter:
        return nn.Parameter(torch.full(shape, fill, dtype=dtype, device=device), requires_grad=False)

    def state_shapes(self) -> Dict[str, tuple]:
        """Name -> (shape of one slot, type)."""
        return {"s": ((self.num_heads, self.v_dim, _pad4(self.head_dim)), torch.float32)}

    @staticmethod
    def _step(md: AttentionMetadata):
        return md.state_slots, md.cu_q, md.seq_lens, md.num_seqs


class GatedLinearAttention(_Recurrent):
    """Forget gate f = lower + (1 - lower) * sigmoid(projection + bias) per channel; keys are 1 - f."""

    def __init__(self, num_heads: int, head_dim: int, v_head_dim: int, eps: float, dtype, device) -> None:
        super().__init__(num_heads, head_dim, v_head_dim, eps, dtype, device)
        self.f_bias = self._param(num_heads * head_dim, device=device)
        self.lower = self._param(num_heads * head_dim, device=device)

    def forward(self, proj: torch.Tensor, offs: Dict[str, int], run: int, out_width: int) -> torch.Tensor:
        ctx = get_forward_context()
        md, state = ctx.attn_metadata, ctx.states[run]
        q, k = ops.gated_linear_prep(proj, offs["q"], offs["f"], self.num_heads, self.head_dim, self.f_bias, self.lower)
        v = proj[:, offs["v"]: offs["v"] + self.num_heads * self.v_dim]
        o = ops.recurrent_scan(q, k, None, v, None, state["s"], self.num_heads, self.v_dim, *self._step(md))
        return ops.head_norm_gate(o, self.out_norm, self.eps, None, out_width)


class DeltaRuleAttention(_Recurrent):
    """Gated delta rule behind short convolutions.  The first ``conv_channels`` columns of the projection
    are q, k and v (each padded); the convolution's weights and its stored inputs have the same columns."""

    def __init__(self, num_heads: int, num_kv_heads: int, head_dim: int, v_head_dim: int, taps: int,
                 conv_channels: int, unit_eps: float, eps: float, dtype, device) -> None:
        super().__init__(num_heads, head_dim, v_head_dim, eps, dtype, device)
        self.num_kv_heads, self.taps, self.channels, self.unit_eps = num_kv_heads, taps, conv_channels, unit_eps
        self.conv_weight = self._param(conv_channels, taps, dtype=dtype, device=device)
        self.a_log = self._param(num_heads, device=device)
        self.dt_bias = self._param(num_heads * head_dim, device=device)

    def state_shapes(self) -> Dict[str, tuple]:
        return {**super().state_shapes(), "conv": ((self.taps - 1, self.channels), self.dtype)}

    def forward(self, proj: torch.Tensor, offs: Dict[str, int], low: torch.Tensor, gate: Optional[torch.Tensor],
                run: int, out_width: int) -> torch.Tensor:
        """``low`` [T, heads * dim]: the decay's low-rank projection; ``gate`` [T, heads * v] before the
        sigmoid."""
        ctx = get_forward_context()
        md, state = ctx.attn_metadata, ctx.states[run]
        q, k, g, v, beta = ops.delta_prep(proj, low, offs, self.num_heads, self.num_kv_heads, self.head_dim, self.v_dim,
                                          self.conv_weight, state["conv"], self.dt_bias, self.a_log, self.unit_eps,
                                          md.seq_idx, *self._step(md))
        o = ops.recurrent_scan(q, k, g, v, beta, state["s"], self.num_heads, self.v_dim, *self._step(md),
                               conv=(proj, state["conv"]))
        return ops.head_norm_gate(o, self.out_norm, self.eps, gate, out_width)


class DecayLinearAttention(_Recurrent):
    """Keys and decays apart: g = sigmoid(z + bias)^(1 / tau) per head and key channel, queries times
    dim^(-1/2); the result is normed per head and multiplied by silu of a gate."""

    def __init__(self, num_heads: int, head_dim: int, v_head_dim: int, tau: float, eps: float, dtype, device) -> None:
        super().__init__(num_heads, head_dim, v_head_dim, eps, dtype, device)
        self.tau = tau
        self.decay_bias = self._param(num_heads * head_dim, device=device)

    def forward(self, q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, z: torch.Tensor, gate: torch.Tensor, run: int,
                out_width: int) -> torch.Tensor:
        """q, k [T, heads * dim], v, gate [T, heads * v] views of the projection, z [T, heads * dim] fp32."""
        ctx = get_forward_context()
        md, state = ctx.attn_metadata, ctx.states[run]
        q, k, g = ops.decay_prep(q, k, z, self.decay_bias, self.num_heads, self.head_dim, self.head_dim ** -0.5, self.tau)
        o = ops.recurrent_scan(q, k, g, v, None, state["s"], self.num_heads, self.v_dim, *self._step(md))
        return ops.head_norm_gate(o, self.out_norm, self.eps, gate, out_width, silu=True)


class TimeMixAttention(_Recurrent):
    """Time mixing: r, k, v, a gate and the decay each read their own blend of the input with the previous
    token's (``blend``), g = exp(-exp(z + w0)), and the current token counts with weight u.  The result is
    divided by its root mean square per head and multiplied by a weight per channel and silu of the gate."""

    BLENDS = ("r", "k", "v", "g", "w")

    def __init__(self, num_heads: int, head_dim: int, width: int, eps: float, dtype, device) -> None:
        super().__init__(num_heads, head_dim, head_dim, eps, dtype, device)
        self.width = width
        self.out_norm = self._param(num_heads, head_dim, fill=1.0, dtype=dtype, device=device)
        self.mu = self._param(len(self.BLENDS), width, dtype=dtype, device=device)
        self.w0 = self._param(num_heads * head_dim, device=device)
        self.u = self._param(num_heads, head_dim, device=device)

    def state_shapes(self) -> Dict[str, tuple]:
        return {**super().state_shapes(), "shift": ((self.width,), torch.float32)}

    def blend(self, h: torch.Tensor, run: int):
        """([5 T, width], offsets): the blends in the order of ``BLENDS``."""
        ctx = get_forward_context()
        md = ctx.attn_metadata
        return ops.token_mix(h, self.mu, ctx.states[run]["shift"], md.seq_idx, *self._step(md))

    def forward(self, r: torch.Tensor, k: torch.Tensor, v: torch.Tensor, z: torch.Tensor, gate: torch.Tensor, run: int,
                scale: float, out: torch.Tensor) -> None:
        """Writes ``scale`` times the result to the rows ``out``."""
        ctx = get_forward_context()
        md, state = ctx.attn_metadata, ctx.states[run]
        r, k, g, bonus = ops.time_mix_prep(r, k, z, self.w0, self.u, self.num_heads, self.head_dim)
        o = ops.recurrent_scan(r, k, g, v, bonus, state["s"], self.num_heads, self.v_dim, *self._step(md), bonus=True)
        ops.head_norm_gate(o, self.out_norm, self.eps, gate, silu=True, scale=scale, out=out)
