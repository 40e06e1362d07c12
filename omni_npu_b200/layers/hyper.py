"""Hyper-connections: several residual streams x_1 .. x_N instead of one.

A sublayer reads u = sum_s in_s x_s and its result y comes back as
x_t <- sum_s mix[s, t] x_s + out_t * (scale * y), all streams at once.  The join of one sublayer, the
reading, layer norm and token shift of the next are one kernel (``ops.hyper_norm``), so a sublayer only
supplies its parameters here.  The streams are fp32, and so is everything in this module but the norm's
result.
"""
from __future__ import annotations

from typing import Optional, Tuple

import torch
from torch import nn

from .. import ops
from ..attention.metadata import AttentionMetadata


class HyperSublayer(nn.Module):
    """Parameters of one sublayer's place between the streams; ``join`` False for the end of the model,
    which only reads (the plain sum of the streams)."""

    def __init__(self, width: int, true_width: int, streams: int, eps: float, dtype, device, join: bool = True,
                 shift: bool = False, out_scale: float = 1.0) -> None:
        super().__init__()

        def param(*shape, fill=0.0, dt=dtype):
            return nn.Parameter(torch.full(shape, fill, dtype=dt, device=device), requires_grad=False)

        self.true_width, self.eps, self.out_scale = true_width, eps, out_scale
        self.norm_weight = param(width, fill=1.0)
        self.norm_bias = param(width)
        self.w_in = param(streams, fill=1.0, dt=torch.float32)
        self.w_mix = self.w_out = self.layer_scale = self.shift = None
        if join:
            self.w_mix = nn.Parameter(torch.eye(streams, dtype=torch.float32, device=device), requires_grad=False)
            self.w_out = param(streams, fill=1.0, dt=torch.float32)
            self.layer_scale = param(width, fill=1.0)
        if shift:
            self.shift = param(width)

    @property
    def streams(self) -> int:
        return self.w_in.shape[0]

    def connection(self):
        return self.layer_scale, self.w_mix, self.w_out

    def read(self, streams: Optional[torch.Tensor], before: Optional["HyperSublayer"], y: Optional[torch.Tensor],
             md: Optional[AttentionMetadata], state: Optional[torch.Tensor] = None, ids: Optional[torch.Tensor] = None,
             table: Optional[torch.Tensor] = None, keep: bool = True) -> Tuple[Optional[torch.Tensor], torch.Tensor]:
        """Join ``y``, the result of the sublayer ``before``, to the streams (or start them from rows
        ``ids`` of ``table``) and return (streams, this sublayer's input).  ``state``: fp32 [slots, width],
        the previous token's input of every sequence, for the token shift."""
        shift = None
        if self.shift is not None:
            shift = (self.shift, state, md.seq_idx, md.state_slots, md.cu_q, md.seq_lens, md.num_seqs)
        return ops.hyper_norm(streams, ids, table, self.streams, y, before.connection() if before is not None else None,
                              self.w_in, self.norm_weight, self.norm_bias, self.eps, self.true_width, self.out_scale,
                              shift, keep)
