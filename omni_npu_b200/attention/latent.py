"""Attention over a cached latent with run-time sizes, in one type (bf16 or fp32) throughout.

A cache row is [normed latent (rank) | rotated key part (rot) | zeros up to whole 16-byte pieces], shared
by all heads.  As for the DeepSeek models (``attention/mla.py``, whose kernels have their sizes built in
or take them from here) there are two paths:

* prompt portions: the rows of every sequence are gathered, brought to per-head keys and values by two
  products, and attended with the variable-length kernel.  The key weight carries an identity block that
  copies the rotated part, so that the product yields whole keys;
* single new tokens: queries are folded into the latent space, attend over the rows themselves, and the
  result is brought back per head.

Queries may come from a latent of their own (``q_rank``); its norm runs with the cache row's (``store``).  A layer
that reads another layer's rows stores none; what that layer gathered for a prompt step is used again.
"""
from __future__ import annotations

from typing import Optional

import torch
from torch import nn

from .. import ops
from .metadata import AttentionMetadata, get_forward_context


class LatentAttention(nn.Module):
    """``num_heads``: heads of this rank.  ``w_uk`` [heads * nope, rank] and ``w_uv`` [heads * v, rank] are
    set before ``build_absorbed``."""

    layer_idx = -1           # (the cache is named at each call; what looks for attention layers finds this one)

    def __init__(self, num_heads: int, nope_dim: int, rope_dim: int, v_head_dim: int, kv_rank: int, scale: float,
                 neox: bool, eps: float, dtype: torch.dtype, device, q_rank: int = 0, own_rows: bool = True,
                 rows_shared: bool = False) -> None:
        super().__init__()
        self.q_rank, self.own_rows, self.rows_shared = q_rank, own_rows, rows_shared
        self.num_heads, self.nope, self.rot, self.v_dim, self.rank = num_heads, nope_dim, rope_dim, v_head_dim, kv_rank
        self.scale, self.neox, self.eps, self.dtype = scale, neox, eps, dtype
        self.qk_dim = nope_dim + rope_dim
        self.row = (kv_rank + rope_dim + 7) // 8 * 8
        self.k_pad, self.v_pad = ops.gated_head_pad(self.qk_dim, dtype), ops.gated_head_pad(v_head_dim, dtype)

        def param(*shape, fill=0.0):
            return nn.Parameter(torch.full(shape, fill, dtype=dtype, device=device), requires_grad=False)

        self.latent_norm = param(kv_rank, fill=1.0) if own_rows else None
        self.query_norm = param(q_rank, fill=1.0) if q_rank else None
        self.w_uk = param(num_heads * nope_dim, kv_rank)
        self.w_uv = param(num_heads * v_head_dim, kv_rank)
        # products of the two paths, derived from the two above
        self.register_buffer("w_key", torch.zeros(num_heads * self.k_pad, self.row, dtype=dtype, device=device), False)
        self.register_buffer("w_value", torch.zeros(num_heads * self.v_pad, self.row, dtype=dtype, device=device), False)
        self.register_buffer("w_fold", torch.zeros(num_heads, kv_rank, nope_dim, dtype=dtype, device=device), False)

    @torch.no_grad()
    def build_absorbed(self) -> None:
        uk = self.w_uk.data.view(self.num_heads, self.nope, self.rank)
        uv = self.w_uv.data.view(self.num_heads, self.v_dim, self.rank)
        key = self.w_key.view(self.num_heads, self.k_pad, self.row)
        key.zero_()
        key[:, : self.nope, : self.rank] = uk
        i = torch.arange(self.rot, device=uk.device)
        key[:, self.nope + i, self.rank + i] = 1
        value = self.w_value.view(self.num_heads, self.v_pad, self.row)
        value.zero_()
        value[:, : self.v_dim, : self.rank] = uv
        self.w_fold.copy_(uk.transpose(1, 2))

    # ------------------------------------------------------------------ forward
    def store(self, z: torch.Tensor, kv_a: Optional[torch.Tensor], cos_sin: torch.Tensor, cache_idx: int) -> torch.Tensor:
        """The queries' latent z [T, q_rank] normed (with zeros up to whole 16-byte rows), and the cache row when the
        layer has its own: views into the projection."""
        ctx = get_forward_context()
        md: AttentionMetadata = ctx.attn_metadata
        c_q = z.new_empty(z.shape[0], (self.q_rank + 7) // 8 * 8)
        ops.latent_prep_(None, kv_a, self.latent_norm, self.eps, ctx.kv_caches[cache_idx], md.positions, md.slot_mapping,
                         cos_sin, self.num_heads, self.nope, self.rot, self.rank, self.neox,
                         low=(z, self.query_norm, c_q))
        return c_q

    def forward(self, q: torch.Tensor, kv_a: Optional[torch.Tensor], cos_sin: torch.Tensor, cache_idx: int,
                out_width: int = 0) -> torch.Tensor:
        """q [T, heads * (nope + rot)] (rotated in place), kv_a [T, rank + rot] or None (the rows are stored
        already): views into the projection.  Returns [T, max(heads * v, out_width)], zero beyond the heads."""
        ctx = get_forward_context()
        md: AttentionMetadata = ctx.attn_metadata
        cache = ctx.kv_caches[cache_idx]
        t, used = q.shape[0], self.num_heads * self.v_dim
        out = q.new_zeros(t, out_width) if out_width > used else q.new_empty(t, used)
        nd = t if not md.is_prefill else md.extra.get("num_decode_seqs", 0)
        q_latent = q.new_empty(t, self.num_heads, self.row) if nd else None
        args = (self.latent_norm, self.eps, cache, md.positions, md.slot_mapping, cos_sin, self.num_heads, self.nope,
                self.rot, self.rank, self.neox)
        ops.latent_prep_(q, kv_a, *args, q_latent, nd)
        if nd:
            self._decode(q[:nd], q_latent[:nd], cache, md, nd, out[:nd])
        if nd < t:
            self._prompt(q[nd:], cache, cache_idx, md, nd, out[nd:])
        return out

    def _decode(self, q, q_latent, cache, md: AttentionMetadata, n: int, out) -> None:
        heads = q[:, : self.num_heads * self.qk_dim].unflatten(1, (self.num_heads, self.qk_dim))
        ops.head_gemm(heads[..., : self.nope], self.w_fold, q_latent[..., : self.rank])
        o = q.new_empty(n, self.num_heads, self.rank)
        ops.latent_decode(q_latent, cache, md.block_tables[:n], md.seq_lens[:n], n, self.num_heads, self.rank,
                          self.scale, o, max_seq_len=md.max_seq_len)
        uv = self.w_uv.view(self.num_heads, self.v_dim, self.rank)
        ops.head_gemm(o, uv, out[:, : self.num_heads * self.v_dim].unflatten(1, (self.num_heads, self.v_dim)))

    def _prompt(self, q, cache, cache_idx: int, md: AttentionMetadata, nd: int, out) -> None:
        n = md.num_seqs - nd
        bt, lens = md.block_tables[nd: md.num_seqs], md.seq_lens[nd: md.num_seqs]
        shared = md.extra.setdefault("latent_prompt", {})           # same for every layer of the step
        if not shared:
            host = md.extra.get("seq_lens_host")
            total = sum((lens.tolist() if host is None else host[nd:]))
            shared.update(total=total, start=(torch.cumsum(lens, 0, dtype=torch.int32) - lens).contiguous())
        rows = shared.get(cache_idx) if not self.own_rows else None
        if rows is None:
            rows = ops.latent_gather(cache, bt, lens, shared["start"], n, shared["total"], md.max_seq_len)
            if self.rows_shared:
                shared[cache_idx] = rows
        k = ops.gemm(rows, self.w_key).view(-1, self.num_heads, 1, self.k_pad)
        v = ops.gemm(rows, self.w_value).view(-1, self.num_heads, 1, self.v_pad)
        cu_q = md.extra["cu_q_prefill"] if nd else md.cu_q
        ops.contiguous_attention(q, k, v, out, cu_q, shared["start"], lens, n,
                                 md.extra["max_q_len_prefill"] if nd else md.max_q_len, self.num_heads, self.qk_dim,
                                 self.v_dim, self.scale)
