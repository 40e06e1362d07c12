"""Grouped-query attention backend over the paged KV cache.

Counterpart of ``NPUAttentionBackend`` (omni_npu/attention/backends/attention.py:114-281):
KV cache shape, metadata handling and the forward that first stores this
step's keys/values (fused with RoPE) and then runs one paged attention call.
Different K and V head sizes are allowed (needed by Pangu Pro MoE).
"""
from __future__ import annotations

from typing import Optional, Tuple

import torch

from .. import ops
from .metadata import AttentionMetadata, get_forward_context


class GQABackend:
    name = "B200_GQA"

    @staticmethod
    def get_name() -> str:
        return GQABackend.name

    @staticmethod
    def get_kv_cache_shape(num_blocks: int, block_size: int, num_kv_heads: int, head_size: int,
                           head_size_v: Optional[int] = None) -> Tuple[Tuple[int, ...], Tuple[int, ...]]:
        hv = head_size_v or head_size
        return ((num_blocks, num_kv_heads, block_size, head_size),
                (num_blocks, num_kv_heads, block_size, hv))

    @staticmethod
    def allocate_kv_cache(num_blocks: int, block_size: int, num_kv_heads: int, head_size: int,
                          dtype: torch.dtype, device: torch.device,
                          head_size_v: Optional[int] = None):
        ks, vs = GQABackend.get_kv_cache_shape(num_blocks, block_size, num_kv_heads, head_size, head_size_v)
        return (torch.zeros(ks, dtype=dtype, device=device), torch.zeros(vs, dtype=dtype, device=device))

    @staticmethod
    def bytes_per_block(block_size: int, num_kv_heads: int, head_size: int, dtype: torch.dtype,
                        head_size_v: Optional[int] = None) -> int:
        hv = head_size_v or head_size
        return block_size * num_kv_heads * (head_size + hv) * dtype.itemsize


class GQAAttention(torch.nn.Module):
    """One layer's attention: RoPE + cache write + paged attention."""

    # gathers the step's keys / values when the step is split over prefill-context-parallel ranks
    supports_prefill_context_parallel = True

    def __init__(self, layer_idx: int, num_heads: int, num_kv_heads: int, head_dim: int,
                 scale: float, rot_dim: int, neox: bool = True, sliding_window: int = 0,
                 head_dim_v: Optional[int] = None) -> None:
        super().__init__()
        self.layer_idx = layer_idx
        self.num_heads = num_heads
        self.num_kv_heads = num_kv_heads
        self.head_dim = head_dim
        self.head_dim_v = head_dim_v or head_dim
        self.scale = scale
        self.rot_dim = rot_dim
        self.neox = neox
        self.window = sliding_window

    def forward(self, q: torch.Tensor, k: torch.Tensor, v: torch.Tensor,
                cos_sin: Optional[torch.Tensor], apply_rope: bool = True) -> torch.Tensor:
        """q [T, Hq*D], k [T, Hk*D], v [T, Hk*Dv] (views into the fused QKV
        projection are fine).  Returns [T, Hq*Dv]."""
        ctx = get_forward_context()
        md: AttentionMetadata = ctx.attn_metadata
        k_cache, v_cache = ctx.kv_caches[self.layer_idx]
        pc = md.extra.get("pcp") if md.is_prefill else None
        if pc is not None:
            # prefill context parallelism: this rank holds the query rows of its token shard; the
            # keys and values of the whole step are gathered, rotated with their own positions and
            # written into the local cache, then the shard attends causally over the cache
            t = q.shape[0]
            pad = pc["pad"]

            def gathered(x):
                x = x.contiguous()
                if t < pad:
                    x = torch.cat([x, x.new_zeros(pad - t, x.shape[1])])
                return pc["group"].all_gather(x, dim=0).index_select(0, pc["gather_idx"])

            k_all, v_all = gathered(k), gathered(v)
            if apply_rope and cos_sin is not None:
                ops.rope_qk_(q, q.new_empty(t, 0), md.positions, cos_sin, self.head_dim, self.rot_dim, self.neox)
                ops.rope_qk_(k_all, k_all.new_empty(k_all.shape[0], 0), pc["positions_all"], cos_sin, self.head_dim,
                             self.rot_dim, self.neox)
            ops.gqa_cache_write(k_all, v_all, k_cache, v_cache, pc["slot_all"])
            return ops.gqa_prefill(q, k_cache, v_cache, md.block_tables, md.cu_q, md.seq_lens,
                                   md.num_seqs, md.max_q_len, self.num_heads, self.scale, True, self.window)
        if apply_rope and cos_sin is not None and md.positions.dim() == 1:
            ops.rope_cache_gqa_(q, k, v, k_cache, v_cache, md.positions, md.slot_mapping, cos_sin,
                                self.head_dim, self.rot_dim, self.neox)
        else:
            ops.gqa_cache_write(k, v, k_cache, v_cache, md.slot_mapping)
        nd = md.extra.get("num_decode_seqs", 0) if md.is_prefill else 0
        if nd:
            # mixed batch: rows [0, nd) are the single new tokens of decoding sequences
            o_dec = ops.gqa_decode(q[:nd], k_cache, v_cache, md.block_tables[:nd], md.seq_lens[:nd], nd,
                                   self.num_heads, self.scale, 1, self.window, max_seq_len=md.max_seq_len)
            o_pre = ops.gqa_prefill(q[nd:], k_cache, v_cache, md.block_tables[nd:], md.extra["cu_q_prefill"],
                                    md.seq_lens[nd:], md.num_seqs - nd, md.extra["max_q_len_prefill"],
                                    self.num_heads, self.scale, True, self.window)
            return torch.cat([o_dec, o_pre], 0)
        if md.is_prefill:
            return ops.gqa_prefill(q, k_cache, v_cache, md.block_tables, md.cu_q, md.seq_lens,
                                   md.num_seqs, md.max_q_len, self.num_heads, self.scale, True,
                                   self.window)
        return ops.gqa_decode(q, k_cache, v_cache, md.block_tables, md.seq_lens, md.num_seqs,
                              self.num_heads, self.scale, md.q_len, self.window,
                              max_seq_len=md.max_seq_len)


class GatedGQAAttention(torch.nn.Module):
    """Attention with any head sizes (queries / keys ``head_dim``, values ``head_dim_v``), rotation of the
    first ``rot_dim`` dimensions, an optional sliding window, an optional sink (a key of score ``sink``
    without a value in every softmax) and an optional output gate.  The cache rows are padded to whole
    tensor-core steps (``ops.gated_head_pad``)."""

    def __init__(self, layer_idx: int, num_heads: int, num_kv_heads: int, head_dim: int, head_dim_v: int,
                 scale: float, rot_dim: int, neox: bool = True, sliding_window: int = 0,
                 sink: Optional[float] = None) -> None:
        super().__init__()
        self.layer_idx = layer_idx
        self.num_heads, self.num_kv_heads = num_heads, num_kv_heads
        self.head_dim, self.head_dim_v = head_dim, head_dim_v
        self.scale, self.rot_dim, self.neox = scale, rot_dim, neox
        self.window, self.sink = sliding_window, sink

    def cache_widths(self, dtype: torch.dtype) -> Tuple[int, int]:
        return ops.gated_head_pad(self.head_dim, dtype), ops.gated_head_pad(self.head_dim_v, dtype)

    def forward(self, q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, gate: Optional[torch.Tensor],
                cos_sin: torch.Tensor, out_width: int = 0) -> torch.Tensor:
        """q [T, Hq*D] (rotated in place), k [T, Hk*D], v [T, Hk*Dv], gate [T, Hq*Dv] or None: views into
        the fused projection.  Returns [T, max(Hq*Dv, out_width)], zero beyond the heads."""
        ctx = get_forward_context()
        md: AttentionMetadata = ctx.attn_metadata
        k_cache, v_cache = ctx.kv_caches[self.layer_idx]
        ops.gated_rope_cache_(q, k, v, k_cache, v_cache, md.positions, md.slot_mapping, cos_sin, self.head_dim,
                              self.head_dim_v, self.rot_dim, self.neox)
        return self._attend(q, gate, md, k_cache, v_cache, out_width)

    def _attend(self, q: torch.Tensor, gate: Optional[torch.Tensor], md: AttentionMetadata, k_cache: torch.Tensor,
                v_cache: torch.Tensor, out_width: int = 0, out: Optional[torch.Tensor] = None) -> torch.Tensor:
        """Attention of this step's rotated queries over the cache (into the rows ``out`` when given)."""
        t, used = q.shape[0], self.num_heads * self.head_dim_v
        if out is None:
            out = q.new_zeros(t, out_width) if out_width > used else q.new_empty(t, used)

        def run(rows: slice, seqs: slice, cu_q, n: int, max_q: int):
            self._run(q[rows], None if gate is None else gate[rows], k_cache, v_cache, out[rows], md.block_tables[seqs],
                      cu_q, md.seq_lens[seqs], n, max_q, md.max_seq_len)

        if not md.is_prefill:
            run(slice(None), slice(None), None, md.num_seqs, md.q_len)
            return out
        nd = md.extra.get("num_decode_seqs", 0)
        if nd:           # rows [0, nd): single new tokens of decoding sequences
            run(slice(0, nd), slice(0, nd), None, nd, 1)
            run(slice(nd, t), slice(nd, None), md.extra["cu_q_prefill"], md.num_seqs - nd,
                md.extra["max_q_len_prefill"])
        else:
            run(slice(None), slice(None), md.cu_q, md.num_seqs, md.max_q_len)
        return out

    def _run(self, q, gate, k_cache, v_cache, out, block_tables, cu_q, seq_lens, n: int, max_q: int, max_seq: int) -> None:
        ops.gated_attention(q, gate, k_cache, v_cache, out, block_tables, cu_q, seq_lens, n, max_q, self.num_heads,
                            self.head_dim, self.head_dim_v, self.scale, self.window, self.sink, max_seq_len=max_seq)


class NormedGQAAttention(GatedGQAAttention):
    """The same with a norm on q and k (``ops.qk_norm_rope_cache``) and, optionally, values blended with those of
    another layer before they are cached.  ``norm`` "projection" has weights over this rank's rows and counts
    the rows of all ranks; ``value_mix`` is the other layer's share."""

    def __init__(self, layer_idx: int, num_heads: int, num_kv_heads: int, head_dim: int, head_dim_v: int, scale: float,
                 rot_dim: int, norm: Optional[str], eps: float, dtype, device, sliding_window: int = 0, group=None) -> None:
        super().__init__(layer_idx, num_heads, num_kv_heads, head_dim, head_dim_v, scale, rot_dim, True, sliding_window)
        self.norm, self.eps, self.group = norm, eps, group
        self.q_norm = self.k_norm = None
        if norm == "projection":
            self.q_norm, self.k_norm = (torch.nn.Parameter(torch.ones(n * head_dim, dtype=dtype, device=device),
                                                           requires_grad=False) for n in (num_heads, num_kv_heads))
        self.value_mix = 0.0

    def forward(self, q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, cos_sin: torch.Tensor, out_width: int = 0,
                v_first: Optional[torch.Tensor] = None, out: Optional[torch.Tensor] = None) -> torch.Tensor:
        """q [T, Hq*D], k [T, Hk*D], v and ``v_first`` [T, Hk*Dv]: views into fused projections.  Returns
        [T, max(Hq*Dv, out_width)], zero beyond the heads, or writes the rows ``out``."""
        ctx = get_forward_context()
        md: AttentionMetadata = ctx.attn_metadata
        k_cache, v_cache = ctx.kv_caches[self.layer_idx]
        sums = None
        if self.norm == "projection" and self.group is not None and self.group.world_size > 1:
            s = torch.stack([x.float().pow(2).sum(-1) for x in (q, k)], 1)
            world = self.group.world_size
            sums = self.group.all_reduce(s), q.shape[1] * world, k.shape[1] * world
        weights = (self.q_norm, self.k_norm) if self.norm == "projection" else None
        q = ops.qk_norm_rope_cache(q, k, v, k_cache, v_cache, md.positions, md.slot_mapping, cos_sin, self.head_dim,
                                   self.head_dim_v, self.rot_dim, self.norm, self.eps, weights, sums, v_first,
                                   self.value_mix)
        return self._attend(q, None, md, k_cache, v_cache, out_width, out)


class MixedScoreAttention(GatedGQAAttention):
    """Attention without rotation whose heads mix their scores before the softmax (``ops.mixed_attention``): q and k
    normed per head with a weight, queries with a temperature that grows with the position, scores capped and lowered
    by a learned distance bias, a learned sink per head.

    ``num_heads`` score heads over ``num_kv_heads`` key heads, whole on every rank; ``out_heads`` output heads over
    ``v_heads`` value heads of this rank.  The constants that multiply scores are kept in fp32."""

    def __init__(self, layer_idx: int, num_heads: int, num_kv_heads: int, out_heads: int, v_heads: int, head_dim: int,
                 head_dim_v: int, scale: float, softcap: float, temperature: Optional[Tuple[float, int]], eps: float, dtype,
                 device) -> None:
        super().__init__(layer_idx, num_heads, num_kv_heads, head_dim, head_dim_v, scale, 0)
        self.out_heads, self.v_heads = out_heads, v_heads
        self.softcap, self.temperature, self.eps = softcap, temperature, eps

        def param(*shape, fill=0.0, dt=torch.float32):
            return torch.nn.Parameter(torch.full(shape, fill, dtype=dt, device=device), requires_grad=False)

        self.q_norm, self.k_norm = param(head_dim, fill=1.0, dt=dtype), param(head_dim, fill=1.0, dt=dtype)
        self.r1, self.r2, self.sink = param(num_heads), param(num_heads), param(out_heads)
        self.talk = param(out_heads, num_heads)
        self.talk_exact = False                  # whether bf16 holds it (set after loading)

    def forward(self, q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, out_width: int = 0) -> torch.Tensor:
        """q [T, Hs*D], k [T, Hk*D], v [T, Hv*Dv]: views into the fused projection.  Returns
        [T, max(Ho*Dv, out_width)], zero beyond the heads."""
        ctx = get_forward_context()
        md: AttentionMetadata = ctx.attn_metadata
        k_cache, v_cache = ctx.kv_caches[self.layer_idx]
        q = ops.qk_norm_rope_cache(q, k, v, k_cache, v_cache, md.positions, md.slot_mapping, None, self.head_dim,
                                   self.head_dim_v, 0, "head_weight", self.eps, (self.q_norm, self.k_norm),
                                   temperature=self.temperature)
        t, used = q.shape[0], self.out_heads * self.head_dim_v
        out = q.new_zeros(t, out_width) if out_width > used else q.new_empty(t, used)
        self._attend(q, None, md, k_cache, v_cache, out=out)
        return out

    def _run(self, q, gate, k_cache, v_cache, out, block_tables, cu_q, seq_lens, n: int, max_q: int, max_seq: int) -> None:
        ops.mixed_attention(q, k_cache, v_cache, out, block_tables, cu_q, seq_lens, n, max_q, self.head_dim, self.head_dim_v,
                            self.scale, self.softcap, (self.r1, self.r2), self.talk, self.sink, max_seq_len=max_seq,
                            talk_exact=self.talk_exact)
