"""Gatosun: a decoder that mixes full attention, attention beside time mixing, and decayed linear attention.

Each layer is a mixer and an optional feed-forward, each on its own RMS norm of the fp32 residual x and added
with one factor: x <- x + m * sublayer(norm(x)).  Mixers are

    attention   grouped-query attention, q / k normed over the whole projection, biases, values blended with
                those of the first such layer                                   (attention/gqa.py)
    parallel    sliding-window attention with unit heads, and time mixing, on one input
                                                                                (attention/gqa.py, recurrent.py)
    gla         linear attention with a decay per head and key channel          (attention/recurrent.py)

The feed-forward is dense (gelu gate, biases) or a mixture of ungated squared-relu experts with group-limited
sigmoid routing and a shared expert.  Sizes and constants are given layer by layer.

Per layer and step: one product for the projections of the input, the mixer's own kernels, one product back,
residual + norm; then two products (grouped ones for the experts) and residual + norm, which also brings the
experts' rows back to their tokens.  The two halves of a parallel mixer write into one row, so that their
output projections are one product: the left weight is the residual kernel's factor, the right one, relative
to it, multiplies the time mixing's result in fp32.

Widths that are not whole 16-byte rows are padded with zeros when the weights are loaded; the norms divide by
the true width.
"""
from __future__ import annotations

import os
from typing import Any, Callable, Dict, Iterable, List, Optional, Tuple

import torch
from torch import nn

from .. import ops
from ..attention.gqa import NormedGQAAttention
from ..attention.recurrent import DecayLinearAttention, TimeMixAttention
from ..config import (AttentionSpec, DecayLinearSpec, DenseSpec, EngineConfig, ExpertSpec, LayerSpec, ModelConfig, MoESpec,
                      ParallelSpec, TimeMixSpec, to_dtype)
from ..layers.embedding import ParallelLMHead, VocabParallelEmbedding
from ..layers.linear import SegmentedLinear
from ..layers.mlp import FusedMLP
from ..layers.moe import FusedMoE
from ..layers.rope import get_rope
from .layered import Mixer, Want, fit, pad8, place_tensors

# Steps of at most this many rows run the two halves of a parallel mixer on two streams.
OVERLAP_ROWS = int(os.environ.get("OMNI_B200_PARALLEL_SUBLAYER_ROWS", "256"))
EXPERT_ACT = "relu2"


# --------------------------------------------------------------------- configuration
def _attention_spec(m: Dict[str, Any], qk_norm: str, window: int = 0, **kw) -> AttentionSpec:
    s = AttentionSpec(num_heads=int(m["heads"]), num_kv_heads=int(m["kv_heads"]), head_dim=int(m["dim"]),
                      v_head_dim=int(m["vdim"]), rotary_dim=int(m["rot"]["dims"]), rope_theta=float(m["rot"]["base"]),
                      scale=float(m["scale"]), rope_neox=True, sliding_window=window, qk_norm=qk_norm, **kw)
    if s.num_heads % s.num_kv_heads or s.rotary_dim % 2 or s.rotary_dim > s.head_dim:
        raise ValueError(f"Gatosun: inconsistent attention sizes {m}")
    return s


def _mixer_spec(kind: str, m: Dict[str, Any], rank: Callable[[str, int], int]):
    if kind == "attention":
        return _attention_spec(m, "projection", bias=True, value_mix=bool(m.get("v_mix", False)))
    if kind == "parallel":
        left, right = m["left"], m["right"]
        window = int(left["mask"]["size"])
        if window < 1:
            raise ValueError(f"Gatosun: window of {window} tokens")
        return ParallelSpec(_attention_spec(left, "head", window),
                            TimeMixSpec(int(right["heads"]), int(right["dim"]), rank("right.w1", int(right["dim"]))),
                            float(m["left_scale"]), float(m["right_scale"]))
    if kind == "gla":
        return DecayLinearSpec(int(m["heads"]), int(m["dim"]), int(m["vdim"]), float(m["tau"]),
                               rank("a1", int(m["dim"])))
    raise ValueError(f"Gatosun: unknown mixer {kind!r}")


def _mlp_spec(d: Optional[Dict[str, Any]]):
    if d is None:
        return None
    if d["kind"] == "dense":
        return DenseSpec(int(d["ff"]), "gelu_tanh", bias=True)
    if d["kind"] != "moe":
        raise ValueError(f"Gatosun: unknown feed-forward {d['kind']!r}")
    r = d["router"]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    shared = d.get("shared")
    spec = MoESpec(int(r["experts"]), int(r["top"]), ExpertSpec(int(d["expert"]["ff"]), EXPERT_ACT),
                   ExpertSpec(int(shared["ff"]), EXPERT_ACT) if shared else None, "sigmoid", renormalize=False,
                   n_group=int(groups["count"]), topk_group=int(groups["keep"]), correction=True)
    if spec.num_experts % spec.n_group or spec.top_k > spec.num_experts // spec.n_group * spec.topk_group:
        raise ValueError(f"Gatosun: inconsistent router {r}")
    return spec


def read_config(d: Dict[str, Any], dtype=None, path: Optional[str] = None) -> ModelConfig:
    """``ModelConfig`` from the design's own config.json keys.  The ranks of the low-rank decays stand in no
    key: they are the rows of the checkpoint's tensors (without a checkpoint, the head size)."""
    from .utils import safetensors_shapes
    shapes = safetensors_shapes(path) if path else {}

    def layer(i: int, x: Dict[str, Any]) -> LayerSpec:
        return LayerSpec(_mixer_spec(x["type"], x["mixer"], lambda name, other: shapes.get(
            f"l{i}.mix.{name}", (other,))[0]), _mlp_spec(x.get("mlp")))

    specs = tuple(layer(i, x) for i, x in enumerate(d["layers"]))
    mixing = [s.attention for s in specs if isinstance(s.attention, AttentionSpec) and s.attention.value_mix]
    if len({a.num_kv_heads * a.v_head_dim for a in mixing}) > 1:
        raise ValueError("Gatosun: layers that blend their values differ in the values' sizes")
    first = specs[0].attention.left if isinstance(specs[0].attention, ParallelSpec) else specs[0].attention
    moes = [s.mlp for s in specs if isinstance(s.mlp, MoESpec)]
    return ModelConfig(
        architecture="Gatosun", model_type="gatosun", hidden_size=int(d["width"]), num_layers=len(specs),
        num_heads=first.num_heads, num_kv_heads=getattr(first, "num_kv_heads", first.num_heads),
        head_dim=first.head_dim, v_head_dim=first.v_head_dim, vocab_size=int(d["vocab"]),
        rms_norm_eps=float(d["norm"]["eps"]), max_position_embeddings=1 << 20, dtype=to_dtype(dtype or "bfloat16"),
        layer_specs=specs, residual_mult=float(d["residual_mult"]),
        num_experts=max((m.num_experts for m in moes), default=0),
        num_experts_per_tok=max((m.top_k for m in moes), default=0), hf_config=d)


# --------------------------------------------------------------------- mixers
def _attention_core(self: Mixer, cfg: ModelConfig, s: AttentionSpec, cache_idx: int, device, max_position: int):
    heads, kv = self.share(s.num_heads), self.share(s.num_kv_heads, "key/value heads")
    self.rotary = get_rope(s.head_dim, s.rotary_dim, max_position, s.rope_theta, s.rope_neox, None, device,
                           exact_angles=True)
    self.attn = NormedGQAAttention(cache_idx, heads, kv, s.head_dim, s.v_head_dim, s.scale, s.rotary_dim, s.qk_norm,
                                   cfg.rms_norm_eps, cfg.dtype, device, s.sliding_window, self.group)
    return {"q": (s.num_heads * s.head_dim, True), "k": (s.num_kv_heads * s.head_dim, True),
            "v": (s.num_kv_heads * s.v_head_dim, True)}


class AttentionMixer(Mixer):
    """``first_values``: whether other layers blend their values with this one's; ``blends``: whether this one does."""

    def __init__(self, cfg: ModelConfig, s: AttentionSpec, cache_idx: int, device, prefix: str, max_position: int,
                 first_values: bool, blends: bool) -> None:
        super().__init__(cfg)
        self.spec, self.first_values, self.blends = s, first_values, blends
        segments = _attention_core(self, cfg, s, cache_idx, device, max_position)
        self.in_proj = SegmentedLinear(self.padded_width, segments, bias=s.bias, dtype=cfg.dtype, device=device,
                                       prefix=f"{prefix}.in_proj")
        self.output_proj(cfg, [self.attn.num_heads * s.v_head_dim], device, prefix, bias=s.bias)
        self.vmix = nn.Parameter(torch.zeros((), dtype=torch.float32, device=device), requires_grad=False)

    def forward(self, h: torch.Tensor, run: int, shared: Dict[str, torch.Tensor]) -> torch.Tensor:
        y = self.in_proj(h)
        q, k, v = (self.in_proj.segment(y, x) for x in ("q", "k", "v"))
        if self.first_values:
            shared["v"] = v
        o = self.attn(q, k, v, self.rotary.cos_sin_cache, self.o_proj.in_local, shared["v"] if self.blends else None)
        return self.o_proj(o)

    def expect(self, want: Want, p: str) -> None:
        self.expect_rows(want, p, self.in_proj)
        self.expect_output(want, p + "o", 0)
        if self.o_proj.bias is not None:
            want[p + "o.b"] = (self.width,), lambda t: self.o_proj.bias.data.copy_(fit(t, self.padded_width))
        if self.attn.norm == "projection":
            self.expect_vector(want, p + "q.norm", self.attn.q_norm, True)
            self.expect_vector(want, p + "k.norm", self.attn.k_norm, True)
        if self.spec.value_mix:
            want[p + "vmix"] = (), lambda t: self.vmix.data.copy_(t)

    def clear_padding(self) -> None:
        super().clear_padding()
        self.clear(self.in_proj, self.width)
        self.attn.value_mix = float(self.vmix)


class ParallelMixer(Mixer):
    def __init__(self, cfg: ModelConfig, s: ParallelSpec, cache_idx: int, device, prefix: str, max_position: int) -> None:
        super().__init__(cfg)
        self.spec = s
        segments = _attention_core(self, cfg, s.left, cache_idx, device, max_position)
        self.in_proj = SegmentedLinear(self.padded_width, segments, dtype=cfg.dtype, device=device,
                                       prefix=f"{prefix}.in_proj")
        heads, d = self.share(s.right.num_heads), s.right.head_dim
        self.mix_rows = heads * d
        self.time = TimeMixAttention(heads, d, self.padded_width, cfg.rms_norm_eps, cfg.dtype, device)

        def param(*shape):
            return nn.Parameter(torch.zeros(*shape, dtype=cfg.dtype, device=device), requires_grad=False)

        # r, k, v and the gate read different blends: one grouped product
        self.rkvg = param(4, pad8(self.mix_rows), self.padded_width)
        self.w1 = param(pad8(s.right.decay_rank), self.padded_width)
        self.low_proj = SegmentedLinear(pad8(s.right.decay_rank), {"z": (s.right.num_heads * d, True)}, dtype=cfg.dtype,
                                        device=device, prefix=f"{prefix}.low_proj")
        self.output_proj(cfg, [self.attn.num_heads * s.left.v_head_dim, self.mix_rows], device, prefix)
        # left_scale * L + right_scale * R = out_scale * (L + right * R); without a left half R alone
        self.out_scale, self.right = (s.left_scale, s.right_scale / s.left_scale) if s.left_scale else (s.right_scale, 1.0)

    def _left(self, h: torch.Tensor, out: torch.Tensor) -> None:
        y = self.in_proj(h)
        q, k, v = (self.in_proj.segment(y, x) for x in ("q", "k", "v"))
        self.attn(q, k, v, self.rotary.cos_sin_cache, out=out)

    def _right(self, h: torch.Tensor, run: int, out: torch.Tensor) -> None:
        t, n = h.shape[0], self.mix_rows
        rows, offsets = self.time.blend(h, run)
        if h.is_cuda and t >= ops.PAIR_MIN_M > 0 and h.dtype == torch.bfloat16:      # large enough for CTA pairs
            r, k, v, g = (ops.gemm(rows[i * t: (i + 1) * t], self.rkvg[i])[:, :n] for i in range(4))
        else:
            r, k, v, g = ops.grouped_gemm(rows[: 4 * t], self.rkvg, offsets[:5])[:, :n].split(t)
        z = self.low_proj(ops.gemm(rows[4 * t:], self.w1, unary="tanh"), out_dtype=torch.float32)
        self.time(r, k, v, z, g, run, self.right, out)

    def forward(self, h: torch.Tensor, run: int, shared: Dict[str, torch.Tensor]) -> torch.Tensor:
        t, cut = h.shape[0], self.starts[1]
        both = h.new_empty(t, self.o_proj.in_local)
        left, right = both[:, : self.parts[0]], both[:, cut:]
        if self.parts[0] < cut:
            both[:, self.parts[0]: cut].zero_()
        if not h.is_cuda or t > OVERLAP_ROWS:
            self._left(h, left)
            self._right(h, run, right)
        else:
            cur, side = torch.cuda.current_stream(h.device), _side_stream(h.device)
            side.wait_stream(cur)
            with torch.cuda.stream(side):
                self._left(h, left)
            self._right(h, run, right)
            cur.wait_stream(side)
        return self.o_proj(both)

    def expect(self, want: Want, p: str) -> None:
        a, w, d = self.time, self.width, self.spec.right.head_dim
        n, heads = self.mix_rows * self.tp, self.spec.right.num_heads
        self.expect_rows(want, p + "left.", self.in_proj)
        self.expect_output(want, p + "left.o", 0)
        p += "right."
        self.expect_output(want, p + "o", 1)
        for i, s in enumerate(a.BLENDS):
            want[f"{p}mu.{s}"] = (w,), lambda t, i=i: a.mu.data[i].copy_(fit(t, self.padded_width))
            if i < 4:
                want[p + s] = (n, w), lambda t, i=i: self.rkvg.data[i, : self.mix_rows, :w].copy_(self.own(t))
        rank = self.spec.right.decay_rank
        want[p + "w1"] = (rank, w), lambda t: self.w1.data[:rank, :w].copy_(t)
        self.expect_low(want, p + "w2", self.low_proj, rank)
        self.expect_vector(want, p + "w0", a.w0, True)
        self.expect_vector(want, p + "u", a.u, True)
        self.expect_vector(want, p + "norm", a.out_norm, True, (heads * d,))

    @torch.no_grad()
    def clear_padding(self) -> None:
        super().clear_padding()
        w, rank = self.width, self.spec.right.decay_rank
        self.clear(self.in_proj, w)
        self.clear(self.low_proj, rank)
        self.rkvg.data[:, self.mix_rows:] = 0
        self.rkvg.data[..., w:] = 0
        self.w1.data[rank:] = 0
        self.w1.data[:, w:] = 0
        self.time.mu.data[:, w:] = 0
        if not self.spec.left_scale:
            self.o_proj.weight.data[:, : self.starts[1]] = 0


class DecayLinearMixer(Mixer):
    def __init__(self, cfg: ModelConfig, s: DecayLinearSpec, device, prefix: str) -> None:
        super().__init__(cfg)
        self.spec = s
        n, e = s.num_heads * s.head_dim, s.num_heads * s.v_head_dim
        heads = self.share(s.num_heads)
        self.in_proj = SegmentedLinear(self.padded_width, {"q": (n, True), "k": (n, True), "v": (e, True), "g": (e, True),
                                                           "a1": (s.decay_rank, False)},
                                       dtype=cfg.dtype, device=device, prefix=f"{prefix}.in_proj")
        self.low_proj = SegmentedLinear(pad8(s.decay_rank), {"z": (n, True)}, dtype=cfg.dtype, device=device,
                                        prefix=f"{prefix}.low_proj")
        self.attn = DecayLinearAttention(heads, s.head_dim, s.v_head_dim, s.tau, cfg.rms_norm_eps, cfg.dtype, device)
        self.output_proj(cfg, [heads * s.v_head_dim], device, prefix)

    def forward(self, h: torch.Tensor, run: int, shared: Dict[str, torch.Tensor]) -> torch.Tensor:
        y = self.in_proj(h)
        q, k, v, g = (self.in_proj.segment(y, x) for x in ("q", "k", "v", "g"))
        a = self.in_proj.offsets["a1"]
        z = self.low_proj(y[:, a: a + self.low_proj.in_features], out_dtype=torch.float32)
        return self.o_proj(self.attn(q, k, v, z, g, run, self.o_proj.in_local))

    def expect(self, want: Want, p: str) -> None:
        self.expect_rows(want, p, self.in_proj)
        self.expect_output(want, p + "o", 0)
        self.expect_low(want, p + "a2", self.low_proj, self.spec.decay_rank)
        self.expect_vector(want, p + "a2.b", self.attn.decay_bias, True)
        self.expect_vector(want, p + "norm", self.attn.out_norm, False)

    def clear_padding(self) -> None:
        super().clear_padding()
        self.clear(self.in_proj, self.width)
        self.clear(self.low_proj, self.spec.decay_rank)


_SIDE_STREAMS: Dict[torch.device, torch.cuda.Stream] = {}


def _side_stream(device: torch.device) -> torch.cuda.Stream:
    if device not in _SIDE_STREAMS:
        _SIDE_STREAMS[device] = torch.cuda.Stream(device)
    return _SIDE_STREAMS[device]


# --------------------------------------------------------------------- the model
class GatosunLayer(nn.Module):
    def __init__(self, engine: EngineConfig, idx: int, cache_idx: int, first_mixing: int, device) -> None:
        super().__init__()
        cfg, spec = engine.model, engine.model.layer_specs[idx]
        self.spec = spec
        w, prefix, positions = pad8(cfg.hidden_size), f"layers.{idx}", engine.scheduler.max_model_len

        def gain():
            return nn.Parameter(torch.zeros(w, dtype=cfg.dtype, device=device), requires_grad=False)

        self.norm1 = gain()
        self.norm2 = gain() if spec.mlp is not None else None
        a, m = spec.attention, spec.mlp
        if isinstance(a, AttentionSpec):
            self.mix = AttentionMixer(cfg, a, cache_idx, device, f"{prefix}.mix", positions, idx == first_mixing,
                                      a.value_mix and idx != first_mixing)
        elif isinstance(a, ParallelSpec):
            self.mix = ParallelMixer(cfg, a, cache_idx, device, f"{prefix}.mix", positions)
        else:
            self.mix = DecayLinearMixer(cfg, a, device, f"{prefix}.mix")
        self.mlp = None
        if isinstance(m, DenseSpec):
            tp = self.mix.tp
            ff = (m.intermediate_size + 8 * tp - 1) // (8 * tp) * 8 * tp
            self.mlp = FusedMLP(w, ff, cfg.dtype, device, prefix=f"{prefix}.mlp", act=m.act, bias=m.bias)
        elif m is not None:
            par = engine.parallel
            self.mlp = FusedMoE(
                m.num_experts, m.top_k, w, pad8(m.expert.intermediate_size), cfg.dtype, device, m.scoring_func,
                m.renormalize, m.scale, m.n_group, m.topk_group, router_bias=m.correction,
                num_shared_experts=1 if m.shared else 0,
                shared_intermediate_size=pad8(m.shared.intermediate_size) if m.shared else None,
                enable_expert_parallel=par.enable_expert_parallel or par.tensor_parallel_size > 1,
                prefix=f"{prefix}.mlp", unary=m.expert.act,
                max_tokens=max(engine.scheduler.max_num_batched_tokens, engine.scheduler.max_num_seqs),
                num_redundant_experts=par.num_redundant_experts)

    def feed_forward(self, h: torch.Tensor):
        """(dense, routed or None), the feed-forward's share of the residual."""
        if isinstance(self.mlp, FusedMoE):
            routed, dense = self.mlp.forward_deferred(h)
            return dense, routed
        return self.mlp(h), None


class GatosunForCausalLM(nn.Module):
    has_recurrent_state = True

    def __init__(self, engine_config: EngineConfig, device=None) -> None:
        super().__init__()
        cfg = self.config = engine_config.model
        self.width, self.padded_width = cfg.hidden_size, pad8(cfg.hidden_size)
        self.embed = VocabParallelEmbedding(cfg.vocab_size, self.padded_width, cfg.dtype, device)
        self.head = ParallelLMHead(cfg.vocab_size, self.padded_width, cfg.dtype, device)
        mixing = [i for i, s in enumerate(cfg.layer_specs)
                  if isinstance(s.attention, AttentionSpec) and s.attention.value_mix]
        layers, caches = [], 0
        for i, s in enumerate(cfg.layer_specs):
            layers.append(GatosunLayer(engine_config, i, caches, mixing[0] if mixing else -1, device))
            caches += isinstance(s.attention, (AttentionSpec, ParallelSpec))
        self.layers = nn.ModuleList(layers)
        self.final_norm = nn.Parameter(torch.zeros(self.padded_width, dtype=cfg.dtype, device=device), requires_grad=False)
        self.num_kv_layers = caches

    # ------------------------------------------------------------------ cache and state
    def _cache_shapes(self, block_size: int) -> List[Tuple[Tuple[int, ...], Tuple[int, ...]]]:
        out = []
        for layer in self.layers:
            if isinstance(layer.mix, DecayLinearMixer):
                continue
            a = layer.mix.attn
            dk, dv = a.cache_widths(self.config.dtype)
            out.append(((a.num_kv_heads, block_size, dk), (a.num_kv_heads, block_size, dv)))
        return out

    def get_kv_cache_spec(self, block_size: int):
        from ..worker.model_runner import KVCacheSpec
        shapes = self._cache_shapes(block_size)
        elems = sum(k[0] * k[1] * (k[2] + v[2]) for k, v in shapes)
        k, v = shapes[0] if shapes else ((), ())
        return KVCacheSpec("gqa", len(shapes), block_size, max(1, elems * self.config.dtype.itemsize), {"k": k, "v": v})

    def allocate_kv_cache(self, num_blocks: int, block_size: int, device):
        # zeros: the padding of the rows stays as it is here
        return [tuple(torch.zeros(num_blocks, *s, dtype=self.config.dtype, device=device) for s in kv)
                for kv in self._cache_shapes(block_size)]

    def allocate_states(self, num_slots: int, device) -> List[Dict[str, torch.Tensor]]:
        """Per layer: the state of its recurrent half (none for attention)."""
        out = []
        for layer in self.layers:
            m = layer.mix
            core = m.time if isinstance(m, ParallelMixer) else m.attn if isinstance(m, DecayLinearMixer) else None
            shapes = core.state_shapes() if core is not None else {}
            out.append({k: torch.zeros(num_slots, *s, dtype=dt, device=device) for k, (s, dt) in shapes.items()})
        return out

    # ---------------------------------------------------------------- forward
    def forward(self, input_ids, positions, inputs_embeds=None, intermediate_tensors=None):
        cfg = self.config
        norm = dict(eps=cfg.rms_norm_eps, weight_offset=0.0, true_width=self.width)
        ids, table = input_ids, self.embed.weight
        if inputs_embeds is not None or self.embed.group.world_size > 1:
            table = inputs_embeds if inputs_embeds is not None else self.embed(input_ids)
            ids = torch.arange(table.shape[0], dtype=torch.int32, device=table.device)
        x = torch.empty(ids.shape[0], self.padded_width, dtype=torch.float32, device=table.device)
        h = ops.embed_residual_norm(x, ids, table, 1.0, self.layers[0].norm1, **norm)
        shared: Dict[str, torch.Tensor] = {}
        trace = self.__dict__.get("layer_outputs")       # hook for tests and debugging: a list
        for i, layer in enumerate(self.layers):
            after = self.layers[i + 1].norm1 if i + 1 < len(self.layers) else self.final_norm
            y, mult = layer.mix(h, i, shared), cfg.residual_mult * layer.mix.out_scale
            if layer.mlp is not None:
                h = ops.residual_add_norm(x, y, None, None, layer.norm2, mult=mult, **norm)
                (y, routed), mult = layer.feed_forward(h), cfg.residual_mult
            else:
                routed = None
            h = ops.residual_add_norm(x, y, None, routed, after, mult=mult, **norm)
            if trace is not None:
                trace.append(x[:, : self.width].clone())
        return h

    def compute_logits(self, hidden: torch.Tensor) -> torch.Tensor:
        return self.head.compute_logits(hidden)

    # ---------------------------------------------------------------- weights
    def load_weights(self, weights: Iterable[Tuple[str, torch.Tensor]]) -> set:
        """Place the checkpoint's tensors (padded with zeros where the parameters are wider).  Unknown names,
        wrong shapes and missing tensors are errors; a norm of a feed-forward that a layer does not have,
        and a blend factor of one that does not blend, are not used."""
        idle = {f"l{i}.norm2" for i, layer in enumerate(self.layers) if layer.mlp is None}
        idle |= {f"l{i}.mix.vmix" for i, layer in enumerate(self.layers) if isinstance(layer.mix, AttentionMixer)}
        return place_tensors(weights, self._expected(), "Gatosun", idle.__contains__)

    def _expected(self) -> Want:
        w, wp, vocab = self.width, self.padded_width, self.config.vocab_size
        want: Want = {}

        def rows(module, n: int, shard=None):
            return (n, w), lambda t: module.weight_loader(module.weight, fit(t, n, wp), shard)

        def norm(name: str, param: nn.Parameter) -> None:
            want[name] = (w,), lambda t: param.data.copy_(fit(t, wp))

        want["embed"], want["head"] = rows(self.embed, vocab), rows(self.head, vocab)
        norm("final.norm", self.final_norm)
        for i, layer in enumerate(self.layers):
            p = f"l{i}."
            norm(p + "norm1", layer.norm1)
            layer.mix.expect(want, p + "mix.")
            if layer.mlp is None:
                continue
            norm(p + "norm2", layer.norm2)
            m = layer.spec.mlp
            (self._expect_dense if isinstance(m, DenseSpec) else self._expect_moe)(want, p + "mlp.", layer.mlp, m)
        return want

    def _expect_dense(self, want: Want, p: str, mlp: FusedMLP, m: DenseSpec) -> None:
        w, wp, ff, gu, down = self.width, self.padded_width, m.intermediate_size, mlp.gate_up_proj, mlp.down_proj
        full = gu.output_sizes[0]
        for j, name in enumerate(("gate", "up")):
            want[p + name] = (ff, w), lambda t, j=j: gu.weight_loader(gu.weight, fit(t, full, wp), j)
            if m.bias:
                want[f"{p}{name}.b"] = (ff,), lambda t, j=j: gu.weight_loader(gu.bias, fit(t, full), j)
        want[p + "down"] = (w, ff), lambda t: down.weight_loader(down.weight, fit(t, wp, full))
        if m.bias:
            want[p + "down.b"] = (w,), lambda t: down.weight_loader(down.bias, fit(t, wp))

    def _expect_moe(self, want: Want, p: str, moe: FusedMoE, m: MoESpec) -> None:
        w, wp = self.width, self.padded_width
        want[p + "router"] = (m.num_experts, w), lambda t: moe.gate.weight_loader(moe.gate.weight, fit(t, t.shape[0], wp))
        want[p + "correction"] = (m.num_experts,), lambda t: moe.e_score_correction_bias.data.copy_(t)

        def expert(prefix: str, ff: int, up, down) -> None:
            fp = pad8(ff)
            want[prefix + "up"] = (ff, w), lambda t: up(fit(t, fp, wp))
            want[prefix + "down"] = (w, ff), lambda t: down(fit(t, wp, fp))

        for e in range(m.num_experts):
            expert(f"{p}e{e}.", m.expert.intermediate_size, lambda t, e=e: moe.weight_loader(moe.w13, t, e, "up"),
                   lambda t, e=e: moe.weight_loader(moe.w2, t, e, "down"))
        if m.shared:
            sh = moe.shared_experts
            expert(p + "shared.", m.shared.intermediate_size, lambda t: sh.up_proj.weight_loader(sh.up_proj.weight, t),
                   lambda t: sh.down_proj.weight_loader(sh.down_proj.weight, t))

    @torch.no_grad()
    def post_load(self) -> None:
        """Host constants, and zeros in the padding whatever filled the parameters (random initialisation
        does)."""
        w = self.width
        for p in (self.embed.weight, self.head.weight):
            p.data[:, w:] = 0
        self.final_norm.data[w:] = 0
        for layer in self.layers:
            layer.norm1.data[w:] = 0
            layer.mix.clear_padding()
            m, mlp = layer.spec.mlp, layer.mlp
            if mlp is None:
                continue
            layer.norm2.data[w:] = 0
            if isinstance(m, DenseSpec):
                mlp.gate_up_proj.weight.data[:, w:] = 0
                mlp.down_proj.weight.data[w:] = 0
                if m.bias:
                    mlp.down_proj.bias.data[w:] = 0
                if mlp.down_proj.tp_size == 1:
                    mlp.down_proj.weight.data[:, m.intermediate_size:] = 0
                continue
            moe, ff = mlp, m.expert.intermediate_size
            moe.gate.weight.data[:, w:] = 0
            moe.w13.data[..., w:] = 0
            moe.w2.data[:, w:] = 0
            moe.w2.data[..., ff:] = 0
            if m.shared:
                moe.shared_experts.up_proj.weight.data[:, w:] = 0
                moe.shared_experts.down_proj.weight.data[w:] = 0
                moe.shared_experts.down_proj.weight.data[:, m.shared.intermediate_size:] = 0
