"""Rivudra: a decoder whose layers run attention and feed-forward side by side on one norm.

    h = norm(x);  x <- x + (mixer(h) + ff(h))

The residual x is fp32; norms store their weight around zero.  The mixer is grouped-query attention with
interleaved partial rotation, a sliding window, a sink of score 0 in every softmax and an element-wise
output gate; the feed-forward is a mixture of clamped gated experts with group-limited softmax routing
and an optional shared expert (or absent).  Sizes and constants are given layer by layer.

Per layer and step: one projection for q, k, v and the gate; rotation + cache write; attention with the
gate in its epilogue; output projection; router, dispatch and two grouped products for the experts.  The
residual kernel then gathers the experts' rows, adds both sublayers to x and applies the NEXT layer's norm
in one pass (``ops.residual_add_norm``), so neither sublayer sum nor combined expert output is written.

Widths that are not whole 16-byte rows are padded with zeros when the weights are loaded; the norms
divide by the true width.
"""
from __future__ import annotations

import os
import re
from typing import Any, Dict, Iterable, List, Optional, Tuple

import torch
from torch import nn

from .. import ops
from ..attention.gqa import GatedGQAAttention
from ..config import AttentionSpec, EngineConfig, ExpertSpec, LayerSpec, ModelConfig, MoESpec, to_dtype
from ..layers.embedding import ParallelLMHead, VocabParallelEmbedding
from ..layers.linear import GatedQKVParallelLinear, RowParallelLinear
from ..layers.moe import FusedMoE
from ..layers.rope import get_rope
from ..parallel import state as pstate
from .utils import IntermediateTensors, PPMissingLayer, build_pipeline_layers

# Steps of at most this many rows run the two sublayers on two streams: each leaves most of the GPU idle
# there, and neither needs the other's result.
OVERLAP_ROWS = int(os.environ.get("OMNI_B200_PARALLEL_SUBLAYER_ROWS", "256"))
SIGMOID_SLOPE = 1.702          # of the experts' gate
SINK_SCORE = 0.0
NORM_WEIGHT_OFFSET = 1.0


# --------------------------------------------------------------------- configuration
def _expert_spec(d: Dict[str, Any]) -> ExpertSpec:
    return ExpertSpec(int(d["ff"]), (SIGMOID_SLOPE, float(d["limit"])))


def _layer_spec(d: Dict[str, Any]) -> LayerSpec:
    if d["type"] != "attention":
        raise ValueError(f"Rivudra: unknown mixer {d['type']!r}")
    m = d["mixer"]
    attn = AttentionSpec(num_heads=int(m["heads"]), num_kv_heads=int(m["kv_heads"]), head_dim=int(m["dim"]),
                         v_head_dim=int(m["vdim"]), rotary_dim=int(m["rot"]["dims"]),
                         rope_theta=float(m["rot"]["base"]), scale=float(m["scale"]), rope_neox=False,
                         sliding_window=int(m["mask"]["size"]), sink=SINK_SCORE, output_gate=True)
    if attn.num_heads % attn.num_kv_heads or attn.rotary_dim % 2 or attn.rotary_dim > attn.head_dim \
            or attn.sliding_window < 1:
        raise ValueError(f"Rivudra: inconsistent attention sizes {m}")
    mlp = d.get("mlp")
    if mlp is None:
        return LayerSpec(attn, None)
    if mlp.get("kind", "moe") != "moe":
        raise ValueError(f"Rivudra: unknown feed-forward {mlp['kind']!r}")
    r = mlp["router"]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    moe = MoESpec(num_experts=int(r["experts"]), top_k=int(r["top"]), expert=_expert_spec(mlp["expert"]),
                  shared=_expert_spec(mlp["shared"]) if mlp.get("shared") else None, scoring_func="softmax",
                  renormalize=True, scale=float(r["scale"]), n_group=int(groups["count"]),
                  topk_group=int(groups["keep"]))
    if moe.num_experts % moe.n_group or moe.top_k > moe.num_experts // moe.n_group * moe.topk_group:
        raise ValueError(f"Rivudra: inconsistent router {r}")
    return LayerSpec(attn, moe)


def read_config(d: Dict[str, Any], dtype=None, path: Optional[str] = None) -> ModelConfig:
    """``ModelConfig`` from the design's own config.json keys."""
    specs = tuple(_layer_spec(x) for x in d["layers"])
    first = specs[0].attention
    moes = [s.mlp for s in specs if s.mlp is not None]
    return ModelConfig(
        architecture="Rivudra", model_type="rivudra", hidden_size=int(d["width"]), num_layers=len(specs),
        num_heads=first.num_heads, num_kv_heads=first.num_kv_heads, head_dim=first.head_dim,
        v_head_dim=first.v_head_dim, rope_theta=first.rope_theta, rope_neox=False,
        sliding_window=first.sliding_window, vocab_size=int(d["vocab"]),
        rms_norm_eps=float(d["norm"]["eps"]), max_position_embeddings=1 << 20,
        dtype=to_dtype(dtype or "bfloat16"), layer_specs=specs, embedding_scale=float(d["embedding"]["scale"]),
        norm_weight_offset=NORM_WEIGHT_OFFSET, num_experts=max((m.num_experts for m in moes), default=0),
        num_experts_per_tok=max((m.top_k for m in moes), default=0), hf_config=d)


def _pad8(n: int) -> int:
    return (n + 7) // 8 * 8


def _fit(t: torch.Tensor, *shape: int) -> torch.Tensor:
    """``t`` with zeros appended up to ``shape``."""
    if tuple(t.shape) == shape:
        return t
    out = t.new_zeros(shape)
    out[tuple(slice(0, n) for n in t.shape)] = t
    return out


# --------------------------------------------------------------------- layers
class RivudraMixer(nn.Module):
    def __init__(self, cfg: ModelConfig, spec: AttentionSpec, layer_idx: int, device, prefix: str,
                 max_position: int) -> None:
        super().__init__()
        self.spec = spec
        width = _pad8(cfg.hidden_size)
        self.qkvg_proj = GatedQKVParallelLinear(width, spec.head_dim, spec.num_heads, spec.num_kv_heads,
                                                head_dim_v=spec.v_head_dim, output_gate=spec.output_gate,
                                                dtype=cfg.dtype, device=device, prefix=f"{prefix}.qkvg_proj")
        tp = self.qkvg_proj.tp_size
        out = spec.num_heads * spec.v_head_dim
        if tp > 1 and (out // tp) % 8:
            raise ValueError(f"Rivudra: {out // tp} value columns per rank are not whole 16-byte rows")
        self.o_proj = RowParallelLinear(out if tp > 1 else _pad8(out), width, dtype=cfg.dtype, device=device,
                                        prefix=f"{prefix}.o_proj")
        self.rotary = get_rope(spec.head_dim, spec.rotary_dim, max_position, spec.rope_theta, spec.rope_neox,
                               None, device, exact_angles=True)
        self.attn = GatedGQAAttention(layer_idx, self.qkvg_proj.num_heads, self.qkvg_proj.num_kv_heads,
                                      spec.head_dim, spec.v_head_dim, spec.scale, spec.rotary_dim, spec.rope_neox,
                                      spec.sliding_window, spec.sink)

    def forward(self, hidden: torch.Tensor) -> torch.Tensor:
        q, k, v, g = self.qkvg_proj(hidden)
        return self.o_proj(self.attn(q, k, v, g, self.rotary.cos_sin_cache, self.o_proj.in_local))


_SIDE_STREAMS: Dict[torch.device, torch.cuda.Stream] = {}


def _side_stream(device: torch.device) -> torch.cuda.Stream:
    if device not in _SIDE_STREAMS:
        _SIDE_STREAMS[device] = torch.cuda.Stream(device)
    return _SIDE_STREAMS[device]


class RivudraLayer(nn.Module):
    def __init__(self, engine: EngineConfig, spec: LayerSpec, layer_idx: int, device) -> None:
        super().__init__()
        cfg = engine.model
        self.spec = spec
        width = _pad8(cfg.hidden_size)
        self.input_gain = nn.Parameter(torch.zeros(width, dtype=cfg.dtype, device=device), requires_grad=False)
        self.mix = RivudraMixer(cfg, spec.attention, layer_idx, device, f"layers.{layer_idx}.mix",
                                engine.scheduler.max_model_len)
        self.mlp = None
        m = spec.mlp
        if m is not None:
            ff = _pad8(m.expert.intermediate_size)
            self.mlp = FusedMoE(
                m.num_experts, m.top_k, width, ff, cfg.dtype, device, m.scoring_func, m.renormalize, m.scale,
                m.n_group, m.topk_group, num_shared_experts=1 if m.shared else 0,
                shared_intermediate_size=_pad8(m.shared.intermediate_size) if m.shared else None,
                enable_expert_parallel=engine.parallel.enable_expert_parallel
                or engine.parallel.tensor_parallel_size > 1, prefix=f"layers.{layer_idx}.mlp",
                max_tokens=max(engine.scheduler.max_num_batched_tokens, engine.scheduler.max_num_seqs),
                num_redundant_experts=engine.parallel.num_redundant_experts, act=m.expert.act,
                shared_act=m.shared.act if m.shared else None)

    def forward(self, hidden: torch.Tensor):
        """The layer's share of the residual from its normed input: (dense, dense or None, routed or None)."""
        if self.mlp is None:
            return self.mix(hidden), None, None
        if not hidden.is_cuda or hidden.shape[0] > OVERLAP_ROWS or self.mix.qkvg_proj.tp_size > 1:
            routed, dense = self.mlp.forward_deferred(hidden)
            return self.mix(hidden), dense, routed
        cur, side = torch.cuda.current_stream(hidden.device), _side_stream(hidden.device)
        side.wait_stream(cur)
        with torch.cuda.stream(side):
            mixed = self.mix(hidden)
        routed, dense = self.mlp.forward_deferred(hidden)
        cur.wait_stream(side)
        return mixed, dense, routed


class RivudraForCausalLM(nn.Module):
    def __init__(self, engine_config: EngineConfig, device=None) -> None:
        super().__init__()
        cfg = self.config = engine_config.model
        self.width, self.padded_width = cfg.hidden_size, _pad8(cfg.hidden_size)
        pp = pstate.get_pp_group()
        self.pp_group = pp if pp.world_size > 1 else None
        self.first = self.pp_group is None or pp.is_first_rank
        self.last = self.pp_group is None or pp.is_last_rank
        self.embed = VocabParallelEmbedding(cfg.vocab_size, self.padded_width, cfg.dtype, device) \
            if self.first else PPMissingLayer()
        self.layers, self.start_layer, self.end_layer = build_pipeline_layers(
            cfg.num_layers, lambda i: RivudraLayer(engine_config, cfg.layer_specs[i], i, device), self.pp_group)
        self.final_gain = nn.Parameter(torch.zeros(self.padded_width, dtype=cfg.dtype, device=device),
                                       requires_grad=False) if self.last else None
        self.head = ParallelLMHead(cfg.vocab_size, self.padded_width, cfg.dtype, device) \
            if self.last else PPMissingLayer()
        self.stage: List[RivudraLayer] = list(self.layers)[self.start_layer:self.end_layer]
        self.num_kv_layers = len(self.stage)

    # ------------------------------------------------------------------ cache
    def _cache_shapes(self, block_size: int) -> List[Tuple[Tuple[int, ...], Tuple[int, ...]]]:
        out = []
        for layer in self.stage:
            a = layer.mix.attn
            dk, dv = a.cache_widths(self.config.dtype)
            out.append(((a.num_kv_heads, block_size, dk), (a.num_kv_heads, block_size, dv)))
        return out

    def get_kv_cache_spec(self, block_size: int):
        from ..worker.model_runner import KVCacheSpec
        shapes = self._cache_shapes(block_size)
        elems = sum(k[0] * k[1] * (k[2] + v[2]) for k, v in shapes)
        k, v = shapes[0] if shapes else ((), ())
        return KVCacheSpec("gqa", len(shapes), block_size, max(1, elems * self.config.dtype.itemsize),
                           {"k": k, "v": v})

    def allocate_kv_cache(self, num_blocks: int, block_size: int, device):
        # zeros: the padding of the rows stays as it is here
        return [(torch.zeros(num_blocks, *k, dtype=self.config.dtype, device=device),
                 torch.zeros(num_blocks, *v, dtype=self.config.dtype, device=device))
                for k, v in self._cache_shapes(block_size)]

    # ---------------------------------------------------------------- forward
    def _gain_after(self, i: int) -> Optional[torch.Tensor]:
        """Norm weight that follows layer ``i`` of this stage (None: the next stage applies it)."""
        return self.stage[i + 1].input_gain if i + 1 < len(self.stage) else self.final_gain

    def forward(self, input_ids, positions, inputs_embeds=None, intermediate_tensors=None):
        cfg = self.config
        norm = dict(eps=cfg.rms_norm_eps, weight_offset=cfg.norm_weight_offset, true_width=self.width)
        gain = self._gain_after(-1)
        hidden = None
        if self.first:
            t = input_ids.shape[0] if inputs_embeds is None else inputs_embeds.shape[0]
            residual = torch.empty(t, self.padded_width, dtype=torch.float32, device=self.embed.weight.device)
            ids, table = input_ids, self.embed.weight
            if inputs_embeds is not None or self.embed.group.world_size > 1:
                table = inputs_embeds if inputs_embeds is not None else self.embed(input_ids)
                ids = torch.arange(t, dtype=torch.int32, device=table.device)
            if gain is not None:
                hidden = ops.embed_residual_norm(residual, ids, table, cfg.embedding_scale, gain, **norm)
            else:                           # a stage without layers passes the embeddings on
                residual.copy_(table[ids.long()].float() * cfg.embedding_scale)
        else:
            residual = intermediate_tensors["residual"]
            if gain is not None:
                hidden = ops.residual_add_norm(residual, None, None, None, gain, **norm)
        for i, layer in enumerate(self.stage):
            a, b, routed = layer(hidden)
            hidden = ops.residual_add_norm(residual, a, b, routed, self._gain_after(i), **norm)
            self._trace(residual)
        if not self.last:
            return IntermediateTensors({"residual": residual})
        return hidden

    def _trace(self, residual: torch.Tensor) -> None:
        """Hook for tests and debugging: the residual stream after a layer (``layer_outputs`` a list)."""
        sink = self.__dict__.get("layer_outputs")
        if sink is not None:
            sink.append(residual[:, : self.width].clone())

    def make_empty_intermediate_tensors(self, num_tokens: int, dtype, device) -> IntermediateTensors:
        return IntermediateTensors({"residual": torch.empty(num_tokens, self.padded_width, dtype=torch.float32,
                                                            device=device)})

    def compute_logits(self, hidden: torch.Tensor) -> torch.Tensor:
        return self.head.compute_logits(hidden)

    # ---------------------------------------------------------------- weights
    def load_weights(self, weights: Iterable[Tuple[str, torch.Tensor]]) -> set:
        """Place the checkpoint's tensors (padded with zeros where the parameters are wider).  Unknown
        names, wrong shapes and missing tensors are errors."""
        want = self._expected()
        loaded = set()
        for name, t in weights:
            if name not in want:
                if self._elsewhere(name):
                    continue
                raise ValueError(f"Rivudra: unknown tensor {name!r}")
            shape, place = want[name]
            if tuple(t.shape) != shape:
                raise ValueError(f"Rivudra: tensor {name!r} is {tuple(t.shape)}, expected {shape}")
            place(t)
            loaded.add(name)
        missing = sorted(set(want) - loaded)
        if missing:
            raise ValueError(f"Rivudra: {len(missing)} tensors missing, first {missing[:3]}")
        return loaded

    def _elsewhere(self, name: str) -> bool:
        """Whether a tensor belongs to another pipeline stage."""
        m = re.match(r"l(\d+)\.", name)
        if m is not None:
            i = int(m.group(1))
            return i < self.config.num_layers and not self.start_layer <= i < self.end_layer
        return (name == "embed" and not self.first) or (name in ("head", "final.norm") and not self.last)

    def _expected(self) -> Dict[str, Tuple[Tuple[int, ...], Any]]:
        """Tensor name -> (shape in the checkpoint, function that puts it in its place)."""
        w, wp, vocab = self.width, self.padded_width, self.config.vocab_size
        want: Dict[str, Tuple[Tuple[int, ...], Any]] = {}

        def rows(module, n: int, shard=None):
            # a projection of the width: columns padded
            return (n, w), lambda t: module.weight_loader(module.weight, _fit(t, n, wp), shard)

        if self.first:
            want["embed"] = rows(self.embed, vocab)
        if self.last:
            want["head"] = rows(self.head, vocab)
            want["final.norm"] = (w,), lambda t: self.final_gain.data.copy_(_fit(t, wp))
        for i, layer in zip(range(self.start_layer, self.end_layer), self.stage):
            p = f"l{i}."
            want[p + "norm1"] = (w,), lambda t, layer=layer: layer.input_gain.data.copy_(_fit(t, wp))
            a, mix = layer.spec.attention, layer.mix
            qkvg = mix.qkvg_proj
            qkvg.weight.data[qkvg.used_rows:].zero_()
            want[p + "mix.q"] = rows(qkvg, a.num_heads * a.head_dim, "q")
            want[p + "mix.k"] = rows(qkvg, a.num_kv_heads * a.head_dim, "k")
            want[p + "mix.v"] = rows(qkvg, a.num_kv_heads * a.v_head_dim, "v")
            want[p + "mix.g"] = rows(qkvg, a.num_heads * a.v_head_dim, "g")
            want[p + "mix.o"] = (w, a.num_heads * a.v_head_dim), lambda t, o=mix.o_proj: o.weight_loader(
                o.weight, _fit(t, wp, o.in_features))
            m, moe = layer.spec.mlp, layer.mlp
            if m is None:
                continue
            p += "mlp."
            want[p + "router"] = rows(moe.gate, m.num_experts)
            for e in range(m.num_experts):
                self._expect_expert(want, f"{p}e{e}.", m.expert.intermediate_size, lambda t, shard, e=e, moe=moe:
                                    moe.weight_loader(moe.w2 if shard == "down" else moe.w13, t, e, shard))
            if m.shared:
                sh = moe.shared_experts
                self._expect_expert(want, p + "shared.", m.shared.intermediate_size, lambda t, shard, sh=sh:
                                    sh.down_proj.weight_loader(sh.down_proj.weight, t) if shard == "down" else
                                    sh.gate_up_proj.weight_loader(sh.gate_up_proj.weight, t, int(shard == "up")))
        return want

    def _expect_expert(self, want, prefix: str, ff: int, place) -> None:
        w, wp, fp = self.width, self.padded_width, _pad8(ff)
        for name in ("gate", "up"):
            want[prefix + name] = (ff, w), lambda t, name=name: place(_fit(t, fp, wp), name)
        want[prefix + "down"] = (w, ff), lambda t: place(_fit(t, wp, fp), "down")

    @torch.no_grad()
    def post_load(self) -> None:
        """Keep the padding at zero whatever filled the parameters (random initialisation does)."""
        w = self.width
        for layer in self.stage:
            a, mix, m, moe = layer.spec.attention, layer.mix, layer.spec.mlp, layer.mlp
            mix.qkvg_proj.weight.data[mix.qkvg_proj.used_rows:].zero_()
            mix.qkvg_proj.weight.data[:, w:].zero_()
            mix.o_proj.weight.data[w:].zero_()
            mix.o_proj.weight.data[:, mix.attn.num_heads * a.v_head_dim:].zero_()
            if m is None:
                continue
            moe.gate.weight.data[:, w:].zero_()
            moe.w13.data[..., w:].zero_()
            moe.w2.data[:, w:].zero_()
            moe.w2.data[..., m.expert.intermediate_size:].zero_()
            if m.shared:
                moe.shared_experts.gate_up_proj.weight.data[:, w:].zero_()
                moe.shared_experts.down_proj.weight.data[w:].zero_()
                moe.shared_experts.down_proj.weight.data[:, m.shared.intermediate_size:].zero_()
        for p in (self.embed, self.head):
            if hasattr(p, "weight"):
                p.weight.data[:, w:].zero_()
