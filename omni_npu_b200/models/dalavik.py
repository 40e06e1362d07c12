"""Dalavik: a decoder with norms on the sublayers' outputs only and a per-layer token input.

The residual x is fp32.  Each layer is a mixer, an optional feed-forward, and a gated row of a second token table,
all reading x itself:

    x <- x + norm1(mixer(x));  x <- x + norm2(ff(x));  x <- x + norm(proj(gelu(gate x) * e_layer[token]))

norm1, norm2 and the final norm treat a row in equal groups.  Mixers are

    latent_attention   attention over a cached latent, queries through a latent of their own; a layer may read
                       the rows that an earlier layer cached                             (attention/latent.py)
    attention          grouped-query attention without rotation whose heads mix their scores
                                                                                        (attention/gqa.py)

Embedding and head share one table.  Sizes and constants are given layer by layer.

Per layer and step: one product for the projections of x, the mixer's own kernels, one product back; norm, add
and the rounded copy of x for the next product in one kernel; two products of the feed-forward, its activation in the
first one's epilogue; two small products around the token row.

Widths that are not whole 16-byte rows are padded with zeros when the weights are loaded; the norms divide by the
true width.
"""
from __future__ import annotations

from typing import Any, Dict, Iterable, List, Optional, Tuple

import torch
from torch import nn

from .. import ops
from ..attention.gqa import MixedScoreAttention
from ..attention.latent import LatentAttention
from ..config import AttentionSpec, DenseSpec, EngineConfig, LatentAttentionSpec, LayerSpec, ModelConfig, to_dtype
from ..layers.embedding import ParallelLMHead
from ..layers.linear import SegmentedLinear
from ..layers.mlp import FusedMLP
from ..layers.rope import get_rope
from .layered import Mixer, Want, fit, pad8, place_tensors


# --------------------------------------------------------------------- configuration
def _mixer_spec(kind: str, m: Dict[str, Any]):
    if kind == "latent_attention":
        rot, source = int(m["rot_dim"]), m.get("kv_from")
        if rot % 2 or int(m["rot"].get("dims", rot)) != rot:
            raise ValueError(f"Dalavik: inconsistent rotation {m}")
        return LatentAttentionSpec(int(m["heads"]), int(m["dim"]), rot, int(m["vdim"]), int(m["kv_rank"]),
                                   float(m["rot"]["base"]), float(m["scale"]), rope_neox=False, q_rank=int(m["q_rank"]),
                                   kv_from=None if source is None else int(source))
    if kind == "attention":
        temp = m.get("q_temp")
        s = AttentionSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), 0, 0.0, float(m["scale"]),
                          qk_norm="head_weight", bias=True, softcap=float(m.get("softcap") or 0.0), distance_bias=True,
                          score_mix=True, head_sink=True,
                          query_temperature=(float(temp["coef"]), int(temp["every"])) if temp else None)
        if s.num_heads % s.num_kv_heads or (temp and s.query_temperature[1] != temp["every"]):
            raise ValueError(f"Dalavik: inconsistent attention sizes {m}")
        return s
    raise ValueError(f"Dalavik: unknown mixer {kind!r}")


def _mlp_spec(d: Optional[Dict[str, Any]]) -> Optional[DenseSpec]:
    if d is None:
        return None
    if d.get("kind", "dense") != "dense":
        raise ValueError(f"Dalavik: unknown feed-forward {d['kind']!r}")
    return DenseSpec(int(d["ff"]), ops.RELU)


def _check_shared_rows(specs: Tuple[LayerSpec, ...]) -> None:
    for i, s in enumerate(specs):
        a = s.attention
        if not isinstance(a, LatentAttentionSpec) or a.kv_from is None:
            continue
        src = specs[a.kv_from].attention if 0 <= a.kv_from < i else None
        if not isinstance(src, LatentAttentionSpec) or src.kv_from is not None:
            raise ValueError(f"Dalavik: layer {i} reads the rows of layer {a.kv_from}, which caches none before it")
        if (src.kv_rank, src.rope_dim, src.rope_theta) != (a.kv_rank, a.rope_dim, a.rope_theta):
            raise ValueError(f"Dalavik: layers {a.kv_from} and {i} share rows of different shapes")


def read_config(d: Dict[str, Any], dtype=None, path: Optional[str] = None) -> ModelConfig:
    """``ModelConfig`` from the design's own config.json keys."""
    specs = tuple(LayerSpec(_mixer_spec(x["type"], x["mixer"]), _mlp_spec(x.get("mlp"))) for x in d["layers"])
    _check_shared_rows(specs)
    width, groups = int(d["width"]), int(d["norm"].get("groups", 1))
    if groups < 1 or width % groups:
        raise ValueError(f"Dalavik: a row of {width} does not split into {groups} groups")
    first = specs[0].attention
    return ModelConfig(
        architecture="Dalavik", model_type="dalavik", hidden_size=width, num_layers=len(specs),
        num_heads=first.num_heads, num_kv_heads=getattr(first, "num_kv_heads", 1), head_dim=first.v_head_dim,
        v_head_dim=first.v_head_dim, vocab_size=int(d["vocab"]), rms_norm_eps=float(d["norm"]["eps"]),
        max_position_embeddings=1 << 20, tie_word_embeddings=True, dtype=to_dtype(dtype or "bfloat16"),
        layer_specs=specs, norm_groups=groups, token_side_dim=int((d.get("token_side") or {"dim": 0})["dim"]), hf_config=d)


# --------------------------------------------------------------------- mixers
class LatentMixer(Mixer):
    """``shared``: whether a later layer reads this one's rows."""

    def __init__(self, cfg: ModelConfig, s: LatentAttentionSpec, cache_idx: int, shared: bool, device, prefix: str,
                 max_position: int) -> None:
        super().__init__(cfg)
        self.spec, self.cache_idx = s, cache_idx
        heads, own = self.share(s.num_heads), s.kv_from is None
        segments = {"dq": (s.q_rank, False)}
        if own:
            segments["dkv"] = (s.kv_rank + s.rope_dim, False)
        self.in_proj = SegmentedLinear(self.padded_width, segments, dtype=cfg.dtype, device=device, prefix=f"{prefix}.in_proj")
        self.q_proj = SegmentedLinear(pad8(s.q_rank), {"uq": (s.num_heads * (s.nope_dim + s.rope_dim), True)},
                                      dtype=cfg.dtype, device=device, prefix=f"{prefix}.q_proj")
        self.rotary = get_rope(s.rope_dim, s.rope_dim, max_position, s.rope_theta, s.rope_neox, None, device,
                               exact_angles=True)
        self.attn = LatentAttention(heads, s.nope_dim, s.rope_dim, s.v_head_dim, s.kv_rank, s.scale, s.rope_neox, self.eps,
                                    cfg.dtype, device, s.q_rank, own, shared)
        self.output_proj(cfg, [heads * s.v_head_dim], device, prefix)

    def forward(self, h: torch.Tensor) -> torch.Tensor:
        y, table = self.in_proj(h), self.rotary.cos_sin_cache
        kv = self.in_proj.segment(y, "dkv") if self.attn.own_rows else None
        c_q = self.attn.store(self.in_proj.segment(y, "dq"), kv, table, self.cache_idx)
        q = self.q_proj.segment(self.q_proj(c_q), "uq")
        return self.o_proj(self.attn(q, None, table, self.cache_idx, self.o_proj.in_local))

    def expect(self, want: Want, p: str) -> None:
        s, a = self.spec, self.attn
        self.expect_rows(want, p, self.in_proj)
        want[p + "uq"] = (s.num_heads * a.qk_dim, s.q_rank), lambda t: self.q_proj.weight_loader(self.q_proj.weight, t, "uq")
        self.expect_vector(want, p + "dq.norm", a.query_norm, False)
        if a.own_rows:
            self.expect_vector(want, p + "dkv.norm", a.latent_norm, False)
        self.expect_vector(want, p + "uk", a.w_uk, True)
        self.expect_vector(want, p + "uv", a.w_uv, True)
        self.expect_output(want, p + "o", 0)

    def clear_padding(self) -> None:
        super().clear_padding()
        self.clear(self.in_proj, self.width)
        self.clear(self.q_proj, self.spec.q_rank)
        self.attn.build_absorbed()


class MixedAttentionMixer(Mixer):
    """Every rank has all heads' scores (the mixture needs them); values and outputs are split by heads."""

    def __init__(self, cfg: ModelConfig, s: AttentionSpec, cache_idx: int, device, prefix: str) -> None:
        super().__init__(cfg)
        self.spec, self.cache_idx = s, cache_idx
        heads, kv = self.share(s.num_heads), self.share(s.num_kv_heads, "key/value heads")
        self.in_proj = SegmentedLinear(
            self.padded_width, {"q": (s.num_heads * s.head_dim, False), "k": (s.num_kv_heads * s.head_dim, False),
                                "v": (s.num_kv_heads * s.v_head_dim, True)},
            bias=s.bias, dtype=cfg.dtype, device=device, prefix=f"{prefix}.in_proj")
        self.attn = MixedScoreAttention(cache_idx, s.num_heads, s.num_kv_heads, heads, kv, s.head_dim, s.v_head_dim, s.scale,
                                        s.softcap, s.query_temperature, self.eps, cfg.dtype, device)
        self.output_proj(cfg, [heads * s.v_head_dim], device, prefix)

    def forward(self, h: torch.Tensor) -> torch.Tensor:
        y = self.in_proj(h)
        q, k, v = (self.in_proj.segment(y, x) for x in ("q", "k", "v"))
        return self.o_proj(self.attn(q, k, v, self.o_proj.in_local))

    def expect(self, want: Want, p: str) -> None:
        a = self.attn
        self.expect_rows(want, p, self.in_proj)
        self.expect_output(want, p + "o", 0)
        for name, param, split in (("q.norm", a.q_norm, False), ("k.norm", a.k_norm, False), ("r1", a.r1, False),
                                   ("r2", a.r2, False), ("sink", a.sink, True), ("talk", a.talk, True)):
            self.expect_vector(want, p + name, param, split)

    @torch.no_grad()
    def clear_padding(self) -> None:
        super().clear_padding()
        self.clear(self.in_proj, self.width)
        self.attn.talk_exact = bool((self.attn.talk.bfloat16().float() == self.attn.talk).all())


# --------------------------------------------------------------------- the model
class TokenSide(nn.Module):
    """The per-layer token input: two small products, whole on every rank, around a gated row of the side table."""

    def __init__(self, width: int, dim: int, offset: int, dtype, device) -> None:
        super().__init__()
        self.dim, self.offset = dim, offset

        def param(*shape):
            return nn.Parameter(torch.zeros(*shape, dtype=dtype, device=device), requires_grad=False)

        self.gate, self.proj, self.norm = param(pad8(dim), width), param(width, pad8(dim)), param(width)

    def forward(self, h: torch.Tensor, ids: torch.Tensor, table: torch.Tensor) -> torch.Tensor:
        return ops.gemm(ops.gelu_rows(ops.gemm(h, self.gate), ids, table, self.offset, self.dim), self.proj)


class DalavikLayer(nn.Module):
    def __init__(self, engine: EngineConfig, idx: int, cache_idx: int, shared: bool, device) -> None:
        super().__init__()
        cfg, spec = engine.model, engine.model.layer_specs[idx]
        self.spec = spec
        w, prefix = pad8(cfg.hidden_size), f"layers.{idx}"

        def gain():
            return nn.Parameter(torch.zeros(w, dtype=cfg.dtype, device=device), requires_grad=False)

        self.norm1, self.norm2 = gain(), gain() if spec.mlp is not None else None
        a = spec.attention
        if isinstance(a, LatentAttentionSpec):
            self.mix = LatentMixer(cfg, a, cache_idx, shared, device, f"{prefix}.mix", engine.scheduler.max_model_len)
        else:
            self.mix = MixedAttentionMixer(cfg, a, cache_idx, device, f"{prefix}.mix")
        self.mlp = self.side = None
        if spec.mlp is not None:
            tp = self.mix.tp
            ff = (spec.mlp.intermediate_size + 8 * tp - 1) // (8 * tp) * 8 * tp
            self.mlp = FusedMLP(w, ff, cfg.dtype, device, prefix=f"{prefix}.mlp", act=spec.mlp.act)
        if cfg.token_side_dim:
            self.side = TokenSide(w, cfg.token_side_dim, idx * cfg.token_side_dim, cfg.dtype, device)


class DalavikForCausalLM(nn.Module):
    def __init__(self, engine_config: EngineConfig, device=None) -> None:
        super().__init__()
        cfg = self.config = engine_config.model
        self.width, self.padded_width = cfg.hidden_size, pad8(cfg.hidden_size)
        self.embed = ParallelLMHead(cfg.vocab_size, self.padded_width, cfg.dtype, device)     # the head as well
        sources = {getattr(s.attention, "kv_from", None) for s in cfg.layer_specs}
        layers: List[DalavikLayer] = []
        caches = 0
        for i, s in enumerate(cfg.layer_specs):
            src = getattr(s.attention, "kv_from", None)
            own = src is None
            layers.append(DalavikLayer(engine_config, i, caches if own else layers[src].mix.cache_idx, i in sources, device))
            caches += own
        self.layers = nn.ModuleList(layers)
        self.num_kv_layers = caches
        self.final_norm = nn.Parameter(torch.zeros(self.padded_width, dtype=cfg.dtype, device=device), requires_grad=False)
        self.side_embed = None
        if cfg.token_side_dim:
            self.side_embed = nn.Parameter(torch.zeros(cfg.vocab_size, cfg.num_layers * cfg.token_side_dim, dtype=cfg.dtype,
                                                       device=device), requires_grad=False)

    # ------------------------------------------------------------------ cache
    def _cache_shapes(self, block_size: int) -> List[Tuple[Tuple[int, ...], ...]]:
        """Per cache: one row per token (latent layers), or the shapes of keys and values."""
        out = []
        for layer in self.layers:
            a = layer.mix.attn
            if isinstance(a, LatentAttention):
                if a.own_rows:
                    out.append(((block_size, a.row),))
            else:
                dk, dv = a.cache_widths(self.config.dtype)
                out.append(((a.num_kv_heads, block_size, dk), (a.v_heads, block_size, dv)))
        return out

    def get_kv_cache_spec(self, block_size: int):
        from ..worker.model_runner import KVCacheSpec
        shapes = self._cache_shapes(block_size)
        elems = sum(torch.Size(s).numel() for cache in shapes for s in cache)
        first = {"latent": shapes[0][0]} if len(shapes[0]) == 1 else dict(zip("kv", shapes[0]))
        return KVCacheSpec("mla" if len(shapes[0]) == 1 else "gqa", len(shapes), block_size,
                           elems * self.config.dtype.itemsize, first)

    def allocate_kv_cache(self, num_blocks: int, block_size: int, device):
        # zeros: the padding of the rows stays as it is here
        out = []
        for cache in self._cache_shapes(block_size):
            t = tuple(torch.zeros(num_blocks, *s, dtype=self.config.dtype, device=device) for s in cache)
            out.append(t if len(t) > 1 else t[0])
        return out

    # ---------------------------------------------------------------- forward
    def forward(self, input_ids, positions, inputs_embeds=None, intermediate_tensors=None):
        cfg, eps = self.config, self.config.rms_norm_eps
        ids, table = input_ids, self.embed.weight
        if inputs_embeds is not None or self.embed.group.world_size > 1:
            table = inputs_embeds if inputs_embeds is not None else self.embed(input_ids)
            ids = torch.arange(table.shape[0], dtype=torch.int32, device=table.device)
        x = torch.empty(ids.shape[0], self.padded_width, dtype=torch.float32, device=table.device)
        trace = self.__dict__.get("layer_outputs")       # hook for tests and debugging: a list
        h = ops.post_norm_residual(x, None, None, 1, eps, self.width, ids, table)

        def add(y, weight, groups, last):
            return ops.post_norm_residual(x, y, weight, groups, eps, self.width,
                                          out_norm=(self.final_norm, cfg.norm_groups) if last else None)

        for i, layer in enumerate(self.layers):
            end = i + 1 == len(self.layers)
            h = add(layer.mix(h), layer.norm1, cfg.norm_groups, end and layer.mlp is None and layer.side is None)
            if layer.mlp is not None:
                h = add(layer.mlp(h), layer.norm2, cfg.norm_groups, end and layer.side is None)
            if layer.side is not None:
                h = add(layer.side(h, input_ids, self.side_embed), layer.side.norm, 1, end)
            if trace is not None:
                trace.append(x[:, : self.width].clone())
        return h

    def compute_logits(self, hidden: torch.Tensor) -> torch.Tensor:
        return self.embed.compute_logits(hidden)

    # ---------------------------------------------------------------- weights
    def load_weights(self, weights: Iterable[Tuple[str, torch.Tensor]]) -> set:
        """Place the checkpoint's tensors (padded with zeros where the parameters are wider).  Unknown names, wrong
        shapes and missing tensors are errors; the norm of a feed-forward that a layer does not have is not used."""
        idle = {f"l{i}.norm2" for i, layer in enumerate(self.layers) if layer.mlp is None}
        return place_tensors(weights, self._expected(), "Dalavik", idle.__contains__)

    def _expected(self) -> Want:
        w, wp, vocab = self.width, self.padded_width, self.config.vocab_size
        want: Want = {"embed": ((vocab, w), lambda t: self.embed.weight_loader(self.embed.weight, fit(t, vocab, wp)))}

        def place(name: str, param: nn.Parameter, *shape: int) -> None:
            want[name] = shape, lambda t: param.data.copy_(fit(t, *param.shape))

        place("final.norm", self.final_norm, w)
        if self.side_embed is not None:
            place("side.embed", self.side_embed, *self.side_embed.shape)
        for i, layer in enumerate(self.layers):
            p = f"l{i}."
            place(p + "norm1", layer.norm1, w)
            layer.mix.expect(want, p + "mix.")
            if layer.mlp is not None:
                place(p + "norm2", layer.norm2, w)
                ff, gu, down = layer.spec.mlp.intermediate_size, layer.mlp.gate_up_proj, layer.mlp.down_proj
                full = gu.output_sizes[0]
                for j, name in enumerate(("gate", "up")):
                    want[f"{p}mlp.{name}"] = (ff, w), lambda t, j=j, gu=gu, full=full: gu.weight_loader(
                        gu.weight, fit(t, full, wp), j)
                want[p + "mlp.down"] = (w, ff), lambda t, down=down, full=full: down.weight_loader(
                    down.weight, fit(t, wp, full))
            if layer.side is not None:
                place(p + "side.gate", layer.side.gate, layer.side.dim, w)
                place(p + "side.proj", layer.side.proj, w, layer.side.dim)
                place(p + "side.norm", layer.side.norm, w)
        return want

    @torch.no_grad()
    def post_load(self) -> None:
        """Derived weights, and zeros in the padding whatever filled the parameters (random initialisation
        does)."""
        w = self.width
        self.embed.weight.data[:, w:] = 0
        self.final_norm.data[w:] = 0
        for layer in self.layers:
            layer.norm1.data[w:] = 0
            layer.mix.clear_padding()
            if layer.mlp is not None:
                layer.norm2.data[w:] = 0
                layer.mlp.gate_up_proj.weight.data[:, w:] = 0
                layer.mlp.down_proj.weight.data[w:] = 0
                if layer.mlp.down_proj.tp_size == 1:
                    layer.mlp.down_proj.weight.data[:, layer.spec.mlp.intermediate_size:] = 0
            if layer.side is not None:
                s = layer.side
                for t in (s.gate.data.T, s.proj.data, s.norm.data):
                    t[w:] = 0
                s.gate.data[s.dim:] = 0
                s.proj.data[:, s.dim:] = 0
