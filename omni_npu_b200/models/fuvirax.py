"""Fuvirax: a decoder that mixes latent attention with two kinds of recurrent layers on several residual
streams.

Each layer is a mixer and an optional feed-forward, each joined to the streams by a hyper-connection
(``layers/hyper.py``).  Mixers read a layer norm whose rows are blended with the previous token's
(token shift) and are one of

    latent_attention   attention over a cached latent        (attention/latent.py)
    hgrn2              linear attention, gate = 1 - key      (attention/recurrent.py)
    channel_delta      gated delta rule, decay per channel   (attention/recurrent.py)

A run of layers may be looped with the same weights; every pass has a cache or state of its own, so
caches and states are numbered by layer RUN.  Embedding and head share one table.

Per sublayer and step: the join / norm / shift kernel, one product for all projections of the input, the
mixer's own kernels, one product back.  The feed-forward is two products, its activation in the first
one's epilogue.

Widths that are not whole 16-byte rows are padded with zeros when the weights are loaded; the norms
divide by the true width.
"""
from __future__ import annotations

from typing import Any, Dict, Iterable, List, Optional, Tuple

import torch
from torch import nn

from ..attention.latent import LatentAttention
from ..attention.metadata import get_forward_context
from ..attention.recurrent import DeltaRuleAttention, GatedLinearAttention
from ..config import (DeltaRuleSpec, DenseSpec, EngineConfig, GatedLinearSpec, LatentAttentionSpec, LayerSpec, LoopSpec,
                      ModelConfig, to_dtype)
from ..layers.embedding import ParallelLMHead
from ..layers.hyper import HyperSublayer
from ..layers.linear import RowParallelLinear, SegmentedLinear
from ..layers.mlp import XieluMLP
from ..layers.rope import get_rope
from ..parallel import state as pstate
from .layered import Want, fit, pad8, place_tensors

UNIT_EPS = 1e-6          # of the unit norm of the delta rule's q and k


# --------------------------------------------------------------------- configuration
def _mixer_spec(kind: str, m: Dict[str, Any], ranks: Tuple[int, int]):
    if kind == "latent_attention":
        spec = LatentAttentionSpec(int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"]),
                                   float(m["rot"]["base"]), float(m["scale"]))
        if spec.rope_dim % 2 or int(m["rot"].get("dims", spec.rope_dim)) != spec.rope_dim:
            raise ValueError(f"Fuvirax: inconsistent rotation {m}")
        return spec
    if kind == "hgrn2":
        return GatedLinearSpec(int(m["heads"]), int(m["dim"]), int(m["vdim"]))
    if kind == "channel_delta":
        spec = DeltaRuleSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), int(m["conv"]), *ranks,
                             unit_eps=UNIT_EPS)
        if spec.num_heads % spec.num_kv_heads or spec.conv_taps < 1:
            raise ValueError(f"Fuvirax: inconsistent sizes {m}")
        return spec
    raise ValueError(f"Fuvirax: unknown mixer {kind!r}")


def read_config(d: Dict[str, Any], dtype=None, path: Optional[str] = None) -> ModelConfig:
    """``ModelConfig`` from the design's own config.json keys.  The ranks of the delta rule's low-rank
    projections stand in no key: they are the rows of the checkpoint's tensors (without a checkpoint, the
    head size)."""
    from .utils import safetensors_shapes
    shapes = safetensors_shapes(path) if path else {}

    def layer(i: int, x: Dict[str, Any]) -> LayerSpec:
        ranks = tuple(shapes.get(f"l{i}.mix.{n}", (x["mixer"].get("dim", 1),))[0] for n in ("a1", "g1"))
        mlp = x.get("mlp")
        if mlp is not None and mlp.get("kind", "dense") != "dense":
            raise ValueError(f"Fuvirax: unknown feed-forward {mlp['kind']!r}")
        return LayerSpec(_mixer_spec(x["type"], x["mixer"], ranks), DenseSpec(int(mlp["ff"])) if mlp else None)

    specs = tuple(layer(i, x) for i, x in enumerate(d["layers"]))
    loop = d.get("loop")
    if loop:
        loop = LoopSpec(int(loop["start"]), int(loop["stop"]), int(loop["times"]))
        if not 0 <= loop.start <= loop.stop <= len(specs) or loop.times < 0:
            raise ValueError(f"Fuvirax: inconsistent loop {loop}")
    first = specs[0].attention
    return ModelConfig(
        architecture="Fuvirax", model_type="fuvirax", hidden_size=int(d["width"]), num_layers=len(specs),
        num_heads=first.num_heads, num_kv_heads=1, head_dim=first.v_head_dim, v_head_dim=first.v_head_dim,
        vocab_size=int(d["vocab"]), rms_norm_eps=float(d["norm"]["eps"]), max_position_embeddings=1 << 20,
        tie_word_embeddings=True, dtype=to_dtype(dtype or "bfloat16"), layer_specs=specs, layer_loop=loop or None,
        residual_streams=int(d.get("streams") or 1), logit_scale=float(d.get("logit_scale", 1.0)), hf_config=d)


# --------------------------------------------------------------------- mixers
class FuviraxMixer(nn.Module):
    """Projections around a mixer's core: one product in, one out."""

    def __init__(self, cfg: ModelConfig, segments: Dict[str, Tuple[int, bool]], out_features: int, device,
                 prefix: str) -> None:
        super().__init__()
        self.width, wp = cfg.hidden_size, pad8(cfg.hidden_size)
        self.in_proj = SegmentedLinear(wp, segments, dtype=cfg.dtype, device=device, prefix=f"{prefix}.in_proj")
        self.tp, self.rank = self.in_proj.tp_size, self.in_proj.tp_rank
        self.true_out = out_features
        if self.tp > 1 and out_features // self.tp % 8:
            raise ValueError(f"Fuvirax: {out_features // self.tp} value columns per rank are not whole 16-byte rows")
        self.o_proj = RowParallelLinear(out_features if self.tp > 1 else pad8(out_features), wp, dtype=cfg.dtype,
                                        device=device, prefix=f"{prefix}.o_proj")

    def heads(self, n: int) -> int:
        """This rank's share of ``n`` heads."""
        if n % self.tp:
            raise ValueError(f"Fuvirax: {n} heads do not split over {self.tp} ranks")
        return n // self.tp

    def own(self, t: torch.Tensor) -> torch.Tensor:
        """This rank's rows of a tensor that is split by heads."""
        n = t.shape[0] // self.tp
        return t.narrow(0, self.rank * n, n)

    def expect(self, want: Want, p: str) -> None:
        proj, o = self.in_proj, self.o_proj
        for name, n in proj.rows.items():
            rows = n * self.tp if proj.sharded[name] else n
            want[p + name] = (rows, self.width), lambda t, name=name: proj.weight_loader(proj.weight, t, name)
        want[p + "o"] = (self.width, self.true_out), lambda t: o.weight_loader(
            o.weight, fit(t, o.out_features, o.in_features))

    def expect_vector(self, want: Want, name: str, param: nn.Parameter, split: bool) -> None:
        shape = (param.shape[0] * (self.tp if split else 1), *param.shape[1:])
        want[name] = shape, lambda t: param.data.copy_(self.own(t) if split else t)

    @torch.no_grad()
    def clear_padding(self) -> None:
        proj, o = self.in_proj, self.o_proj
        proj.weight.data[proj.padding_rows().to(proj.weight.device)] = 0
        proj.weight.data[:, self.width:] = 0
        o.weight.data[self.width:] = 0
        if self.tp == 1:
            o.weight.data[:, self.true_out:] = 0


class LatentMixer(FuviraxMixer):
    def __init__(self, cfg: ModelConfig, s: LatentAttentionSpec, device, prefix: str, max_position: int) -> None:
        super().__init__(cfg, {"q": (s.num_heads * (s.nope_dim + s.rope_dim), True),
                               "dkv": (s.kv_rank + s.rope_dim, False)}, s.num_heads * s.v_head_dim, device, prefix)
        self.rotary = get_rope(s.rope_dim, s.rope_dim, max_position, s.rope_theta, s.rope_neox, None, device,
                               exact_angles=True)
        self.attn = LatentAttention(self.heads(s.num_heads), s.nope_dim, s.rope_dim, s.v_head_dim, s.kv_rank, s.scale,
                                    s.rope_neox, cfg.rms_norm_eps, cfg.dtype, device)

    def forward(self, h: torch.Tensor, run: int, cache_idx: int) -> torch.Tensor:
        y = self.in_proj(h)
        o = self.attn(self.in_proj.segment(y, "q"), self.in_proj.segment(y, "dkv"), self.rotary.cos_sin_cache, cache_idx,
                      self.o_proj.in_local)
        return self.o_proj(o)

    def expect(self, want: Want, p: str) -> None:
        super().expect(want, p)
        self.expect_vector(want, p + "dkv.norm", self.attn.latent_norm, False)
        self.expect_vector(want, p + "uk", self.attn.w_uk, True)
        self.expect_vector(want, p + "uv", self.attn.w_uv, True)

    def clear_padding(self) -> None:
        super().clear_padding()
        self.attn.build_absorbed()


class GatedLinearMixer(FuviraxMixer):
    def __init__(self, cfg: ModelConfig, s: GatedLinearSpec, device, prefix: str) -> None:
        n, e = s.num_heads * s.head_dim, s.num_heads * s.v_head_dim
        super().__init__(cfg, {"q": (n, True), "f": (n, True), "v": (e, True)}, e, device, prefix)
        self.attn = GatedLinearAttention(self.heads(s.num_heads), s.head_dim, s.v_head_dim, cfg.rms_norm_eps, cfg.dtype,
                                         device)

    def forward(self, h: torch.Tensor, run: int, cache_idx: int) -> torch.Tensor:
        return self.o_proj(self.attn(self.in_proj(h), self.in_proj.offsets, run, self.o_proj.in_local))

    def expect(self, want: Want, p: str) -> None:
        super().expect(want, p)
        self.expect_vector(want, p + "f.b", self.attn.f_bias, True)
        self.expect_vector(want, p + "lower", self.attn.lower, True)
        self.expect_vector(want, p + "norm", self.attn.out_norm, False)


class DeltaMixer(FuviraxMixer):
    """The two low-rank projections end in one product with a block-diagonal weight."""

    def __init__(self, cfg: ModelConfig, s: DeltaRuleSpec, device, prefix: str) -> None:
        self.ranks = s.decay_rank, s.gate_rank
        n, e = s.num_heads * s.head_dim, s.num_heads * s.v_head_dim
        super().__init__(cfg, {"q": (s.num_kv_heads * s.head_dim, True), "k": (s.num_kv_heads * s.head_dim, True),
                               "v": (e, True), "b": (s.num_heads, True), "a1": (s.decay_rank, False),
                               "g1": (s.gate_rank, False)}, e, device, prefix)
        self.low_cols = pad8(s.decay_rank), pad8(s.gate_rank)
        self.low_proj = SegmentedLinear(sum(self.low_cols), {"a2": (n, True), "g2": (e, True)}, dtype=cfg.dtype,
                                        device=device, prefix=f"{prefix}.low_proj")
        self.attn = DeltaRuleAttention(self.heads(s.num_heads), self.heads(s.num_kv_heads), s.head_dim, s.v_head_dim,
                                       s.conv_taps, self.in_proj.offsets["b"], s.unit_eps, cfg.rms_norm_eps, cfg.dtype,
                                       device)

    def forward(self, h: torch.Tensor, run: int, cache_idx: int) -> torch.Tensor:
        y = self.in_proj(h)
        a = self.in_proj.offsets["a1"]
        low = self.low_proj(y[:, a: a + sum(self.low_cols)])
        return self.o_proj(self.attn(y, self.in_proj.offsets, self.low_proj.segment(low, "a2"),
                                     self.low_proj.segment(low, "g2"), run, self.o_proj.in_local))

    def expect(self, want: Want, p: str) -> None:
        super().expect(want, p)
        attn, low, offs = self.attn, self.low_proj, self.in_proj.offsets
        for name, col, r in (("a2", 0, self.ranks[0]), ("g2", self.low_cols[0], self.ranks[1])):
            def place(t, name=name, col=col, r=r):
                full = t.new_zeros(t.shape[0], low.in_features)
                full[:, col: col + r] = t
                low.weight_loader(low.weight, full, name)
            want[p + name] = (low.rows[name] * self.tp, r), place
        for name in ("q", "k", "v"):
            n = self.in_proj.rows[name]
            want[f"{p}{name}.conv"] = (n * self.tp, attn.taps), lambda t, o=offs[name], n=n: attn.conv_weight.data[
                o: o + n].copy_(self.own(t))
        self.expect_vector(want, p + "A_log", attn.a_log, True)
        self.expect_vector(want, p + "dt_bias", attn.dt_bias, True)
        self.expect_vector(want, p + "norm", attn.out_norm, False)

    def clear_padding(self) -> None:
        super().clear_padding()
        w, (ra, rg), ca = self.low_proj.weight.data, self.ranks, self.low_cols[0]
        w[self.low_proj.padding_rows().to(w.device)] = 0
        rows = self.low_proj.offsets["g2"]
        w[:rows, ra:] = 0
        w[rows:, :ca] = 0
        w[rows:, ca + rg:] = 0


class FuviraxLayer(nn.Module):
    def __init__(self, engine: EngineConfig, idx: int, device) -> None:
        super().__init__()
        cfg, spec = engine.model, engine.model.layer_specs[idx]
        self.spec = spec
        wp, prefix = pad8(cfg.hidden_size), f"layers.{idx}"
        args = (wp, cfg.hidden_size, cfg.residual_streams, cfg.rms_norm_eps, cfg.dtype, device)
        self.hc1 = HyperSublayer(*args, shift=True)
        a = spec.attention
        if isinstance(a, LatentAttentionSpec):
            self.mix = LatentMixer(cfg, a, device, f"{prefix}.mix", engine.scheduler.max_model_len)
        elif isinstance(a, GatedLinearSpec):
            self.mix = GatedLinearMixer(cfg, a, device, f"{prefix}.mix")
        else:
            self.mix = DeltaMixer(cfg, a, device, f"{prefix}.mix")
        self.hc2 = self.mlp = None
        if spec.mlp is not None:
            self.hc2 = HyperSublayer(*args)
            tp = pstate.get_tp_group().world_size
            ff = (spec.mlp.intermediate_size + 8 * tp - 1) // (8 * tp) * 8 * tp
            self.mlp = XieluMLP(wp, ff, cfg.dtype, device, prefix=f"{prefix}.mlp")

    @property
    def is_latent(self) -> bool:
        return isinstance(self.mix, LatentMixer)


class FuviraxForCausalLM(nn.Module):
    has_recurrent_state = True               # the token shift alone already is one

    def __init__(self, engine_config: EngineConfig, device=None) -> None:
        super().__init__()
        cfg = self.config = engine_config.model
        self.width, self.padded_width = cfg.hidden_size, pad8(cfg.hidden_size)
        self.embed = ParallelLMHead(cfg.vocab_size, self.padded_width, cfg.dtype, device)     # the head as well
        self.layers = nn.ModuleList([FuviraxLayer(engine_config, i, device) for i in range(cfg.num_layers)])
        self.end = HyperSublayer(self.padded_width, self.width, cfg.residual_streams, cfg.rms_norm_eps, cfg.dtype, device,
                                 join=False, out_scale=cfg.logit_scale)
        self.runs: List[FuviraxLayer] = [self.layers[i] for i in cfg.layer_order()]
        self.cache_of_run: List[int] = []
        n = 0
        for layer in self.runs:
            self.cache_of_run.append(n if layer.is_latent else -1)
            n += layer.is_latent
        self.num_kv_layers = n

    # ------------------------------------------------------------------ cache and state
    def get_kv_cache_spec(self, block_size: int):
        from ..worker.model_runner import KVCacheSpec
        rows = [layer.mix.attn.row for layer in self.runs if layer.is_latent]
        return KVCacheSpec("mla", len(rows), block_size, max(1, block_size * sum(rows) * self.config.dtype.itemsize),
                           {"latent": (block_size, rows[0] if rows else 0)})

    def allocate_kv_cache(self, num_blocks: int, block_size: int, device):
        return [torch.zeros(num_blocks, block_size, layer.mix.attn.row, dtype=self.config.dtype, device=device)
                for layer in self.runs if layer.is_latent]

    def allocate_states(self, num_slots: int, device) -> List[Dict[str, torch.Tensor]]:
        """Per layer run: the previous token's mixer input, and the mixer's own state."""
        out = []
        for layer in self.runs:
            shapes = {"shift": ((self.padded_width,), torch.float32)}
            if not layer.is_latent:
                shapes.update(layer.mix.attn.state_shapes())
            out.append({k: torch.zeros(num_slots, *s, dtype=dt, device=device) for k, (s, dt) in shapes.items()})
        return out

    # ---------------------------------------------------------------- forward
    def forward(self, input_ids, positions, inputs_embeds=None, intermediate_tensors=None):
        ctx = get_forward_context()
        md, states = ctx.attn_metadata, ctx.states
        ids, table = input_ids, self.embed.weight
        if inputs_embeds is not None or self.embed.group.world_size > 1:
            table = inputs_embeds if inputs_embeds is not None else self.embed(input_ids)
            ids = torch.arange(table.shape[0], dtype=torch.int32, device=table.device)
        trace = self.__dict__.get("layer_outputs")
        streams = y = before = None

        def enter(sub: HyperSublayer, run: int, keep: bool = True) -> torch.Tensor:
            nonlocal streams, before
            start = dict(ids=ids, table=table) if before is None else {}
            streams, h = sub.read(streams, before, y, md, states[run]["shift"] if run >= 0 else None, keep=keep, **start)
            before = sub
            return h

        for run, layer in enumerate(self.runs):
            h = enter(layer.hc1, run)
            self._trace(trace, streams, run)
            y = layer.mix(h, run, self.cache_of_run[run])
            if layer.mlp is not None:
                y = layer.mlp(enter(layer.hc2, -1))
        h = enter(self.end, -1, keep=trace is not None)
        self._trace(trace, streams, len(self.runs))
        return h

    def _trace(self, sink, streams: torch.Tensor, run: int) -> None:
        """Hook for tests and debugging: the sum of the streams after a layer run (``layer_outputs`` a list)."""
        if sink is not None and run > 0:
            sink.append(streams.sum(1)[:, : self.width].clone())

    def compute_logits(self, hidden: torch.Tensor) -> torch.Tensor:
        return self.embed.compute_logits(hidden)

    # ---------------------------------------------------------------- weights
    def load_weights(self, weights: Iterable[Tuple[str, torch.Tensor]]) -> set:
        """Place the checkpoint's tensors (padded with zeros where the parameters are wider).  Unknown
        names, wrong shapes and missing tensors are errors; what a checkpoint holds for the feed-forward
        place of a layer without one is not used."""
        idle = tuple(f"l{i}.{x}" for i, layer in enumerate(self.layers) if layer.mlp is None
                     for x in ("norm2", "ls2", "hc2."))
        return place_tensors(weights, self._expected(), "Fuvirax", lambda name: name.startswith(idle))

    def _expected(self) -> Want:
        w, wp = self.width, self.padded_width
        want: Want = {"embed": ((self.config.vocab_size, w), lambda t: self.embed.weight_loader(
            self.embed.weight, fit(t, t.shape[0], wp)))}

        def row(name: str, param: nn.Parameter) -> None:
            want[name] = (w,), lambda t: param.data.copy_(fit(t, wp))

        def norm(name: str, sub: HyperSublayer) -> None:
            row(name, sub.norm_weight)
            row(name + ".b", sub.norm_bias)

        norm("final.norm", self.end)
        for i, layer in enumerate(self.layers):
            p = f"l{i}."
            for q, sub in (("1", layer.hc1), ("2", layer.hc2)):
                if sub is None:
                    continue
                norm(f"{p}norm{q}", sub)
                row(f"{p}ls{q}", sub.layer_scale)
                for name, param in (("in", sub.w_in), ("out", sub.w_out), ("mix", sub.w_mix)):
                    want[f"{p}hc{q}.{name}"] = tuple(param.shape), lambda t, param=param: param.data.copy_(t)
            row(p + "shift", layer.hc1.shift)
            layer.mix.expect(want, p + "mix.")
            if layer.mlp is not None:
                ff, up, down = layer.spec.mlp.intermediate_size, layer.mlp.up_proj, layer.mlp.down_proj
                want[p + "mlp.up"] = (ff, w), lambda t, up=up: up.weight_loader(
                    up.weight, fit(t, up.out_features, wp))
                want[p + "mlp.down"] = (w, ff), lambda t, down=down: down.weight_loader(
                    down.weight, fit(t, wp, down.in_features))
                want[p + "mlp.act"] = (2,), lambda t, m=layer.mlp: m.act_params.data.copy_(t)
        return want

    @torch.no_grad()
    def post_load(self) -> None:
        """Derived weights, and zeros in the padding whatever filled the parameters (random
        initialisation does)."""
        w = self.width
        self.embed.weight.data[:, w:] = 0
        for layer in self.layers:
            layer.mix.clear_padding()
            if layer.mlp is None:
                continue
            ff, mlp = layer.spec.mlp.intermediate_size, layer.mlp
            mlp.fix_constants()
            mlp.up_proj.weight.data[:, w:] = 0
            mlp.down_proj.weight.data[w:] = 0
            if mlp.up_proj.tp_size == 1:
                mlp.up_proj.weight.data[ff:] = 0
                mlp.down_proj.weight.data[:, ff:] = 0
