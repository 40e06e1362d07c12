"""Throughput of a design beside the framework's closest existing model at equal size (random weights).

``bench.py --design rivudra`` (``fuvirax``, ``gatosun``, ``dalavik``) runs this on one GPU.  Per size it prints one JSON
line with

* whole steps through the engine (device time of prompt and decode steps, CUDA events): Rivudra and a
  Qwen3-MoE of the same width, heads, experts and window, Fuvirax and a dense DeepSeek-V2 of the same
  width, heads, latent sizes and feed-forward, Gatosun and a Qwen3-MoE of the same width, heads and
  experts (every layer full attention), or Dalavik and a dense DeepSeek-V2 of the same width, heads, latent
  sizes and feed-forward (every layer latent attention);
* single kernels: time, the fraction of the measured roofline (the slower of bytes / copy bandwidth and
  FLOPs / library bf16 GEMM throughput) and the same for the like kernel of the other model.  Between
  iterations a 256 MB buffer is written, so inputs come from HBM.
"""
from __future__ import annotations

import gc
import json
import os
from typing import Callable, Dict, List, Optional, Tuple

import torch

from .. import ops
from ..config import (AttentionSpec, DecayLinearSpec, DeltaRuleSpec, DenseSpec, ExpertSpec, GatedLinearSpec,
                      LatentAttentionSpec, LayerSpec, ModelConfig, MoESpec, ParallelSpec, TimeMixSpec)

LAYERS = 4
CLAMPED = (1.702, 7.0)
# width, q heads, kv heads, head size, window, experts, top-k, expert width
SIZES: Dict[str, Tuple[int, ...]] = {
    "2048x32h/4kv/128 w1024 e128k8 ff768": (2048, 32, 4, 128, 1024, 128, 8, 768),
    "4096x32h/8kv/128 w512 e64k6 ff1536": (4096, 32, 8, 128, 512, 64, 6, 1536),
    "2880x64h/8kv/64 w128 e32k4 ff2880": (2880, 64, 8, 64, 128, 32, 4, 2880),
}
VOCAB = 32768
CONTEXT = 2048


def rivudra(size) -> ModelConfig:
    w, hq, hk, d, win, e, k, ff = size
    ex = ExpertSpec(ff, CLAMPED)
    spec = LayerSpec(AttentionSpec(hq, hk, d, d, d, 1e6, d ** -0.5, False, win, 0.0, True),
                     MoESpec(e, k, ex, ex, n_group=4, topk_group=2))
    return ModelConfig(architecture="Rivudra", model_type="rivudra", hidden_size=w, num_layers=LAYERS, num_heads=hq,
                       num_kv_heads=hk, head_dim=d, vocab_size=VOCAB, max_position_embeddings=1 << 16,
                       layer_specs=(spec,) * LAYERS, embedding_scale=1.0, norm_weight_offset=1.0, num_experts=e,
                       num_experts_per_tok=k)


def qwen3_moe(size) -> ModelConfig:
    w, hq, hk, d, win, e, k, ff = size
    return ModelConfig(architecture="Qwen3MoeForCausalLM", model_type="qwen3_moe", hidden_size=w, num_layers=LAYERS,
                       num_heads=hq, num_kv_heads=hk, head_dim=d, vocab_size=VOCAB, rope_theta=1e6,
                       max_position_embeddings=1 << 16, qk_norm=True, sliding_window=win, num_experts=e,
                       num_experts_per_tok=k, moe_intermediate_size=ff, norm_topk_prob=True)


def model_steps(mc: ModelConfig) -> dict:
    """Device ms of a prompt step of 8 x 1024 tokens and of a decode step of 1 / 16 / 128 sequences."""
    from .. import SamplingParams
    from ..engine.llm import LLM
    llm = LLM(model=mc, device="cuda", max_num_seqs=128, max_num_batched_tokens=8192, max_model_len=CONTEXT + 128,
              compilation_config={"cudagraph_capture_sizes": [1, 16, 128]}, load_format="dummy")
    runner = llm.engine.worker.model_runner
    runner.enable_step_events = True
    g = torch.Generator().manual_seed(0)

    def run(n: int, length: int, out: int, repeat: int):
        prompts = torch.randint(0, mc.vocab_size, (n, length), generator=g).tolist()
        for i in range(repeat + 1):
            if i == 1:
                runner.drain_step_events()
                runner.step_ms_by_kind.clear()
                runner.step_count_by_kind.clear()
            llm.generate(prompts, SamplingParams(max_tokens=out, ignore_eos=True))
        runner.drain_step_events()
        return {k: v / runner.step_count_by_kind[k] for k, v in runner.step_ms_by_kind.items()}

    res = {"prefill_ms_8x1024": round(run(8, 1024, 1, 5)["prefill"], 4)}
    res["prefill_tok_s"] = round(8192 / res["prefill_ms_8x1024"] * 1e3)
    for n in (1, 16, 128):
        ms = run(n, CONTEXT, 64, 1)["decode"]
        res[f"decode_ms_b{n}"] = round(ms, 4)
        res[f"decode_tok_s_b{n}"] = round(n / ms * 1e3)
    ops.check_status()
    llm.engine.shutdown()
    runner.graphs.clear()
    del llm, runner
    from ..layers import moe
    moe._SHARED_BUFFERS.clear()
    gc.collect()
    torch.cuda.empty_cache()
    return res


def _time(fn: Callable[[], object], iters: int = 12) -> float:
    """Median device ms of one call, L2 flushed before it.  The flush also keeps the queue busy, so the
    launch itself is not part of the interval."""
    flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")
    for _ in range(3):
        fn()
    ev = [(torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)) for _ in range(iters)]
    for a, b in ev:
        flush.zero_()
        a.record()
        fn()
        b.record()
    torch.cuda.synchronize()
    return sorted(a.elapsed_time(b) for a, b in ev)[iters // 2]


def _peaks() -> Tuple[float, float]:
    path = os.path.join(os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__)))),
                        "MEASURED_PEAKS.json")
    try:
        with open(path) as f:
            p = json.load(f)
        return p["hbm_gbs"] * 1e9, p["bf16_tflops"] * 1e12
    except Exception:
        return 6.65e12, 1.59e15


def _attention_inputs(size, n: int, rows: int, extra: int, bs: int = 16):
    """n sequences whose last ``rows`` tokens are this step's, CONTEXT - rows earlier ones cached."""
    w, hq, hk, d, win = size[:5]
    per = (CONTEXT + bs - 1) // bs
    dev = dict(device="cuda")
    cols = hq * d + 2 * hk * d + extra
    qkv = torch.randn(n * rows, cols, dtype=torch.bfloat16, **dev)
    kc = torch.randn(n * per, hk, bs, d, dtype=torch.bfloat16, **dev)
    vc = torch.randn(n * per, hk, bs, d, dtype=torch.bfloat16, **dev)
    bt = torch.randperm(n * per, **dev).int().view(n, per)
    pos = torch.arange(CONTEXT - rows, CONTEXT, **dev).repeat(n).int()
    slot = (bt.long().gather(1, (pos.view(n, rows) // bs).long()) * bs + pos.view(n, rows) % bs).int().view(-1)
    return dict(qkv=qkv, kc=kc, vc=vc, bt=bt, pos=pos, slot=slot,
                cu=torch.arange(0, (n + 1) * rows, rows, **dev).int(),
                lens=torch.full((n,), CONTEXT, **dev).int())


def kernels(size) -> List[dict]:
    w, hq, hk, d, win, e, k, ff = size
    bw, fl = _peaks()
    out: List[dict] = []
    bf = dict(dtype=torch.bfloat16, device="cuda")

    def entry(name: str, fn, nbytes: float, flops: float, like: Optional[Tuple] = None):
        ms = _time(fn)
        bound = max(nbytes / bw, flops / fl) * 1e3
        r = {"kernel": name, "ms": round(ms, 4), "roofline": round(bound / ms, 3)}
        if like is not None:
            lms = _time(like[0])
            lb = max(like[1] / bw, like[2] / fl) * 1e3
            r.update(like_ms=round(lms, 4), like_roofline=round(lb / lms, 3),
                     distance=round((lb / lms) / (bound / ms), 2))
        out.append(r)

    cs = torch.randn(CONTEXT + 128, d, device="cuda")
    for kind, n, rows in (("prefill", 8, 1024), ("decode b16", 16, 1), ("decode b128", 128, 1)):
        t = n * rows
        a = _attention_inputs(size, n, rows, hq * d)
        q, kk, vv, g = a["qkv"].split([hq * d, hk * d, hk * d, hq * d], 1)
        o = torch.empty(t, hq * d, **bf)
        moved = t * (2 * hq + 4 * hk) * d * 2
        entry(f"rope + cache, {kind}",
              lambda: ops.gated_rope_cache_(q, kk, vv, a["kc"], a["vc"], a["pos"], a["slot"], cs, d, d, d, False), moved, 0,
              (lambda: ops.rope_cache_gqa_(q, kk, vv, a["kc"], a["vc"], a["pos"], a["slot"], cs, d, d, True), moved, 0))
        # visible (query, key) pairs of one sequence
        def pairs(window):
            return sum(min(window or CONTEXT, p + 1) for p in range(CONTEXT - rows, CONTEXT))
        def keys(window):
            return min(CONTEXT, (window or CONTEXT) + rows - 1)
        kv = n * hk * 2 * d * 2
        pre = kind == "prefill"
        args = (a["kc"], a["vc"])
        def own():
            ops.gated_attention(q, g, *args, o, a["bt"], a["cu"] if pre else None, a["lens"], n, rows, hq, d, d, d ** -0.5,
                                win, 0.0, max_seq_len=CONTEXT)
        def like(window):
            if pre:
                return ops.gqa_prefill(q, *args, a["bt"], a["cu"], a["lens"], n, rows, hq, d ** -0.5, True, window)
            return ops.gqa_decode(q, *args, a["bt"], a["lens"], n, hq, d ** -0.5, 1, window, max_seq_len=CONTEXT)
        mine = (kv * keys(win) + t * hq * d * 2 * 3, 4.0 * n * hq * d * pairs(win))
        for label, window in (("same window", win), ("full context", 0)):
            entry(f"attention, {kind} (like: {label})", own, *mine,
                  (lambda window=window: like(window), kv * keys(window) + t * hq * d * 2 * 2,
                   4.0 * n * hq * d * pairs(window)))
        h = torch.randn(t, w, **bf)
        wq = torch.randn((2 * hq + 2 * hk) * d, w, **bf)
        wl = wq[: (hq + 2 * hk) * d]
        entry(f"input projection, {kind}", lambda: ops.gemm(h, wq), (wq.numel() + h.numel() + t * wq.shape[0]) * 2,
              2.0 * t * wq.numel(), (lambda: ops.gemm(h, wl), (wl.numel() + h.numel() + t * wl.shape[0]) * 2,
                                     2.0 * t * wl.numel()))
        # experts: rows spread evenly
        ids = torch.stack([torch.randperm(e, device="cuda")[:k] for _ in range(min(t, 512))]).repeat(
            (t + 511) // 512, 1)[:t].int()
        counts = torch.bincount(ids.view(-1).long(), minlength=e)
        offs = torch.zeros(e + 1, dtype=torch.int32, device="cuda")
        offs[1:] = counts.cumsum(0)
        live = int((counts > 0).sum())
        x = torch.randn(t * k, w, **bf)
        w13 = torch.randn(e, 2 * ff, w, **bf)
        nb = (live * 2 * ff * w + t * k * (w + ff)) * 2
        entry(f"experts gate/up, {kind}", lambda: ops.grouped_gemm(x, w13, offs, swiglu=True, act=CLAMPED), nb,
              4.0 * t * k * ff * w, (lambda: ops.grouped_gemm(x, w13, offs, swiglu=True), nb, 4.0 * t * k * ff * w))
        entry(f"shared gate/up, {kind}", lambda: ops.gemm(h, w13[0], swiglu=True, act=CLAMPED),
              (2 * ff * w + t * (w + ff)) * 2, 4.0 * t * ff * w,
              (lambda: ops.gemm(h, w13[0], swiglu=True), (2 * ff * w + t * (w + ff)) * 2, 4.0 * t * ff * w))
        del w13
        # end of the layer: routed rows + sublayers + residual + norm, against combine, add and norm
        slots = torch.randperm(t * k, device="cuda").int()
        wt = torch.rand(t, k, device="cuda")
        res, gain = torch.randn(t, w, device="cuda"), torch.randn(w, **bf)
        res16 = res.bfloat16()
        attn_out, shared = torch.randn(t, w, **bf), torch.randn(t, w, **bf)
        from ..layers.moe import _solo_group
        from ..layers.moe_dispatch import DispatchHandle, EpBuffers, ep_combine
        buf = EpBuffers(_solo_group(), torch.device("cuda", torch.cuda.current_device()), e, w, t, k)
        handle = DispatchHandle(ids, wt, slots, t, t * k, offs)
        def other():
            y = ep_combine(None, buf.expert_y, handle, shared, buf)
            ops.fused_add_rms_norm(y, res16, gain, 1e-6)
            ops.fused_add_rms_norm(attn_out, res16, gain, 1e-6)      # (its layer has two norms)
        entry(f"end of layer, {kind}",
              lambda: ops.residual_add_norm(res, attn_out, shared, (x, slots, wt), gain, 1e-6, 1.0, w),
              t * w * (2 * k + 2 + 2 + 4 + 4 + 2), 0,
              (other, t * w * (2 * k + 2 + 2 + 2 * 4 * 2), 0))
        logits = torch.randn(t, e, device="cuda")
        entry(f"routing, {kind}", lambda: ops.moe_topk(logits, None, k, False, 4, 2, True, 1.0), t * (e + 2 * k) * 4, 0,
              (lambda: ops.moe_topk(logits, None, k, False, 1, 1, True, 1.0), t * (e + 2 * k) * 4, 0))
        del a, q, kk, vv, g, o, x, buf
        gc.collect()
        torch.cuda.empty_cache()
    ops.check_status()
    return out


# ----------------------------------------------------------------------------- Fuvirax
# width, heads, head size (states and unrotated keys), value size, rotated keys, latent, feed-forward, streams
FUVIRAX_SIZES: Dict[str, Tuple[int, ...]] = {
    "2048x16h/128 ff8192 s2": (2048, 16, 128, 128, 64, 512, 8192, 2),
    "4096x32h/128 ff12288 s4": (4096, 32, 128, 128, 64, 512, 12288, 4),
    "3072x24h/128 ff8192 s3": (3072, 24, 128, 128, 64, 512, 8192, 3),
}
FUVIRAX_LAYERS = 6           # two of each mixer
LOW_RANK = 128
TAPS = 4
# fp32 multiply-adds per second of the CUDA cores at the maximum clock: what bounds the recurrences
FP32_FLOPS = 148 * 128 * 2 * 1.965e9
# exponentials, logarithms and reciprocals per second of the special function units at that clock
SPECIAL_OPS = 148 * 16 * 1.965e9


def fuvirax(size) -> ModelConfig:
    w, h, d, e, rot, rank, ff, streams = size
    mlp = DenseSpec(ff)
    specs = (LayerSpec(GatedLinearSpec(h, d, e), mlp), LayerSpec(DeltaRuleSpec(h, h, d, e, TAPS, LOW_RANK, LOW_RANK), mlp),
             LayerSpec(LatentAttentionSpec(h, d, rot, e, rank, 1e4, (d + rot) ** -0.5), mlp))
    return ModelConfig(architecture="Fuvirax", model_type="fuvirax", hidden_size=w, num_layers=FUVIRAX_LAYERS, num_heads=h,
                       num_kv_heads=1, head_dim=e, vocab_size=VOCAB, max_position_embeddings=1 << 16,
                       layer_specs=specs * (FUVIRAX_LAYERS // 3), residual_streams=streams, tie_word_embeddings=True)


def deepseek_dense(size) -> ModelConfig:
    w, h, d, e, rot, rank, ff, _ = size
    return ModelConfig(architecture="DeepseekV2ForCausalLM", model_type="deepseek_v2", hidden_size=w,
                       num_layers=FUVIRAX_LAYERS, num_heads=h, num_kv_heads=h, head_dim=d + rot, intermediate_size=ff,
                       vocab_size=VOCAB, max_position_embeddings=1 << 16, rope_neox=False, use_mla=True,
                       kv_lora_rank=rank, qk_nope_head_dim=d, qk_rope_head_dim=rot, v_head_dim=e)


def fuvirax_kernels(size) -> List[dict]:
    from ..attention.latent import LatentAttention
    w, h, d, e, rot, rank, ff, ns = size
    bw, fl = _peaks()
    out: List[dict] = []
    bf = dict(dtype=torch.bfloat16, device="cuda")
    f32 = dict(dtype=torch.float32, device="cuda")
    i32 = dict(dtype=torch.int32, device="cuda")

    def entry(name: str, fn, nbytes: float, flops: float = 0.0, like: Optional[Tuple] = None, peak: float = fl):
        ms = _time(fn)
        bound = max(nbytes / bw, flops / peak) * 1e3
        r = {"kernel": name, "ms": round(ms, 4), "roofline": round(bound / ms, 3)}
        if like is not None:
            lms = _time(like[0])
            lb = max(like[1] / bw, like[2] / fl) * 1e3
            r.update(like_ms=round(lms, 4), like_roofline=round(lb / lms, 3),
                     distance=round((lb / lms) / (bound / ms), 2))
        out.append(r)

    bs, qk, row = 64, d + rot, rank + rot
    for kind, n, rows in (("prefill", 8, 1024), ("decode b1", 1, 1), ("decode b16", 16, 1), ("decode b128", 128, 1)):
        t, pre = n * rows, kind == "prefill"
        ctx = rows if pre else CONTEXT
        x = torch.randn(t, w, **bf)
        gain, bias = torch.randn(w, **bf), torch.randn(w, **bf)
        cu = torch.arange(0, (n + 1) * rows, rows, **i32)
        lens = torch.full((n,), ctx, **i32)
        slots, idx = torch.arange(n, **i32), torch.arange(n, **i32).repeat_interleave(rows)
        states = (slots, cu, lens, n)
        # ---- join + norm (+ token shift) against add + norm
        st = torch.randn(t, ns, w, **f32)
        conn = (gain, torch.eye(ns, **f32), torch.ones(ns, **f32))
        w_in, shift_state = torch.ones(ns, **f32), torch.zeros(n, w, **f32)
        shift = (gain, shift_state, idx, *states)
        res16 = torch.randn(t, w, **bf)
        like_norm = (lambda: ops.fused_add_rms_norm(x, res16, gain, 1e-6), t * w * 2 * 4, 0)
        for label, sh in (("with token shift", shift), ("no shift", None)):
            entry(f"join + norm {label}, {kind}",
                  lambda sh=sh: ops.hyper_norm(st, None, None, ns, x, conn, w_in, gain, bias, 1e-5, w, 1.0, sh),
                  t * w * (8 * ns + 4) + (n * w * 8 if sh else 0), 0, like_norm)
        del st
        # ---- products
        def product(name, cols, like_cols=h * qk):
            a, b = torch.randn(cols, w, **bf), torch.randn(like_cols, w, **bf)
            entry(f"{name}, {kind}", lambda: ops.gemm(x, a), (a.numel() + x.numel() + t * cols) * 2, 2.0 * t * a.numel(),
                  (lambda: ops.gemm(x, b), (b.numel() + x.numel() + t * like_cols) * 2, 2.0 * t * b.numel()))
        delta_cols = h * (2 * d + e) + (h + 7) // 8 * 8 + 2 * LOW_RANK
        product("projection, gated linear (like: q of MLA)", h * (2 * d + e))
        product("projection, delta rule (like: q of MLA)", delta_cols)
        product("projection, latent (like: q of MLA)", h * qk + row)
        up, gu = torch.randn(ff, w, **bf), torch.randn(2 * ff, w, **bf)
        entry(f"up + xielu (like: gate/up + silu), {kind}", lambda: ops.gemm(x, up, xielu=(0.7, 0.9)),
              (up.numel() + x.numel() + t * ff) * 2, 2.0 * t * up.numel(),
              (lambda: ops.gemm(x, gu, swiglu=True), (gu.numel() + x.numel() + t * ff) * 2, 2.0 * t * gu.numel()))
        del up, gu
        # ---- attention inputs: paged latent rows, queries
        per = (ctx + bs - 1) // bs
        cache = torch.randn(n * per, bs, row, **bf)
        bt = torch.randperm(n * per, device="cuda").int().view(n, per)
        pos = torch.arange(ctx - rows, ctx, **i32).repeat(n)
        slot = (bt.long().gather(1, (pos.view(n, rows) // bs).long()) * bs + pos.view(n, rows) % bs).int().view(-1)
        cs = torch.randn(CONTEXT + 128, rot, device="cuda")
        q, kv_a = torch.randn(t, h * qk, **bf), torch.randn(t, row, **bf)
        attn = LatentAttention(h, d, rot, e, rank, qk ** -0.5, True, 1e-5, torch.bfloat16, torch.device("cuda"))
        attn.w_uk.data.normal_(std=0.02)
        attn.w_uv.data.normal_(std=0.02)
        attn.build_absorbed()
        q_lat = torch.empty(t, h, row, **bf)
        def like_prep():
            ops.mla_kv_rmsnorm_rope_cache(kv_a[:, :rank], kv_a[:, rank:], attn.latent_norm, cache, pos, slot, cs, 1e-5, False)
            pe = q.view(t, h, qk)[:, :, d:].reshape(t, h * rot).contiguous()
            ops.rope_qk_(pe, pe.new_empty(t, 0), pos, cs, rot, rot, False)
        moved = t * (2 * row + 2 * h * rot) * 2
        entry(f"latent norm + rotation + cache, {kind}",
              lambda: ops.latent_prep_(q, kv_a, attn.latent_norm, 1e-5, cache, pos, slot, cs, h, d, rot, rank, True,
                                       None if pre else q_lat, 0 if pre else t), moved, 0, (like_prep, moved, 0))
        pairs = n * h * sum(p + 1 for p in range(ctx - rows, ctx))
        if pre:
            start = (torch.cumsum(lens, 0) - lens).int()
            def own_keys():
                r = ops.latent_gather(cache, bt, lens, start, n, t, ctx)
                return ops.gemm(r, attn.w_key), ops.gemm(r, attn.w_value)
            kvb = torch.randn(h * (d + e), rank, **bf)
            def like_keys():
                lat = cache.index_select(0, bt.view(-1).long())
                kv = ops.gemm(lat[..., :rank].reshape(-1, rank).contiguous(), kvb).view(-1, bs, h, d + e)
                pe = lat[..., rank:].unsqueeze(2).expand(-1, bs, h, rot)
                k = torch.cat([kv[..., :d], pe], -1).permute(0, 2, 1, 3).contiguous()
                return k, kv[..., d:].permute(0, 2, 1, 3).contiguous()
            kbytes, kflops = t * (row + h * (qk + e)) * 2 + kvb.numel() * 2, 2.0 * t * kvb.numel()
            entry(f"keys and values from the latents, {kind}", own_keys, kbytes, kflops, (like_keys, kbytes, kflops))
            k, v = own_keys()
            o = torch.empty(t, h * e, **bf)
            lk, lv = like_keys()
            lbt = torch.arange(n * per, **i32).view(n, per)
            abytes, aflops = t * h * (2 * qk + 2 * e) * 2, 2.0 * pairs * (qk + e)
            like_attn = (lambda: ops.gqa_prefill(q, lk, lv, lbt, cu, lens, n, rows, h, 0.07, True, 0), abytes, aflops)
            entry(f"attention, {kind}",
                  lambda: ops.contiguous_attention(q, k.view(-1, h, 1, qk), v.view(-1, h, 1, e), o, cu, start, lens, n, rows,
                                                   h, qk, e, 0.07), abytes, aflops, like_attn)
        else:
            lat_o, o = torch.empty(t, h, rank, **bf), torch.empty(t, h * e, **bf)
            heads = q.view(t, h, qk)
            uv = attn.w_uv.view(h, e, rank)
            offs = torch.arange(0, (h + 1) * t, t, **i32)
            def like_fold():
                qn = heads[..., :d].transpose(0, 1).reshape(h * t, d).contiguous()
                ql = ops.grouped_gemm(qn, attn.w_fold, offs).view(h, t, rank).transpose(0, 1)
                return torch.cat([ql, q_lat[..., rank:]], -1).reshape(t, h * row).contiguous()
            def like_unfold():
                a = lat_o.transpose(0, 1).reshape(h * t, rank).contiguous()
                return ops.grouped_gemm(a, uv, offs).view(h, t, e).transpose(0, 1).reshape(t, h * e).contiguous()
            fb, ff_ = (h * d * rank + t * h * (d + rank)) * 2, 2.0 * t * h * d * rank
            entry(f"queries into the latent space, {kind}",
                  lambda: ops.head_gemm(heads[..., :d], attn.w_fold, q_lat[..., :rank]), fb, ff_, (like_fold, fb, ff_))
            ub, uf = (h * e * rank + t * h * (e + rank)) * 2, 2.0 * t * h * e * rank
            entry(f"results out of the latent space, {kind}", lambda: ops.head_gemm(lat_o, uv, o.view(t, h, e)), ub, uf,
                  (like_unfold, ub, uf))
            abytes, aflops = (n * ctx * row + t * h * (row + rank)) * 2, 2.0 * pairs * (row + rank)
            q_flat = torch.randn(t, h * row, **bf)
            like_attn = (lambda: ops.mla_decode(q_flat, cache, bt, lens, n, h, 0.07, 1, max_seq_len=CONTEXT), abytes, aflops)
            entry(f"attention, {kind}",
                  lambda: ops.latent_decode(q_flat.view(t, h, row), cache, bt, lens, n, h, rank, 0.07, lat_o,
                                            max_seq_len=CONTEXT), abytes, aflops, like_attn)
        # ---- recurrent layers; the like kernel of the scans is attention
        proj = torch.randn(t, delta_cols, **bf)
        fb_, low_ = torch.randn(h * d, **f32), torch.rand(h * d, **f32)
        state = torch.zeros(n, h, e, d, **f32)
        rw = n * h * e * d * 8                                  # the state is read and written once per step
        entry(f"gated linear: q and keys (like: norm + rotation + cache of MLA), {kind}",
              lambda: ops.gated_linear_prep(proj, 0, h * d, h, d, fb_, low_), t * h * d * (4 + 8), 0, (like_prep, moved, 0))
        qf, kf = ops.gated_linear_prep(proj, 0, h * d, h, d, fb_, low_)
        v = proj[:, 2 * h * d: 2 * h * d + h * e]
        entry(f"gated linear: scan (like: attention), {kind}",
              lambda: ops.recurrent_scan(qf, kf, None, v, None, state, h, e, *states),
              t * h * (8 * d + 6 * e) + rw, 5.0 * t * h * d * e, like_attn, FP32_FLOPS)
        offs_ = {"q": 0, "k": h * d, "v": 2 * h * d, "b": h * (2 * d + e)}
        ch = offs_["b"]
        conv_w, conv_state = torch.randn(ch, TAPS, **bf), torch.zeros(n, TAPS - 1, ch, **bf)
        lowp = torch.randn(t, h * (d + e), **bf)
        dt, a_log = torch.randn(h * d, **f32), torch.randn(h, **f32)
        prep = lambda: ops.delta_prep(proj, lowp[:, : h * d], offs_, h, h, d, e, conv_w, conv_state, dt, a_log, 1e-6,  # noqa: E731
                                      idx, *states)
        entry(f"delta rule: convolutions, norms, decays (like: norm + rotation + cache of MLA), {kind}", prep,
              t * h * ((2 * d + e) * 2 + 2 * d + 12 * d + 2 * e), 0, (like_prep, moved, 0))
        qf, kf, gf, vf, beta = prep()
        entry(f"delta rule: scan (like: attention), {kind}",
              lambda: ops.recurrent_scan(qf, kf, gf, vf, beta, state, h, e, *states, conv=(proj, conv_state)),
              t * h * (12 * d + 6 * e) + rw, 7.0 * t * h * d * e, like_attn, FP32_FLOPS)
        low_w = torch.randn(h * (d + e), 2 * LOW_RANK, **bf)
        lp = torch.randn(t, 2 * LOW_RANK, **bf)
        entry(f"delta rule: low-rank product, {kind}", lambda: ops.gemm(lp, low_w),
              (lp.numel() + low_w.numel() + t * h * (d + e)) * 2, 2.0 * t * low_w.numel())
        of, gate, ow = torch.randn(t, h, e, **f32), lowp[:, h * d:], torch.randn(e, **bf)
        flat = torch.randn(t, h * e, **bf)
        fw = torch.randn(h * e, **bf)
        entry(f"head norm + gate (like: norm), {kind}", lambda: ops.head_norm_gate(of, ow, 1e-5, gate, h * e), t * h * e * 8,
              0, (lambda: ops.rms_norm(flat, fw, 1e-6), t * h * e * 4, 0))
        del proj, lowp, cache, q, qf, kf, gf, vf, of
        gc.collect()
        torch.cuda.empty_cache()
    ops.check_status()
    return out


# ----------------------------------------------------------------------------- Gatosun
# width, q heads, kv heads, head size, window, time-mixing heads and size, linear-attention heads, row and column
# size, experts, top-k, expert width
GATOSUN_SIZES: Dict[str, Tuple[int, ...]] = {
    "2048x16h/4kv/128 w1024 t32x64 g4x256/512 e64k6 ff1024": (2048, 16, 4, 128, 1024, 32, 64, 4, 256, 512, 64, 6, 1024),
    "4096x32h/8kv/128 w512 t64x64 g32x128/128 e32k4 ff2048": (4096, 32, 8, 128, 512, 64, 64, 32, 128, 128, 32, 4, 2048),
    "2880x64h/8kv/64 w128 t45x64 g15x96/192 e32k4 ff2880": (2880, 64, 8, 64, 128, 45, 64, 15, 96, 192, 32, 4, 2880),
}
GATOSUN_LAYERS = 6           # two of each mixer
DECAY_RANK = 64


def gatosun(size) -> ModelConfig:
    w, hq, hk, d, win, th, td, gh, gd, ge, e, k, ff = size
    ex = ExpertSpec(ff, "relu2")
    mlp = MoESpec(e, k, ex, ex, "sigmoid", renormalize=False, n_group=4, topk_group=2, correction=True)
    full = AttentionSpec(hq, hk, d, d, d, 1e6, d ** -0.5, True, 0, qk_norm="projection", bias=True, value_mix=True)
    left = AttentionSpec(hq, hk, d, d, d, 1e6, d ** -0.5, True, win, qk_norm="head")
    specs = (LayerSpec(full, mlp), LayerSpec(ParallelSpec(left, TimeMixSpec(th, td, DECAY_RANK), 0.6, 0.5), mlp),
             LayerSpec(DecayLinearSpec(gh, gd, ge, 16.0, DECAY_RANK), mlp))
    return ModelConfig(architecture="Gatosun", model_type="gatosun", hidden_size=w, num_layers=GATOSUN_LAYERS, num_heads=hq,
                       num_kv_heads=hk, head_dim=d, vocab_size=VOCAB, max_position_embeddings=1 << 16,
                       layer_specs=specs * (GATOSUN_LAYERS // 3), residual_mult=0.3, num_experts=e, num_experts_per_tok=k)


def qwen3_moe_full(size) -> ModelConfig:
    w, hq, hk, d, *_, e, k, ff = size
    mc = qwen3_moe((w, hq, hk, d, 0, e, k, ff))
    mc.num_layers = GATOSUN_LAYERS
    return mc


def gatosun_kernels(size) -> List[dict]:
    w, hq, hk, d, win, th, td, gh, gd, ge, e, k, ff = size
    bw, fl = _peaks()
    out: List[dict] = []
    bf, f32, i32 = (dict(dtype=t, device="cuda") for t in (torch.bfloat16, torch.float32, torch.int32))

    def entry(name: str, fn, nbytes: float, flops: float = 0.0, like: Optional[Tuple] = None, peak: float = fl):
        """``like``: (call, bytes, FLOPs[, FLOP rate]) of the like kernel."""
        ms = _time(fn)
        bound = max(nbytes / bw, flops / peak) * 1e3
        r = {"kernel": f"{name}, {kind}", "ms": round(ms, 4), "roofline": round(bound / ms, 3)}
        if like is not None:
            lms = _time(like[0])
            lb = max(like[1] / bw, like[2] / (like[3] if len(like) > 3 else fl)) * 1e3
            r.update(like_ms=round(lms, 4), like_roofline=round(lb / lms, 3),
                     distance=round((lb / lms) / (bound / ms), 2))
        out.append(r)

    def gemm_cost(rows, weight, live=None):
        n, c = weight.shape[-2:]
        return (rows * (n + c) + (live or 1) * n * c) * 2, 2.0 * rows * n * c

    bs, group = 64, 4
    for kind, n, rows in (("prefill", 8, 1024), ("decode b1", 1, 1), ("decode b16", 16, 1), ("decode b128", 128, 1)):
        t, pre = n * rows, kind == "prefill"
        ctx = rows if pre else CONTEXT
        x = torch.randn(t, w, **bf)
        cu, lens = torch.arange(0, (n + 1) * rows, rows, **i32), torch.full((n,), ctx, **i32)
        slots, idx = torch.arange(n, **i32), torch.arange(n, **i32).repeat_interleave(rows)
        states = (slots, cu, lens, n)
        gain = torch.randn(w, **bf)
        res16 = torch.randn(t, w, **bf)
        add_norm = (lambda: ops.fused_add_rms_norm(x, res16, gain, 1e-6), t * w * 8, 0.0)

        def product(name, cols, like_cols, bias=False, act=None, like_act=None, pairs=False):
            a, b = torch.randn(cols, w, **bf), torch.randn(like_cols, w, **bf)
            bb = torch.randn(cols, **bf) if bias else None
            halve = lambda c, cols: (c[0] - t * cols, c[1])                              # noqa: E731
            own, other = gemm_cost(t, a), gemm_cost(t, b)
            entry(name, lambda: ops.gemm(x, a, bb, **(act or {})), *(halve(own, cols) if pairs else own),
                  like=(lambda: ops.gemm(x, b, **(like_act or {})), *(halve(other, like_cols) if like_act else other)))

        # ---- attention: full with projection norms, and windowed with unit heads
        qkv_cols = (hq + 2 * hk) * d
        product("q / k / v with bias (like: q / k / v)", qkv_cols, qkv_cols, bias=True)
        per = (ctx + bs - 1) // bs
        kc, vc = (torch.randn(n * per, hk, bs, d, **bf) for _ in range(2))
        bt = torch.randperm(n * per, device="cuda").int().view(n, per)
        pos = torch.arange(ctx - rows, ctx, **i32).repeat(n)
        slot = (bt.long().gather(1, (pos.view(n, rows) // bs).long()) * bs + pos.view(n, rows) % bs).int().view(-1)
        cs = torch.randn(CONTEXT + 128, d, **f32)
        qkv = torch.randn(t, qkv_cols, **bf)
        q, kk, vv = qkv.split([hq * d, hk * d, hk * d], 1)
        first = torch.randn(t, hk * d, **bf)
        qn, kn, hn = torch.randn(hq * d, **bf), torch.randn(hk * d, **bf), torch.randn(d, **bf)
        moved = t * (2 * hq + 4 * hk) * d * 2

        def like_prep():
            a = ops.rms_norm(q.reshape(-1, d), hn, 1e-6).view(t, -1)
            b = ops.rms_norm(kk.reshape(-1, d), hn, 1e-6).view(t, -1)
            ops.rope_cache_gqa_(a, b, vv, kc, vc, pos, slot, cs, d, d, True)

        prep = lambda norm, wts, vf: ops.qk_norm_rope_cache(q, kk, vv, kc, vc, pos, slot, cs, d, d, d, norm, 1e-6, wts,  # noqa: E731
                                                            None, vf, 0.4)
        entry("projection norm + rotation + values + cache (like: head norms + rotation + cache)",
              lambda: prep("projection", (qn, kn), first), moved + t * hk * d * 2, 0, (like_prep, moved, 0.0))
        entry("rotation + unit heads + cache (like: head norms + rotation + cache)", lambda: prep("head", None, None), moved,
              0, (like_prep, moved, 0.0))
        o = torch.empty(t, hq * d, **bf)
        for name, window in (("full", 0), ("windowed", win)):
            pairs = sum(min(window or ctx, p + 1) for p in range(ctx - rows, ctx))
            cost = (n * hk * 4 * d * min(ctx, (window or ctx) + rows - 1) + t * hq * d * 4, 4.0 * n * hq * d * pairs)

            def own_attn(window=window):
                ops.gated_attention(q, None, kc, vc, o, bt, cu if pre else None, lens, n, rows, hq, d, d, d ** -0.5, window,
                                    None, max_seq_len=ctx)

            def like_attn(window=window):
                if pre:
                    return ops.gqa_prefill(q, kc, vc, bt, cu, lens, n, rows, hq, d ** -0.5, True, window)
                return ops.gqa_decode(q, kc, vc, bt, lens, n, hq, d ** -0.5, 1, window, max_seq_len=ctx)
            entry(f"attention, {name} (like: the same)", own_attn, *cost, like=(like_attn, *cost))
        del kc, vc, qkv, q, kk, vv
        # ---- time mixing
        mu, shift = torch.rand(5, w, **bf), torch.zeros(n, w, **f32)
        entry("blends with the previous token (like: add + norm)", lambda: ops.token_mix(x, mu, shift, idx, *states),
              t * w * 2 * 6 + n * w * 8, 0, add_norm)
        mixed, offs = ops.token_mix(x, mu, shift, idx, *states)
        tm = th * td
        rkvg = torch.randn(4, tm, w, **bf)
        flat = rkvg.view(4 * tm, w)

        def four():
            if pre:
                return [ops.gemm(mixed[i * t: (i + 1) * t], rkvg[i]) for i in range(4)]
            return ops.grouped_gemm(mixed[: 4 * t], rkvg, offs[:5])
        entry("r / k / v / gate of four blends (like: one product)", four,
              (4 * t * (w + tm) + 4 * tm * w) * 2, 8.0 * t * tm * w, (lambda: ops.gemm(x, flat), *gemm_cost(t, flat)))
        w1, w2 = torch.randn(DECAY_RANK, w, **bf), torch.randn(tm, DECAY_RANK, **bf)
        entry("low rank + tanh", lambda: ops.gemm(mixed[4 * t:], w1, unary="tanh"), *gemm_cost(t, w1))
        low = ops.gemm(mixed[4 * t:], w1, unary="tanh")
        entry("decays from the low rank, fp32", lambda: ops.gemm(low, w2, out_dtype=torch.float32),
              gemm_cost(t, w2)[0] + t * tm * 2, gemm_cost(t, w2)[1])
        y4 = torch.randn(4 * t, tm, **bf)
        r, kt, vt, gt = y4.split(t)
        z, w0, u = torch.randn(t, tm, **f32), torch.randn(tm, **f32), torch.randn(th, td, **f32)
        like_lin = torch.randn(t, 2 * tm, **bf)
        entry("time mixing: r, k, decays, bonus (like: q and keys of gated linear attention)",
              lambda: ops.time_mix_prep(r, kt, z, w0, u, th, td), t * tm * (4 + 4 + 12), 0,
              (lambda: ops.gated_linear_prep(like_lin, 0, tm, th, td, w0, w0), t * tm * (4 + 8), 0.0))
        rf, kf, gf, beta = ops.time_mix_prep(r, kt, z, w0, u, th, td)
        state = torch.zeros(n, th, td, td, **f32)
        cost = (t * th * 18 * td + n * th * td * td * 8, 5.0 * t * th * td * td)
        like_cost = (t * th * 14 * td + n * th * td * td * 8, cost[1], FP32_FLOPS)
        entry("time mixing: scan (like: scan of gated linear attention)",
              lambda: ops.recurrent_scan(rf, kf, gf, vt, beta, state, th, td, *states, bonus=True), *cost,
              like=(lambda: ops.recurrent_scan(rf, kf, None, vt, None, state, th, td, *states), *like_cost), peak=FP32_FLOPS)
        of, nw, sw = torch.randn(t, th, td, **f32), torch.randn(th, td, **bf), torch.randn(td, **bf)
        wide = torch.empty(t, hq * d + tm, **bf)
        entry("time mixing: head norm + silu gate (like: head norm + gate)",
              lambda: ops.head_norm_gate(of, nw, 1e-5, gt, silu=True, scale=0.8, out=wide[:, hq * d:]), t * tm * 8, 0,
              (lambda: ops.head_norm_gate(of, sw, 1e-5, gt, tm), t * tm * 8, 0.0))
        both, wo = torch.randn(w, hq * d + tm, **bf), torch.randn(w, hq * d, **bf)
        entry("output of both halves (like: output projection)", lambda: ops.gemm(wide, both), *gemm_cost(t, both),
              like=(lambda: ops.gemm(o, wo), *gemm_cost(t, wo)))
        del mixed, rkvg, flat, y4, rf, kf, gf, of, wide, both
        # ---- decayed linear attention
        gn, gm = gh * gd, gh * ge
        product("projection, decayed linear attention (like: q / k / v)", 2 * gn + 2 * gm + DECAY_RANK, qkv_cols)
        proj = torch.randn(t, 2 * gn + 2 * gm + DECAY_RANK, **bf)
        q2, k2, v2, g2 = proj[:, : 2 * gn + 2 * gm].split([gn, gn, gm, gm], 1)
        z2, b2 = torch.randn(t, gn, **f32), torch.randn(gn, **f32)
        entry("decayed linear: q, k, decays (like: q and keys of gated linear attention)",
              lambda: ops.decay_prep(q2, k2, z2, b2, gh, gd, gd ** -0.5, 16.0), t * gn * (4 + 4 + 12), 0,
              (lambda: ops.gated_linear_prep(proj, 0, gn, gh, gd, b2, b2), t * gn * (4 + 8), 0.0))
        qf, kf, gf = ops.decay_prep(q2, k2, z2, b2, gh, gd, gd ** -0.5, 16.0)
        state = torch.zeros(n, gh, ge, gd, **f32)
        cost = (t * gh * (12 * gd + 6 * ge) + n * gh * gd * ge * 8, 5.0 * t * gh * gd * ge)
        like_cost = (t * gh * (8 * gd + 6 * ge) + n * gh * gd * ge * 8, cost[1], FP32_FLOPS)
        entry("decayed linear: scan (like: scan of gated linear attention)",
              lambda: ops.recurrent_scan(qf, kf, gf, v2, None, state, gh, ge, *states), *cost,
              like=(lambda: ops.recurrent_scan(qf, kf, None, v2, None, state, gh, ge, *states), *like_cost), peak=FP32_FLOPS)
        of, nw = torch.randn(t, gh, ge, **f32), torch.randn(ge, **bf)
        entry("decayed linear: head norm + silu gate (like: head norm + gate)",
              lambda: ops.head_norm_gate(of, nw, 1e-5, g2, gm, silu=True), t * gm * 8, 0,
              (lambda: ops.head_norm_gate(of, nw, 1e-5, g2, gm), t * gm * 8, 0.0))
        del proj, q2, k2, v2, g2, qf, kf, gf, of, state
        # ---- feed-forwards and the residual
        product("gate/up + bias + gelu (like: gate/up + silu)", 4 * ff, 4 * ff, bias=True,
                act=dict(swiglu=True, act=ops.GELU_TANH), like_act=dict(swiglu=True), pairs=True)
        ids = torch.stack([torch.randperm(e, device="cuda")[:k] for _ in range(min(t, 512))]).repeat(
            (t + 511) // 512, 1)[:t].int()
        counts = torch.bincount(ids.view(-1).long(), minlength=e)
        offs = torch.zeros(e + 1, **i32)
        offs[1:] = counts.cumsum(0)
        live = int((counts > 0).sum())
        xr, w13 = torch.randn(t * k, w, **bf), torch.randn(e, 2 * ff, w, **bf)
        up = w13[:, :ff].contiguous()
        nb, nf = gemm_cost(t * k, w13, live)
        entry("experts up + squared relu (like: experts gate/up + silu)",
              lambda: ops.grouped_gemm(xr, up, offs, unary="relu2"), *gemm_cost(t * k, up, live),
              like=(lambda: ops.grouped_gemm(xr, w13, offs, swiglu=True), nb - t * k * 2 * ff, nf))
        del w13, up
        res = torch.randn(t, w, **f32)
        entry("residual + norm (like: add + norm)",
              lambda: ops.residual_add_norm(res, x, None, None, gain, 1e-6, 0.0, w, mult=0.3), t * w * 12, 0, add_norm)
        wt, rslots = torch.rand(t, k, **f32), torch.randperm(t * k, device="cuda").int()
        from ..layers.moe import _solo_group
        from ..layers.moe_dispatch import DispatchHandle, EpBuffers, ep_combine
        buf = EpBuffers(_solo_group(), torch.device("cuda", torch.cuda.current_device()), e, w, t, k)
        handle = DispatchHandle(ids, wt, rslots, t, t * k, offs)

        def like_end():
            ops.fused_add_rms_norm(ep_combine(None, buf.expert_y, handle, x, buf), res16, gain, 1e-6)
        entry("experts' rows + shared + residual + norm (like: combine, add + norm)",
              lambda: ops.residual_add_norm(res, None, x, (xr, rslots, wt), gain, 1e-6, 0.0, w, mult=0.3),
              t * w * (2 * k + 2 + 8 + 2), 0, (like_end, t * w * (2 * k + 2 + 8), 0.0))
        logits, corr = torch.randn(t, e, **f32), torch.randn(e, **f32)
        entry("routing, sigmoid + correction + groups (like: softmax)",
              lambda: ops.moe_topk(logits, corr, k, True, group, 2, False, 1.0), t * (e + 2 * k) * 4, 0,
              (lambda: ops.moe_topk(logits, None, k, False, 1, 1, True, 1.0), t * (e + 2 * k) * 4, 0.0))
        del x, xr, buf, res, res16
        gc.collect()
        torch.cuda.empty_cache()
    ops.check_status()
    return out


# ----------------------------------------------------------------------------- Dalavik
# width, heads, rotated keys, latent, query latent (head and value size of the latent layers: 128), key/value heads, head
# and value size of the mixed-score layers, feed-forward, token input, norm groups
DALAVIK_SIZES: Dict[str, Tuple[int, ...]] = {
    "2048x16h/128 q768 g4x128/128 ff8192 s128": (2048, 16, 64, 512, 768, 4, 128, 128, 8192, 128, 2),
    "4096x32h/128 q1536 g8x128/128 ff12288 s256": (4096, 32, 64, 512, 1536, 8, 128, 128, 12288, 256, 4),
    "3072x24h/128 q1024 g6x96/64 ff8192 s256": (3072, 24, 64, 512, 1024, 6, 96, 64, 8192, 256, 8),
}
DALAVIK_LAYERS = 6           # two of each: own latent rows, shared ones, mixed scores
DALAVIK_HEAD = 128
SOFTCAP, QUERY_TEMPERATURE = 30.0, (0.1, 512)


def dalavik(size) -> ModelConfig:
    w, h, rot, rank, qr, g, d, e, ff, side, groups = size
    hd, mlp = DALAVIK_HEAD, DenseSpec(ff, ops.RELU)

    def lat(source):
        return LayerSpec(LatentAttentionSpec(h, hd, rot, hd, rank, 1e4, (hd + rot) ** -0.5, False, qr, source), mlp)
    mixed = LayerSpec(AttentionSpec(h, g, d, e, 0, 0.0, d ** -0.5, qk_norm="head_weight", bias=True, softcap=SOFTCAP,
                                    query_temperature=QUERY_TEMPERATURE, distance_bias=True, score_mix=True,
                                    head_sink=True), mlp)
    return ModelConfig(architecture="Dalavik", model_type="dalavik", hidden_size=w, num_layers=DALAVIK_LAYERS, num_heads=h,
                       num_kv_heads=1, head_dim=hd, v_head_dim=hd, vocab_size=VOCAB, max_position_embeddings=1 << 16,
                       layer_specs=(lat(None), mixed, lat(0), lat(None), mixed, lat(3)), tie_word_embeddings=True,
                       norm_groups=groups, token_side_dim=side)


def deepseek_query_latent(size) -> ModelConfig:
    w, h, rot, rank, qr, _, _, _, ff, _, _ = size
    hd = DALAVIK_HEAD
    return ModelConfig(architecture="DeepseekV2ForCausalLM", model_type="deepseek_v2", hidden_size=w,
                       num_layers=DALAVIK_LAYERS, num_heads=h, num_kv_heads=h, head_dim=hd + rot, intermediate_size=ff,
                       vocab_size=VOCAB, max_position_embeddings=1 << 16, rope_neox=False, use_mla=True, q_lora_rank=qr,
                       kv_lora_rank=rank, qk_nope_head_dim=hd, qk_rope_head_dim=rot, v_head_dim=hd)


def dalavik_kernels(size) -> List[dict]:
    from ..attention.latent import LatentAttention
    w, h, rot, rank, qr, kvh, d, e, ff, side, groups = size
    hd = DALAVIK_HEAD
    bw, fl = _peaks()
    out: List[dict] = []
    bf = dict(dtype=torch.bfloat16, device="cuda")
    f32 = dict(dtype=torch.float32, device="cuda")
    i32 = dict(dtype=torch.int32, device="cuda")

    def bound(nbytes: float, flops: float = 0.0, fp32: float = 0.0, special: float = 0.0) -> float:
        return max(nbytes / bw, flops / fl, fp32 / FP32_FLOPS, special / SPECIAL_OPS) * 1e3

    def entry(name: str, fn, cost, like=None, like_cost=None):
        ms, b = _time(fn), bound(*cost)
        r = {"kernel": f"{name}, {kind}", "ms": round(ms, 4), "roofline": round(b / ms, 3)}
        if like is not None:
            lms, lb = _time(like), bound(*(like_cost or cost))
            r.update(like_ms=round(lms, 4), like_roofline=round(lb / lms, 3), distance=round((lb / lms) / (b / ms), 2))
        out.append(r)

    bs, qk, row = 64, hd + rot, rank + rot
    for kind, n, rows in (("prefill", 8, 1024), ("decode b1", 1, 1), ("decode b16", 16, 1), ("decode b128", 128, 1)):
        t, pre = n * rows, kind == "prefill"
        ctx = rows if pre else CONTEXT
        x, gain = torch.randn(t, w, **bf), torch.randn(w, **bf)
        res, res16 = torch.randn(t, w, **f32), torch.randn(t, w, **bf)

        def add_norm():
            ops.fused_add_rms_norm(x, res16, gain, 1e-6)
        entry("norm of the result + add (like: add + norm)",
              lambda: ops.post_norm_residual(res, x, gain, groups, 1e-6, w), (t * w * 12,), add_norm, (t * w * 8,))
        entry("the same + final norm (like: add + norm)",
              lambda: ops.post_norm_residual(res, x, gain, 1, 1e-6, w, out_norm=(gain, groups)), (t * w * 12,), add_norm,
              (t * w * 8,))

        def cost(a, b, cols=None):
            return (a.numel() + b.numel() + a.shape[0] * (cols or b.shape[0])) * 2, 2.0 * a.shape[0] * b.numel()

        def product(name, a, cols, like_cols, like_a=None, bias=False, act=None, like_act=None):
            la = a if like_a is None else like_a
            wa, wb = torch.randn(cols, a.shape[1], **bf), torch.randn(like_cols, la.shape[1], **bf)
            bb = torch.randn(cols, **bf) if bias else None
            entry(name, lambda: ops.gemm(a, wa, bb, **(act or {})), cost(a, wa, cols // 2 if act else None),
                  lambda: ops.gemm(la, wb, **(like_act or {})), cost(la, wb, like_cols // 2 if like_act else None))
        qkv = (h + kvh) * d + kvh * e
        product("query and key latents (like: the same of MLA)", x, qr + row, qr + row)
        product("query latent alone (like: both latents of MLA)", x, qr, qr + row)
        zq = torch.randn(t, qr, **bf)
        product("queries from their latent (like: the same of MLA)", zq, h * qk, h * qk)
        product("q / k / v with bias (like: q of MLA)", x, qkv, h * qk, zq, bias=True)
        product("gate / up + relu (like: gate / up + silu)", x, 2 * ff, 2 * ff, act=dict(swiglu=True, act=ops.RELU),
                like_act=dict(swiglu=True))
        sp = (side + 7) // 8 * 8
        product("token input: gate (like: router of 128 experts)", x, sp, 128)
        z = torch.randn(t, sp, **bf)
        low = torch.randn(t, 2 * LOW_RANK, **bf)
        product("token input: back (like: low-rank product of Fuvirax)", z, w, h * 2 * hd, low)
        ids, table = torch.randint(0, VOCAB, (t,), **i32), torch.randn(VOCAB, side * DALAVIK_LAYERS, **bf)
        gu = torch.randn(t, 2 * sp, **bf)
        entry("token input: gated rows (like: silu(gate) * up)", lambda: ops.gelu_rows(z, ids, table, side, side),
              (t * side * 6,), lambda: ops.silu_and_mul(gu))
        del gu, table

        # ---- latent attention
        cu, lens = torch.arange(0, (n + 1) * rows, rows, **i32), torch.full((n,), ctx, **i32)
        per = (ctx + bs - 1) // bs
        cache = torch.randn(n * per, bs, row, **bf)
        bt = torch.randperm(n * per, device="cuda").int().view(n, per)
        pos = torch.arange(ctx - rows, ctx, **i32).repeat(n)
        slot = (bt.long().gather(1, (pos.view(n, rows) // bs).long()) * bs + pos.view(n, rows) % bs).int().view(-1)
        cs = torch.randn(CONTEXT + 128, rot, device="cuda")
        q, y = torch.randn(t, h * qk, **bf), torch.randn(t, qr + row, **bf)
        low, kv_a, c_q = y[:, :qr], y[:, qr:], torch.empty(t, qr, **bf)
        low_c = low.contiguous()
        attn = LatentAttention(h, hd, rot, hd, rank, qk ** -0.5, False, 1e-5, torch.bfloat16, torch.device("cuda"), qr)
        attn.w_uk.data.normal_(std=0.02)
        attn.w_uv.data.normal_(std=0.02)
        attn.build_absorbed()
        q_lat = torch.empty(t, h, row, **bf)

        def like_norms():
            ops.rms_norm(low_c, attn.query_norm, 1e-5)
            ops.mla_kv_rmsnorm_rope_cache(kv_a[:, :rank], kv_a[:, rank:], attn.latent_norm, cache, pos, slot, cs, 1e-5, False)

        def like_rotate():
            pe = q.view(t, h, qk)[:, :, hd:].reshape(t, h * rot).contiguous()
            ops.rope_qk_(pe, pe.new_empty(t, 0), pos, cs, rot, rot, False)
        prep = (attn.latent_norm, 1e-5, cache, pos, slot, cs, h, hd, rot, rank, False)
        entry("norms of both latents + rotation + cache (like: norm; norm + rotation + cache)",
              lambda: ops.latent_prep_(None, kv_a, *prep, low=(low, attn.query_norm, c_q)), (t * (2 * row + 2 * qr) * 2,),
              like_norms)
        entry("norm of the query latent (like: norm)",
              lambda: ops.latent_prep_(None, None, *prep, low=(low, attn.query_norm, c_q)), (t * qr * 4,),
              lambda: ops.rms_norm(low_c, attn.query_norm, 1e-5))
        entry("rotation of the queries (like: the same)",
              lambda: ops.latent_prep_(q, None, *prep, None if pre else q_lat, 0 if pre else t), (t * h * rot * 4,),
              like_rotate)
        pairs = n * h * sum(p + 1 for p in range(ctx - rows, ctx))
        if pre:
            start = (torch.cumsum(lens, 0) - lens).int()
            gathered = ops.latent_gather(cache, bt, lens, start, n, t, ctx)

            def own_keys():
                r = ops.latent_gather(cache, bt, lens, start, n, t, ctx)
                return ops.gemm(r, attn.w_key), ops.gemm(r, attn.w_value)
            kvb = torch.randn(h * 2 * hd, rank, **bf)

            def like_keys():
                lat = cache.index_select(0, bt.view(-1).long())
                kv = ops.gemm(lat[..., :rank].reshape(-1, rank).contiguous(), kvb).view(-1, bs, h, 2 * hd)
                pe = lat[..., rank:].unsqueeze(2).expand(-1, bs, h, rot)
                k = torch.cat([kv[..., :hd], pe], -1).permute(0, 2, 1, 3).contiguous()
                return k, kv[..., hd:].permute(0, 2, 1, 3).contiguous()
            kc_ = t * (row + h * (qk + hd)) * 2 + kvb.numel() * 2, 2.0 * t * kvb.numel()
            entry("keys and values from the latents (like: the same)", own_keys, kc_, like_keys)
            entry("keys and values from shared rows (like: with the gather)",
                  lambda: (ops.gemm(gathered, attn.w_key), ops.gemm(gathered, attn.w_value)), kc_, like_keys)
            k, v = own_keys()
            o = torch.empty(t, h * hd, **bf)
            lk, lv = like_keys()
            lbt = torch.arange(n * per, **i32).view(n, per)
            entry("latent attention (like: the same)",
                  lambda: ops.contiguous_attention(q, k.view(-1, h, 1, qk), v.view(-1, h, 1, hd), o, cu, start, lens, n, rows,
                                                   h, qk, hd, 0.07), (t * h * (2 * qk + 2 * hd) * 2, 2.0 * pairs * (qk + hd)),
                  lambda: ops.gqa_prefill(q, lk, lv, lbt, cu, lens, n, rows, h, 0.07, True, 0))
            del k, v, lk, lv, gathered
        else:
            lat_o, o = torch.empty(t, h, rank, **bf), torch.empty(t, h * hd, **bf)
            heads, uv = q.view(t, h, qk), attn.w_uv.view(h, hd, rank)
            offs = torch.arange(0, (h + 1) * t, t, **i32)

            def like_fold():
                qn = heads[..., :hd].transpose(0, 1).reshape(h * t, hd).contiguous()
                ql = ops.grouped_gemm(qn, attn.w_fold, offs).view(h, t, rank).transpose(0, 1)
                return torch.cat([ql, q_lat[..., rank:]], -1).reshape(t, h * row).contiguous()

            def like_unfold():
                a = lat_o.transpose(0, 1).reshape(h * t, rank).contiguous()
                return ops.grouped_gemm(a, uv, offs).view(h, t, hd).transpose(0, 1).reshape(t, h * hd).contiguous()
            fc = (h * hd * rank + t * h * (hd + rank)) * 2, 2.0 * t * h * hd * rank
            entry("queries into the latent space (like: the same)",
                  lambda: ops.head_gemm(heads[..., :hd], attn.w_fold, q_lat[..., :rank]), fc, like_fold)
            entry("results out of the latent space (like: the same)", lambda: ops.head_gemm(lat_o, uv, o.view(t, h, hd)), fc,
                  like_unfold)
            q_flat = torch.randn(t, h * row, **bf)
            entry("latent attention (like: the same)",
                  lambda: ops.latent_decode(q_flat.view(t, h, row), cache, bt, lens, n, h, rank, 0.07, lat_o,
                                            max_seq_len=CONTEXT),
                  ((n * ctx * row + t * h * (row + rank)) * 2, 2.0 * pairs * (row + rank)),
                  lambda: ops.mla_decode(q_flat, cache, bt, lens, n, h, 0.07, 1, max_seq_len=CONTEXT))
        del cache, q, y, q_lat, attn
        # ---- attention with mixed scores; the like kernels are those of grouped-query attention
        kc, vc = torch.randn(n * per, kvh, bs, d, **bf), torch.randn(n * per, kvh, bs, e, **bf)
        lvc = vc if e == d else torch.randn(n * per, kvh, bs, d, **bf)
        y = torch.randn(t, qkv, **bf)
        q, kk, vv = y.split([h * d, kvh * d, kvh * e], 1)
        lv_ = torch.randn(t, kvh * d, **bf)
        hn, cs = torch.randn(d, **bf), torch.randn(CONTEXT + 128, d, **f32)

        def like_prep():
            a = ops.rms_norm(q.reshape(-1, d), hn, 1e-6).view(t, -1)
            b = ops.rms_norm(kk.reshape(-1, d), hn, 1e-6).view(t, -1)
            ops.rope_cache_gqa_(a, b, lv_, kc, lvc, pos, slot, cs, d, d, True)
        entry("head norms + query temperature + cache (like: head norms + rotation + cache)",
              lambda: ops.qk_norm_rope_cache(q, kk, vv, kc, vc, pos, slot, None, d, e, 0, "head_weight", 1e-6, (hn, hn),
                                             temperature=QUERY_TEMPERATURE), (t * (2 * (h + kvh) * d + 2 * kvh * e) * 2,),
              like_prep, (t * (2 * h + 4 * kvh) * d * 2,))
        o, lo = torch.empty(t, h * e, **bf), torch.empty(t, h * d, **bf)
        r1, r2, sink = torch.rand(h, **f32), torch.rand(h, **f32) * 0.1, torch.randn(h, **f32)
        talk = (torch.eye(h, **f32) + 0.1 * torch.randn(h, h, **f32)).bfloat16().float()
        qc = q.contiguous()

        def like_attn():
            if not pre and d == 128:
                return ops.gqa_decode(qc, kc, lvc, bt, lens, n, h, d ** -0.5, 1, 0, max_seq_len=ctx)
            if d == e == 128:
                return ops.gqa_prefill(qc, kc, vc, bt, cu, lens, n, rows, h, d ** -0.5, True, 0)
            return ops.gated_attention(qc, None, kc, vc, o, bt, cu if pre else None, lens, n, rows, h, d, e, d ** -0.5, 0, None,
                                       max_seq_len=ctx)
        kv = n * kvh * ctx * 2
        le = e if pre or d != 128 else d
        entry("attention with mixed scores (like: grouped-query attention)",
              lambda: ops.mixed_attention(qc, kc, vc, o, bt, cu if pre else None, lens, n, rows, d, e, d ** -0.5, SOFTCAP,
                                          (r1, r2), talk, sink, max_seq_len=ctx, talk_exact=True),
              (kv * (d + e) + t * h * (d + e) * 2, 2.0 * pairs * (d + e), 2.0 * pairs * h, 3.0 * pairs), like_attn,
              (kv * (d + le) + t * h * (d + le) * 2, 2.0 * pairs * (d + le), 0.0, 1.0 * pairs))
        del kc, vc, lvc, y, q, kk, vv, qc, res
        gc.collect()
        torch.cuda.empty_cache()
    ops.check_status()
    return out


DESIGNS = {
    "rivudra": (SIZES, LAYERS, kernels, {"rivudra": rivudra, "qwen3-moe": qwen3_moe}),
    "fuvirax": (FUVIRAX_SIZES, FUVIRAX_LAYERS, fuvirax_kernels, {"fuvirax": fuvirax, "deepseek-v2 dense": deepseek_dense}),
    "gatosun": (GATOSUN_SIZES, GATOSUN_LAYERS, gatosun_kernels, {"gatosun": gatosun, "qwen3-moe": qwen3_moe_full}),
    "dalavik": (DALAVIK_SIZES, DALAVIK_LAYERS, dalavik_kernels,
                {"dalavik": dalavik, "deepseek-v2 dense": deepseek_query_latent}),
}


def run(design: str, only: Optional[str] = None) -> None:
    sizes, layers, kernel_table, models = DESIGNS[design]
    ops.load_extension(required=True)
    for name, size in sizes.items():
        if only and only not in name:
            continue
        line = {"design": design, "size": name, "layers": layers, "dtype": "bf16", "data": "random",
                "l2_policy": "kernels: 256 MB written before each; steps: weights and cache above L2",
                "kernels": kernel_table(size), "steps": {k: model_steps(make(size)) for k, make in models.items()}}
        print(json.dumps(line), flush=True)
