"""Throughput of a design beside the framework's closest existing model at equal size (random weights).

``bench.py --design rivudra`` runs this on one GPU.  Per size it prints one JSON line with

* whole steps through the engine (device time of prompt and decode steps, CUDA events): Rivudra and a
  Qwen3-MoE of the same width, heads, experts and window;
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
from ..config import AttentionSpec, ExpertSpec, LayerSpec, ModelConfig, MoESpec

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


def run(design: str, only: Optional[str] = None) -> None:
    if design != "rivudra":
        raise SystemExit(f"no comparison for design {design!r}")
    ops.load_extension(required=True)
    for name, size in SIZES.items():
        if only and only not in name:
            continue
        line = {"design": design, "size": name, "layers": LAYERS, "dtype": "bf16", "data": "random",
                "l2_policy": "kernels: 256 MB written before each; steps: weights and cache above L2",
                "kernels": kernels(size), "steps": {"rivudra": model_steps(rivudra(size)),
                                                    "qwen3-moe": model_steps(qwen3_moe(size))}}
        print(json.dumps(line), flush=True)
