"""Replays a trace of token ids through the engine, step by step, and returns logits.

The trace says which tokens of which requests each step brings; nothing is sampled.  Everything below
that decision is the engine's own: the scheduler's block pool and batch (``schedule_portions``), the
model runner's step (``execute_with_logits``: staging, prefill or captured decode graph, kernels) and the
paged cache.  ``bin/trace_run`` is the command line.

Steps come as JSON objects, one a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["b"]}

``entries``: the next tokens of requests (a request is admitted at its first entry) and the places among
them whose logits are wanted; ``end``: requests whose cache blocks and slot are given back after the step.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict, List, Optional, Sequence

import torch

from ..config import ModelConfig
from .llm import LLMEngine, build_engine_config
from .request import Request, SamplingParams


class TraceReplay:
    def __init__(self, model_dir: str, dtype: str = "bfloat16", max_tokens: int = 8192, max_live: int = 4,
                 block_size: int = 16, device: str = "cuda", **engine_args) -> None:
        mc = ModelConfig.from_pretrained(model_dir, dtype=dtype)
        blocks = (max_tokens + block_size - 1) // block_size
        cfg = build_engine_config(mc, model_path=model_dir, max_num_seqs=max_live, max_num_batched_tokens=max_tokens,
                                  max_model_len=max_tokens, block_size=block_size, num_gpu_blocks=blocks,
                                  device=device, **engine_args)
        self.engine = LLMEngine(cfg, before_capture=lambda runner: setattr(runner, "keep_logits", True))
        self.runner = self.engine.worker.model_runner
        self.vocab = mc.vocab_size
        self.live: Dict[str, Request] = {}

    def step(self, entries: Sequence[dict], end: Sequence[str] = ()) -> Optional[torch.Tensor]:
        """Run one step; logits fp32 [wanted, vocab] in the order of the entries, None if none are wanted."""
        sched = self.engine.scheduler
        portions, index = [], {}
        for e in entries:
            tokens = [int(t) for t in e["tokens"]]
            if not tokens:
                continue
            if min(tokens) < 0 or max(tokens) >= self.vocab:
                raise ValueError(f"request {e['id']}: token id outside the vocabulary of {self.vocab}")
            req = self.live.get(e["id"])
            if req is None:
                req = self.live[e["id"]] = Request(e["id"], [], SamplingParams(ignore_eos=True))
            req.prompt_token_ids.extend(tokens)
            portions.append((req, len(tokens)))
        logits = None
        if portions:
            out = sched.schedule_portions(portions)
            row = 0
            for s in out.seqs:
                index[s.request.request_id] = row
                row += s.num_new_tokens
            rows: List[int] = [index[e["id"]] + int(w) for e in entries for w in e.get("want", ())]
            if out.kind == "decode":
                for s in out.seqs:             # rows of the decode batch are entered at admission
                    self.runner.input_batch.add_request(s.request)
            logits = self.runner.execute_with_logits(out, rows)
            sched.commit_portions(out)
        for rid in end:
            req = self.live.pop(rid, None)
            if req is not None:
                sched.abort_request(rid)
                self.runner.input_batch.remove_request(rid)
        return logits

    def check(self) -> None:
        if self.engine.device.type == "cuda":
            from .. import ops
            ops.check_status(self.engine.device)


def main(argv: Optional[Sequence[str]] = None) -> int:
    ap = argparse.ArgumentParser("trace_run", description="replay a trace of token ids and write logits")
    ap.add_argument("--model", required=True, help="directory with config.json and safetensors weights")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="directory for <step>.f32 (little-endian fp32 [wanted, vocab])")
    ap.add_argument("--max-tokens", type=int, required=True, help="cache pool: tokens that live requests hold at most")
    ap.add_argument("--max-live", type=int, default=4, help="requests alive at any time")
    ap.add_argument("--block-size", type=int, default=16)
    args = ap.parse_args(argv)
    replay = TraceReplay(args.model, args.dtype, args.max_tokens, args.max_live, args.block_size)
    for line in sys.stdin:
        if not line.strip():
            continue
        d = json.loads(line)
        logits = replay.step(d["entries"], d.get("end", ()))
        replay.check()
        if logits is not None:
            path = os.path.join(args.out, f"{d['step']}.f32")
            logits.contiguous().numpy().astype("<f4").tofile(path)
        print(f"done {d['step']}", flush=True)
    return 0
