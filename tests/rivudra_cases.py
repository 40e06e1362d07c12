"""Small random Rivudra models and the checks that the CPU and GPU tests share: the framework's step
function, cache and scheduler against the plain implementation in rivudra_oracle.py."""
from __future__ import annotations

import json
import os
from typing import Dict, List, Sequence, Tuple

import torch
from safetensors.torch import save_file

import rivudra_oracle as oracle


def attn_layer(heads, kv, dim, vdim, rot, window, base=5000.0, scale=None, mlp=None) -> dict:
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "mask": {"size": window},
                      "rot": {"base": base, "dims": rot}, "scale": dim ** -0.5 if scale is None else scale}}


def moe(experts, top, ff, limit, groups=1, keep=1, scale=1.0, shared=None) -> dict:
    d = {"kind": "moe", "expert": {"ff": ff, "limit": limit},
         "router": {"experts": experts, "top": top, "scale": scale, "groups": {"count": groups, "keep": keep}}}
    if shared is not None:
        d["shared"] = {"ff": shared[0], "limit": shared[1]}
    return d


def model(width, vocab, layers, emb=3.0, eps=1e-4) -> dict:
    return {"architecture": "Rivudra", "width": width, "vocab": vocab, "embedding": {"scale": emb},
            "norm": {"eps": eps}, "layers": layers}


# unequal layers; a layer without a feed-forward; partial rotation; one group and several; no shared expert
VARIED = model(96, 203, [
    attn_layer(4, 2, 24, 40, 16, 10, mlp=moe(8, 3, 40, 0.8, 4, 2, 1.7, shared=(24, 1.1))),
    attn_layer(5, 1, 16, 16, 8, 33, base=900.0, scale=0.4),
    attn_layer(3, 3, 48, 24, 48, 17, mlp=moe(6, 1, 16, 2.5, shared=None)),
])
# nothing is a whole 16-byte row: width, head sizes, expert widths, vocabulary
RAGGED = model(100, 77, [
    attn_layer(3, 1, 20, 12, 6, 21, mlp=moe(9, 4, 20, 1.2, 3, 2, 0.6, shared=(28, 0.7))),
    attn_layer(2, 2, 36, 44, 36, 5, mlp=moe(5, 2, 12, 0.5, shared=(12, 0.5))),
])
# the head size of the tcgen05 prompt kernel, and windows around its tiles
HEAD128 = model(256, 320, [
    attn_layer(4, 2, 128, 128, 64, 65, mlp=moe(16, 4, 64, 1.3, 4, 3, 2.2, shared=(128, 1.9))),
    attn_layer(6, 2, 128, 128, 128, 150, mlp=moe(16, 2, 64, 1.0, 2, 1)),
])
# head sizes above 128, and beyond the tensor-core kernels
WIDE = model(128, 150, [
    attn_layer(4, 1, 192, 136, 100, 40, mlp=moe(4, 2, 32, 1.0, 2, 1)),
    attn_layer(2, 1, 272, 64, 272, 30),
    attn_layer(20, 1, 32, 64, 32, 70),
])


def shapes(cfg: dict) -> Dict[str, Tuple[int, ...]]:
    w = cfg["width"]
    out = {"embed": (cfg["vocab"], w), "head": (cfg["vocab"], w), "final.norm": (w,)}
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}."
        out[p + "norm1"] = (w,)
        for name, n in (("q", m["heads"] * m["dim"]), ("k", m["kv_heads"] * m["dim"]),
                        ("v", m["kv_heads"] * m["vdim"]), ("g", m["heads"] * m["vdim"])):
            out[p + "mix." + name] = (n, w)
        out[p + "mix.o"] = (w, m["heads"] * m["vdim"])
        f = layer["mlp"]
        if f is None:
            continue
        out[p + "mlp.router"] = (f["router"]["experts"], w)
        experts = [(f"e{e}", f["expert"]["ff"]) for e in range(f["router"]["experts"])]
        for name, ff in experts + ([("shared", f["shared"]["ff"])] if f.get("shared") else []):
            for t, s in (("gate", (ff, w)), ("up", (ff, w)), ("down", (w, ff))):
                out[f"{p}mlp.{name}.{t}"] = s
    return out


def weights(cfg: dict, seed: int) -> Dict[str, torch.Tensor]:
    """bf16 weights that leave no mechanism idle: attention scores of a few units, router logits far
    apart, activations beyond their limits, norm weights away from zero."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, s in shapes(cfg).items():
        gain = {"q": 1.6, "k": 1.6, "g": 2.0, "router": 3.0, "gate": 1.5, "up": 1.5}.get(name.rsplit(".", 1)[-1], 1.0)
        t = torch.randn(s, generator=g) * (0.3 if len(s) == 1 else gain * s[1] ** -0.5)
        if name == "embed":
            t = torch.randn(s, generator=g)
        out[name] = t.to(torch.bfloat16)
    return out


def write_model(path, cfg: dict, seed: int = 0) -> Dict[str, torch.Tensor]:
    w = weights(cfg, seed)
    save_file(w, os.path.join(path, "model.safetensors"))
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    return w


def tokens(n: int, vocab: int, seed: int) -> List[int]:
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def close(got: torch.Tensor, want: torch.Tensor, dtype: str) -> None:
    """Every position in fp32; in bf16 a router's close call may fall the other way at a few."""
    assert got.shape == want.shape
    d = got.double() - want.double()
    err = (d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / want.double().std()
    if dtype == "float32":
        assert float(err.max()) < 2e-5, float(err.max())
    else:
        assert float(err.median()) < 0.03, float(err.median())
        assert float((err > 0.12).double().mean()) <= 0.06, err.topk(min(5, err.numel()))


class Driver:
    """Requests with their oracle logits, fed in portions through a replay of the engine."""
    oracle = oracle
    close = staticmethod(close)

    def __init__(self, path, cfg, w, device, dtype, max_tokens=512, **kw) -> None:
        from omni_npu_b200.engine.trace_replay import TraceReplay
        self.cfg, self.w, self.dtype = cfg, w, dtype
        self.replay = TraceReplay(str(path), dtype, max_tokens, device=device, **kw)
        self.req, self.at = {}, {}
        self.got: List[torch.Tensor] = []
        self.want: List[torch.Tensor] = []

    def add(self, rid: str, n: int, seed: int) -> None:
        toks = tokens(n, self.cfg["vocab"], seed)
        self.req[rid], self.at[rid] = (toks, self.oracle.forward(toks, self.w, self.cfg)), 0

    def step(self, portions: Dict[str, int]) -> None:
        entries, end, rows = [], [], []
        for rid, n in portions.items():
            toks, logits = self.req[rid]
            lo = self.at[rid]
            hi = min(len(toks), lo + n)
            entries.append({"id": rid, "tokens": toks[lo:hi], "want": list(range(hi - lo))})
            rows.append(logits[lo:hi])
            self.at[rid] = hi
            if hi == len(toks):
                end.append(rid)
        self.got.append(self.replay.step(entries, end))
        self.want.append(torch.cat(rows))

    def left(self, rid: str) -> int:
        return len(self.req[rid][0]) - self.at[rid]

    def finish(self) -> None:
        self.replay.check()
        pool = self.replay.engine.scheduler.pool
        assert pool.num_free == pool.num_blocks - pool.num_reserved, "cache blocks were not given back"
        self.close(torch.cat(self.got), torch.cat(self.want), self.dtype)


# ---------------------------------------------------------------------------- whole-model checks
def check_prompts(d: Driver, lengths: Sequence[int]) -> None:
    for i, n in enumerate(lengths):
        d.add(f"p{i}", n, i)
        d.step({f"p{i}": n})
    d.finish()


def check_decode(d: Driver, prefix: int, total: int) -> None:
    """A short prompt, then token by token across page borders and past every window."""
    d.add("a", total, 11)
    d.step({"a": prefix})
    while d.left("a"):
        d.step({"a": 1})
    d.finish()


def check_portions(d: Driver, sizes: Sequence[int], total: int) -> None:
    d.add("a", total, 12)
    i = 0
    while d.left("a"):
        d.step({"a": sizes[i % len(sizes)]})
        i += 1
    d.finish()


def check_mixed(d: Driver, rounds: int = 3) -> None:
    """Unequal requests at once: portions beside single tokens, pauses, pages and slots used again."""
    for r in range(rounds):
        names = [f"r{r}.{i}" for i in range(4)]
        for i, (rid, n) in enumerate(zip(names, (37, 3, 64, 21))):
            d.add(rid, n + 5 * r, 100 * r + i)
        d.step({names[0]: 20})
        d.step({names[0]: 1, names[1]: 2})
        d.step({names[2]: 33, names[0]: 1, names[1]: 1})
        d.step({names[3]: 2, names[0]: 1})
        k = 0
        while any(d.left(x) for x in names):
            k += 1
            live = [x for j, x in enumerate(names) if d.left(x) and (k + j) % 4]        # one sits each step out
            if live:
                d.step({x: (1, 2, 7, 16)[(k + 3 * j) % 4] if x == names[2] else 1 for j, x in enumerate(live)})
    d.finish()


def check_generate(path, cfg, w, device, oracle=oracle, **kw) -> None:
    """Greedy generation through ``LLM.generate``: continuous batching over a small cache."""
    from omni_npu_b200 import LLM, SamplingParams
    prompts = [tokens(n, cfg["vocab"], 50 + n) for n in (1, 19, 40, 7, 28, 2)]
    llm = LLM(model=str(path), dtype="float32", device=device, max_num_seqs=3, max_num_batched_tokens=24,
              max_model_len=96, **kw)
    outs = llm.generate(prompts, SamplingParams(max_tokens=14, temperature=0.0, ignore_eos=True))
    for p, o in zip(prompts, outs):
        seq = list(p)
        for got in o.output_token_ids:
            logits = oracle.forward(seq, w, cfg)[-1]
            assert float(logits.max() - logits[got]) < 1e-3 * max(1.0, float(logits.std()))   # the greedy token, or its equal
            seq.append(got)
        assert len(o.output_token_ids) == 14


# ---------------------------------------------------------------------------- mechanism checks
def paged(x: torch.Tensor, width: int, bs: int, seed: int):
    """[T, G, d] laid out over shuffled cache blocks: (cache [blocks, G, bs, width], block table [1, n])."""
    t, g, dd = x.shape
    n = (t + bs - 1) // bs
    order = torch.randperm(n + 3, generator=torch.Generator().manual_seed(seed))[:n]
    cache = torch.zeros(n + 3, g, bs, width, dtype=x.dtype)
    for j in range(t):
        cache[order[j // bs], :, j % bs, :dd] = x[j]
    return cache, order.int().unsqueeze(0)


def check_window(device, dtype, heads, kv, dim, vdim, window, t, bs, queries, planted, variant=0, splits=0) -> None:
    """The last ``queries`` rows of a sequence of ``t`` tokens, as a prompt portion and one by one.  Key
    ``planted`` outweighs all others by far for every query that sees it."""
    from omni_npu_b200 import ops
    g = torch.Generator().manual_seed(window * 1000 + t)
    q, k, v = (torch.randn(t, n, dd, generator=g) for n, dd in ((heads, dim), (kv, dim), (kv, vdim)))
    q[..., 0] = q[..., 0].abs() + 2.0
    k[..., 0] = 0.0
    k[planted] = 0.0
    k[planted, :, 0] = 6.0 * dim ** 0.5
    gate = torch.randn(t, heads * vdim, generator=g) * 2
    q, k, v, gate = (x.to(dtype) for x in (q, k, v, gate))
    scale = dim ** -0.5
    want = oracle.attention(q.double(), k.double(), v.double(), scale, window) * torch.sigmoid(gate.double())
    kc, bt = paged(k, ops.gated_head_pad(dim, dtype), bs, 1)
    vc, _ = paged(v, ops.gated_head_pad(vdim, dtype), bs, 1)
    kc, vc, bt = kc.to(device), vc.to(device), bt.to(device)
    rows = slice(t - queries, t)
    qd, gd = q[rows].reshape(queries, -1).to(device), gate[rows].to(device)
    i32 = dict(dtype=torch.int32, device=device)
    tol = 2e-5 if dtype == torch.float32 else 0.03

    def compare(out, ref):
        assert float((out.double().cpu() - ref).abs().max()) < tol * max(1.0, float(ref.abs().max()))

    out = torch.empty(queries, heads * vdim, dtype=dtype, device=device)
    ops.gated_attention(qd, gd, kc, vc, out, bt, torch.tensor([0, queries], **i32), torch.tensor([t], **i32), 1,
                        queries, heads, dim, vdim, scale, window, 0.0, max_seq_len=t, variant=variant)
    compare(out, want[rows])
    for i in sorted({t - 1, t - queries, *(x for x in (planted + window - 1, planted + window, planted)
                                           if t - queries <= x < t)}):
        one = torch.empty(1, heads * vdim, dtype=dtype, device=device)
        r = i - (t - queries)
        ops.gated_attention(qd[r:r + 1], gd[r:r + 1], kc, vc, one, bt, None, torch.tensor([i + 1], **i32), 1, 1, heads,
                            dim, vdim, scale, window, 0.0, max_seq_len=t, splits=splits, variant=variant)
        compare(one, want[i:i + 1])


def check_rope(device, dtype, heads, kv, dim, vdim, rot, base) -> None:
    from omni_npu_b200 import ops
    from omni_npu_b200.layers.rope import get_rope
    t, bs = 9, 8
    g = torch.Generator().manual_seed(rot)
    pos = torch.tensor([0, 1, 2, 7, 8, 63, 500, 4097, 5999])
    slots = torch.tensor([3, 30, 31, -1, 0, 17, 5, 8, 9])
    q, k, v = (torch.randn(t, n, dd, generator=g).to(dtype) for n, dd in ((heads, dim), (kv, dim), (kv, vdim)))
    rope = get_rope(dim, rot, 6000, base, False, None, torch.device(device), exact_angles=True)
    kc = torch.zeros(4, kv, bs, ops.gated_head_pad(dim, dtype), dtype=dtype, device=device)
    vc = torch.zeros(4, kv, bs, ops.gated_head_pad(vdim, dtype), dtype=dtype, device=device)
    qd = q.reshape(t, -1).clone().to(device)
    ops.gated_rope_cache_(qd, k.reshape(t, -1).to(device), v.reshape(t, -1).to(device), kc, vc, pos.int().to(device),
                          slots.int().to(device), rope.cos_sin_cache, dim, vdim, rot, False)
    tol = 3e-6 if dtype == torch.float32 else 0.03
    want_q = oracle.rotate_interleaved(q.double(), pos, rot, base)
    want_k = oracle.rotate_interleaved(k.double(), pos, rot, base)
    err = (qd.view(t, heads, dim).double().cpu() - want_q).abs().amax((1, 2))
    assert float(err.max()) < tol, err
    for j in range(t):
        s = int(slots[j])
        if s >= 0:
            assert float((kc[s // bs, :, s % bs, :dim].double().cpu() - want_k[j]).abs().max()) < tol
            assert torch.equal(vc[s // bs, :, s % bs, :vdim].cpu(), v[j])
    written = int((slots >= 0).sum()) * kv * dim
    assert int((kc != 0).sum()) <= written and float(kc[..., dim:].abs().sum()) == 0.0


def check_glu(device, dtype, m, ff, width, limit) -> None:
    from omni_npu_b200 import ops
    from omni_npu_b200.ops import ref
    g = torch.Generator().manual_seed(ff)
    h = torch.randn(m, width, generator=g).to(dtype)
    wg, wu = ((torch.randn(ff, width, generator=g) * 2 * width ** -0.5).to(dtype) for _ in range(2))
    want = oracle.clamped_glu(h.double() @ wg.double().T, h.double() @ wu.double().T, limit)
    w = ref.interleave_gate_up(wg, wu).to(device)
    got = ops.gemm(h.to(device), w, swiglu=True, act=(oracle.SIGMOID_SLOPE, limit))
    tol = 1e-4 if dtype == torch.float32 else 0.03
    assert float((got.double().cpu() - want).abs().max()) < tol * float(want.abs().max())
    assert float((h.double() @ wg.double().T).max()) > limit             # the clamps were at work


def check_moe(device, dtype, t, cfg_mlp, width) -> None:
    """The expert layer alone, and its last step fused into the residual kernel."""
    from omni_npu_b200 import ops
    from omni_npu_b200.layers.moe import FusedMoE
    r = cfg_mlp["router"]
    cfg = model(width, 8, [attn_layer(1, 1, 8, 8, 8, 4, mlp=cfg_mlp)])
    w = {k[len("l0.mlp."):]: v for k, v in weights(cfg, 3).items() if k.startswith("l0.mlp.")}
    act = (oracle.SIGMOID_SLOPE, cfg_mlp["expert"]["limit"])
    sh = cfg_mlp.get("shared")
    layer = FusedMoE(r["experts"], r["top"], width, cfg_mlp["expert"]["ff"], dtype, torch.device(device), "softmax",
                     True, r["scale"], r["groups"]["count"], r["groups"]["keep"], num_shared_experts=1 if sh else 0,
                     shared_intermediate_size=sh["ff"] if sh else None, enable_expert_parallel=False,
                     max_tokens=max(t, 64), act=act, shared_act=(oracle.SIGMOID_SLOPE, sh["limit"]) if sh else None)
    layer.gate.weight.data.copy_(w["router"])
    for e in range(r["experts"]):
        for name in ("gate", "up", "down"):
            layer.weight_loader(layer.w2 if name == "down" else layer.w13, w[f"e{e}.{name}"], e, name)
    if sh:
        layer.shared_experts.gate_up_proj.weight_loader(layer.shared_experts.gate_up_proj.weight, w["shared.gate"], 0)
        layer.shared_experts.gate_up_proj.weight_loader(layer.shared_experts.gate_up_proj.weight, w["shared.up"], 1)
        layer.shared_experts.down_proj.weight_loader(layer.shared_experts.down_proj.weight, w["shared.down"])
    g = torch.Generator().manual_seed(t)
    h = torch.randn(t, width, generator=g).to(dtype)
    x = torch.randn(t, width, generator=g)
    a = torch.randn(t, width, generator=g).to(dtype)
    gain = (torch.randn(width, generator=g) * 0.3).to(dtype)
    want = x.double() + a.double() + oracle.moe(h.double(), {k: v.double() for k, v in w.items()}, cfg_mlp)
    routed, dense = layer.forward_deferred(h.to(device))
    res = x.clone().to(device)
    out = ops.residual_add_norm(res, a.to(device), dense, routed, gain.to(device), 1e-5, 1.0, width)
    err = (res.double().cpu() - want).abs().amax(-1) / want.std()
    bad = float((err > (1e-5 if dtype == torch.float32 else 0.05)).double().mean())
    assert bad <= (0.0 if dtype == torch.float32 else 0.04), (bad, float(err.max()))
    norm = oracle.rms_norm(res.double().cpu(), gain.double(), 1e-5)
    assert float((out.double().cpu() - norm).abs().max()) < (1e-5 if dtype == torch.float32 else 0.02) * \
        float(norm.abs().max())
