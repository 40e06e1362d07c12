"""Small random Dalavik models and the checks that the CPU and GPU tests share: the framework's step function, cache
and scheduler against the plain implementation in dalavik_oracle.py."""
from __future__ import annotations

import json
import os
from typing import Dict, Optional, Tuple

import torch
from safetensors.torch import save_file

import dalavik_oracle as oracle
import rivudra_cases as base
from fuvirax_cases import rel
from rivudra_cases import check_decode, check_mixed, check_portions, check_prompts, paged, tokens       # noqa: F401


# ---------------------------------------------------------------------------- configurations
def dense(ff) -> dict:
    return {"kind": "dense", "ff": ff}


def latent(heads, dim, rot, vdim, rank, q_rank, kv_from=None, scale=None, theta=3000.0, mlp=None) -> dict:
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "q_rank": q_rank,
         "rot": {"base": theta, "dims": rot}, "scale": (dim + rot) ** -0.5 if scale is None else scale}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mlp": mlp, "mixer": m}


def attention(heads, kv, dim, vdim, softcap=20.0, coef=0.4, every=16, scale=None, mlp=None) -> dict:
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "softcap": softcap,
                      "q_temp": {"coef": coef, "every": every}, "scale": 0.7 * dim ** -0.5 if scale is None else scale}}


def model(width, vocab, layers, groups=1, side=16, eps=1e-5) -> dict:
    return {"architecture": "Dalavik", "width": width, "vocab": vocab, "norm": {"eps": eps, "groups": groups},
            "token_side": {"dim": side}, "layers": layers}


# both mixers, rows read by two later layers, layers without a feed-forward (the last one too), one head per group
VARIED = model(96, 203, [
    attention(4, 2, 24, 40, mlp=dense(56)),
    latent(4, 24, 16, 40, 56, 48, mlp=dense(40)),
    latent(2, 40, 16, 24, 56, 32, kv_from=1),
    attention(3, 3, 16, 16, softcap=5.0, coef=-0.2, every=7),
    latent(3, 16, 8, 32, 24, 16, theta=500.0, mlp=dense(24)),
    latent(6, 8, 16, 8, 56, 80, kv_from=1, scale=0.6),
], groups=3)
# nothing is a whole 16-byte row: width, groups, head sizes, ranks, side width, vocabulary; seven heads
RAGGED = model(100, 77, [
    latent(3, 20, 6, 12, 28, 18, scale=0.4, mlp=dense(36)),
    attention(7, 1, 18, 22, mlp=dense(20), every=1),
    latent(5, 14, 6, 10, 28, 26, kv_from=0, mlp=dense(12)),
    attention(2, 1, 36, 14),
], groups=4, side=10)
# sizes of a real model's heads
LARGE = model(256, 320, [
    attention(8, 2, 128, 128, softcap=30.0, mlp=dense(512)),
    latent(6, 128, 64, 128, 512, 192, mlp=dense(128)),
    attention(32, 4, 64, 64, every=64),
    latent(8, 64, 64, 64, 512, 256, kv_from=1, mlp=dense(256)),
    attention(18, 6, 96, 64, mlp=dense(64)),
], groups=2, side=64)
# head sizes above 128 and beyond the tensor-core kernels, many heads, every head with its own keys
WIDE = model(128, 150, [
    attention(4, 1, 192, 136, mlp=dense(64)),
    latent(2, 200, 72, 48, 520, 264, mlp=dense(64)),
    attention(2, 1, 272, 64),
    attention(20, 20, 32, 32, mlp=dense(24)),
    attention(48, 4, 24, 136),
], groups=8, side=8)


def shapes(cfg: dict) -> Dict[str, Tuple[int, ...]]:
    w, side = cfg["width"], cfg["token_side"]["dim"]
    out = {"embed": (cfg["vocab"], w), "side.embed": (cfg["vocab"], side * len(cfg["layers"])), "final.norm": (w,)}
    for i, layer in enumerate(cfg["layers"]):
        m, f, p = layer["mixer"], layer["mlp"], f"l{i}."
        h, d, e = m["heads"], m["dim"], m["vdim"]
        out[p + "norm1"] = (w,)
        if layer["type"] == "attention":
            g = m["kv_heads"]
            mix = {"q": (h * d, w), "q.b": (h * d,), "k": (g * d, w), "k.b": (g * d,), "v": (g * e, w), "v.b": (g * e,),
                   "q.norm": (d,), "k.norm": (d,), "r1": (h,), "r2": (h,), "talk": (h, h), "sink": (h,)}
        else:
            r, rq = m["kv_rank"], m["q_rank"]
            mix = {"dq": (rq, w), "dq.norm": (rq,), "uq": (h * (d + m["rot_dim"]), rq), "uk": (h * d, r), "uv": (h * e, r)}
            if "kv_from" not in m:
                mix.update({"dkv": (r + m["rot_dim"], w), "dkv.norm": (r,)})
        mix["o"] = (w, h * e)
        out.update({f"{p}mix.{k}": s for k, s in mix.items()})
        if f:
            out[p + "norm2"] = (w,)
            out.update({p + "mlp.gate": (f["ff"], w), p + "mlp.up": (f["ff"], w), p + "mlp.down": (w, f["ff"])})
        out.update({p + "side.gate": (side, w), p + "side.proj": (w, side), p + "side.norm": (w,)})
    return out


def weights(cfg: dict, seed: int) -> Dict[str, torch.Tensor]:
    """bf16 weights that leave no mechanism idle: scores of a few units, some near their cap, mixtures away from the
    identity, biases and sinks that count."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, s in shapes(cfg).items():
        last = name.rsplit(".", 1)[-1]
        n, u = torch.randn(s, generator=g), torch.rand(s, generator=g)
        if "embed" in name:
            t = n
        elif last.startswith("norm"):
            t = 0.8 + 0.3 * n
            if name.endswith((".q.norm", ".k.norm")):
                t = 1.6 + 0.6 * n
        elif last == "talk":
            t = 0.7 * torch.eye(s[0]) + 0.6 * n * s[0] ** -0.5
        elif last == "r1":
            t = 0.2 + 0.8 * u
        elif last == "r2":
            t = 0.05 + 0.4 * u
        elif last == "sink":
            t = 1 + 2 * n
        elif last == "b":
            t = 0.4 * n
        else:
            t = n * {"uq": 1.6, "uk": 1.6, "gate": 1.5, "up": 1.5}.get(last, 1.0) * s[-1] ** -0.5
        out[name] = t.to(torch.bfloat16)
    return out


def write_model(path, cfg: dict, seed: int = 0) -> Dict[str, torch.Tensor]:
    w = weights(cfg, seed)
    save_file(w, os.path.join(path, "model.safetensors"))
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    return w


class Driver(base.Driver):
    oracle = oracle


def check_generate(path, cfg, w, device, **kw) -> None:
    base.check_generate(path, cfg, w, device, oracle=oracle, **kw)


# ---------------------------------------------------------------------------- attention with mixed scores
def check_prep(device, dtype, n, kv, dim, vdim, temp: Optional[dict], rot=0, base_=3000.0, eps=1e-3) -> None:
    """Weighted norm per head and query temperature at far positions, cache rows; padded rows (slot -1) store
    nothing."""
    from omni_npu_b200 import ops
    from omni_npu_b200.layers.rope import get_rope
    from gatosun_oracle import rotate_halves
    t, bs = 9, 8
    g = torch.Generator().manual_seed(dim + n)
    pos = torch.tensor([0, 6, 7, 14, 15, 63, 500, 4097, 5999])
    slots = torch.tensor([3, 30, 31, -1, 0, 17, 5, 8, 9])
    y = torch.randn(t, (n + kv) * dim + kv * vdim + 16, generator=g).to(dtype)
    q, k, v = y[:, : n * dim], y[:, n * dim: (n + kv) * dim], y[:, (n + kv) * dim: (n + kv) * dim + kv * vdim]
    qw, kw = ((1 + 0.3 * torch.randn(dim, generator=g)).to(dtype) for _ in range(2))
    kc = torch.zeros(4, kv, bs, ops.gated_head_pad(dim, dtype), dtype=dtype, device=device)
    vc = torch.zeros(4, kv, bs, ops.gated_head_pad(vdim, dtype), dtype=dtype, device=device)
    table = get_rope(dim, rot, 6000, base_, True, None, torch.device(device), exact_angles=True).cos_sin_cache if rot else None
    yd = y.to(device)
    part = lambda a, m: yd[:, a: a + m]                                                  # noqa: E731
    got = ops.qk_norm_rope_cache(part(0, n * dim), part(n * dim, kv * dim), part((n + kv) * dim, kv * vdim), kc, vc,
                                 pos.int().to(device), slots.int().to(device), table, dim, vdim, rot, "head_weight", eps,
                                 (qw.to(device), kw.to(device)), temperature=(temp["coef"], temp["every"]) if temp else None)
    wq, wk = oracle.normed_queries_keys(q.double().view(t, n, dim), k.double().view(t, kv, dim), qw.double(), kw.double(),
                                        eps, temp, pos)
    if rot:
        wq, wk = (rotate_halves(x, pos, rot, base_) for x in (wq, wk))
    tol = 3e-6 if dtype == torch.float32 else 0.05
    assert float((got.double().cpu().view(t, n, dim) - wq).abs().max()) < tol * max(1.0, float(wq.abs().max()) / 4)
    for j in range(t):
        s = int(slots[j])
        if s >= 0:
            assert float((kc[s // bs, :, s % bs, :dim].double().cpu() - wk[j]).abs().max()) < tol
            assert torch.equal(vc[s // bs, :, s % bs, :vdim].cpu(), v[j].view(kv, vdim))
    assert int((kc != 0).sum()) <= int((slots >= 0).sum()) * kv * dim and float(kc[..., dim:].abs().sum()) == 0.0
    assert float(vc[..., vdim:].abs().sum()) == 0.0


def score_constants(n: int, g: torch.Generator, bias=True, sink=True):
    talk = 0.8 * torch.eye(n) + 0.5 * torch.randn(n, n, generator=g) * n ** -0.5
    r = (0.3 + 0.5 * torch.rand(n, generator=g), 0.1 + 0.3 * torch.rand(n, generator=g)) if bias else None
    return r, talk, (torch.randn(n, generator=g) * 2 if sink else None)


def check_mixed_scores(device, dtype, n, kv, dim, vdim, t, bs, queries, planted, softcap=20.0, bias=True, sink=True,
                       variant=0, splits=0, ranks=1, exact=False) -> None:
    """The last ``queries`` rows of a sequence, as a prompt portion and one by one.  Every head's score of key
    ``planted`` is close to the cap for every query that sees it, and the mixture is such that it outweighs the rest.
    ``ranks`` > 1: the output heads of each of so many ranks.  ``exact``: a mixture that bf16 holds."""
    from omni_npu_b200 import ops
    g = torch.Generator().manual_seed(1000 * n + t + planted)
    q, k, v = (torch.randn(t, m, dd, generator=g) for m, dd in ((n, dim), (kv, dim), (kv, vdim)))
    q[..., 0] = q[..., 0].abs() + 2.0
    k[..., 0] = 0.0
    k[planted] = 0.0
    k[planted, :, 0] = 9.0 * dim ** 0.5
    q, k, v = (x.to(dtype) for x in (q, k, v))
    r, talk, sinks = score_constants(n, g, bias, sink)
    talk = talk + (1 - talk.sum(1, keepdim=True)).clamp(min=0) / n                       # every row adds up to one or more
    if exact:
        talk = talk.bfloat16().float()
    scale = dim ** -0.5
    d64 = lambda x: None if x is None else x.double()                                    # noqa: E731
    want = oracle.mixed_attend(q.double(), k.double(), v.double(), scale, softcap, *(map(d64, r) if r else (None, None)),
                               d64(talk), d64(sinks))
    kc, bt = paged(k, ops.gated_head_pad(dim, dtype), bs, 1)
    vc, _ = paged(v, ops.gated_head_pad(vdim, dtype), bs, 1)
    rows = slice(t - queries, t)
    dd = lambda x: None if x is None else x.to(device)                                   # noqa: E731
    qd, bt, kc = q[rows].reshape(queries, -1).to(device), bt.to(device), kc.to(device)
    i32 = dict(dtype=torch.int32, device=device)
    tol = 2e-5 if dtype == torch.float32 else 0.03
    for rank in range(ranks):
        ho, hv = n // ranks, kv // ranks
        own = slice(rank * ho, rank * ho + ho)
        vr = vc[:, rank * hv: rank * hv + hv].contiguous().to(device)
        consts = (dd(talk[own]).contiguous(), dd(sinks[own].contiguous()) if sink else None)
        ref = want[:, rank * ho * vdim: (rank + 1) * ho * vdim]

        def run(q_, cu, lens, b, m, sp=0):
            wide = torch.full((q_.shape[0], ho * vdim + 24), 7.0, dtype=dtype, device=device)
            ops.mixed_attention(q_, kc, vr, wide[:, : ho * vdim], bt, cu, lens, b, m, dim, vdim, scale, softcap,
                                tuple(map(dd, r)) if r else None, *consts, max_seq_len=t, variant=variant, splits=sp,
                                talk_exact=exact)
            assert float((wide[:, ho * vdim:] - 7.0).abs().max()) == 0.0
            return wide[:, : ho * vdim].double().cpu()

        def compare(out, w_):
            assert float((out - w_).abs().max()) < tol * max(1.0, float(want.abs().max()))

        compare(run(qd, torch.tensor([0, queries], **i32), torch.tensor([t], **i32), 1, queries), ref[rows])
        for i in sorted({x for x in (t - queries, planted - 1, planted, planted + 1, planted + bs, t - 1)
                         if t - queries <= x < t}):
            j = i - (t - queries)
            for sp in sorted({1, splits}):
                compare(run(qd[j: j + 1], None, torch.tensor([i + 1], **i32), 1, 1, sp), ref[i: i + 1])


def check_mixed_batch(device, dtype, n, kv, dim, vdim, lens, portions, bs=16) -> None:
    """Portions of unequal sequences in one call, with and without their scores cut into several runs; decode rows of
    all sequences in one call."""
    from omni_npu_b200 import ops
    g = torch.Generator().manual_seed(n + dim)
    r, talk, sinks = score_constants(n, g)
    seqs = [tuple(torch.randn(t, m, dd, generator=g).to(dtype) for m, dd in ((n, dim), (kv, dim), (kv, vdim))) for t in lens]
    scale, cap = dim ** -0.5, 8.0
    want = [oracle.mixed_attend(*(x.double() for x in s), scale, cap, *(x.double() for x in r), talk.double(), sinks.double())
            for s in seqs]
    i32 = dict(dtype=torch.int32, device=device)
    blocks = [(t + bs - 1) // bs for t in lens]
    order = torch.randperm(sum(blocks), generator=g)
    bt = torch.zeros(len(lens), max(blocks), dtype=torch.int32)
    caches = [torch.zeros(sum(blocks), kv, bs, ops.gated_head_pad(w, dtype), dtype=dtype) for w in (dim, vdim)]
    at = 0
    for i, t in enumerate(lens):
        bt[i, : blocks[i]] = order[at: at + blocks[i]]
        at += blocks[i]
        for c, x in zip(caches, seqs[i][1:]):
            for j in range(t):
                c[bt[i, j // bs], :, j % bs, : x.shape[-1]] = x[j]
    kc, vc, bt = caches[0].to(device), caches[1].to(device), bt.to(device)
    consts = (tuple(x.to(device) for x in r), talk.to(device), sinks.to(device))
    tol = 2e-5 if dtype == torch.float32 else 0.03

    def run(counts, cu):
        q = torch.cat([s[0][len(s[0]) - c:] for s, c in zip(seqs, counts)]).flatten(1).to(device)
        out = torch.empty(q.shape[0], n * vdim, dtype=dtype, device=device)
        ops.mixed_attention(q, kc, vc, out, bt, cu, torch.tensor(lens, **i32), len(lens), max(counts), dim, vdim, scale, cap,
                            *consts, max_seq_len=max(lens))
        ref = torch.cat([w[len(w) - c:] for w, c in zip(want, counts)])
        assert float((out.double().cpu() - ref).abs().max()) < tol * max(1.0, float(ref.abs().max()))

    cu = torch.tensor([0, *torch.tensor(portions).cumsum(0).tolist()], **i32)
    run(portions, cu)
    keep = ops.MIXED_SCORE_BYTES
    try:
        for tiles in (1, 3):                             # so many query tiles at a time
            ops.MIXED_SCORE_BYTES = tiles * 16 * n * ((max(lens) + 63) // 64 * 64) * 4
            run(portions, cu)
    finally:
        ops.MIXED_SCORE_BYTES = keep
    run([1] * len(lens), None)


# ---------------------------------------------------------------------------- latent attention
def check_shared_rows(device, dtype, n, dim, rot, vdim, rank, q_rank, planted, t=90, bs=16, prompt=50) -> None:
    """Two layers on one cache: the first stores the rows, the second only reads them with weights of its own; key
    ``planted`` stands out for both.  A prompt portion, a second one, then single tokens."""
    from omni_npu_b200 import ops
    from omni_npu_b200.attention.latent import LatentAttention
    from omni_npu_b200.attention.metadata import AttentionMetadata, set_forward_context
    from omni_npu_b200.layers.rope import get_rope
    g = torch.Generator().manual_seed(rank + planted)
    eps, theta = 1e-4, 700.0
    m = {"heads": n, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "q_rank": q_rank, "rot": {"base": theta},
         "scale": (dim + rot) ** -0.5}
    width = q_rank + rank + rot
    h = torch.randn(t, width, generator=g)
    h[:, q_rank] = 0.0
    h[planted, q_rank: q_rank + rank] = 0.0
    h[planted, q_rank] = 3.0                             # all of the planted token's latent in one direction
    h = h.to(dtype)
    eye = torch.eye(width).double()
    ws = []
    for _ in range(2):
        w = {"uq": torch.randn(n * (dim + rot), q_rank, generator=g) * q_rank ** -0.5,
             "uk": torch.randn(n * dim, rank, generator=g) * rank ** -0.5,
             "uv": torch.randn(n * vdim, rank, generator=g) * rank ** -0.5, "dq.norm": 1 + 0.3 * torch.randn(q_rank, generator=g)}
        ws.append({k: v.to(dtype) for k, v in w.items()})
    norm = (1 + 0.3 * torch.randn(rank, generator=g)).to(dtype)
    o64 = dict(dq=eye[:q_rank], dkv=eye[q_rank:], o=torch.eye(n * vdim).double())
    o64["dkv.norm"] = norm.double()
    rows = oracle.latent_rows(h.double(), o64, m, eps)
    want = [oracle.latent_attention(h.double(), {**{k: v.double() for k, v in w.items()}, **o64}, m, eps, rows) for w in ws]
    rope = get_rope(rot, rot, t + 8, theta, False, None, torch.device(device), exact_angles=True)
    layers = [LatentAttention(n, dim, rot, vdim, rank, m["scale"], False, eps, dtype, device, q_rank, i == 0, i == 0)
              for i in range(2)]
    for a, w in zip(layers, ws):
        a.w_uk.data.copy_(w["uk"])
        a.w_uv.data.copy_(w["uv"])
        a.query_norm.data.copy_(w["dq.norm"])
        a.build_absorbed()
    layers[0].latent_norm.data.copy_(norm)
    assert layers[1].latent_norm is None
    blocks = (t + bs - 1) // bs
    order = torch.randperm(blocks + 2, generator=g)[:blocks].int()
    cache = torch.zeros(blocks + 2, bs, layers[0].row, dtype=dtype, device=device)
    i32 = dict(dtype=torch.int32, device=device)
    got = [[], []]
    cuts = [0, prompt, prompt + 2, *range(prompt + 3, t + 1)]
    for lo, hi in zip(cuts, cuts[1:]):
        pos = torch.arange(lo, hi)
        md = AttentionMetadata(is_prefill=hi - lo > 1, num_seqs=1, num_tokens=hi - lo, max_q_len=hi - lo, max_seq_len=hi,
                               q_len=1 if hi - lo == 1 else 0, positions=pos.to(**i32),
                               slot_mapping=(order[pos // bs] * bs + pos % bs).to(**i32),
                               block_tables=order.view(1, -1).to(device), seq_lens=torch.tensor([hi], **i32),
                               cu_q=torch.tensor([0, hi - lo], **i32))
        md.extra["seq_lens_host"] = [hi]
        x = h[lo:hi].to(device)
        with set_forward_context(md, [cache]):
            for i, (a, w) in enumerate(zip(layers, ws)):
                c_q = a.store(x[:, :q_rank], x[:, q_rank:] if i == 0 else None, rope.cos_sin_cache, 0)
                assert c_q.shape[1] % 8 == 0 and float(c_q[:, q_rank:].abs().sum()) == 0.0
                q = (c_q[:, :q_rank].float() @ w["uq"].float().T.to(device)).to(dtype)
                got[i].append(a(q, None, rope.cos_sin_cache, 0).double().cpu())
    tol = 3e-5 if dtype == torch.float32 else 0.04
    for out, ref in zip(got, want):
        assert float((torch.cat(out) - ref).abs().max()) < tol * max(1.0, float(ref.abs().max()))


# ---------------------------------------------------------------------------- residual, feed-forward, token input
def check_post_norm(device, dtype, t, width, groups, out_groups) -> None:
    """Norm of a sublayer's result in groups, added in fp32; groups of very different sizes of number.  Padding stays
    zero."""
    from omni_npu_b200 import ops
    g = torch.Generator().manual_seed(width + groups)
    wp, eps = (width + 7) // 8 * 8, 1e-3
    pad = lambda z: torch.nn.functional.pad(z, (0, wp - width))                          # noqa: E731
    sizes = torch.logspace(-2, 1, groups).repeat_interleave(width // groups)
    y = (torch.randn(t, width, generator=g) * sizes).to(dtype)
    x = torch.randn(t, width, generator=g) * 50
    w, ow = ((1 + 0.3 * torch.randn(width, generator=g)).to(dtype) for _ in range(2))
    want = x.double() + oracle.group_norm(y.double(), w.double(), groups, eps)
    tol = 2e-6 if dtype == torch.float32 else 0.01
    for out_norm in (None, (pad(ow).to(device), out_groups)):
        res = pad(x).to(device)
        h = ops.post_norm_residual(res, pad(y).to(device), pad(w).to(device), groups, eps, width, out_norm=out_norm)
        assert rel(res[:, :width], want) < 2e-6 and float(res[:, width:].abs().sum()) == 0.0
        ref = want if out_norm is None else oracle.group_norm(want, ow.double(), out_groups, eps)
        assert h.dtype == dtype and rel(h[:, :width], ref) < tol and float(h[:, width:].abs().sum()) == 0.0
    table = pad(torch.randn(11, width, generator=g).to(dtype)).to(device)
    ids = torch.randint(0, 11, (t,), generator=g).int().to(device)
    res = torch.full((t, wp), 9.0, device=device)
    h = ops.post_norm_residual(res, None, None, 1, eps, width, ids, table)
    assert torch.equal(h, table[ids.long()]) and torch.equal(res, h.float())


def check_token_rows(device, dtype, t, dim, layers, layer) -> None:
    from omni_npu_b200 import ops
    g = torch.Generator().manual_seed(dim + t)
    width = (dim + 7) // 8 * 8
    z = (torch.randn(t, width, generator=g) * 3).to(dtype)
    table = torch.randn(13, dim * layers, generator=g).to(dtype)
    ids = torch.randint(0, 13, (t,), generator=g).int()
    got = ops.gelu_rows(z.to(device), ids.to(device), table.to(device), layer * dim, dim)
    want = oracle.gelu_tanh(z[:, :dim].double()) * table[ids.long(), layer * dim: (layer + 1) * dim].double()
    assert rel(got[:, :dim], want) < (2e-6 if dtype == torch.float32 else 0.01)
    assert got.shape == z.shape and float(got[:, dim:].abs().sum()) == 0.0


def check_relu_gate(device, dtype, m, ff, width) -> None:
    from omni_npu_b200 import ops
    from omni_npu_b200.ops import ref
    g = torch.Generator().manual_seed(ff + m)
    h = torch.randn(m, width, generator=g).to(dtype)
    wg, wu = ((torch.randn(ff, width, generator=g) * 2 * width ** -0.5).to(dtype) for _ in range(2))
    got = ops.gemm(h.to(device), ref.interleave_gate_up(wg, wu).to(device), swiglu=True, act=ops.RELU)
    want = torch.clamp(h.double() @ wg.double().T, min=0) * (h.double() @ wu.double().T)
    assert rel(got, want) < (1e-5 if dtype == torch.float32 else 0.012)


