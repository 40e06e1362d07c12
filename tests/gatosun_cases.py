"""Small random Gatosun models and the checks that the CPU and GPU tests share: the framework's step function,
cache, state slots and scheduler against the plain implementation in gatosun_oracle.py."""
from __future__ import annotations

import json
import os
from typing import Dict, Optional, Tuple

import torch
from safetensors.torch import save_file

import fuvirax_cases as states
import gatosun_oracle as oracle
import rivudra_cases as base
from fuvirax_cases import Step, cuts, rel
from rivudra_cases import check_decode, check_mixed, check_portions, check_prompts, paged, tokens       # noqa: F401


# ---------------------------------------------------------------------------- configurations
def dense(ff) -> dict:
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, groups=1, keep=1, shared=None) -> dict:
    d = {"kind": "moe", "expert": {"ff": ff},
         "router": {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep}}}
    if shared:
        d["shared"] = {"ff": shared}
    return d


def heads(n, kv, dim, vdim, rot, base=3000.0, scale=None, window=0) -> dict:
    d = {"heads": n, "kv_heads": kv, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": rot},
         "scale": dim ** -0.5 if scale is None else scale}
    if window:
        d["mask"] = {"size": window}
    return d


def attention(*a, v_mix: Optional[bool] = True, mlp=None, **kw) -> dict:
    m = heads(*a, **kw)
    if v_mix is not None:
        m["v_mix"] = v_mix
    return {"type": "attention", "mlp": mlp, "mixer": m}


def parallel(left, right, left_scale=0.7, right_scale=0.4, mlp=None) -> dict:
    return {"type": "parallel", "mlp": mlp, "mixer": {"left": left, "right": {"heads": right[0], "dim": right[1]},
                                                      "left_scale": left_scale, "right_scale": right_scale}}


def gla(n, dim, vdim, tau=8.0, mlp=None) -> dict:
    return {"type": "gla", "mlp": mlp, "mixer": {"heads": n, "dim": dim, "vdim": vdim, "tau": tau}}


def model(width, vocab, layers, mult=0.5, eps=1e-4) -> dict:
    return {"architecture": "Gatosun", "width": width, "vocab": vocab, "residual_mult": mult, "norm": {"eps": eps},
            "layers": layers}


# every mixer and feed-forward, layers without one, blended values around a layer that does not blend, a weight of
# zero and a negative one, several groups kept
VARIED = model(96, 203, [
    parallel(heads(4, 2, 24, 40, 16, window=10), (3, 20), mlp=dense(56)),
    attention(6, 2, 24, 16, 8, mlp=moe(8, 3, 40, 4, 2, shared=24)),
    attention(4, 4, 16, 24, 16, v_mix=False, base=700.0),
    gla(3, 20, 28, 5.0, mlp=moe(6, 2, 24, 3, 2)),
    attention(2, 1, 48, 32, 48, scale=0.2, mlp=dense(40)),
    parallel(heads(3, 3, 16, 16, 4, window=33), (2, 36), 1.0, -0.8),
    parallel(heads(2, 1, 32, 8, 32, window=1), (4, 12), 0.0, 0.9, mlp=moe(5, 5, 16, shared=32)),
])
# nothing is a whole 16-byte row: width, head sizes, ranks, expert widths, vocabulary
RAGGED = model(100, 77, [
    gla(3, 18, 22, 1.0, mlp=moe(9, 4, 20, 3, 2, shared=28)),
    parallel(heads(3, 1, 20, 12, 6, window=21), (5, 10), mlp=dense(36)),
    attention(2, 2, 36, 44, 36, v_mix=None, mlp=dense(20)),
    attention(5, 5, 22, 14, 10, mlp=moe(4, 1, 12, 2, 1)),
    attention(3, 1, 30, 70, 2),
], mult=1.0)
# the head size of the tcgen05 prompt kernel, windows around its tiles, states above 64 rows
LARGE = model(256, 320, [
    attention(8, 2, 128, 128, 64, mlp=dense(512)),
    parallel(heads(4, 2, 128, 128, 128, window=65), (2, 128), mlp=moe(16, 4, 64, 4, 3, shared=128)),
    gla(4, 96, 160, 16.0, mlp=moe(16, 2, 64, 2, 1)),
    attention(4, 2, 64, 128, 32, mlp=moe(32, 6, 64, 8, 4, shared=64)),
    parallel(heads(6, 2, 128, 128, 32, window=150), (4, 64)),
])
# head sizes above 128, and beyond the tensor-core kernels
WIDE = model(128, 150, [
    attention(4, 1, 192, 136, 96, mlp=dense(64)),
    parallel(heads(2, 1, 272, 64, 16, window=30), (1, 264), mlp=moe(4, 2, 32, 2, 1)),
    gla(1, 300, 72, 3.0),
    attention(20, 1, 32, 136, 32, mlp=dense(24)),
])


def rank(i: int) -> int:
    """Rank of layer i's low-rank decay: no config key has it."""
    return 5 + 4 * i


def shapes(cfg: dict) -> Dict[str, Tuple[int, ...]]:
    w = cfg["width"]
    out = {"embed": (cfg["vocab"], w), "head": (cfg["vocab"], w), "final.norm": (w,)}
    for i, layer in enumerate(cfg["layers"]):
        m, f, p = layer["mixer"], layer["mlp"], f"l{i}."
        out[p + "norm1"] = (w,)
        if f:
            out[p + "norm2"] = (w,)

        def qkv(m):
            return {"q": (m["heads"] * m["dim"], w), "k": (m["kv_heads"] * m["dim"], w),
                    "v": (m["kv_heads"] * m["vdim"], w), "o": (w, m["heads"] * m["vdim"])}

        if layer["type"] == "attention":
            mix = qkv(m)
            mix.update({k + ".b": (s[0],) for k, s in list(mix.items())})
            mix.update({k + ".norm": (mix[k][0],) for k in "qk"})
            if m.get("v_mix"):
                mix["vmix"] = ()
        elif layer["type"] == "parallel":
            mix = {"left." + k: s for k, s in qkv(m["left"]).items()}
            h, d = m["right"]["heads"], m["right"]["dim"]
            right = {"mu." + s: (w,) for s in "rkvgw"}
            right.update({s: (h * d, w) for s in "rkvg"})
            right.update({"w1": (rank(i), w), "w2": (h * d, rank(i)), "w0": (h * d,), "u": (h, d), "norm": (h * d,),
                          "o": (w, h * d)})
            mix.update({"right." + k: s for k, s in right.items()})
        else:
            h, d, e = m["heads"], m["dim"], m["vdim"]
            mix = {"q": (h * d, w), "k": (h * d, w), "v": (h * e, w), "g": (h * e, w), "o": (w, h * e), "norm": (e,),
                   "a1": (rank(i), w), "a2": (h * d, rank(i)), "a2.b": (h * d,)}
        out.update({f"{p}mix.{k}": s for k, s in mix.items()})
        if f and f["kind"] == "dense":
            for k, s in (("gate", (f["ff"], w)), ("up", (f["ff"], w)), ("down", (w, f["ff"]))):
                out[f"{p}mlp.{k}"], out[f"{p}mlp.{k}.b"] = s, (s[0],)
        elif f:
            n = f["router"]["experts"]
            out[p + "mlp.router"], out[p + "mlp.correction"] = (n, w), (n,)
            each = [(f"e{e}", f["expert"]["ff"]) for e in range(n)]
            for k, ff in each + ([("shared", f["shared"]["ff"])] if f.get("shared") else []):
                out[f"{p}mlp.{k}.up"], out[f"{p}mlp.{k}.down"] = (ff, w), (w, ff)
    return out


def weights(cfg: dict, seed: int) -> Dict[str, torch.Tensor]:
    """bf16 weights that leave no mechanism idle: scores of a few units, decays from a token to hundreds, negative
    choice scores, biases and blends away from zero."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, s in shapes(cfg).items():
        last = name.rsplit(".", 1)[-1]
        n, u = torch.randn(s, generator=g), torch.rand(s, generator=g)
        if name == "embed":
            t = 2 * n
        elif "norm" in name:
            t = 1 + 0.3 * n
        elif ".mu." in name or last == "vmix":
            t = 0.15 + 0.7 * u
        elif name.endswith("a2.b"):
            t = 3 * n + 2
        elif last == "w0":
            t = 2 * n - 2
        elif last == "u":
            t = n
        elif last == "correction":
            t = 0.4 * n - 0.9
        elif last == "b":
            t = 0.4 * n
        else:
            gain = {"q": 1.6, "k": 1.6, "router": 2.5, "gate": 1.5, "up": 1.5, "w1": 2.0, "a1": 1.5}.get(last, 1.0)
            t = n * gain * s[-1] ** -0.5
        out[name] = t.to(torch.bfloat16)
    return out


def write_model(path, cfg: dict, seed: int = 0) -> Dict[str, torch.Tensor]:
    w = weights(cfg, seed)
    save_file(w, os.path.join(path, "model.safetensors"))
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    return w


class Driver(states.Driver):
    oracle = oracle
    close = staticmethod(base.close)


def check_generate(path, cfg, w, device, **kw) -> None:
    base.check_generate(path, cfg, w, device, oracle=oracle, **kw)


# ---------------------------------------------------------------------------- attention
def check_prep(device, dtype, n, kv, dim, vdim, rot, norm, mixed, base=3000.0, eps=1e-3) -> None:
    """Norm, rotation and blended values into cache rows at far positions; padded rows (slot -1) store nothing."""
    from omni_npu_b200 import ops
    from omni_npu_b200.layers.rope import get_rope
    t, bs = 9, 8
    g = torch.Generator().manual_seed(rot * 10 + n)
    pos = torch.tensor([0, 1, 2, 7, 8, 63, 500, 4097, 5999])
    slots = torch.tensor([3, 30, 31, -1, 0, 17, 5, 8, 9])
    pad8 = lambda x: (x + 7) // 8 * 8                                                    # noqa: E731
    ko, vo = pad8(n * dim), pad8(n * dim) + pad8(kv * dim)
    y, other = (torch.randn(t, vo + pad8(kv * vdim) + 8, generator=g).to(dtype) for _ in range(2))
    qw, kw = ((1 + 0.3 * torch.randn(m * dim, generator=g)).to(dtype) for m in (n, kv))
    rope = get_rope(dim, rot, 6000, base, True, None, torch.device(device), exact_angles=True)
    kc = torch.zeros(4, kv, bs, ops.gated_head_pad(dim, dtype), dtype=dtype, device=device)
    vc = torch.zeros(4, kv, bs, ops.gated_head_pad(vdim, dtype), dtype=dtype, device=device)
    yd, od = y.to(device), other.to(device)
    part = lambda z, a, m: z[:, a: a + m]                                                # noqa: E731
    got = ops.qk_norm_rope_cache(part(yd, 0, n * dim), part(yd, ko, kv * dim), part(yd, vo, kv * vdim), kc, vc,
                                 pos.int().to(device), slots.int().to(device), rope.cos_sin_cache, dim, vdim, rot, norm,
                                 eps, (qw.to(device), kw.to(device)) if norm == "projection" else None, None,
                                 part(od, vo, kv * vdim) if mixed else None, 0.3)
    q, k, v = part(y, 0, n * dim).double(), part(y, ko, kv * dim).double(), part(y, vo, kv * vdim).double()
    if norm == "projection":
        q, k = oracle.rms(q, eps) * qw.double(), oracle.rms(k, eps) * kw.double()
    q, k = (oracle.rotate_halves(x.reshape(t, -1, dim), pos, rot, base) for x in (q, k))
    if norm == "head":
        q, k = oracle.rms(q, eps), oracle.rms(k, eps)
    v = oracle.mix_values(v, part(other, vo, kv * vdim).double() if mixed else None, 0.3).view(t, kv, vdim)
    tol = 3e-6 if dtype == torch.float32 else 0.04
    assert float((got.double().cpu().view(t, n, dim) - q).abs().max()) < tol
    for j in range(t):
        s = int(slots[j])
        if s >= 0:
            assert float((kc[s // bs, :, s % bs, :dim].double().cpu() - k[j]).abs().max()) < tol
            assert float((vc[s // bs, :, s % bs, :vdim].double().cpu() - v[j]).abs().max()) < tol
    assert int((kc != 0).sum()) <= int((slots >= 0).sum()) * kv * dim and float(kc[..., dim:].abs().sum()) == 0.0
    assert float(vc[..., vdim:].abs().sum()) == 0.0


def check_visible(device, dtype, n, kv, dim, vdim, window, t, bs, queries, planted, variant=0, splits=0) -> None:
    """The last ``queries`` rows of a sequence, as a prompt portion and one by one, without sink or gate.  Key
    ``planted`` outweighs all others by far for every query that sees it; the rows land inside wider ones."""
    from omni_npu_b200 import ops
    g = torch.Generator().manual_seed(window * 1000 + t + planted)
    q, k, v = (torch.randn(t, m, dd, generator=g) for m, dd in ((n, dim), (kv, dim), (kv, vdim)))
    q[..., 0] = q[..., 0].abs() + 2.0
    k[..., 0] = 0.0
    k[planted] = 0.0
    k[planted, :, 0] = 6.0 * dim ** 0.5
    q, k, v = (x.to(dtype) for x in (q, k, v))
    scale = dim ** -0.5
    want = oracle.attend(q.double(), k.double(), v.double(), scale, window)
    kc, bt = paged(k, ops.gated_head_pad(dim, dtype), bs, 1)
    vc, _ = paged(v, ops.gated_head_pad(vdim, dtype), bs, 1)
    kc, vc, bt = kc.to(device), vc.to(device), bt.to(device)
    rows = slice(t - queries, t)
    qd = q[rows].reshape(queries, -1).to(device)
    i32 = dict(dtype=torch.int32, device=device)
    tol = 2e-5 if dtype == torch.float32 else 0.03

    def run(q_, cu, lens, b, m):
        wide = torch.full((q_.shape[0], n * vdim + 24), 7.0, dtype=dtype, device=device)
        ops.gated_attention(q_, None, kc, vc, wide[:, : n * vdim], bt, cu, lens, b, m, n, dim, vdim, scale, window, None,
                            max_seq_len=t, variant=variant, splits=splits if cu is None else 0)
        assert float((wide[:, n * vdim:] - 7.0).abs().max()) == 0.0
        return wide[:, : n * vdim]

    out = run(qd, torch.tensor([0, queries], **i32), torch.tensor([t], **i32), 1, queries)
    assert float((out.double().cpu() - want[rows]).abs().max()) < tol * max(1.0, float(want.abs().max()))
    edges = {t - 1, t - queries, planted, *((planted + window - 1, planted + window) if window else ())}
    for i in sorted(x for x in edges if t - queries <= x < t):
        r = i - (t - queries)
        one = run(qd[r: r + 1], None, torch.tensor([i + 1], **i32), 1, 1)
        assert float((one.double().cpu() - want[i: i + 1]).abs().max()) < tol * max(1.0, float(want.abs().max()))


# ---------------------------------------------------------------------------- recurrent layers
def check_token_mix(device, dtype, width, lengths=(23, 9, 40), plan=(3, 1, 17, 2), names="rkvgw") -> None:
    from omni_npu_b200 import ops
    g = torch.Generator().manual_seed(width)
    slot = [2, 0, 3]
    hs = [torch.randn(n, width, generator=g).to(dtype) for n in lengths]
    mu = torch.rand(len(names), width, generator=g).to(dtype)
    state = torch.randn(5, width, generator=g).to(device)                       # what other sequences left
    tol = 1e-6 if dtype == torch.float32 else 0.01
    for step in cuts(list(lengths), plan):
        st = Step(device, [(a, b - a) for _, a, b in step], [slot[i] for i, _, _ in step])
        h = torch.cat([hs[i][a:b] for i, a, b in step]).to(device)
        rows, offs = ops.token_mix(h, mu.to(device), state, st.idx, *st.states)
        assert offs.tolist() == [j * h.shape[0] for j in range(len(names) + 1)]
        for j in range(len(names)):
            want = torch.cat([oracle.token_mix(hs[i].double(), mu[j].double())[a:b] for i, a, b in step])
            assert rel(rows[j * h.shape[0]: (j + 1) * h.shape[0]], want) < tol
        for i, a, b in step:
            assert torch.equal(state[slot[i]].cpu(), hs[i][b - 1].float())
    # a sequence without a slot (a padded row of a captured step) leaves every state alone
    before = state.clone()
    st = Step(device, [(4, 1), (0, 2)], [-1, -1])
    ops.token_mix(hs[2][:3].to(device), mu.to(device), state, st.idx, *st.states)
    assert torch.equal(before, state)


def check_scan(device, dtype, kind, n, dim, vdim, plan=(2, 1, 30, 5), lengths=(70, 3, 45)) -> None:
    """Decayed linear attention ("decay") or time mixing ("bonus") behind their projections, cut into portions, in
    slots that held other sequences."""
    from omni_npu_b200 import ops
    g = torch.Generator().manual_seed(dim)
    slot = [1, 3, 0]
    bonus = kind == "bonus"
    e, m, pad8 = n * vdim, n * dim, lambda x: (x + 7) // 8 * 8
    off = [0, pad8(m), 2 * pad8(m), 2 * pad8(m) + pad8(e)]
    projs = [torch.randn(t, off[3] + pad8(e), generator=g).to(dtype) * 1.5 for t in lengths]
    zs = [torch.randn(t, pad8(m), generator=g) * 2 for t in lengths]
    bias = torch.randn(m, generator=g) * 2 + (-2 if bonus else 2)
    u = torch.randn(n, dim, generator=g)
    nw = (1 + 0.3 * torch.randn(*((n, vdim) if bonus else (vdim,)), generator=g)).to(dtype)
    tau, eps, scale = 6.0, 1e-4, -0.7
    dd = lambda x: x.to(device)                                                          # noqa: E731
    state = dd(torch.randn(5, n, vdim, (dim + 3) // 4 * 4, generator=g))
    tol = 5e-5 if dtype == torch.float32 else 0.02
    want = []
    for x, z in zip(projs, zs):
        x, t = x.double(), x.shape[0]
        q, k = x[:, :m].reshape(t, n, dim), x[:, off[1]: off[1] + m].reshape(t, n, dim)
        v, gate = x[:, off[2]: off[2] + e].reshape(t, n, vdim), x[:, off[3]: off[3] + e]
        z = z[:, :m].double() + bias.double()
        if bonus:
            o = oracle.bonus_scan(q, k, v, torch.exp(-torch.exp(z)).view(t, n, dim), u.double())
        else:
            o = oracle.decay_scan(q * dim ** -0.5, k, v, (oracle.sigmoid(z) ** (1 / tau)).view(t, n, dim))
        want.append((o, (oracle.rms(o, eps) * nw.double()).reshape(t, e) * oracle.silu(gate) * (scale if bonus else 1.0)))
    for step in cuts(list(lengths), plan):
        st = Step(device, [(a, b - a) for _, a, b in step], [slot[i] for i, _, _ in step])
        proj, z = (dd(torch.cat([y[i][a:b] for i, a, b in step])) for y in (projs, zs))
        q, k, v, gate = (proj[:, a: a + c] for a, c in zip(off, (m, m, e, e)))
        if bonus:
            q, k, dec, beta = ops.time_mix_prep(q, k, z, dd(bias), dd(u), n, dim)
        else:
            (q, k, dec), beta = ops.decay_prep(q, k, z, dd(bias), n, dim, dim ** -0.5, tau), None
        o = ops.recurrent_scan(q, k, dec, v, beta, state, n, vdim, *st.states, bonus=bonus)
        if bonus:
            wide = torch.full((o.shape[0], e + 16), 7.0, dtype=dtype, device=device)
            y = ops.head_norm_gate(o, dd(nw), eps, gate, silu=True, scale=scale, out=wide[:, 8: 8 + pad8(e)])
            assert float((wide[:, :8] - 7.0).abs().max()) == 0.0
        else:
            y = ops.head_norm_gate(o, dd(nw), eps, gate, pad8(e), silu=True)
        assert rel(o, torch.cat([want[i][0][a:b] for i, a, b in step])) < 1e-4
        assert rel(y[:, :e], torch.cat([want[i][1][a:b] for i, a, b in step])) < tol
        assert float(y[:, e:].abs().sum()) == 0.0


# ---------------------------------------------------------------------------- products and experts
def check_products(device, dtype, m, ff, width) -> None:
    """Activations and biases in the epilogues: gated gelu behind biases, squared relu, tanh."""
    from omni_npu_b200 import ops
    from omni_npu_b200.ops import ref
    g = torch.Generator().manual_seed(ff + m)
    h = torch.randn(m, width, generator=g).to(dtype)
    wg, wu = ((torch.randn(ff, width, generator=g) * 2 * width ** -0.5).to(dtype) for _ in range(2))
    bg, bu = (torch.randn(ff, generator=g).to(dtype) for _ in range(2))
    zg, zu = h.double() @ wg.double().T, h.double() @ wu.double().T
    tol = 1e-5 if dtype == torch.float32 else 0.012
    dd = lambda x: x.to(device)                                                          # noqa: E731
    bias = torch.stack([bg.view(-1, 8), bu.view(-1, 8)], 1).reshape(-1)
    got = ops.gemm(dd(h), dd(ref.interleave_gate_up(wg, wu)), dd(bias), swiglu=True, act=ops.GELU_TANH)
    assert rel(got, oracle.gelu_tanh(zg + bg.double()) * (zu + bu.double())) < tol
    assert rel(ops.gemm(dd(h), dd(wg), unary="relu2"), oracle.relu_squared(zg)) < tol
    assert rel(ops.gemm(dd(h), dd(wg), unary="tanh"), torch.tanh(zg)) < tol
    cut = m // 3
    offs = torch.tensor([0, cut, cut, m], dtype=torch.int32)
    got = ops.grouped_gemm(dd(h), dd(torch.stack([wg, wu, wu])), dd(offs), unary="relu2")
    assert rel(got, oracle.relu_squared(torch.cat([zg[:cut], zu[cut:]]))) < tol
    plain = ops.grouped_gemm(dd(h), dd(torch.stack([wg, wu, wu])), dd(offs))
    assert rel(plain, torch.cat([zg[:cut], zu[cut:]])) < tol


def check_moe(device, dtype, t, cfg_mlp, width, mult=0.6) -> None:
    """The expert layer alone, its last step fused into the residual kernel.  All choice scores are negative, so
    that an expert of a closed group would win if it counted as zero."""
    from omni_npu_b200 import ops
    from omni_npu_b200.layers.moe import FusedMoE
    r, sh = cfg_mlp["router"], cfg_mlp.get("shared")
    cfg = model(width, 8, [gla(1, 8, 8, mlp=cfg_mlp)])
    w = {k[len("l0.mlp."):]: v for k, v in weights(cfg, 3).items() if k.startswith("l0.mlp.")}
    w["correction"] = (w["correction"] - 1.5).to(torch.bfloat16)
    layer = FusedMoE(r["experts"], r["top"], width, cfg_mlp["expert"]["ff"], dtype, torch.device(device), "sigmoid", False,
                     1.0, r["groups"]["count"], r["groups"]["keep"], router_bias=True, num_shared_experts=1 if sh else 0,
                     shared_intermediate_size=sh["ff"] if sh else None, enable_expert_parallel=False,
                     max_tokens=max(t, 64), unary="relu2")
    layer.gate.weight.data.copy_(w["router"])
    layer.e_score_correction_bias.data.copy_(w["correction"])
    for e in range(r["experts"]):
        layer.weight_loader(layer.w13, w[f"e{e}.up"], e, "up")
        layer.weight_loader(layer.w2, w[f"e{e}.down"], e, "down")
    if sh:
        layer.shared_experts.up_proj.weight.data.copy_(w["shared.up"])
        layer.shared_experts.down_proj.weight.data.copy_(w["shared.down"])
    g = torch.Generator().manual_seed(t)
    h = torch.randn(t, width, generator=g).to(dtype)
    x = torch.randn(t, width, generator=g)
    gain = (torch.randn(width, generator=g) * 0.3).to(dtype)
    wd = {k: v.double() for k, v in w.items()}
    assert float((oracle.sigmoid(h.double() @ wd["router"].T) + wd["correction"]).max()) < 0
    want = x.double() + mult * oracle.moe(h.double(), wd, cfg_mlp)
    routed, rest = layer.forward_deferred(h.to(device))
    res = x.clone().to(device)
    out = ops.residual_add_norm(res, None, rest, routed, gain.to(device), 1e-5, 0.0, width, mult=mult)
    err = (res.double().cpu() - want).abs().amax(-1) / want.std()
    bad = float((err > (2e-5 if dtype == torch.float32 else 0.05)).double().mean())
    assert bad <= (0.0 if dtype == torch.float32 else 0.04), (bad, float(err.max()))
    norm = oracle.rms(res.double().cpu(), 1e-5) * gain.double()
    assert rel(out, norm) < (1e-5 if dtype == torch.float32 else 0.02)
