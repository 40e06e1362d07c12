"""Small random Fuvirax models and the checks that the CPU and GPU tests share: the framework's step
function, cache, state slots and scheduler against the plain implementation in fuvirax_oracle.py."""
from __future__ import annotations

import json
import os
from typing import Dict, List, Tuple

import torch
from safetensors.torch import save_file

import fuvirax_oracle as oracle
import rivudra_cases as base
from rivudra_cases import check_decode, check_mixed, check_portions, check_prompts, tokens       # noqa: F401


def dense(ff) -> dict:
    return {"kind": "dense", "ff": ff}


def latent(heads, dim, rot, vdim, rank, scale=None, theta=3000.0, mlp=None) -> dict:
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank,
                      "rot": {"base": theta, "dims": rot}, "scale": (dim + rot) ** -0.5 if scale is None else scale}}


def hgrn2(heads, dim, vdim, mlp=None) -> dict:
    return {"type": "hgrn2", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim}}


def delta(heads, kv, dim, vdim, conv, mlp=None) -> dict:
    return {"type": "channel_delta", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}}


def model(width, vocab, layers, streams=2, loop=None, scale=0.8, eps=1e-4) -> dict:
    d = {"architecture": "Fuvirax", "width": width, "vocab": vocab, "streams": streams, "logit_scale": scale,
         "norm": {"eps": eps}, "layers": layers}
    if loop:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


# every mixer, a layer without a feed-forward, shared q / k heads, a loop in the middle over a cached layer
VARIED = model(96, 203, [
    hgrn2(3, 20, 24),
    delta(4, 2, 24, 40, 3, mlp=dense(56)),
    latent(4, 24, 16, 40, 56, mlp=dense(40)),
    hgrn2(2, 36, 64, mlp=dense(72)),
], streams=3, loop=(1, 3, 2))
# nothing is a whole 16-byte row, one stream, no convolution to speak of, no loop
RAGGED = model(100, 77, [
    latent(3, 20, 6, 12, 28, scale=0.4, mlp=dense(36)),
    delta(3, 1, 18, 22, 1, mlp=dense(20)),
    hgrn2(5, 10, 14, mlp=dense(12)),
], streams=1, scale=1.0)
# the sizes of the DeepSeek cache row, rows above 64 in the states
LARGE = model(256, 320, [
    delta(4, 4, 128, 128, 4, mlp=dense(256)),
    latent(6, 128, 64, 128, 512, mlp=dense(128)),
    hgrn2(2, 160, 96, mlp=dense(512)),
], streams=4, loop=(0, 2, 2))
# beyond the tensor-core kernels, the longest convolution, many streams
WIDE = model(128, 150, [
    latent(2, 200, 72, 48, 520, mlp=dense(64)),
    delta(2, 1, 264, 40, 8, mlp=dense(64)),
    latent(18, 16, 8, 24, 136),
    hgrn2(1, 300, 72, mlp=dense(32)),
], streams=7, loop=(3, 4, 3))


def ranks(i: int) -> Tuple[int, int]:
    """Ranks of layer i's low-rank projections (decay, gate): no config key has them."""
    return 5 + 3 * i, 12 + i


def shapes(cfg: dict) -> Dict[str, Tuple[int, ...]]:
    w, n = cfg["width"], cfg["streams"]
    out = {"embed": (cfg["vocab"], w), "final.norm": (w,), "final.norm.b": (w,)}
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}."
        for q in ("1", "2") if layer["mlp"] else ("1",):
            out.update({f"{p}norm{q}": (w,), f"{p}norm{q}.b": (w,), f"{p}ls{q}": (w,), f"{p}hc{q}.in": (n,),
                        f"{p}hc{q}.out": (n,), f"{p}hc{q}.mix": (n, n)})
        out[p + "shift"] = (w,)
        h, d, e = m["heads"], m["dim"], m["vdim"]
        mix = {"o": (w, h * e)}
        if layer["type"] == "latent_attention":
            r = m["kv_rank"]
            mix.update({"q": (h * (d + m["rot_dim"]), w), "dkv": (r + m["rot_dim"], w), "dkv.norm": (r,),
                        "uk": (h * d, r), "uv": (h * e, r)})
        elif layer["type"] == "hgrn2":
            mix.update({"q": (h * d, w), "f": (h * d, w), "f.b": (h * d,), "lower": (h * d,), "v": (h * e, w),
                        "norm": (e,)})
        else:
            g, (ra, rg) = m["kv_heads"], ranks(i)
            mix.update({"q": (g * d, w), "k": (g * d, w), "v": (h * e, w), "q.conv": (g * d, m["conv"]),
                        "k.conv": (g * d, m["conv"]), "v.conv": (h * e, m["conv"]), "b": (h, w), "A_log": (h,),
                        "norm": (e,), "a1": (ra, w), "a2": (h * d, ra), "dt_bias": (h * d,), "g1": (rg, w),
                        "g2": (h * e, rg)})
        out.update({f"{p}mix.{k}": s for k, s in mix.items()})
        if layer["mlp"]:
            ff = layer["mlp"]["ff"]
            out.update({p + "mlp.up": (ff, w), p + "mlp.down": (w, ff), p + "mlp.act": (2,)})
    return out


def weights(cfg: dict, seed: int) -> Dict[str, torch.Tensor]:
    """bf16 weights that leave no mechanism idle: scores of a few units, forget gates and decays from short
    to hundreds of tokens, norm biases and shifts away from zero, unequal streams."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, s in shapes(cfg).items():
        last = name.rsplit(".", 1)[-1]
        n = torch.randn(s, generator=g)
        u = torch.rand(s, generator=g)
        if name == "embed":
            t = n
        elif "norm" in name:
            t = 0.3 * n if last == "b" else 1 + 0.3 * n
        elif last in ("ls1", "ls2"):
            t = 0.7 + 0.6 * u
        elif ".hc" in name:
            t = {"in": 0.3 + u, "out": 0.4 + u}.get(last, 0.3 * n)
            if last == "mix":
                t = t + 0.9 * torch.eye(s[0])
        elif last == "shift":
            t = u
        elif name.endswith("f.b"):
            t = 3 * n + 1
        elif last == "lower":
            t = u * u
        elif last == "A_log":
            t = -3 * u
        elif last == "dt_bias":
            t = 2 * n - 2
        elif last == "conv":
            t = n * s[1] ** -0.5
        elif last == "act":
            t = n
        else:
            gain = {"q": 2.0, "dkv": 1.5, "uk": 2.0, "f": 1.5, "a1": 1.5, "b": 2.0, "up": 1.5}.get(last, 1.0)
            t = n * gain * s[-1] ** -0.5
        out[name] = t.to(torch.bfloat16)
    return out


def write_model(path, cfg: dict, seed: int = 0) -> Dict[str, torch.Tensor]:
    w = weights(cfg, seed)
    save_file(w, os.path.join(path, "model.safetensors"))
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    return w


def close(got: torch.Tensor, want: torch.Tensor, dtype: str) -> None:
    assert got.shape == want.shape
    d = got.double() - want.double()
    err = (d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / want.double().std()
    assert float(err.max()) < (5e-5 if dtype == "float32" else 0.15), err.topk(min(5, err.numel()))
    if dtype != "float32":
        assert float(err.median()) < 0.04, float(err.median())


class Driver(base.Driver):
    oracle = oracle
    close = staticmethod(close)

    def finish(self) -> None:
        slots = self.replay.engine.scheduler.state_pool
        assert slots.num_free == slots.num_slots, "state slots were not given back"
        super().finish()


def check_generate(path, cfg, w, device, **kw) -> None:
    base.check_generate(path, cfg, w, device, oracle=oracle, **kw)


# ---------------------------------------------------------------------------- mechanism checks
class Step:
    """Portions of several sequences as one step: their places, lengths and state slots on the device."""

    def __init__(self, device, portions, slots) -> None:
        """``portions``: (tokens before this step, tokens in it) per sequence."""
        i32 = dict(dtype=torch.int32, device=device)
        n = [b for _, b in portions]
        self.num_seqs, self.tokens = len(n), sum(n)
        self.cu = torch.tensor([0, *torch.tensor(n).cumsum(0).tolist()], **i32)
        self.lens = torch.tensor([a + b for a, b in portions], **i32)
        self.slots = torch.tensor(slots, **i32)
        self.idx = torch.repeat_interleave(torch.arange(len(n)), torch.tensor(n)).to(**i32)

    @property
    def states(self):
        return self.slots, self.cu, self.lens, self.num_seqs


def cuts(lengths: List[int], plan) -> List[List[Tuple[int, int, int]]]:
    """Steps of (sequence, from, to): each sequence in portions of the sizes in ``plan``, all sequences side
    by side, one of them left out now and then."""
    at, out, k = [0] * len(lengths), [], 0
    while any(a < n for a, n in zip(at, lengths)):
        step = []
        for i, n in enumerate(lengths):
            k += 1
            if at[i] < n and k % 5:
                m = min(plan[(k + i) % len(plan)], n - at[i])
                step.append((i, at[i], at[i] + m))
                at[i] += m
        if step:
            out.append(step)
    return out


def rel(got: torch.Tensor, want: torch.Tensor) -> float:
    return float((got.double().cpu() - want).abs().max() / want.abs().max().clamp_min(1e-9))


def check_hyper(device, dtype, streams, width, true, plan=(3, 1, 17, 2)) -> None:
    """Join, reading, norm, scale and token shift over sequences cut into portions; slots that held other
    sequences before; the start from an embedding table."""
    from omni_npu_b200 import ops
    g = torch.Generator().manual_seed(streams * 1000 + true)
    lengths, slot = [23, 9, 40], [2, 0, 3]

    def rand(*s):
        return torch.randn(*s, generator=g)

    def vec(x):
        return torch.nn.functional.pad(x, (0, width - true)).to(dtype)

    xs = [rand(streams, n, true) * 4 + 1 for n in lengths]
    ys = [vec(rand(n, true)) for n in lengths]
    ls, mix, w_out, w_in = vec(rand(true)), rand(streams, streams), rand(streams), rand(streams)
    nw, nb, mu = vec(1 + 0.3 * rand(true)), vec(rand(true)), vec(torch.rand(true, generator=g))
    eps, scale = 1e-3, 0.6
    dd = lambda x: x.to(device)                                                          # noqa: E731
    state = dd(rand(5, width))
    tol = 2e-5 if dtype == torch.float32 else 0.02

    def want_of(x):
        u = sum(w_in[s].double() * x[s] for s in range(streams))
        h = oracle.layer_norm(u, nw[:true].double(), nb[:true].double(), eps) * scale
        return h, oracle.token_shift(h, mu[:true].double())

    for step in cuts(lengths, plan):
        st = Step(device, [(a, b - a) for _, a, b in step], [slot[i] for i, _, _ in step])
        x = torch.cat([xs[i][:, a:b] for i, a, b in step], 1).transpose(0, 1)
        x = torch.nn.functional.pad(x, (0, width - true)).contiguous()
        y = torch.cat([ys[i][a:b] for i, a, b in step])
        new, h = ops.hyper_norm(dd(x), None, None, streams, dd(y), (dd(ls), dd(mix), dd(w_out)), dd(w_in), dd(nw), dd(nb),
                                eps, true, scale, (dd(mu), state, st.idx, *st.states))
        row = 0
        for i, a, b in step:
            full = torch.stack([sum(mix[s, t].double() * xs[i][s].double() for s in range(streams))
                                + w_out[t].double() * (ys[i].double() * ls.double())[:, :true] for t in range(streams)])
            n = b - a
            assert rel(new[row:row + n, :, :true].transpose(0, 1), full[:, a:b]) < 2e-6
            h_all, want = want_of(full)
            assert rel(h[row:row + n, :true], want[a:b]) < tol
            assert rel(state[slot[i], :true], h_all[b - 1]) < 2e-5
            row += n
        assert float(h[:, true:].abs().sum()) == 0.0
    # from a table, without a shift, nothing kept
    table, ids = vec(rand(30, true)), torch.randint(0, 30, (11,), generator=g)
    none, h = ops.hyper_norm(None, dd(ids.int()), dd(table), streams, None, None, dd(w_in), dd(nw), dd(nb), eps, true,
                             scale, None, False)
    assert none is None
    x = table[ids, :true].double().expand(streams, -1, -1)
    assert rel(h[:, :true], want_of(x)[0]) < tol
    st = Step(device, [(0, 4), (0, 1), (0, 6)], [1, -1, 4])
    kept, h = ops.hyper_norm(None, dd(ids.int()), dd(table), streams, None, None, dd(w_in), dd(nw), dd(nb), eps, true,
                             scale, (dd(mu), state, st.idx, *st.states))
    assert torch.equal(kept.cpu()[:, :, :true], table[ids, None, :true].float().expand(-1, streams, -1))
    for a, b in ((0, 4), (4, 5), (5, 11)):
        assert rel(h[a:b, :true], want_of(x[:, a:b])[1]) < tol


def check_gated_linear(device, dtype, heads, dim, vdim, plan=(2, 1, 30, 5)) -> None:
    from omni_npu_b200 import ops
    g = torch.Generator().manual_seed(dim)
    lengths, slot = [70, 3, 45], [1, 3, 0]
    n, e = heads * dim, heads * vdim
    off = {"q": 8, "f": 8 + (n + 7) // 8 * 8, "v": 8 + 2 * ((n + 7) // 8 * 8)}
    projs = [torch.randn(t, off["v"] + (e + 7) // 8 * 8, generator=g).to(dtype) * 2 for t in lengths]
    bias, low = torch.randn(n, generator=g) * 3, torch.rand(n, generator=g) ** 2
    nw = (1 + 0.3 * torch.randn(vdim, generator=g)).to(dtype)
    state = torch.randn(5, heads, vdim, (dim + 3) // 4 * 4, generator=g).to(device)        # what other sequences left
    width = (e + 7) // 8 * 8
    tol = 5e-5 if dtype == torch.float32 else 0.02
    want = []
    for x in projs:
        x = x.double()
        t = x.shape[0]
        f = low.double() + (1 - low.double()) * oracle.sigmoid(x[:, off["f"]: off["f"] + n] + bias.double())
        o = oracle.gated_linear_scan(oracle.silu(x[:, off["q"]: off["q"] + n]).view(t, heads, dim), f.view(t, heads, dim),
                                     x[:, off["v"]: off["v"] + e].view(t, heads, vdim))
        want.append((o, (oracle.rms(o, 1e-4) * nw.double()).reshape(t, e)))
    for step in cuts(lengths, plan):
        st = Step(device, [(a, b - a) for _, a, b in step], [slot[i] for i, _, _ in step])
        proj = torch.cat([projs[i][a:b] for i, a, b in step]).to(device)
        q, k = ops.gated_linear_prep(proj, off["q"], off["f"], heads, dim, bias.to(device), low.to(device))
        o = ops.recurrent_scan(q, k, None, proj[:, off["v"]: off["v"] + e], None, state, heads, vdim, *st.states)
        y = ops.head_norm_gate(o, nw.to(device), 1e-4, None, width)
        assert rel(o, torch.cat([want[i][0][a:b] for i, a, b in step])) < 1e-4
        assert rel(y[:, :e], torch.cat([want[i][1][a:b] for i, a, b in step])) < tol
        assert float(y[:, e:].abs().sum()) == 0.0


def check_delta(device, dtype, heads, kv, dim, vdim, taps, plan=(2, 1, 30, 5)) -> None:
    from omni_npu_b200 import ops
    g = torch.Generator().manual_seed(dim * 10 + taps)
    lengths, slot = [70, 3, 45], [1, 3, 0]
    pad8 = lambda n: (n + 7) // 8 * 8                                                    # noqa: E731
    n, e, c = heads * dim, heads * vdim, kv * dim
    offs = {"q": 0, "k": pad8(c), "v": 2 * pad8(c)}
    offs["b"] = ch = offs["v"] + pad8(e)
    projs = [torch.randn(t, ch + pad8(heads), generator=g).to(dtype) * 1.5 for t in lengths]
    lows = [torch.randn(t, n, generator=g).to(dtype) * 2 for t in lengths]
    gates = [torch.randn(t, e, generator=g).to(dtype) * 2 for t in lengths]
    conv_w = (torch.randn(ch, taps, generator=g) * taps ** -0.5).to(dtype)
    dt, a_log = torch.randn(n, generator=g) * 2 - 2, -3 * torch.rand(heads, generator=g)
    nw = (1 + 0.3 * torch.randn(vdim, generator=g)).to(dtype)
    dd = lambda x: x.to(device)                                                          # noqa: E731
    state = dd(torch.randn(5, heads, vdim, (dim + 3) // 4 * 4, generator=g))
    conv_state = dd(torch.randn(5, taps - 1, ch, generator=g).to(dtype))
    tol = 5e-5 if dtype == torch.float32 else 0.02
    want = []
    for x, lo, gt in zip(projs, lows, gates):
        x, t = x.double(), x.shape[0]

        def conv(name, cols):
            o = offs[name]
            return oracle.short_conv(x[:, o: o + cols], conv_w[o: o + cols].double())

        q = (oracle.unit(conv("q", c).view(t, kv, dim)) * dim ** -0.5).repeat_interleave(heads // kv, 1)
        k = oracle.unit(conv("k", c).view(t, kv, dim)).repeat_interleave(heads // kv, 1)
        v = conv("v", e).view(t, heads, vdim)
        rate = oracle.softplus(lo.double() + dt.double()).view(t, heads, dim)
        dec = torch.exp(-torch.exp(a_log.double())[None, :, None] * rate)
        o = oracle.delta_scan(q, k, v, dec, oracle.sigmoid(x[:, ch: ch + heads]))
        want.append((o, (oracle.rms(o, 1e-4) * nw.double()).reshape(t, e) * oracle.sigmoid(gt.double())))
    for step in cuts(lengths, plan):
        st = Step(device, [(a, b - a) for _, a, b in step], [slot[i] for i, _, _ in step])
        proj, low, gate = (dd(torch.cat([z[i][a:b] for i, a, b in step])) for z in (projs, lows, gates))
        q, k, dec, v, beta = ops.delta_prep(proj, low, offs, heads, kv, dim, vdim, dd(conv_w), conv_state, dd(dt), dd(a_log),
                                            oracle.UNIT_EPS, st.idx, *st.states)
        o = ops.recurrent_scan(q, k, dec, v, beta, state, heads, vdim, *st.states, conv=(proj, conv_state))
        y = ops.head_norm_gate(o, dd(nw), 1e-4, gate, pad8(e))
        assert rel(o, torch.cat([want[i][0][a:b] for i, a, b in step])) < (1e-4 if dtype == torch.float32 else 0.01)
        assert rel(y[:, :e], torch.cat([want[i][1][a:b] for i, a, b in step])) < tol
        for i, a, b in step:                       # the newest inputs, oldest first, zeros before the start
            kept = torch.cat([torch.zeros(taps - 1, ch, dtype=dtype), projs[i][:b, :ch]])[b:]
            assert torch.equal(conv_state[slot[i]].cpu(), kept)


def check_latent(device, dtype, heads, dim, rot, vdim, rank, planted, t=200, bs=16, prompt=120, splits=0) -> None:
    """One layer's attention: a prompt in two portions, then token by token, over shuffled pages.  The key
    at ``planted`` outweighs all others for every query that sees it."""
    from omni_npu_b200 import ops
    from omni_npu_b200.attention.latent import LatentAttention
    from omni_npu_b200.attention.metadata import AttentionMetadata, set_forward_context
    from omni_npu_b200.layers.rope import get_rope
    g = torch.Generator().manual_seed(planted * 100 + dim)
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "rot": {"base": 900.0},
         "scale": (dim + rot) ** -0.5}

    def rand(*s):
        return torch.randn(*s, generator=g)

    w = {"dkv.norm": 1 + 0.3 * rand(rank), "uk": rand(heads * dim, rank) * rank ** -0.5,
         "uv": rand(heads * vdim, rank) * rank ** -0.5}
    q, down = rand(t, heads, dim + rot) * 0.5, rand(t, rank + rot)
    c = oracle.rms(down[planted, :rank], 1e-5) * w["dkv.norm"]
    key = (w["uk"] @ c).view(heads, dim)
    q[..., :dim] += key / key.pow(2).sum(-1, keepdim=True) * 14 / m["scale"]
    q = q.reshape(t, -1).to(dtype)
    down = down.to(dtype)
    w = {k: v.to(dtype) for k, v in w.items()}
    want = oracle.latent_core(q.double(), down.double(), {k: v.double() for k, v in w.items()}, m, 1e-5)
    attn = LatentAttention(heads, dim, rot, vdim, rank, m["scale"], True, 1e-5, dtype, torch.device(device))
    attn.latent_norm.data.copy_(w["dkv.norm"])
    attn.w_uk.data.copy_(w["uk"])
    attn.w_uv.data.copy_(w["uv"])
    attn.build_absorbed()
    cos_sin = get_rope(rot, rot, t, 900.0, True, None, torch.device(device), exact_angles=True).cos_sin_cache
    n = (t + bs - 1) // bs
    pages = torch.randperm(n + 3, generator=g)[:n]
    cache = (rand(n + 3, bs, attn.row) * 50).to(dtype).to(device)             # what other sequences left
    i32 = dict(dtype=torch.int32, device=device)

    def run(a: int, b: int) -> torch.Tensor:
        pos = torch.arange(a, b)
        md = AttentionMetadata(
            is_prefill=b - a > 1, num_seqs=1, num_tokens=b - a, max_q_len=b - a, max_seq_len=b if b - a > 1 else t, q_len=1,
            positions=pos.to(**i32), slot_mapping=(pages[pos // bs] * bs + pos % bs).to(**i32),
            block_tables=pages.to(**i32).view(1, -1), seq_lens=torch.tensor([b], **i32),
            cu_q=torch.tensor([0, b - a], **i32))
        if b - a > 1:
            md.extra["seq_lens_host"] = [b]
        with set_forward_context(md, [cache]):
            return attn(q[a:b].clone().to(device), down[a:b].to(device), cos_sin, 0)

    got = torch.cat([run(0, prompt // 3), run(prompt // 3, prompt), *(run(i, i + 1) for i in range(prompt, t))])
    assert rel(got, want) < (1e-4 if dtype == torch.float32 else 0.04)
    if device != "cpu" and splits and dtype != torch.float32:
        qs = torch.randn(3, heads, attn.row, generator=g).to(dtype).to(device)
        lens, bt = torch.tensor([t, 1, 77], **i32), pages.to(**i32).view(1, -1).repeat(3, 1)
        outs = []
        for s in (1, splits):
            o = torch.empty(3, heads, rank, dtype=dtype, device=device)
            ops.latent_decode(qs, cache, bt, lens, 3, heads, rank, m["scale"], o, splits=s)
            outs.append(o.double().cpu())
        assert rel(outs[1], outs[0]) < 0.02


def check_xielu(device, dtype, m, ff, width, p, q) -> None:
    from omni_npu_b200.layers.mlp import XieluMLP
    from omni_npu_b200 import ops
    g = torch.Generator().manual_seed(ff)
    mlp = XieluMLP(width, ff, dtype, torch.device(device))
    mlp.act_params.data.copy_(torch.tensor([p, q]))
    mlp.fix_constants()
    h = torch.randn(m, width, generator=g).to(dtype)
    up = (torch.randn(ff, width, generator=g) * 2 * width ** -0.5).to(dtype)
    want = oracle.xielu(h.double() @ up.double().T, torch.tensor(p).double(), torch.tensor(q).double())
    got = ops.gemm(h.to(device), up.to(device), xielu=mlp.constants)
    assert rel(got, want) < (1e-5 if dtype == torch.float32 else 0.01)
