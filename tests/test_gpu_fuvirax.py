"""Fuvirax's kernels and steps on the GPU, in bf16 and entirely in fp32, against the plain implementation."""
import json
import os
import subprocess
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import fuvirax_cases as cases                                           # noqa: E402
import fuvirax_oracle as oracle                                         # noqa: E402

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
MODELS = {"varied": cases.VARIED, "ragged": cases.RAGGED, "large": cases.LARGE, "wide": cases.WIDE}
DTYPES = {"bfloat16": torch.bfloat16, "float32": torch.float32}


@pytest.fixture(params=sorted(MODELS))
def setup(request, tmp_path):
    cfg = MODELS[request.param]
    return tmp_path, cfg, cases.write_model(tmp_path, cfg, seed=6)


def driver(setup, dtype, **kw):
    path, cfg, w = setup
    return cases.Driver(path, cfg, w, "cuda", dtype, **kw)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
def test_prompts(setup, dtype):
    cases.check_prompts(driver(setup, dtype), (1, 2, 5, 63, 129, 200))


@pytest.mark.parametrize("dtype", sorted(DTYPES))
def test_long_decoding(setup, dtype):
    cases.check_decode(driver(setup, dtype), 3, 150)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("sizes", [(2,), (1, 7, 2, 90)])
def test_portions(setup, dtype, sizes):
    cases.check_portions(driver(setup, dtype), sizes, 150)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("block_size", [16, 64])
def test_mixed_batches_reuse_pages_and_slots(setup, dtype, block_size):
    cases.check_mixed(driver(setup, dtype, max_tokens=320, block_size=block_size), rounds=2)


def test_mixed_batches_without_graphs(setup):
    cases.check_mixed(driver(setup, "bfloat16", max_tokens=256, enforce_eager=True), rounds=1)


@pytest.mark.parametrize("mixed", [False, True])
def test_generation(setup, mixed):
    path, cfg, w = setup
    cases.check_generate(path, cfg, w, "cuda", num_gpu_blocks=9, enable_mixed_batches=mixed)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("streams,width,true", [(1, 24, 24), (2, 256, 256), (3, 48, 43), (4, 4104, 4099), (8, 1032, 1032)])
def test_hyper_connections_and_token_shift(dtype, streams, width, true):
    cases.check_hyper("cuda", DTYPES[dtype], streams, width, true)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
def test_token_shift_in_long_portions(dtype):
    """Portions longer than a CTA's run of tokens, many CTAs per portion."""
    from omni_npu_b200 import ops
    g = torch.Generator().manual_seed(1)
    t, n, w = 2600, 2, 64
    x = torch.randn(t, n, w, generator=g)
    y, ls, mu, nw, nb = (torch.randn(*s, generator=g).to(DTYPES[dtype]) for s in ((t, w), (w,), (w,), (w,), (w,)))
    mix, w_out, w_in = torch.randn(n, n, generator=g), torch.randn(n, generator=g), torch.randn(n, generator=g)
    portions = [(0, 1), (0, 1203), (0, 7), (0, 1389)]
    st = cases.Step("cuda", portions, [3, 0, -1, 1])
    state = torch.randn(4, w, generator=g).cuda()
    new, h = ops.hyper_norm(x.cuda(), None, None, n, y.cuda(), (ls.cuda(), mix.cuda(), w_out.cuda()), w_in.cuda(), nw.cuda(),
                            nb.cuda(), 1e-4, w, 1.0, (mu.cuda(), state, st.idx, *st.states))
    full = torch.einsum("tsw,sr->trw", x.double(), mix.double()) + w_out.double()[None, :, None] * \
        (y.double() * ls.double())[:, None]
    u = oracle.layer_norm(torch.einsum("tsw,s->tw", full, w_in.double()), nw.double(), nb.double(), 1e-4)
    a = 0
    for (_, m), slot in zip(portions, (3, 0, -1, 1)):
        assert cases.rel(h[a:a + m], oracle.token_shift(u[a:a + m], mu.double())) < (2e-5 if dtype == "float32" else 0.02)
        if slot >= 0:
            assert cases.rel(state[slot], u[a + m - 1]) < 2e-5
        a += m
    assert cases.rel(new, full) < 2e-6


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("heads,dim,vdim", [(2, 8, 12), (3, 10, 7), (2, 64, 64), (4, 128, 96), (1, 200, 136), (1, 500, 40)])
def test_gated_linear_attention(dtype, heads, dim, vdim):
    cases.check_gated_linear("cuda", DTYPES[dtype], heads, dim, vdim)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("heads,kv,dim,vdim,taps", [(2, 2, 8, 12, 4), (6, 2, 10, 7, 2), (3, 1, 5, 9, 1), (2, 1, 64, 72, 8),
                                                    (4, 2, 128, 128, 4), (2, 2, 130, 300, 3), (1, 1, 400, 24, 5)])
def test_delta_rule(dtype, heads, kv, dim, vdim, taps):
    cases.check_delta("cuda", DTYPES[dtype], heads, kv, dim, vdim, taps)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("heads,dim,rot,vdim,rank", [(3, 12, 8, 20, 28), (16, 128, 64, 128, 512), (18, 40, 24, 72, 136),
                                                     (5, 56, 40, 88, 250), (2, 200, 72, 48, 520), (1, 7, 2, 9, 11)])
@pytest.mark.parametrize("planted", [0, 15, 16, 64, 119, 120, 150])
def test_latent_attention(dtype, heads, dim, rot, vdim, rank, planted):
    cases.check_latent("cuda", DTYPES[dtype], heads, dim, rot, vdim, rank, planted, bs=16 if planted % 2 else 64, splits=5)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("m", [1, 7, 130, 1500])
def test_xielu(dtype, m):
    cases.check_xielu("cuda", DTYPES[dtype], m, 72, 200, 0.7, -1.3)
    cases.check_xielu("cuda", DTYPES[dtype], m, 1024, 512, -2.0, 0.4)


def test_trace_command(tmp_path):
    """bin/trace_run from the outside: lines in, files out."""
    cfg = cases.VARIED
    w = cases.write_model(tmp_path, cfg, seed=2)
    toks = cases.tokens(20, cfg["vocab"], 1)
    lines = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:17], "want": [16, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": toks[:2], "want": [1]},
                                     {"id": "a", "tokens": toks[17:18], "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": toks[18:], "want": [0, 1]}], "end": ["a"]}]
    out = tmp_path / "out"
    out.mkdir()
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out",
                        str(out), "--max-tokens", "128"], input="\n".join(map(json.dumps, lines)) + "\n", text=True,
                       capture_output=True, timeout=280)
    assert r.returncode == 0, r.stderr[-2000:]
    ref = oracle.forward(toks, w, cfg)
    for step, rows in ((0, ref[[16, 3]]), (1, torch.stack([ref[1], ref[17]])), (2, ref[18:])):
        got = torch.frombuffer(bytearray((out / f"{step}.f32").read_bytes()), dtype=torch.float32)
        cases.close(got.view(rows.shape), rows, "float32")
