"""Rivudra's kernels and steps on the GPU, in bf16 and entirely in fp32, against the plain implementation."""
import json
import os
import subprocess
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import rivudra_cases as cases                                           # noqa: E402
import rivudra_oracle as oracle                                         # noqa: E402

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
MODELS = {"varied": cases.VARIED, "ragged": cases.RAGGED, "head128": cases.HEAD128, "wide": cases.WIDE}
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
    cases.check_prompts(driver(setup, dtype), (1, 2, 5, 63, 129, 300))


@pytest.mark.parametrize("dtype", sorted(DTYPES))
def test_long_decoding(setup, dtype):
    cases.check_decode(driver(setup, dtype), 3, 180)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("sizes", [(2,), (16, 1), (1, 7, 2, 90)])
def test_portions(setup, dtype, sizes):
    cases.check_portions(driver(setup, dtype), sizes, 210)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("block_size", [16, 64])
def test_mixed_batches_reuse_pages(setup, dtype, block_size):
    cases.check_mixed(driver(setup, dtype, max_tokens=320, block_size=block_size))


def test_mixed_batches_without_graphs(setup):
    cases.check_mixed(driver(setup, "bfloat16", max_tokens=256, enforce_eager=True), rounds=1)


@pytest.mark.parametrize("mixed", [False, True])
def test_generation(setup, mixed):
    path, cfg, w = setup
    cases.check_generate(path, cfg, w, "cuda", num_gpu_blocks=9, enable_mixed_batches=mixed)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("heads,kv,dim,vdim", [(6, 2, 24, 40), (4, 1, 128, 128), (20, 1, 64, 64), (3, 1, 200, 144),
                                               (2, 2, 12, 20), (32, 8, 128, 128), (150, 1, 16, 16)])
@pytest.mark.parametrize("window", [1, 16, 63, 64, 65, 130])
def test_window_edges(dtype, heads, kv, dim, vdim, window):
    t = 200
    for planted in (0, 64, 128, 150):
        cases.check_window("cuda", DTYPES[dtype], heads, kv, dim, vdim, window, t, 16, 137, planted)
    if dtype == "bfloat16" and dim == 128:
        cases.check_window("cuda", torch.bfloat16, heads, kv, dim, vdim, window, t, 32, 199, 64, variant=1)


@pytest.mark.parametrize("splits", [1, 2, 4, 8, 0])
@pytest.mark.parametrize("window", [700, 1024, 3000])
def test_split_decoding(window, splits):
    for planted in (0, 1500 - window if window < 1500 else 3, 1499, 1000):
        cases.check_window("cuda", torch.bfloat16, 8, 2, 128, 96, window, 1500, 16, 3, planted, splits=splits)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("rot,dim,vdim", [(2, 24, 20), (24, 24, 20), (64, 128, 128), (38, 51, 33)])
def test_rotation(dtype, rot, dim, vdim):
    cases.check_rope("cuda", DTYPES[dtype], 3, 1, dim, vdim, rot, 700.0)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("m", [1, 7, 130, 1500])
def test_clamped_glu(dtype, m):
    cases.check_glu("cuda", DTYPES[dtype], m, 72, 200, 0.6)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("t", [1, 5, 33, 400])
def test_expert_layer(dtype, t):
    cases.check_moe("cuda", DTYPES[dtype], t, cases.moe(12, 3, 24, 0.7, 4, 2, 1.4, shared=(16, 1.2)), 48)
    cases.check_moe("cuda", DTYPES[dtype], t, cases.moe(40, 6, 136, 0.7), 256)


@pytest.mark.parametrize("width,true", [(104, 100), (256, 256), (4096, 4096), (12288, 12281)])
@pytest.mark.parametrize("dtype", sorted(DTYPES))
def test_embedding_and_norm(width, true, dtype):
    from omni_npu_b200 import ops
    g = torch.Generator().manual_seed(width)
    table = torch.randn(50, width, generator=g)
    table[:, true:] = 0
    gain = torch.randn(width, generator=g) * 0.3
    table, gain = table.to(DTYPES[dtype]), gain.to(DTYPES[dtype])
    ids = torch.randint(0, 50, (9,), generator=g)
    res = torch.empty(9, width, device="cuda")
    out = ops.embed_residual_norm(res, ids.int().cuda(), table.cuda(), 7.5, gain.cuda(), 1e-5, 1.0, true)
    x = table[ids].double() * 7.5
    assert torch.allclose(res.double().cpu(), x, rtol=1e-6)
    want = oracle.rms_norm(x[:, :true], gain[:true].double(), 1e-5)
    err = (out.double().cpu()[:, :true] - want).abs().max()
    assert float(err) < (1e-5 if dtype == "float32" else 0.01) * float(want.abs().max())


@pytest.mark.parametrize("groups,keep,top", [(1, 1, 5), (4, 1, 3), (4, 3, 7), (12, 5, 5)])
def test_routing(groups, keep, top):
    from omni_npu_b200 import ops
    logits = torch.randn(40, 12, generator=torch.Generator().manual_seed(groups)) * 2
    ids, w = ops.moe_topk(logits.cuda(), None, top, False, groups, keep, True, 1.3)
    got = torch.zeros(40, 12).scatter_(1, ids.long().cpu(), w.cpu())
    assert float((got.double() - oracle.route(logits.double(), top, groups, keep, 1.3)).abs().max()) < 1e-5


def test_trace_command(tmp_path):
    """bin/trace_run from the outside: lines in, files out."""
    cfg = cases.VARIED
    w = cases.write_model(tmp_path, cfg, seed=2)
    toks = cases.tokens(20, cfg["vocab"], 1)
    lines = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:17], "want": [16, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[17:18], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": toks[:2], "want": [1]},
                                     {"id": "a", "tokens": toks[18:19], "want": [0]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "a", "tokens": toks[19:], "want": [0]}], "end": ["a"]}]
    out = tmp_path / "out"
    out.mkdir()
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out",
                        str(out), "--max-tokens", "128"], input="\n".join(map(json.dumps, lines)) + "\n", text=True,
                       capture_output=True, timeout=280)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    assert not (out / "1.f32").exists()
    ref = oracle.forward(toks, w, cfg)
    for step, rows in ((0, ref[[16, 3]]), (2, torch.stack([ref[1], ref[18]])), (3, ref[19:20])):
        got = torch.frombuffer(bytearray((out / f"{step}.f32").read_bytes()), dtype=torch.float32)
        cases.close(got.view(rows.shape), rows, "float32")
