"""Gatosun's kernels and steps on the GPU, in bf16 and entirely in fp32, against the plain implementation."""
import json
import os
import subprocess
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import gatosun_cases as cases                                           # noqa: E402
import gatosun_oracle as oracle                                         # noqa: E402

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


def test_residual_stays_32_bit(setup):
    d = driver(setup, "float32")
    _, cfg, w = setup
    toks, want = cases.tokens(90, cfg["vocab"], 4), []
    oracle.forward(toks, w, cfg, layers_out=want)
    d.replay.runner.model.layer_outputs = got = []
    d.replay.step([{"id": "a", "tokens": toks, "want": []}])
    for x, y in zip(got, want):
        assert x.dtype == torch.float32 and cases.rel(x, y) < 2e-5


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("norm,mixed", [("projection", True), ("projection", False), ("head", False), ("head", True),
                                        (None, False)])
@pytest.mark.parametrize("shape", [(4, 2, 24, 16, 16), (3, 1, 18, 22, 6), (32, 8, 128, 128, 128), (5, 5, 272, 40, 96),
                                   (2, 1, 64, 64, 24)])
def test_norm_rotation_and_values(dtype, shape, norm, mixed):
    cases.check_prep("cuda", DTYPES[dtype], *shape, norm, mixed)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("shape", [(4, 2, 24, 20), (8, 2, 128, 128), (6, 1, 96, 48), (2, 2, 200, 72), (3, 1, 272, 40)])
@pytest.mark.parametrize("window,planted", [(0, 0), (0, 127), (0, 128), (1, 150), (40, 120), (40, 160), (40, 161), (65, 135),
                                            (65, 136), (200, 1)])
def test_visible_keys(dtype, shape, window, planted):
    for variant, splits in ((0, 0), (1, 4), (2, 0)) if dtype == "bfloat16" else ((0, 0),):
        cases.check_visible("cuda", DTYPES[dtype], *shape, window, 201, 16 if planted % 2 else 64, 170, planted, variant,
                            splits)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("width", [24, 1032, 4104])
def test_blends_with_the_previous_token(dtype, width):
    cases.check_token_mix("cuda", DTYPES[dtype], width)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("names", ["r", "rk", "rkvgw"])
def test_blends_in_long_portions(dtype, names):
    """Portions longer than a thread's run of tokens, in one step."""
    cases.check_token_mix("cuda", DTYPES[dtype], 64, (2203, 1, 2800), (3000, 1900), names)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("kind", ["decay", "bonus"])
@pytest.mark.parametrize("heads,dim,vdim", [(2, 8, 12), (3, 10, 7), (2, 64, 64), (4, 128, 96), (1, 200, 136), (1, 500, 40)])
def test_recurrent_layers(dtype, kind, heads, dim, vdim):
    cases.check_scan("cuda", DTYPES[dtype], kind, heads, dim, vdim)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("m", [1, 7, 130, 1500])
def test_products(dtype, m):
    cases.check_products("cuda", DTYPES[dtype], m, 72, 200)
    cases.check_products("cuda", DTYPES[dtype], m, 1024, 512)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("t", [1, 33, 300])
@pytest.mark.parametrize("mlp", [cases.moe(8, 3, 24, 4, 2, shared=16), cases.moe(6, 1, 16), cases.moe(6, 2, 8, 6, 3),
                                 cases.moe(64, 6, 128, 8, 4, shared=256)])
def test_experts(dtype, t, mlp):
    cases.check_moe("cuda", DTYPES[dtype], t, mlp, 96)


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
        cases.Driver.close(got.view(rows.shape), rows, "float32")
