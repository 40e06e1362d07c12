"""Dalavik's kernels and steps on the GPU, in bf16 and entirely in fp32, against the plain implementation."""
import json
import os
import subprocess
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import dalavik_cases as cases                                           # noqa: E402
import dalavik_oracle as oracle                                         # noqa: E402

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
def test_mixed_batches_reuse_pages(setup, dtype, block_size):
    cases.check_mixed(driver(setup, dtype, max_tokens=320, block_size=block_size), rounds=2)


def test_mixed_batches_without_graphs(setup):
    cases.check_mixed(driver(setup, "bfloat16", max_tokens=256, enforce_eager=True), rounds=1)


@pytest.mark.parametrize("mixed,prefix", [(False, False), (True, False), (False, True)])
def test_generation(setup, mixed, prefix):
    path, cfg, w = setup
    cases.check_generate(path, cfg, w, "cuda", num_gpu_blocks=9, enable_mixed_batches=mixed, enable_prefix_caching=prefix)


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
@pytest.mark.parametrize("temp,rot", [({"coef": 0.4, "every": 8}, 0), ({"coef": -0.1, "every": 1}, 8), (None, 0)])
@pytest.mark.parametrize("shape", [(4, 2, 24, 16), (3, 1, 18, 22), (32, 8, 128, 128), (5, 5, 272, 40)])
def test_norm_and_query_temperature(dtype, shape, temp, rot):
    cases.check_prep("cuda", DTYPES[dtype], *shape, temp, rot)


# one head; odd heads over one; groups beyond eight heads; pages of 8; many heads; sizes at the edges of the kernels
SHAPES = [(1, 1, 16, 16), (4, 2, 24, 20), (7, 1, 18, 22), (8, 2, 128, 128), (12, 4, 96, 64), (24, 2, 80, 112),
          (32, 8, 128, 128), (64, 8, 64, 64), (16, 4, 256, 256), (3, 1, 272, 40), (2, 2, 40, 200)]


@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("planted", [0, 31, 32, 127, 144, 199])
def test_mixed_scores(shape, planted):
    cases.check_mixed_scores("cuda", torch.bfloat16, *shape, 201, 8 if planted % 2 else 64, 170, planted, splits=5,
                             exact=planted in (0, 127, 199))


@pytest.mark.parametrize("shape", SHAPES[1:6])
@pytest.mark.parametrize("variant", [1, 2])
def test_mixed_scores_by_kernel(shape, variant):
    for planted in (16, 130):
        cases.check_mixed_scores("cuda", torch.bfloat16, *shape, 150, 16, 75, planted, variant=variant, splits=3)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("kw", [dict(softcap=0.0), dict(bias=False), dict(sink=False), dict(ranks=2)])
def test_mixed_scores_without_a_part(dtype, kw):
    for planted in (0, 64, 90):
        cases.check_mixed_scores("cuda", DTYPES[dtype], 6, 2, 48, 32, 100, 16, 60, planted, splits=2, **kw)


@pytest.mark.parametrize("shape", SHAPES[:6])
def test_mixed_scores_in_32_bit(shape):
    for planted in (0, 63, 98):
        cases.check_mixed_scores("cuda", torch.float32, *shape, 100, 16, 60, planted)


def test_mixed_scores_of_long_sequences():
    """Far keys over many key ranges and shares."""
    for planted in (3, 1030, 2040):
        cases.check_mixed_scores("cuda", torch.bfloat16, 6, 3, 64, 32, 2050, 16, 40, planted, splits=61)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("shape", [(5, 1, 12, 20), (8, 4, 64, 128), (40, 8, 32, 32)])
def test_mixed_scores_of_a_batch(dtype, shape):
    cases.check_mixed_batch("cuda", DTYPES[dtype], *shape, [140, 7, 325, 64, 33], [100, 7, 2, 17, 1])


def test_mixed_scores_of_many_portions():
    """More sequences than a warp has lanes."""
    lens = [1 + (37 * i) % 50 for i in range(45)]
    cases.check_mixed_batch("cuda", torch.bfloat16, 4, 2, 32, 32, lens, [1 + n // 2 for n in lens])


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("shape", [(3, 20, 8, 12, 28, 18), (4, 128, 64, 128, 512, 384), (18, 16, 6, 24, 136, 72)])
@pytest.mark.parametrize("planted", [0, 15, 49, 51])
def test_layers_on_shared_rows(dtype, shape, planted):
    cases.check_shared_rows("cuda", DTYPES[dtype], *shape, planted, bs=16 if planted % 2 else 64)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("width,groups,out_groups", [(96, 3, 1), (100, 4, 10), (100, 1, 4), (48, 48, 6), (2880, 8, 2),
                                                     (16384, 1, 16), (12000, 30, 1000)])
def test_norm_of_a_result(dtype, width, groups, out_groups):
    cases.check_post_norm("cuda", DTYPES[dtype], 33, width, groups, out_groups)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("dim,layer", [(16, 0), (10, 3), (256, 2)])
def test_token_rows(dtype, dim, layer):
    cases.check_token_rows("cuda", DTYPES[dtype], 77, dim, 4, layer)


@pytest.mark.parametrize("dtype", sorted(DTYPES))
@pytest.mark.parametrize("m", [1, 7, 130, 1500])
def test_relu_gate(dtype, m):
    cases.check_relu_gate("cuda", DTYPES[dtype], m, 72, 200)
    cases.check_relu_gate("cuda", DTYPES[dtype], m, 1024, 512)


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
