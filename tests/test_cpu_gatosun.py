"""Gatosun on the CPU references: configuration, weight loading, cache and state slots, scheduler, batching and
generation against the plain implementation (gatosun_oracle.py)."""
import copy
import json
import os
import sys

import pytest
import torch
from safetensors.torch import save_file

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import gatosun_cases as cases                                           # noqa: E402
import gatosun_oracle as oracle                                         # noqa: E402

MODELS = {"varied": cases.VARIED, "ragged": cases.RAGGED}


@pytest.fixture(params=sorted(MODELS))
def setup(request, tmp_path):
    cfg = MODELS[request.param]
    return tmp_path, cfg, cases.write_model(tmp_path, cfg, seed=5)


def driver(setup, **kw):
    path, cfg, w = setup
    return cases.Driver(path, cfg, w, "cpu", "float32", **kw)


def test_prompts(setup):
    cases.check_prompts(driver(setup), (1, 2, 5, 40, 70))


def test_long_decoding(setup):
    cases.check_decode(driver(setup), 3, 70)


@pytest.mark.parametrize("sizes", [(2,), (1, 7, 2, 30)])
def test_portions(setup, sizes):
    cases.check_portions(driver(setup), sizes, 60)


@pytest.mark.parametrize("block_size", [8, 16])
def test_mixed_batches_reuse_pages_and_slots(setup, block_size):
    cases.check_mixed(driver(setup, max_tokens=192, block_size=block_size), rounds=2)


@pytest.mark.parametrize("mixed", [False, True])
def test_generation(setup, mixed):
    path, cfg, w = setup
    # a cache of nine blocks: requests wait for each other and are preempted
    cases.check_generate(path, cfg, w, "cpu", num_gpu_blocks=9, enable_mixed_batches=mixed)


def test_residual_after_every_layer(setup):
    d = driver(setup)
    _, cfg, w = setup
    toks, want = cases.tokens(30, cfg["vocab"], 4), []
    oracle.forward(toks, w, cfg, layers_out=want)
    d.replay.runner.model.layer_outputs = got = []
    d.replay.step([{"id": "a", "tokens": toks, "want": []}])
    assert len(got) == len(want) == len(cfg["layers"])
    for x, y in zip(got, want):
        assert float((x.double() - y).abs().max()) < 2e-5 * float(y.abs().max())


@pytest.mark.parametrize("norm,mixed", [("projection", True), ("projection", False), ("head", False), (None, True)])
@pytest.mark.parametrize("shape", [(4, 2, 24, 16, 16), (3, 1, 18, 22, 6)])
def test_norm_rotation_and_values(shape, norm, mixed):
    cases.check_prep("cpu", torch.float32, *shape, norm, mixed)


@pytest.mark.parametrize("window,planted", [(0, 0), (0, 15), (0, 40), (1, 30), (17, 20), (17, 31), (17, 32)])
def test_visible_keys(window, planted):
    cases.check_visible("cpu", torch.float32, 4, 2, 24, 20, window, 60, 16, 48, planted)


@pytest.mark.parametrize("width", [24, 104])
def test_blends_with_the_previous_token(width):
    cases.check_token_mix("cpu", torch.float32, width)


@pytest.mark.parametrize("kind", ["decay", "bonus"])
@pytest.mark.parametrize("heads,dim,vdim", [(2, 8, 12), (3, 10, 7)])
def test_recurrent_layers(kind, heads, dim, vdim):
    cases.check_scan("cpu", torch.float32, kind, heads, dim, vdim)


def test_products():
    cases.check_products("cpu", torch.float32, 9, 24, 40)


@pytest.mark.parametrize("mlp", [cases.moe(8, 3, 24, 4, 2, shared=16), cases.moe(6, 1, 16), cases.moe(6, 2, 8, 6, 3)])
def test_experts(mlp):
    cases.check_moe("cpu", torch.float32, 40, mlp, 48)


def test_config_reader_and_registry(tmp_path):
    from omni_npu_b200.config import AttentionSpec, DecayLinearSpec, DenseSpec, ModelConfig, ParallelSpec, TimeMixSpec
    from omni_npu_b200.models.registry import resolve_model_cls, runs_on_core_library
    cases.write_model(tmp_path, cases.VARIED)
    mc = ModelConfig.from_pretrained(str(tmp_path), dtype="float32")
    assert resolve_model_cls(mc.architecture).__name__ == "GatosunForCausalLM" and runs_on_core_library("Gatosun")
    s = mc.layer_specs
    assert s[0].attention == ParallelSpec(AttentionSpec(4, 2, 24, 40, 16, 3000.0, 24 ** -0.5, True, 10, qk_norm="head"),
                                          TimeMixSpec(3, 20, cases.rank(0)), 0.7, 0.4)
    assert s[0].mlp == DenseSpec(56, "gelu_tanh", True) and s[2].mlp is None
    assert s[1].attention == AttentionSpec(6, 2, 24, 16, 8, 3000.0, 24 ** -0.5, True, qk_norm="projection", bias=True,
                                           value_mix=True)
    assert s[3].attention == DecayLinearSpec(3, 20, 28, 5.0, cases.rank(3)) and not s[2].attention.value_mix
    m = s[1].mlp
    assert (m.num_experts, m.top_k, m.n_group, m.topk_group, m.renormalize, m.correction) == (8, 3, 4, 2, False, True)
    assert (m.expert.intermediate_size, m.expert.act, m.shared.intermediate_size) == (40, "relu2", 24)
    assert mc.residual_mult == 0.5
    assert mc.kv_bytes_per_token() == 4 * (2 * 64 + 2 * 40 + 4 * 40 + 80 + 3 * 32 + 40)
    for key, value, text in (("type", "mamba", "mamba"), ("mlp", {"kind": "sparse"}, "sparse")):
        bad = copy.deepcopy(cases.VARIED)
        bad["layers"][1][key] = value
        with pytest.raises(ValueError, match=text):
            ModelConfig.from_hf_dict(bad)
    bad = copy.deepcopy(cases.VARIED)
    bad["layers"][4]["mixer"]["vdim"] = 24
    with pytest.raises(ValueError, match="blend their values"):
        ModelConfig.from_hf_dict(bad)


def test_wrong_checkpoints_are_refused(tmp_path):
    from omni_npu_b200.engine.trace_replay import TraceReplay
    good = cases.write_model(tmp_path, cases.VARIED)
    file = str(tmp_path / "model.safetensors")
    # (l2 neither blends its values nor has a feed-forward: tensors in those places are idle)
    save_file({**good, "l2.norm2": torch.ones(96), "l2.mix.vmix": torch.ones(())}, file)
    TraceReplay(str(tmp_path), "float32", 64, device="cpu")
    for change, text in ((lambda w: w.pop("l0.mix.right.u"), "missing"),
                         (lambda w: w.__setitem__("l3.mix.dt_bias", torch.zeros(2)), "unknown"),
                         (lambda w: w.__setitem__("l1.mlp.e7.down", torch.zeros(96, 39)), "expected")):
        w = dict(good)
        change(w)
        save_file(w, file)
        with pytest.raises(ValueError, match=text):
            TraceReplay(str(tmp_path), "float32", 64, device="cpu")


def test_first_values_come_from_the_first_layer_that_blends(tmp_path):
    """That layer's own factor is not used; a layer that does not blend leaves the values alone."""
    cfg = cases.model(48, 40, [cases.attention(2, 1, 16, 8, 8, v_mix=False), cases.attention(2, 2, 16, 8, 8),
                               cases.attention(4, 1, 16, 16, 8), cases.gla(2, 8, 8), cases.attention(2, 1, 8, 16, 4)])
    w = cases.write_model(tmp_path, cfg, seed=1)
    toks = cases.tokens(12, 40, 1)
    a = oracle.forward(toks, w, cfg)
    w["l1.mix.vmix"] = w["l1.mix.vmix"] * 0
    assert torch.equal(a, oracle.forward(toks, w, cfg))
    w["l4.mix.vmix"] = w["l4.mix.vmix"] * 0
    assert not torch.allclose(a, oracle.forward(toks, w, cfg), rtol=1e-3)
    for seed in (1, 2):
        w = cases.write_model(tmp_path, cfg, seed=seed)
        cases.check_portions(cases.Driver(tmp_path, cfg, w, "cpu", "float32"), (5, 1, 2), 40)


def test_what_a_recurrent_state_rules_out(setup):
    from omni_npu_b200 import LLM
    with pytest.raises(ValueError, match="recurrent state"):
        LLM(model=str(setup[0]), dtype="float32", device="cpu", max_num_seqs=2, max_model_len=64, enable_prefix_caching=True)


def test_sampling_and_logprobs(setup):
    """A seeded request draws the same tokens in any company; log-probabilities are those of the oracle."""
    from omni_npu_b200 import LLM, SamplingParams
    path, cfg, w = setup
    llm = LLM(model=str(path), dtype="float32", device="cpu", max_num_seqs=3, max_model_len=96)
    prompt = cases.tokens(12, cfg["vocab"], 3)
    sp = SamplingParams(max_tokens=6, temperature=0.8, seed=7, ignore_eos=True)
    alone = llm.generate([prompt], sp)[0].output_token_ids
    others = [cases.tokens(20, cfg["vocab"], 8), prompt, cases.tokens(3, cfg["vocab"], 9)]
    assert llm.generate(others, sp)[1].output_token_ids == alone
    out = llm.generate([prompt], SamplingParams(max_tokens=1, logprobs=3, ignore_eos=True))[0]
    want = torch.log_softmax(oracle.forward(prompt, w, cfg)[-1], -1)
    assert abs(out.logprobs[0][0] - float(want[out.output_token_ids[0]])) < 1e-3


def test_server_command_line_takes_the_model(setup):
    from omni_npu_b200 import LLM
    from omni_npu_b200.serving.api_server import make_parser
    args = make_parser().parse_args(["--model", str(setup[0]), "--max-num-seqs", "2"])
    llm = LLM(model=args.model, dtype="float32", device="cpu", max_num_seqs=args.max_num_seqs, max_model_len=128)
    assert type(llm.engine.worker.get_model()).__name__ == "GatosunForCausalLM"


def test_random_weights(setup):
    """A model without a checkpoint (load_format dummy) runs, its padding at zero."""
    from omni_npu_b200 import LLM, SamplingParams
    from omni_npu_b200.config import ModelConfig
    llm = LLM(model=ModelConfig.from_hf_dict(setup[1], dtype="float32"), device="cpu", max_num_seqs=2, max_model_len=64,
              load_format="dummy")
    assert len(llm.generate([[1, 2, 3]], SamplingParams(max_tokens=4, ignore_eos=True))[0].output_token_ids) == 4


def test_two_ranks(tmp_path):
    """Tensor parallel: heads of every mixer and feed-forward columns split over two ranks, experts dealt out; the
    norm over a whole projection counts both ranks' rows."""
    from dist_utils import run_ranks
    cfg = cases.model(96, 203, [
        cases.attention(4, 2, 24, 16, 8, mlp=cases.dense(36)),
        cases.parallel(cases.heads(4, 2, 24, 40, 16, window=10), (2, 20), mlp=cases.moe(8, 3, 40, 4, 2, shared=24)),
        cases.gla(2, 20, 28, mlp=cases.dense(40)),
        cases.attention(2, 2, 32, 16, 32)])
    (tmp_path / "model").mkdir()
    w = cases.write_model(tmp_path / "model", cfg, seed=9)
    prompts = [cases.tokens(n, cfg["vocab"], n) for n in (20, 33, 50)]
    (tmp_path / "prompts.json").write_text(json.dumps(prompts))
    (tmp_path / "pipeline_parallel").write_text("1")
    res = run_ranks("tp_engine", 2, str(tmp_path))
    assert res[0]["tokens"] == res[1]["tokens"]
    for p, out in zip(prompts, res[0]["tokens"]):
        seq = list(p)
        for t in out:
            logits = oracle.forward(seq, w, cfg)[-1]
            assert float(logits.max() - logits[t]) < 1e-3 * float(logits.std())
            seq.append(t)


@pytest.mark.parametrize("layer", [cases.attention(2, 1, 16, 8, 8), cases.gla(2, 8, 12, mlp=cases.dense(16)),
                                   cases.parallel(cases.heads(2, 2, 16, 8, 8, window=5), (2, 8), 0.3, 0.0)])
def test_models_of_one_mixer(tmp_path, layer):
    """A model without a cache, one without a recurrent layer, one whose right half counts for nothing."""
    cfg = cases.model(32, 40, [layer] * 2)
    w = cases.write_model(tmp_path, cfg, seed=3)
    cases.check_mixed(cases.Driver(tmp_path, cfg, w, "cpu", "float32", max_tokens=192), rounds=1)
    cases.check_generate(tmp_path, cfg, w, "cpu", num_gpu_blocks=24)
