"""Dalavik on the CPU references: configuration, weight loading, cache, scheduler, batching and generation against the
plain implementation (dalavik_oracle.py)."""
import copy
import json
import os
import sys

import pytest
import torch
from safetensors.torch import save_file

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import dalavik_cases as cases                                           # noqa: E402
import dalavik_oracle as oracle                                         # noqa: E402

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
def test_mixed_batches_reuse_pages(setup, block_size):
    cases.check_mixed(driver(setup, max_tokens=192, block_size=block_size), rounds=2)


@pytest.mark.parametrize("mixed,prefix", [(False, False), (True, False), (False, True)])
def test_generation(setup, mixed, prefix):
    path, cfg, w = setup
    # a cache of nine blocks: requests wait for each other and are preempted
    cases.check_generate(path, cfg, w, "cpu", num_gpu_blocks=9, enable_mixed_batches=mixed, enable_prefix_caching=prefix)


def test_generation_with_drafts(setup):
    """Prompt look-up drafts are verified as short portions: the tokens stay the greedy ones."""
    path, cfg, w = setup
    cases.check_generate(path, cfg, w, "cpu", num_gpu_blocks=24,
                         speculative_config={"method": "ngram", "num_speculative_tokens": 3})


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


@pytest.mark.parametrize("temp,rot", [({"coef": 0.4, "every": 8}, 0), ({"coef": -0.1, "every": 1}, 8), (None, 0)])
@pytest.mark.parametrize("shape", [(4, 2, 24, 16), (3, 1, 18, 22)])
def test_norm_and_query_temperature(shape, temp, rot):
    cases.check_prep("cpu", torch.float32, *shape, temp, rot)


@pytest.mark.parametrize("planted", [0, 15, 16, 40, 59])
@pytest.mark.parametrize("kw", [{}, dict(softcap=0.0), dict(bias=False), dict(sink=False), dict(ranks=2)])
def test_mixed_scores(planted, kw):
    cases.check_mixed_scores("cpu", torch.float32, 4, 2, 24, 20, 60, 16, 48, planted, **kw)


def test_mixed_scores_of_a_batch():
    cases.check_mixed_batch("cpu", torch.float32, 5, 1, 12, 20, [40, 7, 25], [20, 7, 2])


@pytest.mark.parametrize("planted", [0, 15, 49, 51])
def test_layers_on_shared_rows(planted):
    cases.check_shared_rows("cpu", torch.float32, 3, 20, 8, 12, 28, 18, planted)


@pytest.mark.parametrize("width,groups,out_groups", [(96, 3, 1), (100, 4, 10), (100, 1, 4), (48, 48, 6)])
def test_norm_of_a_result(width, groups, out_groups):
    cases.check_post_norm("cpu", torch.float32, 9, width, groups, out_groups)


@pytest.mark.parametrize("dim,layer", [(16, 0), (10, 3)])
def test_token_rows(dim, layer):
    cases.check_token_rows("cpu", torch.float32, 9, dim, 4, layer)


def test_relu_gate():
    cases.check_relu_gate("cpu", torch.float32, 9, 24, 40)


def test_config_reader_and_registry(tmp_path):
    from omni_npu_b200.config import AttentionSpec, DenseSpec, LatentAttentionSpec, ModelConfig
    from omni_npu_b200.models.registry import resolve_model_cls, runs_on_core_library
    cases.write_model(tmp_path, cases.VARIED)
    mc = ModelConfig.from_pretrained(str(tmp_path), dtype="float32")
    assert resolve_model_cls(mc.architecture).__name__ == "DalavikForCausalLM" and runs_on_core_library("Dalavik")
    s = mc.layer_specs
    assert s[0].attention == AttentionSpec(4, 2, 24, 40, 0, 0.0, 0.7 * 24 ** -0.5, qk_norm="head_weight", bias=True,
                                           query_temperature=(0.4, 16), softcap=20.0, distance_bias=True, score_mix=True,
                                           head_sink=True)
    assert s[0].mlp == DenseSpec(56, "relu") and s[3].mlp is None and s[3].attention.query_temperature == (-0.2, 7)
    assert s[1].attention == LatentAttentionSpec(4, 24, 16, 40, 56, 3000.0, 40 ** -0.5, False, 48)
    assert s[2].attention.kv_from == 1 and s[5].attention.scale == 0.6
    assert (mc.norm_groups, mc.token_side_dim) == (3, 16)
    assert mc.kv_bytes_per_token() == 4 * (2 * 64 + 72 + 3 * 32 + 32)          # layers 2 and 5 cache nothing
    for layer, key, value, text in ((0, "type", "mamba", "mamba"), (1, "mlp", {"kind": "sparse"}, "sparse"),
                                    (2, "kv_from", 0, "caches none"), (2, "kv_from", 2, "caches none"),
                                    (5, "kv_from", 4, "different shapes"), (5, "kv_from", 2, "caches none"),
                                    (0, "kv_heads", 3, "inconsistent"), (1, "rot_dim", 8, "inconsistent")):
        bad = copy.deepcopy(cases.VARIED)
        where = bad["layers"][layer]
        (where if key in where else where["mixer"])[key] = value
        with pytest.raises(ValueError, match=text):
            ModelConfig.from_hf_dict(bad)
    with pytest.raises(ValueError, match="groups"):
        ModelConfig.from_hf_dict({**cases.VARIED, "norm": {"eps": 1e-5, "groups": 5}})


def test_wrong_checkpoints_are_refused(tmp_path):
    from omni_npu_b200.engine.trace_replay import TraceReplay
    good = cases.write_model(tmp_path, cases.VARIED)
    file = str(tmp_path / "model.safetensors")
    # (l2 has no feed-forward: a norm for one is idle)
    save_file({**good, "l2.norm2": torch.ones(96)}, file)
    TraceReplay(str(tmp_path), "float32", 64, device="cpu")
    for change, text in ((lambda w: w.pop("l0.mix.talk"), "missing"),
                         (lambda w: w.__setitem__("l2.mix.dkv", torch.zeros(72, 96)), "unknown"),
                         (lambda w: w.__setitem__("l1.side.proj", torch.zeros(96, 15)), "expected")):
        w = dict(good)
        change(w)
        save_file(w, file)
        with pytest.raises(ValueError, match=text):
            TraceReplay(str(tmp_path), "float32", 64, device="cpu")


def test_layers_that_share_rows_have_one_cache(setup):
    d = driver(setup)
    runner, (_, cfg, _) = d.replay.runner, setup
    own = [i for i, x in enumerate(cfg["layers"]) if "kv_from" not in x["mixer"]]
    assert len(runner.kv_caches) == runner.model.num_kv_layers == len(own)
    assert runner.get_kv_cache_spec().bytes_per_block == sum(
        t[0].numel() * t.element_size() for c in runner.kv_caches for t in (c if isinstance(c, tuple) else (c,)))
    for x, layer in zip(cfg["layers"], runner.model.layers):
        if "kv_from" in x["mixer"]:
            assert layer.mix.cache_idx == runner.model.layers[x["mixer"]["kv_from"]].mix.cache_idx


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
    assert type(llm.engine.worker.get_model()).__name__ == "DalavikForCausalLM"


def test_random_weights(setup):
    """A model without a checkpoint (load_format dummy) runs, its padding at zero."""
    from omni_npu_b200 import LLM, SamplingParams
    from omni_npu_b200.config import ModelConfig
    llm = LLM(model=ModelConfig.from_hf_dict(setup[1], dtype="float32"), device="cpu", max_num_seqs=2, max_model_len=64,
              load_format="dummy")
    model = llm.engine.worker.get_model()
    for layer in model.layers:
        for p in (layer.side.gate, layer.mix.in_proj.weight):
            assert float(p[:, model.width:].abs().sum()) == 0.0
    assert len(llm.generate([[1, 2, 3]], SamplingParams(max_tokens=4, ignore_eos=True))[0].output_token_ids) == 4


def test_two_ranks(tmp_path):
    """Tensor parallel: heads and feed-forward columns split over two ranks; every rank mixes all heads' scores."""
    from dist_utils import run_ranks
    cfg = cases.model(96, 203, [
        cases.attention(4, 2, 24, 40, mlp=cases.dense(36)), cases.latent(4, 24, 16, 40, 56, 48, mlp=cases.dense(40)),
        cases.latent(2, 8, 16, 24, 56, 20, kv_from=1), cases.attention(6, 2, 16, 16, mlp=cases.dense(24))], groups=2)
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


@pytest.mark.parametrize("layer", [cases.attention(2, 1, 16, 8), cases.latent(2, 8, 8, 16, 24, 12, mlp=cases.dense(16))])
def test_models_of_one_mixer(tmp_path, layer):
    cfg = cases.model(32, 40, [layer] * 2, side=8)
    w = cases.write_model(tmp_path, cfg, seed=3)
    cases.check_mixed(cases.Driver(tmp_path, cfg, w, "cpu", "float32", max_tokens=192), rounds=1)
    cases.check_generate(tmp_path, cfg, w, "cpu", num_gpu_blocks=24)


def test_first_tokens_and_equal_weights(tmp_path):
    """A sequence of one token, whose only key competes with the sink; a mixture that is the identity."""
    cfg = cases.model(32, 40, [cases.attention(2, 2, 16, 8), cases.latent(2, 8, 8, 16, 24, 12)], side=8)
    w = cases.write_model(tmp_path, cfg, seed=4)
    w["l0.mix.talk"] = torch.eye(2, dtype=torch.bfloat16)
    w["l0.mix.sink"] = torch.tensor([-30.0, 30.0], dtype=torch.bfloat16)
    save_file(w, str(tmp_path / "model.safetensors"))
    cases.check_decode(cases.Driver(tmp_path, cfg, w, "cpu", "float32"), 1, 20)
