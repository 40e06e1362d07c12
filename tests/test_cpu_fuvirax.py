"""Fuvirax on the CPU references: configuration, weight loading, cache and state slots, scheduler, batching and
generation against the plain implementation (fuvirax_oracle.py)."""
import copy
import json
import os
import sys

import pytest
import torch
from safetensors.torch import save_file

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import fuvirax_cases as cases                                           # noqa: E402
import fuvirax_oracle as oracle                                         # noqa: E402

MODELS = {"varied": cases.VARIED, "ragged": cases.RAGGED}


@pytest.fixture(params=sorted(MODELS))
def setup(request, tmp_path):
    cfg = MODELS[request.param]
    return tmp_path, cfg, cases.write_model(tmp_path, cfg, seed=5)


def driver(setup, **kw):
    path, cfg, w = setup
    return cases.Driver(path, cfg, w, "cpu", "float32", **kw)


def test_prompts(setup):
    cases.check_prompts(driver(setup), (1, 2, 5, 40, 90))


def test_long_decoding(setup):
    cases.check_decode(driver(setup), 3, 90)


@pytest.mark.parametrize("sizes", [(2,), (16,), (1, 7, 2, 30)])
def test_portions(setup, sizes):
    cases.check_portions(driver(setup), sizes, 75)


@pytest.mark.parametrize("block_size", [8, 16])
def test_mixed_batches_reuse_pages_and_slots(setup, block_size):
    cases.check_mixed(driver(setup, max_tokens=192, block_size=block_size), rounds=2)


@pytest.mark.parametrize("mixed", [False, True])
def test_generation(setup, mixed):
    path, cfg, w = setup
    # a cache of nine blocks: requests wait for each other and are preempted
    cases.check_generate(path, cfg, w, "cpu", num_gpu_blocks=9, enable_mixed_batches=mixed)


def test_streams_after_every_layer_run(setup):
    d = driver(setup)
    _, cfg, w = setup
    toks, want = cases.tokens(30, cfg["vocab"], 4), []
    oracle.forward(toks, w, cfg, layers_out=want)
    d.replay.runner.model.layer_outputs = got = []
    d.replay.step([{"id": "a", "tokens": toks, "want": []}])
    assert len(got) == len(want) == len(oracle.layer_order(cfg))
    for x, y in zip(got, want):
        assert float((x.double() - y).abs().max()) < 2e-5 * float(y.abs().max())


@pytest.mark.parametrize("streams,width,true", [(1, 24, 24), (3, 48, 43)])
def test_hyper_connections_and_token_shift(streams, width, true):
    cases.check_hyper("cpu", torch.float32, streams, width, true)


@pytest.mark.parametrize("heads,dim,vdim", [(2, 8, 12), (3, 10, 7)])
def test_gated_linear_attention(heads, dim, vdim):
    cases.check_gated_linear("cpu", torch.float32, heads, dim, vdim)


@pytest.mark.parametrize("heads,kv,dim,vdim,taps", [(2, 2, 8, 12, 4), (6, 2, 10, 7, 2), (3, 1, 5, 9, 1), (2, 1, 12, 8, 7)])
def test_delta_rule(heads, kv, dim, vdim, taps):
    cases.check_delta("cpu", torch.float32, heads, kv, dim, vdim, taps)


@pytest.mark.parametrize("planted", [0, 15, 16, 119, 120, 150])
def test_latent_attention(planted):
    cases.check_latent("cpu", torch.float32, 3, 12, 8, 20, 28, planted, t=170)


def test_xielu():
    cases.check_xielu("cpu", torch.float32, 9, 24, 40, 0.7, -1.3)


def test_config_reader_and_registry(tmp_path):
    from omni_npu_b200.config import DeltaRuleSpec, GatedLinearSpec, LatentAttentionSpec, ModelConfig
    from omni_npu_b200.models.registry import resolve_model_cls, runs_on_core_library
    cases.write_model(tmp_path, cases.VARIED)
    mc = ModelConfig.from_pretrained(str(tmp_path), dtype="float32")
    assert resolve_model_cls(mc.architecture).__name__ == "FuviraxForCausalLM" and runs_on_core_library("Fuvirax")
    specs = mc.layer_specs
    assert specs[0].attention == GatedLinearSpec(3, 20, 24) and specs[0].mlp is None
    assert specs[1].attention == DeltaRuleSpec(4, 2, 24, 40, 3, *cases.ranks(1)) and specs[1].mlp.intermediate_size == 56
    assert specs[2].attention == LatentAttentionSpec(4, 24, 16, 40, 56, 3000.0, 40 ** -0.5)
    assert mc.layer_order() == [0, 1, 2, 1, 2, 3] and (mc.residual_streams, mc.logit_scale) == (3, 0.8)
    assert mc.kv_bytes_per_token() == 4 * 2 * (56 + 16)              # two runs of the one cached layer
    for key, value, text in (("type", "mamba", "mamba"), ("mlp", {"kind": "moe"}, "moe")):
        bad = copy.deepcopy(cases.VARIED)
        bad["layers"][1][key] = value
        with pytest.raises(ValueError, match=text):
            ModelConfig.from_hf_dict(bad)


@pytest.mark.parametrize("loop", [None, (0, 3, 1), (2, 3, 4), (0, 1, 0)])
def test_layer_order(loop):
    from omni_npu_b200.config import ModelConfig
    cfg = cases.model(8, 8, cases.RAGGED["layers"], loop=loop)
    assert ModelConfig.from_hf_dict(cfg).layer_order() == oracle.layer_order(cfg)


def test_wrong_checkpoints_are_refused(tmp_path):
    from omni_npu_b200.engine.trace_replay import TraceReplay
    good = cases.write_model(tmp_path, cases.VARIED)
    file = str(tmp_path / "model.safetensors")
    # (l0 has no feed-forward: tensors in its place are idle)
    save_file({**good, "l0.norm2": torch.ones(96), "l0.hc2.in": torch.ones(3)}, file)
    TraceReplay(str(tmp_path), "float32", 64, device="cpu")
    for change, text in ((lambda w: w.pop("l1.mix.g2"), "missing"),
                         (lambda w: w.__setitem__("l2.mix.dt_bias", torch.zeros(2)), "unknown"),
                         (lambda w: w.__setitem__("l3.mlp.down", torch.zeros(96, 71)), "expected")):
        w = dict(good)
        change(w)
        save_file(w, file)
        with pytest.raises(ValueError, match=text):
            TraceReplay(str(tmp_path), "float32", 64, device="cpu")


def test_state_slots():
    from omni_npu_b200.engine.block_manager import StateSlotPool
    pool = StateSlotPool(3)
    a = [pool.allocate() for _ in range(3)]
    assert sorted(a) == [0, 1, 2] and pool.num_free == 0
    with pytest.raises(RuntimeError, match="out of state"):
        pool.allocate()
    pool.free(a[1])
    with pytest.raises(RuntimeError, match="twice"):
        pool.free(a[1])
    assert pool.allocate() == a[1]


def test_what_a_recurrent_state_rules_out(setup):
    from omni_npu_b200 import LLM
    for kw in ({"enable_prefix_caching": True},
               {"speculative_config": {"method": "ngram", "num_speculative_tokens": 2}}):
        with pytest.raises(ValueError, match="recurrent state"):
            LLM(model=str(setup[0]), dtype="float32", device="cpu", max_num_seqs=2, max_model_len=64, **kw)


def test_replay_refuses_what_does_not_fit(setup):
    d = driver(setup, max_tokens=64)
    for i in range(4):
        d.replay.step([{"id": f"x{i}", "tokens": [1, 2], "want": []}])
    with pytest.raises(RuntimeError, match="live"):
        d.replay.step([{"id": "y", "tokens": [1], "want": []}])


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
    assert type(llm.engine.worker.get_model()).__name__ == "FuviraxForCausalLM"


def test_random_weights(setup):
    """A model without a checkpoint (load_format dummy) runs, its padding at zero."""
    from omni_npu_b200 import LLM, SamplingParams
    from omni_npu_b200.config import ModelConfig
    llm = LLM(model=ModelConfig.from_hf_dict(setup[1], dtype="float32"), device="cpu", max_num_seqs=2, max_model_len=64,
              load_format="dummy")
    assert len(llm.generate([[1, 2, 3]], SamplingParams(max_tokens=4, ignore_eos=True))[0].output_token_ids) == 4


def test_two_ranks(tmp_path):
    """Tensor parallel: heads of every mixer and feed-forward columns split over two ranks."""
    from dist_utils import run_ranks
    cfg = cases.model(96, 203, [
        cases.delta(4, 2, 24, 40, 3, mlp=cases.dense(56)),
        cases.latent(4, 24, 16, 40, 56, mlp=cases.dense(36)),
        cases.hgrn2(2, 36, 64)], streams=2, loop=(0, 2, 2))
    (tmp_path / "model").mkdir()
    w = cases.write_model(tmp_path / "model", cfg, seed=9)
    prompts = [cases.tokens(n, cfg["vocab"], n) for n in (20, 33, 70)]
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
