"""Rivudra on the CPU references: configuration, weight loading, cache, scheduler, batching and generation
against the plain implementation (rivudra_oracle.py)."""
import copy
import json
import os
import sys

import pytest
import torch
from safetensors.torch import save_file

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import rivudra_cases as cases                                           # noqa: E402
import rivudra_oracle as oracle                                         # noqa: E402

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
    cases.check_decode(driver(setup), 3, 120)


@pytest.mark.parametrize("sizes", [(2,), (16,), (1, 7, 2, 30)])
def test_portions(setup, sizes):
    cases.check_portions(driver(setup), sizes, 75)


@pytest.mark.parametrize("block_size", [8, 16])
def test_mixed_batches_reuse_pages(setup, block_size):
    cases.check_mixed(driver(setup, max_tokens=192, block_size=block_size))


@pytest.mark.parametrize("mixed", [False, True])
def test_generation(setup, mixed):
    path, cfg, w = setup
    # a cache of nine blocks: requests wait for each other and are preempted
    cases.check_generate(path, cfg, w, "cpu", num_gpu_blocks=9, enable_mixed_batches=mixed)


def test_generation_with_prefix_cache(setup):
    path, cfg, w = setup
    cases.check_generate(path, cfg, w, "cpu", enable_prefix_caching=True)


def test_residual_after_every_layer(setup):
    d = driver(setup)
    _, cfg, w = setup
    toks, want = cases.tokens(30, cfg["vocab"], 4), []
    oracle.forward(toks, w, cfg, layers_out=want)
    d.replay.runner.model.layer_outputs = got = []
    d.replay.step([{"id": "a", "tokens": toks, "want": []}])
    assert len(got) == len(want)
    for x, y in zip(got, want):
        assert float((x.double() - y).abs().max()) < 2e-5 * float(y.abs().max())


@pytest.mark.parametrize("window,t,planted", [(1, 20, 10), (2, 40, 31), (16, 60, 15), (17, 60, 16), (40, 60, 0)])
def test_window_edges(window, t, planted):
    for p in (planted, min(t - 1, planted + 1)):
        cases.check_window("cpu", torch.float32, 6, 2, 24, 40, window, t, 8, t, p)


@pytest.mark.parametrize("rot", [2, 10, 24])
def test_rotation(rot):
    cases.check_rope("cpu", torch.float32, 3, 1, 24, 20, rot, 700.0)


def test_clamped_experts():
    cases.check_glu("cpu", torch.float32, 9, 24, 40, 0.6)
    cases.check_moe("cpu", torch.float32, 23, cases.moe(12, 3, 24, 0.7, 4, 2, 1.4, shared=(16, 1.2)), 48)


@pytest.mark.parametrize("groups,keep,top", [(1, 1, 5), (4, 1, 3), (4, 3, 7), (12, 5, 5)])
def test_routing(groups, keep, top):
    from omni_npu_b200 import ops
    logits = torch.randn(40, 12, generator=torch.Generator().manual_seed(groups)) * 2
    ids, w = ops.moe_topk(logits, None, top, False, groups, keep, True, 1.3)
    got = torch.zeros(40, 12).scatter_(1, ids.long(), w)
    want = oracle.route(logits.double(), top, groups, keep, 1.3)
    assert float((got.double() - want).abs().max()) < 1e-5


def test_sink_at_the_first_token():
    """Position 0 sees itself and the sink alone: p = e^s / (1 + e^s)."""
    from omni_npu_b200 import ops
    for s in (-8.0, 0.0, 3.0):
        q, k = torch.tensor([[s, 0.0]]), torch.tensor([[[1.0, 0.0]]])
        v = torch.tensor([[[2.0, -4.0]]])
        kc, bt = cases.paged(k, 2, 4, 0)
        vc, _ = cases.paged(v, 2, 4, 0)
        out = torch.empty(1, 2)
        ops.gated_attention(q, None, kc, vc, out, bt, None, torch.tensor([1], dtype=torch.int32), 1, 1, 1, 2, 2, 1.0, 5,
                            0.0)
        assert torch.allclose(out[0], v[0, 0] * torch.sigmoid(torch.tensor(s)), atol=1e-6)


def test_config_reader_and_registry():
    from omni_npu_b200.config import ModelConfig
    from omni_npu_b200.models.registry import resolve_model_cls, runs_on_core_library
    mc = ModelConfig.from_hf_dict(cases.VARIED, dtype="float32")
    assert resolve_model_cls(mc.architecture).__name__ == "RivudraForCausalLM" and runs_on_core_library("Rivudra")
    a, m = mc.layer_specs[0].attention, mc.layer_specs[0].mlp
    assert (a.num_heads, a.num_kv_heads, a.head_dim, a.v_head_dim, a.rotary_dim, a.sliding_window) == (4, 2, 24, 40, 16, 10)
    assert (m.num_experts, m.top_k, m.n_group, m.topk_group, m.scale) == (8, 3, 4, 2, 1.7)
    assert m.expert.act == (1.702, 0.8) and m.shared.act == (1.702, 1.1) and m.shared.intermediate_size == 24
    assert mc.layer_specs[1].mlp is None and mc.layer_specs[2].mlp.shared is None
    assert mc.kv_bytes_per_token() == 4 * (2 * 64 + 32 + 3 * 72)
    bad = copy.deepcopy(cases.VARIED)
    bad["layers"][0]["type"] = "recurrent"
    with pytest.raises(ValueError, match="recurrent"):
        ModelConfig.from_hf_dict(bad)
    with pytest.raises(ValueError, match="no config reader"):
        ModelConfig.from_hf_dict({"architecture": "Nobody"})


def test_wrong_checkpoints_are_refused(tmp_path):
    from omni_npu_b200.engine.trace_replay import TraceReplay
    good = cases.write_model(tmp_path, cases.VARIED)
    file = str(tmp_path / "model.safetensors")
    for change, text in ((lambda w: w.pop("l1.mix.g"), "missing"),
                         (lambda w: w.__setitem__("l1.mlp.router", torch.zeros(2, 96)), "unknown"),
                         (lambda w: w.__setitem__("l0.mlp.e3.down", torch.zeros(96, 41)), "expected")):
        w = dict(good)
        change(w)
        save_file(w, file)
        with pytest.raises(ValueError, match=text):
            TraceReplay(str(tmp_path), "float32", 64, device="cpu")


def test_replay_refuses_what_does_not_fit(setup):
    path, cfg, _ = setup
    d = driver(setup, max_tokens=64)
    with pytest.raises(ValueError, match="vocabulary"):
        d.replay.step([{"id": "a", "tokens": [cfg["vocab"]], "want": []}])
    for i in range(4):
        d.replay.step([{"id": f"x{i}", "tokens": [1, 2], "want": []}])
    with pytest.raises(RuntimeError, match="live"):
        d.replay.step([{"id": "y", "tokens": [1], "want": []}])


def test_server_command_line_takes_the_model(setup):
    from omni_npu_b200 import LLM
    from omni_npu_b200.serving.api_server import make_parser
    args = make_parser().parse_args(["--model", str(setup[0]), "--max-num-seqs", "2"])
    llm = LLM(model=args.model, dtype="float32", device="cpu", max_num_seqs=args.max_num_seqs, max_model_len=128)
    assert type(llm.engine.worker.get_model()).__name__ == "RivudraForCausalLM"


def test_config_file_is_plain_json(setup):
    with open(setup[0] / "config.json") as f:
        assert json.load(f)["architecture"] == "Rivudra"


@pytest.mark.parametrize("pp", [1, 2])
def test_two_ranks(tmp_path, pp, monkeypatch):
    """Tensor parallel (heads and experts sharded, one key/value head replicated) and two pipeline stages
    (the fp32 residual crosses the boundary)."""
    from dist_utils import run_ranks
    monkeypatch.delenv("OMNI_B200_PP_LAYER_PARTITION", raising=False)
    cfg = cases.model(96, 203, [
        cases.attn_layer(4, 2, 24, 40, 16, 10, mlp=cases.moe(8, 3, 40, 0.8, 4, 2, 1.7, shared=(24, 1.1))),
        cases.attn_layer(6, 1, 16, 16, 8, 33),
        cases.attn_layer(2, 2, 48, 24, 48, 17, mlp=cases.moe(6, 1, 16, 2.5))])
    (tmp_path / "model").mkdir()
    w = cases.write_model(tmp_path / "model", cfg, seed=9)
    prompts = [cases.tokens(n, cfg["vocab"], n) for n in (20, 33, 70)]
    (tmp_path / "prompts.json").write_text(json.dumps(prompts))
    (tmp_path / "pipeline_parallel").write_text(str(pp))
    res = run_ranks("tp_engine", 2, str(tmp_path))
    assert res[0]["tokens"] == res[1]["tokens"]
    for p, out in zip(prompts, res[0]["tokens"]):
        seq = list(p)
        for t in out:
            logits = oracle.forward(seq, w, cfg)[-1]
            assert float(logits.max() - logits[t]) < 1e-3
            seq.append(t)
