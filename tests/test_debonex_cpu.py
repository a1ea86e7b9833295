"""Debonex family on the CPU: parsing, loading, and every schedule against the plain statement (``debonex_oracle``)."""
import json
import math
import os
import subprocess
import sys

import pytest
import torch

import debonex_cases as cases
import debonex_oracle as oracle
from tensorrt_edge_llm_b200 import ops
from tensorrt_edge_llm_b200.config import ModelConfig

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.fixture(scope="module")
def ckpt(tmp_path_factory):
    made = {}

    def get(name, sharp=1.0):
        if (name, sharp) not in made:
            made[name, sharp] = cases.save_checkpoint(tmp_path_factory.mktemp(name), *cases.weights(name, sharp))
        return made[name, sharp]
    return get


# ---- configuration -----------------------------------------------------------------------------------------


def test_config_round_trip_and_projection_ranks(ckpt):
    cfg = ModelConfig.from_pretrained(ckpt("mixed"))
    assert cfg.layer_types == ["channel_delta", "attention", "attention", "channel_delta"] and cfg.mlp_types == ["mlp", "mlp", "none", "mlp"]
    d = cfg.layer_specs[0].delta
    assert (d.decay_rank, d.gate_rank, d.k_pad, d.v_pad, d.conv_kernel) == (8, 12, 64, 32, 3)          # ranks come from the tensors
    assert cfg.kv_geometry() == [(1, 128 + 64), (2, 128)] and cfg.kv_planes() == [1, 2] and cfg.is_hybrid
    assert cfg.layer_specs[2].attention.temp_every == 30 and cfg.embedding_mult == 2.0 and cfg.logits_mult == 1.5
    again = ModelConfig.from_dict(json.loads(json.dumps(cfg.to_dict())))
    assert again.layer_specs == cfg.layer_specs
    assert not ModelConfig.from_pretrained(ckpt("latent")).is_hybrid


@pytest.mark.parametrize("name", sorted(cases.CONFIGS))
def test_native_engine_config_sizes(name, ckpt):
    """The native configuration derives the cache and state sizes that the Python managers allocate."""
    from tensorrt_edge_llm_b200.checkpoint.artifacts import runtime_config_dict
    from tensorrt_edge_llm_b200.runtime import native as rt
    from tensorrt_edge_llm_b200.runtime.kv_cache import KVCacheManager
    cfg = ModelConfig.from_pretrained(ckpt(name))
    c = rt.LLMEngineConfig.from_runtime_config(json.dumps(runtime_config_dict(cfg, 2, 64, 128, 1), default=str))
    kv = KVCacheManager(cfg, 2, 64, max_seats=1, max_pages_per_seq=2)
    state = 0 if kv.recurrent is None else kv.recurrent.bytes()
    assert c.validate() == "" and c.is_hybrid() == cfg.is_hybrid and c.num_attention_layers() == cfg.num_attn_layers
    assert c.kv_bytes_per_token() == kv.bytes_per_token
    assert c.recurrent_state_bytes_per_seat() == state


@pytest.mark.parametrize("change", ["mixer", "mlp", "rot", "heads", "temp"])
def test_config_refuses_what_it_does_not_know(change):
    hf = cases.CONFIGS["mixed"]()
    if change == "mixer":
        hf["layers"][0]["type"] = "other"
    elif change == "mlp":
        hf["layers"][0]["mlp"]["kind"] = "moe"
    elif change == "rot":
        hf["layers"][1]["mixer"]["rot"]["dims"] = 16
    elif change == "heads":
        hf["layers"][0]["mixer"]["kv_heads"] = 3
    else:
        hf["layers"][2]["mixer"]["q_temp"]["every"] = 0
    with pytest.raises(ValueError):
        ModelConfig.from_hf_dict(hf)


# ---- mechanisms alone --------------------------------------------------------------------------------------


def test_tanh_norm_and_stream():
    x, a, w, b = (torch.randn(3, 8) for _ in range(4))
    table, ids = torch.randn(5, 8), torch.tensor([4, 0, 2])
    alpha = torch.tensor(0.8)
    y, h = ops.stream_norm(x, w[0], 1e-3, delta=a, alpha=alpha, bias=b[0], dtype=torch.float32)
    want = oracle.dynamic_tanh((x + a).double(), {"n.alpha": alpha.double(), "n": w[0].double(), "n.b": b[0].double()}, "n")
    assert torch.allclose(y, x + a) and torch.allclose(h.double(), want, atol=1e-6)
    y, _ = ops.stream_norm(None, w[0], 1e-3, alpha=alpha, bias=b[0], ids=ids, table=table, table_mult=3.0, dtype=torch.float32)
    assert torch.allclose(y, table[ids] * 3.0)


def test_query_temperature_steps():
    t = ops.query_temperature(300, 0.5, 128)
    assert float(t[0]) == 1.0 and float(t[126]) == 1.0                                    # positions before the first full block
    assert abs(float(t[127]) - (1 + 0.5 * math.log(2))) < 1e-6 and abs(float(t[255]) - (1 + 0.5 * math.log(3))) < 1e-6
    assert torch.allclose(t.double(), oracle.query_temperature(300, 0.5, 128), atol=1e-6)


@pytest.mark.parametrize("shape", [(4, 2, 40, 24, 3), (1, 1, 16, 16, 1), (3, 3, 64, 130, 8)])
def test_channel_delta(shape):
    assert cases.delta_case("cpu", torch.float32, *shape, [9, 1, 4], past=[5, 1, 2]) < 1e-5
    assert cases.delta_case("cpu", torch.float32, *shape, [12, 12], keep=1) < 1e-5


@pytest.mark.parametrize("needle", [None, 0, 63, 64, 69])
def test_latent_attention(needle):
    assert cases.latent_case("cpu", torch.float32, 3, 40, 24, 56, 72, [70, 1, 9], [0, 69, 64], needle=needle) < 1e-4


@pytest.mark.parametrize("loud", [None, 0, 64])
def test_unit_attention_with_temperature(loud):
    assert cases.unit_case("cpu", torch.float32, 6, 2, 48, 80, [70, 1, 9], [0, 69, 64], 0.4, 30, loud) < 1e-4


@pytest.mark.parametrize("part", ["tap", "decay", "order", "rotation", "norm", "temperature", "head"])
def test_planted_mistakes_would_show(part, monkeypatch):
    """Each mechanism matters in the test models: an oracle with one of them slightly wrong leaves the tolerance by far."""
    cfg, w = cases.weights("mixed")
    toks = list(cases.prompt(cfg["vocab"], 70, 1))
    w = dict(w)
    if part == "tap":
        w["l0.mix.k.conv"] = w["l0.mix.k.conv"].flip(1)
    elif part == "decay":
        monkeypatch.setattr(oracle, "channel_decay", lambda h, w, p, n, d, real=oracle.channel_decay: real(h, w, p, n, d).mean(-1, keepdim=True).expand(-1, n, d))
    elif part == "order":
        def read_first(q, k, v, g, beta):
            s, out = torch.zeros(k.shape[1], v.shape[1], dtype=torch.float64), torch.zeros(v.shape, dtype=torch.float64)
            for t in range(k.shape[0]):
                s = g[t][:, None] * s
                out[t] = s.T @ q[t]
                s = s + torch.outer(k[t], beta[t] * (v[t] - s.T @ k[t]))
            return out
        monkeypatch.setattr(oracle, "delta_recurrence", read_first)
    elif part == "rotation":
        monkeypatch.setattr(oracle, "rotate_pairs", lambda x, dims, base: x)
    elif part == "norm":
        monkeypatch.setattr(oracle, "rms_norm", lambda x, eps, gain=1.0: x * gain)
    elif part == "temperature":
        monkeypatch.setattr(oracle, "query_temperature", lambda t, c, e: torch.ones(t, dtype=torch.float64))
    else:
        w["head"] = w["embed"]
    wrong = oracle.forward(cfg, w, toks)
    assert float(cases.row_errors(wrong, cases.expected("mixed", 1.0, 70, 1)).max()) > 3 * cases.TOL["bfloat16"]


# ---- the model through the runner --------------------------------------------------------------------------


@pytest.mark.parametrize("name", sorted(cases.CONFIGS))
def test_prompt_in_one_step_and_layer_taps(name, ckpt):
    r = cases.make_runner(ckpt(name), "cpu", "float32")
    assert cases.replay(r, name, 1.0, {"a": (90, 1)}, [[("a", 90)]]) < cases.TOL["float32"]
    cfg, w = cases.weights(name)
    trace, toks = [], list(cases.prompt(cfg["vocab"], 90, 1))
    oracle.forward(cfg, w, toks, trace)
    meta = r._meta([0], [90])
    _, taps = r.model.hidden_states(torch.tensor(toks, dtype=torch.int32), meta, r.cache, capture_layers=range(len(trace)))
    assert len(taps) == len(trace)
    for a, b in zip(taps, trace):
        assert float((a.double() - b).abs().max() / b.abs().max()) < 1e-4


@pytest.mark.parametrize("sharp", [1.0, 4.0])
@pytest.mark.parametrize("name", sorted(cases.CONFIGS))
def test_portions_and_decoding(name, sharp, ckpt):
    r = cases.make_runner(ckpt(name, sharp), "cpu", "float32")
    n = 150
    for sizes in ([64, 40, 1], [2, 3, 37], [24, 40]):
        steps = [[("a", c)] for c in cases.portions(n, sizes)]
        assert cases.replay(r, name, sharp, {"a": (n, 2)}, steps) < cases.TOL["float32"], sizes
    assert cases.replay(r, name, sharp, {"a": (n, 2)}, [[("a", 1)] for _ in range(n)]) < cases.TOL["float32"]


@pytest.mark.parametrize("name", sorted(cases.CONFIGS))
def test_unequal_requests_share_steps_pages_and_slots(name, ckpt):
    r = cases.make_runner(ckpt(name), "cpu", "float32", pages=6, seats=3)
    req = {"a": (130, 3), "b": (1, 4), "c": (25, 5), "d": (90, 6), "e": (66, 7)}
    steps = [[("a", 60), ("b", 1), ("c", 20)], [("c", 1), ("a", 2)], [("d", 33), ("a", 1), ("c", 3)], [("c", 1), ("d", 40), ("a", 66)],
             [("a", 1)], [("d", 17), ("e", 64)], [("e", 2)]]
    assert cases.replay(r, name, 1.0, req, steps) < cases.TOL["float32"]
    assert r.kv.native is None or r.kv.native.allocator().free_pages == 6
    assert cases.replay(r, name, 1.0, req, steps) < cases.TOL["float32"]        # all pages and rows a second time


def test_bf16_stays_close(ckpt):
    r = cases.make_runner(ckpt("mixed"), "cpu", "bfloat16")
    assert cases.replay(r, "mixed", 1.0, {"a": (70, 8)}, [[("a", 50)]] + [[("a", 1)]] * 20) < cases.TOL["bfloat16"]


def test_recurrent_replay_advances_by_the_accepted_rows(ckpt):
    """Speculative commit: a recorded step of four rows, rolled back, replayed over its first two."""
    r = cases.make_runner(ckpt("mixed"), "cpu", "float32")
    cfg, _ = cases.weights("mixed")
    p = list(cases.prompt(cfg["vocab"], 30, 9))
    r.step([0], [p[:20]])
    saved = r.kv.recurrent.snapshot([0])
    r.kv.recurrent.begin_record()
    r.step([0], [p[20:24]])
    rec = r.kv.recurrent.end_record()
    r.kv.recurrent.restore([0], saved)
    r.kv.rewind(0, 20)
    meta = r._meta([0], [2])
    assert r.model.replay_recurrent(rec, torch.arange(2), meta, r.cache) == 2
    r.kv.commit(0, 2)
    got = r.step([0], [p[22:30]], logits_all=True)
    assert cases.error(got, cases.expected("mixed", 1.0, 30, 9)[22:]) < cases.TOL["float32"]


# ---- generation, command line ------------------------------------------------------------------------------


@pytest.mark.parametrize("engine", [False, True])
def test_greedy_generation(engine, ckpt):
    from tensorrt_edge_llm_b200.runtime.llm import LLM
    from tensorrt_edge_llm_b200.runtime.runner import SamplingParams
    cfg, w = cases.weights("mixed")
    prompts = [list(cases.prompt(cfg["vocab"], n, n)) for n in (100, 3, 20)]
    kw = {"enable_in_flight_batching": True, "scheduling": {"mode": "mixed", "max_chunk_tokens": 64, "max_num_tokens": 72}} if engine else {}
    llm = LLM(ckpt("mixed"), device="cpu", dtype="float32", max_batch_size=2, max_input_len=128, max_kv_cache_capacity=128, **kw)
    try:
        outs = llm.generate(prompts, SamplingParams(max_tokens=6))
        for p, o in zip(prompts, outs):
            assert list(o.token_ids) == oracle.greedy(cfg, w, p, 6)
    finally:
        llm.close()


def test_prefix_cache_restores_state(ckpt):
    """A prompt that shares its first pages with an earlier one starts from their pages and state rows."""
    from tensorrt_edge_llm_b200.runtime.llm import LLM
    from tensorrt_edge_llm_b200.runtime.runner import SamplingParams
    cfg, w = cases.weights("mixed")
    base = list(cases.prompt(cfg["vocab"], 64, 11))
    tails = [list(cases.prompt(cfg["vocab"], 9, s)) for s in (12, 13)]
    llm = LLM(ckpt("mixed"), device="cpu", dtype="float32", max_batch_size=2, max_input_len=128, max_kv_cache_capacity=192,
              enable_in_flight_batching=True, enable_prefix_cache=True)
    try:
        for k, t in enumerate(tails):
            o = llm.generate([base + t], SamplingParams(max_tokens=4))[0]
            assert list(o.token_ids) == oracle.greedy(cfg, w, base + t, 4)
            assert o.reused_input_tokens == (64 if k else 0)
    finally:
        llm.close()


def test_prepared_artifacts_load_the_same_model(ckpt, tmp_path):
    from tensorrt_edge_llm_b200.checkpoint.artifacts import write_artifacts
    write_artifacts(ckpt("mixed"), str(tmp_path / "engine"))
    r = cases.make_runner(str(tmp_path / "engine"), "cpu", None)
    assert cases.replay(r, "mixed", 1.0, {"a": (40, 1)}, [[("a", 40)]]) < cases.TOL["bfloat16"]


def test_trace_runner_and_infer_command(ckpt, tmp_path):
    cfg, w = cases.weights("mixed")
    a, b = (list(cases.prompt(cfg["vocab"], n, s)) for n, s in ((70, 1), (30, 2)))
    lines = [{"step": 0, "entries": [{"id": "a", "tokens": a[:50], "want": [0, 49]}, {"id": "b", "tokens": b[:3], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[3:], "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[50:], "want": [19]}], "end": ["a"]}]
    out = tmp_path / "out"
    out.mkdir()
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", ckpt("mixed"), "--dtype", "float32", "--out", str(out), "--max-tokens",
                        "192", "--device", "cpu"], input="\n".join(json.dumps(x) for x in lines), capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr
    want = oracle.forward(cfg, w, a)
    for f, rows in (("0.f32", [0, 49]), ("2.f32", [69])):
        got = torch.frombuffer(bytearray((out / f).read_bytes()), dtype=torch.float32).view(len(rows), cfg["vocab"])
        assert cases.error(got, want[rows]) < cases.TOL["float32"]
    req = tmp_path / "req.json"
    req.write_text(json.dumps({"temperature": 0.0, "max_generate_length": 3, "requests": [{"input_ids": a[:20]}]}))
    p = subprocess.run([sys.executable, "-m", "tensorrt_edge_llm_b200.cli", "infer", ckpt("mixed"), "--input-file", str(req), "--output-file",
                        str(tmp_path / "res.json"), "--device", "cpu", "--dtype", "float32"], capture_output=True, text=True, timeout=300, cwd=ROOT)
    assert p.returncode == 0, p.stderr
    assert json.loads((tmp_path / "res.json").read_text())["responses"][0]["output_ids"] == oracle.greedy(cfg, w, a[:20], 3)


def test_parallel_deployments_are_refused():
    from tensorrt_edge_llm_b200.model import AutoModel
    cfg = ModelConfig.from_hf_dict(cases.CONFIGS["mixed"]())
    with pytest.raises((NotImplementedError, ValueError)):
        AutoModel.from_config(cfg.for_rank(0, 3))
