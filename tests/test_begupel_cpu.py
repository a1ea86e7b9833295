"""Begupel family on the CPU: parsing, loading, and every schedule against the plain statement (``begupel_oracle``)."""
import json
import os
import subprocess
import sys

import pytest
import torch

import begupel_cases as cases
import begupel_oracle as oracle
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


def test_config_round_trip(ckpt):
    cfg = ModelConfig.from_pretrained(ckpt("mixed"))
    assert cfg.layer_types == ["parallel", "lightning", "lightning", "parallel"] and cfg.mlp_types == ["mlp", "none", "mlp", "none"]
    a, d, l = cfg.layer_specs[0].attention, cfg.layer_specs[0].delta, cfg.layer_specs[2].lightning
    assert (a.window, a.rotary_dim, a.rope_factor, a.rope_theta, a.pad) == (37, 24, 2.5, 500.0, 64) and a.row_norm and a.rotated_values
    assert (d.conv_kernel, d.k_pad, d.v_pad) == (3, 64, 32) and d.head_decay and d.silu_gate
    assert (l.k_pad, l.v_pad, l.decay) == (128, 256, [0.5, 0.875])
    assert (cfg.norm_groups, cfg.input_conv, cfg.final_logit_softcapping) == (12, 3, 6.0)
    assert (cfg.bigram_buckets, cfg.bigram_mul_prev, cfg.bigram_mul_cur) == (61, 13, 29)
    assert (cfg.layer_specs[3].attention_mult, cfg.layer_specs[3].delta_mult) == (1.3, 0.4)
    assert cfg.kv_geometry() == [(2, 64), (3, 64)] and cfg.num_attn_layers == 2 and cfg.is_hybrid
    again = ModelConfig.from_dict(json.loads(json.dumps(cfg.to_dict())))
    assert again.layer_specs == cfg.layer_specs


@pytest.mark.parametrize("name", sorted(cases.CONFIGS))
def test_native_engine_config_sizes(name, ckpt):
    """The native configuration derives the cache and state sizes that the Python managers allocate."""
    from tensorrt_edge_llm_b200.checkpoint.artifacts import runtime_config_dict
    from tensorrt_edge_llm_b200.runtime import native as rt
    from tensorrt_edge_llm_b200.runtime.kv_cache import KVCacheManager
    cfg = ModelConfig.from_pretrained(ckpt(name))
    c = rt.LLMEngineConfig.from_runtime_config(json.dumps(runtime_config_dict(cfg, 2, 64, 128, 1), default=str))
    kv = KVCacheManager(cfg, 2, 64, max_seats=1, max_pages_per_seq=2)
    assert c.validate() == "" and c.is_hybrid() and c.num_attention_layers() == cfg.num_attn_layers
    assert c.kv_bytes_per_token() == kv.bytes_per_token
    assert c.recurrent_state_bytes_per_seat() == kv.recurrent.bytes()


@pytest.mark.parametrize("change", ["mixer", "mlp", "rot", "heads", "delta heads", "window", "decays", "decay", "groups", "taps"])
def test_config_refuses_what_it_does_not_know(change):
    hf = cases.CONFIGS["mixed"]()
    l = hf["layers"]
    if change == "mixer":
        l[0]["type"] = "other"
    elif change == "mlp":
        l[0]["mlp"]["kind"] = "moe"
    elif change == "rot":
        l[0]["mixer"]["left"]["rot"]["dims"] = 42
    elif change == "heads":
        l[0]["mixer"]["left"]["kv_heads"] = 4
    elif change == "delta heads":
        l[0]["mixer"]["right"]["kv_heads"] = 3
    elif change == "window":
        l[0]["mixer"]["left"]["mask"]["size"] = 0
    elif change == "decays":
        l[1]["mixer"]["decay"] = [0.5]
    elif change == "decay":
        l[1]["mixer"]["decay"][0] = 1.5
    elif change == "groups":
        hf["norm"]["groups"] = 7
    else:
        hf["canon"]["taps"] = 0
    with pytest.raises(ValueError):
        ModelConfig.from_hf_dict(hf)


# ---- mechanisms alone --------------------------------------------------------------------------------------


@pytest.mark.parametrize("width, groups, taps", [(24, 3, 4), (40, 4, 1), (256, 2, 3), (64, 1, 8)])
def test_stream_conv_and_bigram(width, groups, taps):
    assert max(cases.stream_case("cpu", torch.float32, width, groups, taps, [9, 1, 20], behind=3)) < 1e-5
    for ids in (False, True):
        for lens, past in (([9, 1, 20], None), ([12, 3, 30], [5, 2, 1]), ([2, 2], [1, 1])):
            assert max(cases.stream_case("cpu", torch.float32, width, groups, taps, lens, past, ids=ids)) < 1e-5


def test_stream_norms():
    x, d, w, o = torch.randn(5, 36), torch.randn(5, 36) * 3, torch.randn(36), torch.randn(36)
    y, h = ops.stream_post(x, d, w, 4, 1e-3, cases._meta([0], [5], None, "cpu"), torch.float32, out_norm=o)
    want = x.double() + oracle.group_norm(d.double(), w.double(), 4, 1e-3)
    assert torch.allclose(y.double(), want, atol=1e-5) and torch.allclose(h.double(), oracle.group_norm(want, o.double(), 4, 1e-3), atol=1e-5)


def test_glu_and_softcap():
    x = torch.randn(5, 48)
    assert torch.allclose(ops.glu(x, "relu"), torch.relu(x[:, :24]) * x[:, 24:])
    assert torch.allclose(ops.softcap_(x.clone() * 30, 7.0).double(), oracle.softcap(x.double() * 30, 7.0), atol=1e-5)


@pytest.mark.parametrize("needle", [None, 0, 20, 63, 64])
@pytest.mark.parametrize("window", [1, 37, 64, 500])
def test_windowed_attention_with_rotated_values(window, needle):
    assert cases.attention_case("cpu", torch.float32, 6, 2, 48, 24, window, 32, [70, 1, 9], [0, 69, 64], factor=2.5, needle=needle) < 1e-4
    assert cases.attention_case("cpu", torch.float32, 3, 3, 24, 80, window, 8, [2, 1], [63, 36], needle=needle) < 1e-4


@pytest.mark.parametrize("shape", [(4, 2, 40, 24, 3), (1, 1, 16, 16, 1), (3, 3, 64, 130, 8)])
def test_delta_with_head_decays(shape):
    assert cases.delta_case("cpu", torch.float32, *shape, [9, 2, 4], past=[5, 1, 2]) < 1e-5
    assert cases.delta_case("cpu", torch.float32, *shape, [12, 12], keep=1) < 1e-5


@pytest.mark.parametrize("shape", [(3, 24, 40), (1, 72, 136), (4, 64, 128)])
def test_lightning(shape):
    for kw in (dict(past=[5, 1, 2]), dict(loud=0), dict(decay=([0.0, 1.0, 0.5, 1.0][:shape[0]]))):
        assert max(cases.lightning_case("cpu", torch.float32, *shape, [9, 2, 4], **kw)) < 1e-5


@pytest.mark.parametrize("part", ["prefix", "buckets", "canon", "norm groups", "window", "values", "factor", "row norm", "decay", "lightning decay",
                                  "write first", "gate", "scales", "bias", "cap", "lightning norm"])
def test_planted_mistakes_would_show(part, monkeypatch):
    """Each mechanism matters in the test models: an oracle with one of them slightly wrong leaves the tolerance by far."""
    cfg, w = cases.weights("mixed", 3.0)
    cfg, w, n = json.loads(json.dumps(cfg)), dict(w), 70
    right = cases.expected("mixed", 3.0, n, 1)
    toks, attn = list(cases.prompt(cfg["vocab"], n, 1)), [l["mixer"]["left"] for l in cfg["layers"] if l["type"] == "parallel"]
    real = {k: getattr(oracle, k) for k in ("bigram_rows", "turn", "rms_norm", "group_norm", "silu", "delta_recurrence", "head_decay")}
    if part == "prefix":
        monkeypatch.setattr(oracle, "bigram_rows", lambda t, b, p, c: [(t[i - 1] * p + x * c) % b if i else c * x % b for i, x in enumerate(t)])
    elif part == "buckets":
        monkeypatch.setattr(oracle, "bigram_rows", lambda t, b, p, c: real["bigram_rows"](t, b, c, p))
    elif part == "canon":
        for i in range(4):
            w[f"l{i}.canon1"] = w[f"l{i}.canon1"].flip(1)
    elif part == "norm groups":
        cfg["norm"]["groups"] = 1
    elif part == "window":
        for a in attn:
            a["mask"]["size"] += 1
    elif part == "values":
        monkeypatch.setattr(oracle, "turn", lambda x, dims, base, factor=1.0, back=False: x if back else real["turn"](x, dims, base, factor))
    elif part == "factor":
        for a in attn:
            a["rot"]["scaling"]["factor"] *= 1.3
    elif part == "row norm":
        def norm_by_head(h, c, w, p, eps):
            t = h.shape[0]
            q, k = (oracle.rms_norm((h @ w[f"{p}.{m}"].T).reshape(t, n, -1), eps, w[f"{p}.{m}.norm"].reshape(n, -1))
                    for m, n in (("q", c["heads"]), ("k", c["kv_heads"])))
            v = (h @ w[p + ".v"].T).reshape(t, c["kv_heads"], -1)
            return oracle.attention_heads(q, k, v, c).reshape(t, -1) @ w[p + ".o"].T
        monkeypatch.setattr(oracle, "attention", norm_by_head)
    elif part == "decay":
        monkeypatch.setattr(oracle, "head_decay", lambda z, a, b: real["head_decay"](z, a, b) ** 1.2)
    elif part == "lightning decay":
        for l in cfg["layers"]:
            if l["type"] == "lightning":
                l["mixer"]["decay"] = l["mixer"]["decay"][::-1]
    elif part == "write first":
        def read_first(q, k, v, g, beta):
            return torch.cat([torch.zeros_like(v[:1]), real["delta_recurrence"](q[1:], k[:-1], v[:-1], g[:-1], beta[:-1])])
        monkeypatch.setattr(oracle, "delta_recurrence", read_first)
    elif part == "gate":
        monkeypatch.setattr(oracle, "silu", torch.sigmoid)
    elif part == "scales":
        for l in cfg["layers"]:
            if l["type"] == "parallel":
                l["mixer"]["left_scale"], l["mixer"]["right_scale"] = l["mixer"]["right_scale"], l["mixer"]["left_scale"]
    elif part == "bias":
        w["l0.mlp.down.b"] = torch.zeros_like(w["l0.mlp.down.b"])
    elif part == "cap":
        cfg["logit_softcap"] = 1e9
    else:
        w["l1.mix.norm"] = w["l1.mix.norm"].roll(1)
    wrong = oracle.forward(cfg, w, toks)
    worst = float(cases.row_errors(wrong, right).max())
    assert worst > 1.5 * cases.TOL["bfloat16"] and worst > 500 * cases.TOL["float32"]


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
    for sizes in ([64, 40, 1], [2, 3, 37]):
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
    assert r.model.replay_recurrent(rec, torch.arange(2), meta, r.cache) == 4
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


def test_deployments_that_are_refused(ckpt):
    from tensorrt_edge_llm_b200.model import AutoModel
    cfg = ModelConfig.from_hf_dict(cases.CONFIGS["wide"]())
    with pytest.raises((NotImplementedError, ValueError)):
        AutoModel.from_config(cfg.for_rank(0, 2))
    with pytest.raises(ValueError, match="range of float16"):
        cases.make_runner(ckpt("wide"), "cpu", "float16")
    r = cases.make_runner(ckpt("wide"), "cpu", "float32")
    with pytest.raises(NotImplementedError):
        r.prefill_embeds([0], [torch.zeros(3, cfg.hidden_size)])
