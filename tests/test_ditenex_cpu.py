"""Ditenex family on the CPU: parsing, loading, and every schedule against the plain statement (``ditenex_oracle``)."""
import json
import os
import subprocess
import sys

import pytest
import torch

import ditenex_cases as cases
import ditenex_oracle as oracle
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
    assert cfg.layer_types == ["attention"] * 5 and cfg.mlp_types == ["mlp", "moe", "none", "moe", "mlp"]
    a, b, e = cfg.layer_specs[0].attention, cfg.layer_specs[1].attention, cfg.layer_specs[1].moe
    assert (a.num_heads, a.num_kv_heads, a.head_dim, a.v_head_dim, a.window, a.pad) == (6, 2, 40, 56, 37, 64)
    assert a.mixed_scores and a.distance_bias and a.qkv_bias and a.out_gate and not a.value_mix and b.value_mix and b.scale == 40 ** -0.5
    assert (e.num_experts, e.top_k, e.intermediate_size, e.groups, e.keep_groups, e.weight_scale, e.shared_size) == (9, 3, 40, 3, 2, 1.7, 48)
    assert (e.router, e.limit, e.alpha, e.up_offset) == ("sigmoid_groups", 0.0, 1.0, 0.0) and cfg.layer_specs[3].moe.shared_size == 0
    assert (cfg.layer_specs[0].ff, cfg.layer_specs[0].ff_act, cfg.residual_mult, cfg.max_position_embeddings) == (72, "xielu", 0.4, 400)
    assert cfg.token_shift and cfg.learned_positions and cfg.is_hybrid and cfg.tie_word_embeddings
    assert cfg.kv_geometry() == [(2, 64), (3, 64), (3, 64), (1, 128), (3, 128)] and cfg.num_attn_layers == 5
    again = ModelConfig.from_dict(json.loads(json.dumps(cfg.to_dict())))
    assert again.layer_specs == cfg.layer_specs and again.token_shift


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
    assert c.recurrent_state_bytes_per_seat() == kv.recurrent.bytes() == 4 * cfg.hidden_size * len(cfg.layer_specs)


@pytest.mark.parametrize("change", ["mixer", "mlp", "heads", "window", "groups", "keep", "top", "values"])
def test_config_refuses_what_it_does_not_know(change):
    hf = cases.CONFIGS["mixed"]()
    l = hf["layers"]
    if change == "mixer":
        l[0]["type"] = "other"
    elif change == "mlp":
        l[0]["mlp"]["kind"] = "other"
    elif change == "heads":
        l[0]["mixer"]["kv_heads"] = 4
    elif change == "window":
        l[0]["mixer"]["mask"]["size"] = 0
    elif change == "groups":
        l[1]["mlp"]["router"]["groups"]["count"] = 2
    elif change == "keep":
        l[1]["mlp"]["router"]["groups"]["keep"] = 4
    elif change == "top":
        l[1]["mlp"]["router"]["top"] = 7
    else:
        l[1]["mixer"]["vdim"] = 32
    with pytest.raises(ValueError):
        ModelConfig.from_hf_dict(hf)


# ---- mechanisms alone --------------------------------------------------------------------------------------


@pytest.mark.parametrize("width", [24, 40, 256])
def test_stream_norms_and_token_shift(width):
    for kw in (dict(), dict(top=3), dict(top=2, dense=False), dict(ids=True), dict(shift=False)):
        for lens, past in (([9, 1, 20], None), ([12, 3, 30], [5, 2, 1]), ([2, 2], [1, 1])):
            assert max(cases.sandwich_case("cpu", torch.float32, width, lens, past, **kw)) < 1e-5


@pytest.mark.parametrize("needle", [None, 0, 20, 63, 64])
@pytest.mark.parametrize("window", [1, 37, 64, 500])
def test_mixed_attention(window, needle):
    assert cases.attention_case("cpu", torch.float32, 6, 2, 48, 24, window, [70, 1, 9], [0, 69, 64], needle=needle) < 1e-4
    assert cases.attention_case("cpu", torch.float32, 3, 3, 24, 80, window, [2, 1], [63, 36], needle=needle, join=False, gate=False) < 1e-4


def test_activations():
    x, p, q = torch.randn(50, 16) * 4, torch.tensor(0.7).double(), torch.tensor(-0.4).double()
    coef = torch.stack([oracle.softplus(p), 0.5 + oracle.softplus(q)]).float()
    assert torch.allclose(ops.xielu(x, coef).double(), oracle.xielu(x.double(), p, q), atol=1e-5)
    g, u = x.double().chunk(2, -1)
    assert torch.allclose(ops.glu(x, "silu").double(), g * torch.sigmoid(g) * u, atol=1e-5)


@pytest.mark.parametrize("experts, top, groups, keep", [(8, 2, 2, 1), (9, 3, 3, 2), (6, 1, 6, 2), (5, 5, 1, 1)])
def test_router(experts, top, groups, keep):
    z, corr = torch.randn(40, experts) * 3, torch.randn(experts) * 0.3 - 2.0
    w, idx = ops.moe_route_sigmoid_groups(z, corr, top, groups, keep, 1.7)
    for t in range(z.shape[0]):
        s = torch.sigmoid(z[t].double())
        want = oracle.chosen_experts(s + corr.double(), top, groups, keep)
        assert idx[t].tolist() == want and torch.allclose(w[t].double(), s[want] * 1.7, rtol=1e-5)


def _shift_own(x, amount):
    """A shift that feeds on its own result."""
    rows = [x[0] * (1 - amount)]
    for t in range(1, x.shape[0]):
        rows.append(x[t] + (rows[-1] - x[t]) * amount)
    return torch.stack(rows)


@pytest.mark.parametrize("part", ["positions", "shift", "shift of shifted", "shift first", "talk", "talk of weights", "slopes", "bias behind the mixing", "window",
                                  "first values", "value share", "gate", "bias", "residual", "post norm", "xielu", "groups", "closed groups", "correction",
                                  "router scale", "shared"])
def test_planted_mistakes_would_show(part, monkeypatch):
    """Each mechanism matters in the test models: an oracle with one of them slightly wrong leaves the tolerance by far."""
    cfg, w = cases.weights("mixed", 3.0)
    cfg, w, n = json.loads(json.dumps(cfg)), dict(w), 70
    right = cases.expected("mixed", 3.0, n, 1)
    toks, layers = list(cases.prompt(cfg["vocab"], n, 1)), cfg["layers"]
    real = {k: getattr(oracle, k) for k in ("token_shift", "mix_heads", "head_scores", "window_weights", "mix_values", "chosen_experts", "attention", "routed")}
    moes = [i for i, l in enumerate(layers) if l["mlp"] and l["mlp"]["kind"] == "moe"]
    if part == "positions":
        w["pos"] = w["pos"].roll(1, 0)
    elif part == "shift":
        monkeypatch.setattr(oracle, "token_shift", lambda h, s: h)
    elif part == "shift of shifted":
        monkeypatch.setattr(oracle, "token_shift", _shift_own)
    elif part == "shift first":
        monkeypatch.setattr(oracle, "token_shift", lambda h, s: torch.cat([h[:1], real["token_shift"](h, s)[1:]]))
    elif part == "talk":
        monkeypatch.setattr(oracle, "mix_heads", lambda s, t: real["mix_heads"](s, t.T))
    elif part == "talk of weights":
        monkeypatch.setattr(oracle, "mix_heads", lambda s, t: s)
    elif part == "slopes":
        monkeypatch.setattr(oracle, "distance_slopes", lambda h: torch.tensor([2.0 ** (-8.0 * i / h) for i in range(h)], dtype=torch.float64))
    elif part == "bias behind the mixing":
        def late(q, k, v, talk, scale, window):
            zero = real["head_scores"](q * 0, k, scale)
            a = real["window_weights"](real["mix_heads"](real["head_scores"](q, k, scale) - zero, talk) + zero, window)
            group = q.shape[1] // v.shape[1]
            return torch.stack([a[h] @ v[:, h // group] for h in range(q.shape[1])], 1)
        monkeypatch.setattr(oracle, "attend", late)
    elif part == "window":
        for l in layers:
            l["mixer"]["mask"]["size"] += 1
    elif part == "first values":
        layers[0]["mixer"]["v_mix"] = False
        def from_layer_behind(h, c, w_, p, first):
            out, f = real["attention"](h, {**c, "v_mix": c["v_mix"] and p != "l1.mix"}, w_, p, first)
            return out, f
        monkeypatch.setattr(oracle, "attention", from_layer_behind)
    elif part == "value share":
        monkeypatch.setattr(oracle, "mix_values", lambda v, f, s: real["mix_values"](v, f, 1 - s))
    elif part == "gate":
        for i in range(len(layers)):
            w[f"l{i}.mix.g"] = torch.zeros_like(w[f"l{i}.mix.g"])
    elif part == "bias":
        w["l0.mix.k.b"], w["l0.mix.v.b"] = torch.zeros_like(w["l0.mix.k.b"]), torch.zeros_like(w["l0.mix.v.b"])
    elif part == "residual":
        cfg["residual_mult"] = 0.42
    elif part == "post norm":
        w["l2.norm1b"] = w["l2.norm1b"].roll(1)
    elif part == "xielu":
        w["l0.mlp.act"] = w["l0.mlp.act"].flip(0)
    elif part == "groups":
        monkeypatch.setattr(oracle, "chosen_experts", lambda s, top, count, keep: real["chosen_experts"](s, top, 1, 1))
    elif part == "closed groups":
        def zeros(s, top, count, keep):
            best = real["chosen_experts"](s, s.numel() // count * keep, count, keep)
            masked = torch.zeros_like(s)
            masked[best] = s[best]
            return masked.topk(top).indices.tolist()
        monkeypatch.setattr(oracle, "chosen_experts", zeros)
    elif part == "correction":
        for i in moes:
            w[f"l{i}.mlp.correction"] = torch.zeros_like(w[f"l{i}.mlp.correction"])
    elif part == "router scale":
        for i in moes:
            layers[i]["mlp"]["router"]["scale"] *= 1.3
    else:
        for i in moes:
            layers[i]["mlp"].pop("shared", None)
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
    assert r.model.replay_recurrent(rec, torch.arange(2), meta, r.cache) == 5
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


def test_no_position_beyond_the_table(ckpt):
    """The last position has a row; a sequence that needs one more is refused before anything is written."""
    from tensorrt_edge_llm_b200.runtime.llm import LLM
    from tensorrt_edge_llm_b200.runtime.runner import SamplingParams
    cfg, _ = cases.weights("mixed")
    n = cfg["max_positions"]
    r = cases.make_runner(ckpt("mixed"), "cpu", "float32")
    r.step([0], [list(cases.prompt(cfg["vocab"], n, 1))])
    with pytest.raises(ValueError, match="positions"):
        r.step([0], [[1]])
    for engine, reason in ((True, "TOO_LONG"), (False, "positions")):
        llm = LLM(ckpt("mixed"), device="cpu", dtype="float32", max_batch_size=1, max_input_len=n, max_kv_cache_capacity=2 * n, enable_in_flight_batching=engine)
        try:
            assert llm.kv.max_tokens == n
            with pytest.raises((RuntimeError, ValueError), match=reason):
                llm.generate([list(cases.prompt(cfg["vocab"], n - 2, 2))], SamplingParams(max_tokens=10))
        finally:
            llm.close()


def test_embedding_rows_as_prompts(ckpt):
    """Prompts given as embedding rows get their position rows too."""
    cfg, _ = cases.weights("mixed")
    r = cases.make_runner(ckpt("mixed"), "cpu", "float32")
    p = list(cases.prompt(cfg["vocab"], 20, 3))
    got = r.prefill_embeds([0], [r.model.model.embed_tokens.weight[p]])
    assert cases.error(got, cases.expected("mixed", 1.0, 20, 3)[-1:]) < cases.TOL["float32"]
