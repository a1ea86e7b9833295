"""Dimesun family on the CPU: parsing, loading, and every schedule against the plain statement (``dimesun_oracle``)."""
import json
import math
import os
import subprocess
import sys

import pytest
import torch

import dimesun_cases as cases
import dimesun_oracle as oracle
from tensorrt_edge_llm_b200 import ops
from tensorrt_edge_llm_b200.config import ModelConfig
from tensorrt_edge_llm_b200.ops.meta import build_step_meta

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.fixture(scope="module")
def ckpt(tmp_path_factory):
    made = {}

    def get(name, sharp=1.0):
        if (name, sharp) not in made:
            made[name, sharp] = cases.save_checkpoint(tmp_path_factory.mktemp(name), *cases.weights(name, sharp))
        return made[name, sharp]
    return get


# ---- mechanisms alone --------------------------------------------------------------------------------------


def test_config_runs_and_round_trip():
    hf = cases.CONFIGS["mixed"]()
    cfg = ModelConfig.from_hf_dict(hf)
    assert cfg.layer_run_ids == [i for i, _, _ in oracle.schedule(hf)] == [0, 1, 2, 1, 2, 3]
    assert cfg.num_hidden_layers == 6 and cfg.layer_types.count("attention") == 3 and cfg.mlp_types == ["moe", "moe", "none", "moe", "none", "none"]
    assert cfg.kv_geometry() == [(2, 64), (2, 64), (4, 128)] and cfg.is_hybrid
    again = ModelConfig.from_dict(json.loads(json.dumps(cfg.to_dict())))
    assert again.layer_specs == cfg.layer_specs and again.layer_run_ids == cfg.layer_run_ids
    assert not ModelConfig.from_hf_dict(cases.CONFIGS["attention_only"]()).is_hybrid


@pytest.mark.parametrize("name", sorted(cases.CONFIGS))
def test_native_engine_config_sizes(name):
    """The native configuration derives the cache and state sizes that the Python managers allocate."""
    from tensorrt_edge_llm_b200.checkpoint.artifacts import runtime_config_dict
    from tensorrt_edge_llm_b200.runtime import native as rt
    from tensorrt_edge_llm_b200.runtime.kv_cache import KVCacheManager
    cfg = ModelConfig.from_hf_dict(cases.CONFIGS[name]())
    c = rt.LLMEngineConfig.from_runtime_config(json.dumps(runtime_config_dict(cfg, 2, 64, 128, 1), default=str))
    kv = KVCacheManager(cfg, 2, 64, max_seats=1, max_pages_per_seq=2)
    state = 0 if kv.recurrent is None else kv.recurrent.bytes()
    assert c.validate() == "" and c.is_hybrid() == cfg.is_hybrid and c.num_attention_layers() == cfg.num_attn_layers
    assert c.kv_bytes_per_token() == kv.bytes_per_token
    assert c.recurrent_state_bytes_per_seat() == state


@pytest.mark.parametrize("change", ["mixer", "mlp", "loop", "rot"])
def test_config_refuses_what_it_does_not_know(change):
    hf = cases.CONFIGS["mixed"]()
    if change == "mixer":
        hf["layers"][0]["type"] = "other"
    elif change == "mlp":
        hf["layers"][0]["mlp"]["kind"] = "dense"
    elif change == "loop":
        hf["loop"]["stop"] = 9
    else:
        hf["layers"][1]["mixer"]["rot"]["dims"] = 50
    with pytest.raises(ValueError):
        ModelConfig.from_hf_dict(hf)


def test_router_takes_the_softmax_over_the_chosen():
    z = torch.tensor([[1.0, 3.0, 2.0, 3.0], [0.0, -50.0, -49.0, -1.0]])
    w, idx = ops.moe_route_chosen(z, 2)
    assert idx.tolist() == [[1, 3], [0, 3]]
    for r in range(2):
        i, p = oracle.route(z[r].double(), 2)
        assert torch.allclose(w[r].double(), p, atol=1e-6)


def test_clamped_unit_and_experts():
    g, u = torch.tensor([[-9.0, 0.5, 9.0]]), torch.tensor([[5.0, -5.0, 0.25]])
    got = ops.ref.clamped_glu(torch.cat([g, u], -1), 1.0, 1.702)
    assert torch.allclose(got.double(), oracle.clamped_glu(g.double(), u.double(), 1.0), atol=1e-6)


def test_stream_norm_adds_both_sublayers_and_the_step():
    x, a, b, s, w = (torch.randn(*n) for n in ((3, 8), (3, 8), (3, 8), (8,), (8,)))
    y, h = ops.stream_norm(x, w, 1e-3, delta=a, routed=b, mult=0.7, step=s, offset=1.0, dtype=torch.float32)
    want = x + 0.7 * (a + b) + s
    assert torch.allclose(y, want, atol=1e-6)
    assert torch.allclose(h.double(), oracle.rms_norm(want.double(), 1 + w.double(), 1e-3), atol=1e-5)


@pytest.mark.parametrize("chunk", [1, 2, 64, 63, 65, 100])
def test_chunked_attention_edges(chunk):
    cases_edges(chunk, "cpu", torch.float32)


def cases_edges(chunk, device, dtype, d=64, hq=2, hkv=1):
    """One key stands out far above the rest.  A row that may see it returns its value, any other row does not: checked for the rows
    just inside and just outside its block, for a prompt and for single decoded rows, at page borders."""
    n, page = 200, 64
    g = torch.Generator().manual_seed(0)
    table = torch.tensor([[5, 2, 7, 0]], dtype=torch.int32)
    for j in sorted({0, 1, 63, 64, 65, 127, 128, chunk - 1, chunk, 2 * chunk - 1} & set(range(n))):
        kv = torch.randn(8, 2, hkv, page, d, generator=g) * 0.05
        kv[:, 1] = 0.0
        loud = torch.zeros(d)
        loud[0] = 8.0
        kv[table[0, j // page], 0, :, j % page] = loud
        kv[table[0, j // page], 1, :, j % page] = 1.0
        kv = kv.to(device, dtype)
        q = torch.zeros(n, hq, d)
        q[:, :, 0] = 4.0
        sinks = torch.zeros(hq, device=device)
        see = torch.tensor([oracle.chunk_visible(i, j, chunk) for i in range(n)])
        meta = build_step_meta([n], [0], table, page, device=device)
        out = ops.paged_attention(q.to(device, dtype), kv, meta, 1.0, None, sinks, chunk=chunk).float().cpu()
        assert torch.allclose(out[:, 0, 0], see.float(), atol=2e-2), (chunk, j)
        for i in {j, j + 1, n - 1, (j // chunk + 1) * chunk - 1, (j // chunk + 1) * chunk} & set(range(n)):
            meta = build_step_meta([1], [i], table, page, device=device)
            o = ops.paged_attention(q[:1].to(device, dtype), kv, meta, 1.0, None, sinks, chunk=chunk).float().cpu()
            assert abs(float(o[0, 0, 0]) - float(see[i])) < 2e-2, (chunk, j, i)


def test_zero_sink_keeps_a_share():
    """A lone key with score s gets exp(s) / (1 + exp(s)) of the weight, not all of it."""
    kv = torch.zeros(1, 2, 1, 64, 64)
    kv[:, 0, :, 0, 0], kv[:, 1] = 1.0, 1.0
    meta = build_step_meta([1], [0], torch.zeros(1, 1, dtype=torch.int32), 64)
    for s in (-2.0, 0.0, 3.0):
        q = torch.zeros(1, 1, 64)
        q[0, 0, 0] = s
        o = ops.paged_attention(q, kv, meta, 1.0, None, torch.zeros(1), chunk=8)
        assert abs(float(o[0, 0, 0]) - math.exp(s) / (1 + math.exp(s))) < 1e-6


def mlstm_case(device, dtype, heads, dk, dv, cap, lens, kernel=None, past=None, hot=None):
    """Packed rows for :func:`ops.mlstm` at padded sizes and the recurrence of the oracle over the same numbers, in two halves when
    ``past`` splits them.  ``hot``: a token whose input gate is wide open (its key must dominate what follows)."""
    from tensorrt_edge_llm_b200.config import MlstmConfig
    mc = MlstmConfig(heads, dk, dv, cap)
    kp, vp, t = mc.k_pad, mc.v_pad, sum(lens)
    g = torch.Generator().manual_seed(7)
    rows = torch.zeros(t, 2 * heads * (kp + vp))
    q, k = (rows[:, i * heads * kp:(i + 1) * heads * kp].view(t, heads, kp) for i in range(2))
    v, gate = (rows[:, heads * (2 * kp + i * vp):heads * (2 * kp + (i + 1) * vp)].view(t, heads, vp) for i in range(2))
    for x, n in ((q, dk), (k, dk), (v, dv), (gate, dv)):
        x[:, :, :n] = torch.randn(t, heads, n, generator=g)
    pre = torch.randn(t, 2 * heads, generator=g) * 2
    pre[:, heads:] += 3
    if hot is not None:
        pre[hot, :heads] = 50.0
    rows = rows.to(dtype)
    norm = torch.zeros(heads * vp)
    norm.view(heads, vp)[:, :dv] = torch.randn(heads, dv, generator=g) * 0.2 + 1
    want, r0 = [], 0
    f = lambda x: x.to(dtype).double()
    log_i, log_f = oracle.soft_cap(pre[:, :heads].double(), cap), torch.nn.functional.logsigmoid(oracle.soft_cap(pre[:, heads:].double(), cap))
    for n in lens:
        o = torch.stack([oracle.mlstm_recurrence(f(q[r0:r0 + n, h, :dk]) * dk ** -0.5, f(k[r0:r0 + n, h, :dk]), f(v[r0:r0 + n, h, :dv]),
                                                 log_i[r0:r0 + n, h], log_f[r0:r0 + n, h]) for h in range(heads)], 1)
        o = oracle.rms_norm(o, 1.0, 1e-6) * norm.view(heads, vp)[:, :dv].double() * torch.sigmoid(f(gate[r0:r0 + n, :, :dv]))
        want.append(o)
        r0 += n
    state = torch.full((6, heads, kp, vp), 9.0, device=device)          # rows hold leftovers of earlier requests
    nstate = torch.full((6, heads, kp + 1), 9.0, device=device)
    slots = [4, 1, 3, 0][:len(lens)]
    table = torch.zeros(len(lens), 1, dtype=torch.int32)
    kw = {} if kernel is None else {"kernel": kernel}
    fn = ops.mlstm if kernel is None else ops.cuda_ops().mlstm
    rows, pre, norm = rows.to(device), pre.to(device), norm.to(device)
    starts = [sum(lens[:i]) for i in range(len(lens))]
    cuts = [[0] * len(lens), lens] if past is None else [[0] * len(lens), past, lens]
    got = torch.zeros(t, heads * vp)
    for lo, hi in zip(cuts, cuts[1:]):
        idx = torch.cat([torch.arange(s + a, s + b) for s, a, b in zip(starts, lo, hi)]).to(device)
        meta = build_step_meta([b - a for a, b in zip(lo, hi)], lo, table, 64, slot_ids=slots, device=device)
        out = fn(rows[idx].contiguous(), pre[idx].contiguous(), norm, state, nstate, meta, dk ** -0.5, cap, 1e-6, dv, **kw)
        got[idx.cpu()] = out.float().cpu()
    got = got.view(t, heads, vp)
    assert float(got[:, :, dv:].abs().max()) == 0.0 if vp > dv else True
    w = torch.cat(want)
    return float((got[:, :, :dv].double() - w).pow(2).mean().sqrt() / w.std())


@pytest.mark.parametrize("shape", [(2, 40, 24, 9.0), (1, 64, 130, 4.0), (2, 130, 64, 15.0)])
def test_mlstm_recurrence(shape):
    assert mlstm_case("cpu", torch.float32, *shape, [9, 1, 4], past=[5, 1, 2], hot=3) < 1e-5


# ---- the model through the runner --------------------------------------------------------------------------


@pytest.mark.parametrize("name", sorted(cases.CONFIGS))
def test_prompt_in_one_step_and_layer_taps(name, ckpt):
    r = cases.make_runner(ckpt(name), "cpu", "float32")
    assert cases.replay(r, name, 1.0, {"a": (90, 1)}, [[("a", 90)]]) < cases.TOL["float32"]
    cfg, w = cases.weights(name)
    trace = []
    toks = list(cases.prompt(cfg["vocab"], 90, 1))
    oracle.forward(cfg, w, toks, trace)
    meta = r._meta([0], [90])
    _, taps = r.model.hidden_states(torch.tensor(toks, dtype=torch.int32), meta, r.cache, capture_layers=range(len(trace)))
    assert len(taps) == len(trace)
    for a, b in zip(taps, trace):
        assert float((a.double() - b).abs().max() / b.abs().max()) < 1e-4


@pytest.mark.parametrize("sharp", [1.0, 3.0])
@pytest.mark.parametrize("name", sorted(cases.CONFIGS))
def test_portions_and_decoding(name, sharp, ckpt):
    r = cases.make_runner(ckpt(name, sharp), "cpu", "float32")
    n = 150
    for sizes in ([64, 40, 1], [2, 3, 37], [24, 40]):
        steps = [[("a", c)] for c in cases.portions(n, sizes)]
        assert cases.replay(r, name, sharp, {"a": (n, 2)}, steps) < cases.TOL["float32"], sizes
    steps = [[("a", 1)] for _ in range(n)]
    assert cases.replay(r, name, sharp, {"a": (n, 2)}, steps) < cases.TOL["float32"]


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
    cfg, w = cases.weights("loop_all")
    a, b = (list(cases.prompt(cfg["vocab"], n, s)) for n, s in ((70, 1), (30, 2)))
    lines = [{"step": 0, "entries": [{"id": "a", "tokens": a[:50], "want": [0, 49]}, {"id": "b", "tokens": b[:3], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[3:], "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[50:], "want": [19]}], "end": ["a"]}]
    out = tmp_path / "out"
    out.mkdir()
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", ckpt("loop_all"), "--dtype", "float32", "--out", str(out), "--max-tokens",
                        "192", "--device", "cpu"], input="\n".join(json.dumps(x) for x in lines), capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr
    assert [x for x in p.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    assert sorted(os.listdir(out)) == ["0.f32", "2.f32"]
    want = oracle.forward(cfg, w, a)
    for f, rows in (("0.f32", [0, 49]), ("2.f32", [69])):
        got = torch.frombuffer(bytearray((out / f).read_bytes()), dtype=torch.float32).view(len(rows), cfg["vocab"])
        assert cases.error(got, want[rows]) < cases.TOL["float32"]
    req = tmp_path / "req.json"
    req.write_text(json.dumps({"temperature": 0.0, "max_generate_length": 3, "requests": [{"input_ids": a[:20]}]}))
    p = subprocess.run([sys.executable, "-m", "tensorrt_edge_llm_b200.cli", "infer", ckpt("loop_all"), "--input-file", str(req), "--output-file",
                        str(tmp_path / "res.json"), "--device", "cpu", "--dtype", "float32"], capture_output=True, text=True, timeout=300, cwd=ROOT)
    assert p.returncode == 0, p.stderr
    assert json.loads((tmp_path / "res.json").read_text())["responses"][0]["output_ids"] == oracle.greedy(cfg, w, a[:20], 3)


def test_parallel_and_quantised_deployments_are_refused():
    from tensorrt_edge_llm_b200.model import AutoModel
    cfg = ModelConfig.from_hf_dict(cases.CONFIGS["mixed"]())
    with pytest.raises((NotImplementedError, ValueError)):
        AutoModel.from_config(cfg.for_rank(0, 2))
