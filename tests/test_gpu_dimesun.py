"""Dimesun family on the GPU: every kernel against the plain statement, then whole models in bf16 and in true fp32."""
import pytest
import torch

import dimesun_cases as cases
import dimesun_oracle as oracle
from test_dimesun_cpu import cases_edges, mlstm_case

pytestmark = pytest.mark.gpu
DEV = "cuda"
DTYPES = {"bfloat16": torch.bfloat16, "float16": torch.float16, "float32": torch.float32}


@pytest.fixture(scope="module")
def ckpt(tmp_path_factory):
    made = {}

    def get(name, sharp=1.0):
        if (name, sharp) not in made:
            made[name, sharp] = cases.save_checkpoint(tmp_path_factory.mktemp(name), *cases.weights(name, sharp))
        return made[name, sharp]
    return get


@pytest.fixture(autouse=True)
def no_timed_out_waits():
    yield
    from tensorrt_edge_llm_b200.ops import cuda as cu
    cu.Workspace.get(torch.device(DEV, torch.cuda.current_device())).check_status()


# ---- kernels ------------------------------------------------------------------------------------------------


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("d, hq, hkv", [(64, 2, 1), (128, 4, 2), (128, 3, 1), (256, 2, 2), (320, 2, 1)])
def test_chunked_attention_edges(d, hq, hkv, dtype):
    """Tile, decode and CUDA-core kernels: a loud key is seen exactly inside its block."""
    for chunk in (1, 63, 64, 65, 100, 128):
        cases_edges(chunk, DEV, DTYPES[dtype], d, hq, hkv)


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("hq, hkv, d, dv, chunk", [(8, 2, 128, 128, 70), (6, 2, 48, 32, 40), (5, 1, 96, 128, 1000)])
def test_chunked_attention_values(hq, hkv, d, dv, chunk, dtype):
    """A mixed batch (prompt portions beside single rows) against the softmax of the oracle."""
    from tensorrt_edge_llm_b200 import ops
    from tensorrt_edge_llm_b200.config import AttentionConfig
    from tensorrt_edge_llm_b200.ops.meta import build_step_meta
    dt, pad = DTYPES[dtype], AttentionConfig(hq, hkv, d, dv).pad
    g = torch.Generator().manual_seed(3)
    past, lens = [137, 0, 64], [1, 130, 9]
    table = torch.randperm(12, generator=g)[:9].reshape(3, 3).to(torch.int32)
    kv = torch.zeros(12, 2, hkv, 64, pad)
    kv[:, 0, :, :, :d], kv[:, 1, :, :, :dv] = torch.randn(12, hkv, 64, d, generator=g), torch.randn(12, hkv, 64, dv, generator=g)
    q = torch.zeros(sum(lens), hq, pad)
    q[:, :, :d] = torch.randn(sum(lens), hq, d, generator=g)
    kv, q = kv.to(dt), q.to(dt)
    meta = build_step_meta(lens, past, table, 64, device=DEV)
    got = ops.paged_attention(q.to(DEV), kv.to(DEV), meta, 0.3, None, torch.zeros(hq, device=DEV), chunk=chunk).float().cpu()
    want, r = torch.zeros(sum(lens), hq, dv, dtype=torch.float64), 0
    for s, (p0, n) in enumerate(zip(past, lens)):
        for i in range(p0, p0 + n):
            js = [j for j in range(i + 1) if oracle.chunk_visible(i, j, chunk)]
            for h in range(hq):
                page, off = table[s, [j // 64 for j in js]].long(), torch.tensor([j % 64 for j in js])
                k, v = (kv[page, x, h // (hq // hkv), off].double() for x in (0, 1))
                want[r, h] = oracle.sink_softmax(k @ q[r, h].double() * 0.3) @ v[:, :dv]
            r += 1
    assert float((got[:, :, :dv].double() - want).abs().max()) < (1e-5 if dtype == "float32" else 3e-2)
    if dtype == "bfloat16":
        # with fp32 weights only the result is rounded (a plain 16-bit P·V product misses the rounded value of about half the elements)
        for rows, m in ((slice(0, sum(lens)), meta), (slice(0, 1), build_step_meta([1], past[:1], table[:1], 64, device=DEV))):
            exact = ops.paged_attention(q[rows].to(DEV), kv.to(DEV), m, 0.3, None, torch.zeros(hq, device=DEV), chunk=chunk, fp32_weights=True).cpu()
            same = exact[:, :, :dv] == want[rows].to(torch.bfloat16)
            assert float(same.double().mean()) > 0.97


@pytest.mark.parametrize("kernel", ["chunk", "scan"])
@pytest.mark.parametrize("heads, dk, dv, cap", [(2, 48, 40, 9.0), (1, 128, 128, 15.0), (2, 100, 200, 4.0), (1, 64, 384, 30.0)])
def test_mlstm_prompts(heads, dk, dv, cap, kernel):
    """Ragged prompts over several 128-token chunks, cut in the middle of one, in state rows that held other requests; an early token
    with an open gate stays in the memory."""
    assert mlstm_case(DEV, torch.bfloat16, heads, dk, dv, cap, [300, 17, 129, 1], kernel) < 3e-3
    assert mlstm_case(DEV, torch.bfloat16, heads, dk, dv, cap, [290, 20, 257], kernel, past=[131, 18, 129], hot=5) < 3e-3
    if kernel == "scan":
        assert mlstm_case(DEV, torch.float32, heads, dk, dv, cap, [150, 20], None, past=[131, 19], hot=5) < 2e-5


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("heads, dk, dv", [(2, 48, 40), (3, 128, 128), (1, 200, 300)])
def test_mlstm_decode(heads, dk, dv, dtype):
    tol = 3e-3 if dtype == "bfloat16" else 2e-5
    assert mlstm_case(DEV, DTYPES[dtype], heads, dk, dv, 8.0, [1, 1, 1], "decode") < tol          # first tokens
    assert mlstm_case(DEV, DTYPES[dtype], heads, dk, dv, 8.0, [41, 18], None, past=[40, 17]) < tol


def test_mlstm_chunk_keeps_32_bits_where_it_has_to():
    """State after a prompt: the chunk kernel's split operands against the fp32 walk (a 16-bit rounding of the decays, the gated values
    or the state would show at 1e-3)."""
    from tensorrt_edge_llm_b200.ops import cuda as cu
    from tensorrt_edge_llm_b200.ops.meta import build_step_meta
    g = torch.Generator().manual_seed(1)
    n, d, t = 2, 128, 700
    rows = torch.randn(t, 8 * n * d // 2, generator=g).bfloat16().to(DEV)
    gates = (torch.randn(t, 2 * n, generator=g) * 2 + torch.tensor([0.0] * n + [4.0] * n)).to(DEV)
    meta = build_step_meta([t], [0], torch.zeros(1, 11, dtype=torch.int32), 64, device=DEV)
    out = {}
    for k in ("chunk", "scan"):
        s, m = torch.zeros(1, n, d, d, device=DEV), torch.zeros(1, n, d + 1, device=DEV)
        cu.mlstm(rows, gates, torch.ones(n * d, device=DEV), s, m, meta, d ** -0.5, 15.0, 1e-6, d, kernel=k)
        out[k] = (s, m)
    for a, b in zip(out["chunk"], out["scan"]):
        assert float((a - b).pow(2).mean().sqrt() / b.pow(2).mean().sqrt()) < 2e-5


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("t, width, n", [(1, 64, 5), (9, 72, 131), (130, 256, 8), (700, 136, 300)])
def test_products_with_fp32_results(t, width, n, dtype):
    from tensorrt_edge_llm_b200 import ops
    g = torch.Generator().manual_seed(2)
    x, w, b = torch.randn(t, width, generator=g).to(DTYPES[dtype]), torch.randn(n, width, generator=g).to(DTYPES[dtype]), torch.randn(n, generator=g)
    got = ops.linear_f32(x.to(DEV), w.to(DEV), b.to(DEV))
    want = x.double() @ w.double().T + b.double()
    assert got.dtype == torch.float32 and float((got.cpu().double() - want).abs().max() / want.std()) < 1e-5


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("t, width, e, top, ff", [(3, 72, 5, 5, 40), (200, 256, 64, 8, 64), (65, 192, 33, 1, 136)])
def test_experts_into_the_stream(t, width, e, top, ff, dtype):
    from tensorrt_edge_llm_b200 import ops
    from tensorrt_edge_llm_b200.config import LAYER_ATTENTION, AttentionConfig, LayerConfig, ModelConfig, MoeConfig
    from tensorrt_edge_llm_b200.models.qwen3_moe import GatedExperts
    dt = DTYPES[dtype]
    spec = MoeConfig(e, top, ff, 0.7)
    cfg = ModelConfig(model_type="dimesun", hidden_size=width, num_hidden_layers=1, dtype=dtype, layer_types=[LAYER_ATTENTION],
                      layer_specs=[LayerConfig(LAYER_ATTENTION, AttentionConfig(), None, spec)])
    c = cases.moe(e, top, ff, 0.7)
    w = {k: v.to(dt) for k, v in oracle.random_weights(cases.small_config([("attention", cases.attn_mixer(1, 1, 64), c)], width=width)).items()}
    m = GatedExperts(cfg, spec, "m")
    assert m.load_checkpoint(lambda n: w["l0.mlp.e{}.{}".format(n.split(".")[2], n.split(".")[3][:-5])])
    m = m.to(DEV)
    g = torch.Generator().manual_seed(4)
    x, a, s = torch.randn(t, width, generator=g).to(dt), torch.randn(t, width, generator=g).to(dt), torch.randn(t, width, generator=g)
    z = (x.double() @ w["l0.mlp.router"].double().T + w["l0.mlp.router.b"].double()).float()
    step, nw = torch.randn(width, generator=g), torch.randn(width, generator=g) * 0.2
    y, h = ops.stream_norm(s.to(DEV), nw.to(DEV), 1e-5, delta=a.to(DEV), routed=m(x.to(DEV), z.to(DEV)), mult=0.6, step=step.to(DEV), offset=1.0, dtype=dt)
    want = s.double() + 0.6 * (a.double() + oracle.experts(x.double(), c, {k: v.double() for k, v in w.items()}, "l0.mlp")) + step.double()
    tol = 1e-5 if dtype == "float32" else 1e-2
    assert float((y.cpu().double() - want).abs().max() / want.std()) < tol
    assert float((h.cpu().double() - oracle.rms_norm(want, 1 + nw.double(), 1e-5)).abs().max()) < (5e-5 if dtype == "float32" else 5e-2)


# ---- the model through the runner ---------------------------------------------------------------------------


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(cases.CONFIGS))
def test_prompts_portions_and_decoding(name, dtype, ckpt):
    r = cases.make_runner(ckpt(name), DEV, dtype)
    tol, n = cases.TOL[dtype], 300
    req = {"a": (n, 20)}
    for sizes in ([n], [270, 1], [24, 40, 128], [2, 3, 37]):
        cut = cases.portions(n, sizes) if sizes != [270, 1] else [270] + [1] * 30
        assert cases.replay(r, name, 1.0, req, [[("a", c)] for c in cut]) < tol, sizes


@pytest.mark.parametrize("name", ["mixed", "loop_all", "attention_only"])
def test_sharp_attention_in_prompts_and_decoding(name, ckpt):
    r = cases.make_runner(ckpt(name, 3.0), DEV, "float32")
    req = {"a": (150, 2)}
    for cut in ([150], [1] * 150, cases.portions(150, [2, 3, 37])):
        assert cases.replay(r, name, 3.0, req, [[("a", c)] for c in cut]) < cases.TOL["float32"]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(cases.CONFIGS))
def test_unequal_requests_share_steps_pages_and_slots(name, dtype, ckpt):
    r = cases.make_runner(ckpt(name), DEV, dtype, pages=6, seats=3)
    req = {"a": (130, 3), "b": (1, 4), "c": (25, 5), "d": (90, 6), "e": (66, 7)}
    steps = [[("a", 60), ("b", 1), ("c", 20)], [("c", 1), ("a", 2)], [("d", 33), ("a", 1), ("c", 3)], [("c", 1), ("d", 40), ("a", 66)],
             [("a", 1)], [("d", 17), ("e", 64)], [("e", 2)]]
    for _ in range(2):
        assert cases.replay(r, name, 1.0, req, steps) < cases.TOL[dtype]


def test_batch_and_cut_do_not_change_16_bit_logits_beyond_rounding(ckpt):
    """The same rows alone, cut and beside others, compared with each other."""
    name = "mlstm_only"
    r = cases.make_runner(ckpt(name), DEV, "bfloat16")
    cfg, _ = cases.weights(name)
    p, other = (list(cases.prompt(cfg["vocab"], n, s)) for n, s in ((200, 30), (77, 31)))
    alone = r.step([0], [p], logits_all=True).double().cpu()
    r.kv.free(0)
    parts = [r.step([2, 1], [p[:90], other], logits_all=True)[:90], r.step([2], [p[90:199]], logits_all=True), r.step([2], [p[199:]], logits_all=True)]
    assert float(cases.row_errors(torch.cat(parts), alone).quantile(0.9)) < 2e-2


@pytest.mark.parametrize("mode", ["static", "engine", "engine, no graphs"])
def test_greedy_generation(mode, ckpt):
    """fp32 generation equals the oracle's, token by token, from the static path and from the request engine, captured decode steps
    included (a decode graph's warm-up must leave the recurrent state alone)."""
    from tensorrt_edge_llm_b200.runtime.llm import LLM
    from tensorrt_edge_llm_b200.runtime.runner import SamplingParams
    cfg, w = cases.weights("mixed")
    prompts = [list(cases.prompt(cfg["vocab"], n, n)) for n in (100, 3, 20)]
    kw = {} if mode == "static" else {"enable_in_flight_batching": True, "scheduling": {"mode": "mixed", "max_chunk_tokens": 64, "max_num_tokens": 72}}
    llm = LLM(ckpt("mixed"), device=DEV, dtype="float32", max_batch_size=2, max_input_len=128, max_kv_cache_capacity=192, **kw)
    if "no graphs" in mode:
        llm.runner.use_cuda_graphs = False
    try:
        for p, o in zip(prompts, llm.generate(prompts, SamplingParams(max_tokens=12))):
            assert list(o.token_ids) == oracle.greedy(cfg, w, p, 12)
        if mode == "engine":
            assert llm.session.graph_steps > 0
    finally:
        llm.close()


def test_long_decoding_through_graphs(ckpt):
    """Two hundred decoded tokens across page and chunk borders: captured steps against the eager runner."""
    name = "loop_all"
    cfg, _ = cases.weights(name)
    r = cases.make_runner(ckpt(name), DEV, "float32")
    prompts = [list(cases.prompt(cfg["vocab"], n, n)) for n in (120, 61)]
    first = r.prefill([0, 1], prompts).argmax(-1).to(torch.int32)
    toks = r.decode_greedy([0, 1], first, 200).cpu()
    full = [p + [int(f)] + t.tolist() for p, f, t in zip(prompts, first.cpu(), toks)]
    for s in (0, 1):
        r.kv.free(s)
    for s, f in enumerate(full):
        lg = r.step([s], [f[:-1]], logits_all=True)
        assert lg[-200:].argmax(-1).tolist() == f[-200:]


def test_hybrid_graph_decode_keeps_recurrent_state():
    """The decode graph of the other hybrid stacks: capture must not advance the state either."""
    from tensorrt_edge_llm_b200.config import hybrid_nemotron_config
    from tensorrt_edge_llm_b200.model import AutoModel
    from tensorrt_edge_llm_b200.runtime.kv_cache import KVCacheManager
    from tensorrt_edge_llm_b200.runtime.runner import ModelRunner
    cfg = hybrid_nemotron_config(num_hidden_layers=6, hidden_size=256, intermediate_size=512, vocab_size=512, num_attention_heads=2,
                                 num_key_value_heads=1, dtype="bfloat16")
    model = AutoModel.from_config(cfg, device=DEV, random_init=0)
    r = ModelRunner(model, KVCacheManager(cfg, 8, 64, max_seats=2, max_pages_per_seq=4, device=DEV))
    p = list(range(3, 40))
    first = r.prefill([0], [p]).argmax(-1).to(torch.int32)
    graph = r.decode_greedy([0], first, 6).cpu()
    states = [t[0].clone() for t in r.kv.recurrent.pools()]
    r.kv.free(0)
    r.use_cuda_graphs = False
    r.prefill([0], [p])
    r.decode_greedy([0], first, 1)
    for t in graph[0, :5].tolist():
        r.step([0], [[t]])
    for a, b in zip(states, (t[0] for t in r.kv.recurrent.pools())):
        assert torch.allclose(a.float(), b.float(), atol=1e-3, rtol=1e-2)
