"""Debonex family on the GPU: every kernel against the plain statement, then whole models in bf16 and in true fp32."""
import pytest
import torch

import debonex_cases as cases
import debonex_oracle as oracle

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
@pytest.mark.parametrize("t, width", [(1, 64), (9, 72), (130, 2048), (3, 5120)])
def test_tanh_norm_and_stream(t, width, dtype):
    from tensorrt_edge_llm_b200 import ops
    dt, g = DTYPES[dtype], torch.Generator().manual_seed(1)
    table, ids = torch.randn(50, width, generator=g).to(dt), torch.randint(0, 50, (t,), generator=g)
    a, w, b, alpha = torch.randn(t, width, generator=g).to(dt), torch.randn(width, generator=g), torch.randn(width, generator=g), torch.tensor(0.6)
    dev = lambda x: x.to(DEV)
    x, h0 = ops.stream_norm(None, dev(w), 1e-5, ids=dev(ids), table=dev(table), table_mult=3.0, alpha=dev(alpha), bias=dev(b), dtype=dt)
    y, h1 = ops.stream_norm(x, dev(w), 1e-5, delta=dev(a), alpha=dev(alpha), bias=dev(b), dtype=dt)
    s = table[ids].double() * 3
    n = {"n": w.double(), "n.b": b.double(), "n.alpha": alpha.double()}
    tol = 1e-5 if dtype == "float32" else 3e-2
    assert torch.allclose(x.cpu().double(), s, atol=1e-5) and torch.allclose(y.cpu().double(), s + a.double(), atol=1e-5)
    assert torch.allclose(h0.cpu().double(), oracle.dynamic_tanh(s, n, "n"), atol=tol, rtol=tol)
    assert torch.allclose(h1.cpu().double(), oracle.dynamic_tanh(s + a.double(), n, "n"), atol=tol, rtol=tol)


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_geglu(dtype):
    from tensorrt_edge_llm_b200 import ops
    x = (torch.randn(37, 2 * 192, generator=torch.Generator().manual_seed(2)) * 2).to(DTYPES[dtype])
    want = oracle.gelu_tanh(x[:, :192].double()) * x[:, 192:].double()
    assert torch.allclose(ops.geglu(x.to(DEV)).cpu().double(), want, atol=1e-5 if dtype == "float32" else 2e-2, rtol=1e-5 if dtype == "float32" else 1e-2)


SHAPES = [(4, 2, 40, 24, 3), (1, 1, 16, 16, 1), (3, 3, 128, 128, 4), (2, 1, 136, 200, 8), (8, 8, 64, 128, 2)]


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("shape", SHAPES)
def test_channel_delta_prompts(shape, dtype):
    """Ragged prompts, cut in the middle, in state rows that held other requests; a value written early stays in the memory."""
    tol = 6e-3 if dtype == "bfloat16" else 2e-5
    assert cases.delta_case(DEV, DTYPES[dtype], *shape, [150, 17, 65, 2]) < tol
    assert cases.delta_case(DEV, DTYPES[dtype], *shape, [150, 20, 75], past=[71, 18, 74]) < tol
    assert cases.delta_case(DEV, DTYPES[dtype], *shape, [90, 90], keep=3) < tol


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("shape", SHAPES)
def test_channel_delta_decoding(shape, dtype):
    tol = 6e-3 if dtype == "bfloat16" else 2e-5
    assert cases.delta_case(DEV, DTYPES[dtype], *shape, [1, 1, 1]) < tol                              # first tokens
    assert cases.delta_case(DEV, DTYPES[dtype], *shape, [41, 18, 2], past=[40, 17, 1]) < tol


@pytest.mark.parametrize("heads", [16, 48])
def test_channel_delta_slices(heads):
    """Many (sequence, head) pairs take wider column slices per warp: the same numbers."""
    assert cases.delta_case(DEV, torch.bfloat16, heads, heads, 128, 128, 4, [20] * 4) < 6e-3
    assert cases.delta_case(DEV, torch.float32, heads, heads, 128, 128, 4, [9, 30, 1], past=[4, 20, 0]) < 2e-5


LATENT = [(16, 128, 64, 128, 512), (3, 40, 24, 56, 72), (5, 64, 32, 64, 192), (40, 64, 64, 128, 256), (2, 200, 8, 96, 64)]


@pytest.mark.parametrize("kernel", ["folded", "folded-64", "folded-128", "expanded", "simt"])
@pytest.mark.parametrize("heads, dim, rot, dv, rank", LATENT)
def test_latent_attention_kernels(heads, dim, rot, dv, rank, kernel):
    """Both tensor-core forms and the CUDA-core one: prompts, portions behind a past, page borders, single rows."""
    tol = 4e-2
    for lens, past in (([300, 1, 65], [0, 0, 0]), ([2, 130, 9], [129, 64, 1]), ([1, 1, 1], [127, 128, 400])):
        if kernel == "expanded" and max(lens) == 1:
            continue
        assert cases.latent_case(DEV, torch.bfloat16, heads, dim, rot, dv, rank, lens, past, kernel) < tol, (lens, past)


@pytest.mark.parametrize("needle", [0, 63, 64, 127, 128, 255])
@pytest.mark.parametrize("kernel", ["folded-64", "folded-128"])
def test_latent_needle_in_tiles(needle, kernel):
    for past in ([needle, 700, 256], [needle + 1, 129, 383]):
        assert cases.latent_case(DEV, torch.bfloat16, 4, 64, 32, 64, 128, [1, 3, 2], past, kernel, needle=needle) < 8e-2


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("needle", [0, 63, 64, 128, 255])
def test_latent_needle(needle, dtype):
    """One key far above all others, at page and tile borders and first: seen by every later row, near and far, and by no earlier one."""
    tol = 8e-2 if dtype == "bfloat16" else 1e-3
    for lens, past in (([300, 70], [0, 0]), ([1, 1, 2], [700, needle, 256]), ([130, 1, 4], [needle, 300, 64])):
        assert cases.latent_case(DEV, DTYPES[dtype], 4, 64, 32, 64, 128, lens, past, needle=needle) < tol


def test_latent_mixed_step_and_other_sizes():
    """Prompt portions beside single rows in one step (both forms in one call), fp32 and fp16 rows, a value size beyond the expanded form."""
    for dt, tol in ((torch.bfloat16, 4e-2), (torch.float16, 1e-2), (torch.float32, 2e-4)):
        assert cases.latent_case(DEV, dt, 16, 128, 64, 128, 512, [1, 200, 1, 40], [200, 3, 64, 0]) < tol
    assert cases.latent_case(DEV, torch.bfloat16, 2, 64, 32, 192, 128, [150, 1], [0, 30]) < 4e-2


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("loud", [None, 0, 63, 64, 200])
@pytest.mark.parametrize("hq, hkv, d, dv", [(8, 2, 128, 128), (6, 2, 48, 80), (2, 2, 200, 32)])
def test_unit_attention(hq, hkv, d, dv, loud, dtype):
    tol = 4e-2 if dtype == "bfloat16" else 2e-4
    assert cases.unit_case(DEV, DTYPES[dtype], hq, hkv, d, dv, [210, 3, 1], [0, 207, 230], 0.4, 30, loud) < tol
    assert cases.unit_case(DEV, DTYPES[dtype], hq, hkv, d, dv, [1, 1], [300, 201], 0.4, 30, loud) < tol


# ---- the model through the runner ---------------------------------------------------------------------------


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(cases.CONFIGS))
def test_prompts_portions_and_decoding(name, dtype, ckpt):
    r = cases.make_runner(ckpt(name), DEV, dtype)
    tol, n = cases.TOL[dtype], 300
    for sizes in ([n], [270, 1], [24, 40, 128], [2, 3, 37]):
        cut = cases.portions(n, sizes) if sizes != [270, 1] else [270] + [1] * 30
        assert cases.replay(r, name, 1.0, {"a": (n, 20)}, [[("a", c)] for c in cut]) < tol, sizes


@pytest.mark.parametrize("name", ["mixed", "latent", "attention"])
def test_sharp_attention_in_prompts_and_decoding(name, ckpt):
    r = cases.make_runner(ckpt(name, 4.0), DEV, "float32")
    for cut in ([150], [1] * 150, cases.portions(150, [2, 3, 37])):
        assert cases.replay(r, name, 4.0, {"a": (150, 2)}, [[("a", c)] for c in cut]) < cases.TOL["float32"]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(cases.CONFIGS))
def test_unequal_requests_share_steps_pages_and_slots(name, dtype, ckpt):
    r = cases.make_runner(ckpt(name), DEV, dtype, pages=6, seats=3)
    req = {"a": (130, 3), "b": (1, 4), "c": (25, 5), "d": (90, 6), "e": (66, 7)}
    steps = [[("a", 60), ("b", 1), ("c", 20)], [("c", 1), ("a", 2)], [("d", 33), ("a", 1), ("c", 3)], [("c", 1), ("d", 40), ("a", 66)],
             [("a", 1)], [("d", 17), ("e", 64)], [("e", 2)]]
    for _ in range(2):
        assert cases.replay(r, name, 1.0, req, steps) < cases.TOL[dtype]


@pytest.mark.parametrize("mode", ["static", "engine", "engine, no graphs"])
def test_greedy_generation(mode, ckpt):
    """fp32 generation equals the oracle's, token by token, from the static path and from the request engine, captured decode steps
    included."""
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


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_through_graphs(dtype, ckpt):
    """Two hundred decoded tokens across page borders: captured steps, then the same tokens through one eager step."""
    name = "mixed"
    cfg, w = cases.weights(name)
    r = cases.make_runner(ckpt(name), DEV, dtype)
    prompts = [list(cases.prompt(cfg["vocab"], n, n)) for n in (120, 61)]
    first = r.prefill([0, 1], prompts).argmax(-1).to(torch.int32)
    toks = r.decode_greedy([0, 1], first, 200).cpu()
    full = [p + [int(f)] + t.tolist() for p, f, t in zip(prompts, first.cpu(), toks)]
    for s in (0, 1):
        r.kv.free(s)
    for n, p in enumerate(full):
        want = oracle.forward(cfg, w, p)
        got = r.step([0], [p], logits_all=True)
        r.kv.free(0)
        assert cases.error(got, want) < cases.TOL[dtype]
        lo = len(prompts[n]) - 1
        picked = want[lo:-1].gather(1, torch.tensor(p[lo + 1:])[:, None])[:, 0]
        assert float((want[lo:-1].max(-1).values - picked).max() / want.std()) < 4 * cases.TOL[dtype]     # greedy up to rounding
