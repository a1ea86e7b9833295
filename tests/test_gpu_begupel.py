"""Begupel family on the GPU: every kernel against the plain statement, then whole models in bf16 and in true fp32."""
import pytest
import torch

import begupel_cases as cases
import begupel_oracle as oracle

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
@pytest.mark.parametrize("width, groups, taps", [(24, 3, 4), (40, 4, 1), (256, 2, 3), (64, 1, 8), (2048, 4, 4), (4096, 32, 5), (5120, 2, 2), (1032, 6, 3)])
def test_stream_conv_and_bigram(width, groups, taps, dtype):
    """Rows of one portion in several blocks, portions shorter than the convolution, single rows; state rows held other requests."""
    tol = (1e-5, 1e-5) if dtype == "float32" else (1e-5, 8e-3)
    assert max(cases.stream_case(DEV, DTYPES[dtype], width, groups, taps, [40, 1, 20], behind=37)) < tol[1]
    for ids in (False, True):
        for lens, past in (([40, 1, 20], None), ([33, 9, 30], [17, 2, 1]), ([2, 2], [1, 1]), ([7, 100, 3], [6, 99, 2])):
            x, h = cases.stream_case(DEV, DTYPES[dtype], width, groups, taps, lens, past, ids=ids)
            assert x < tol[0] and h < tol[1], (ids, lens, x, h)


def test_stream_long_blocks():
    """Enough rows for blocks of 16 and of 32."""
    for n in (3000, 10000):
        assert max(cases.stream_case(DEV, torch.float32, 64, 2, 4, [n, 5, 700], [n - 9, 2, 300])) < 1e-5


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("width, groups", [(128, 1), (768, 3), (2048, 4), (4096, 1)])
def test_stream_many_rows(width, groups, dtype):
    """One row per warp."""
    for behind in (0, 40):
        x, h = cases.stream_case(DEV, DTYPES[dtype], width, groups, 4, [1203, 5], behind=behind)
        assert x < 1e-5 and h < (8e-3 if dtype == "bfloat16" else 1e-5)


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("t, width, groups", [(1, 64, 2), (9, 72, 12), (130, 2048, 4), (3, 5120, 1), (5, 40, 4)])
def test_stream_norms(t, width, groups, dtype):
    from tensorrt_edge_llm_b200 import ops
    g, dt = torch.Generator().manual_seed(1), DTYPES[dtype]
    x, d = torch.randn(t, width, generator=g), (torch.randn(t, width, generator=g) * 3).to(dt)
    w, o = torch.randn(width, generator=g), torch.randn(width, generator=g)
    dev, tol, meta = (lambda v: v.to(DEV)), 1e-5 if dtype == "float32" else 3e-2, cases._meta([0], [t], None, DEV)
    want = x.double() + oracle.group_norm(d.double(), w.double(), groups, 1e-3)
    y, h = ops.stream_post(dev(x), dev(d), dev(w), groups, 1e-3, meta, dt)
    assert torch.allclose(y.cpu().double(), want, atol=1e-5) and torch.allclose(h.cpu().double(), want, atol=tol, rtol=tol)
    y, h = ops.stream_post(dev(x), dev(d), dev(w), groups, 1e-3, meta, dt, out_norm=dev(o))
    assert torch.allclose(y.cpu().double(), want, atol=1e-5)
    assert torch.allclose(h.cpu().double(), oracle.group_norm(want, o.double(), groups, 1e-3), atol=tol, rtol=tol)


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_glu_and_softcap(dtype):
    from tensorrt_edge_llm_b200 import ops
    x = (torch.randn(37, 2 * 192, generator=torch.Generator().manual_seed(2)) * 2).to(DTYPES[dtype])
    tol = 1e-5 if dtype == "float32" else 2e-2
    want = torch.relu(x[:, :192].double()) * x[:, 192:].double()
    assert torch.allclose(ops.glu(x.to(DEV), "relu").cpu().double(), want, atol=tol, rtol=tol)
    y = x.float() * 20
    assert torch.allclose(ops.softcap_(y.to(DEV), 7.0).cpu().double(), oracle.softcap(y.double(), 7.0), atol=1e-5)


HEADS = [(8, 2, 128, 128, 96), (6, 2, 48, 24, 32), (3, 3, 24, 80, 8), (2, 1, 200, 136, 128), (16, 1, 64, 64, 32), (20, 4, 128, 72, 64)]


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("window", [1, 37, 64, 129, 1000])
@pytest.mark.parametrize("hq, hkv, d, dv, dims", HEADS)
def test_windowed_attention_with_rotated_values(hq, hkv, d, dv, dims, window, dtype):
    """Prompts, portions behind a past, single rows far behind the window's start; page and tile borders."""
    tol = 4e-2 if dtype == "bfloat16" else 2e-4
    for lens, past in (([210, 3, 1], [0, 207, 230]), ([1, 1], [400, 64]), ([2, 130], [129, 64])):
        assert cases.attention_case(DEV, DTYPES[dtype], hq, hkv, d, dv, window, dims, lens, past, factor=2.5) < tol, (lens, past)


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("needle", [0, 63, 64, 127, 200])
@pytest.mark.parametrize("hq, hkv, d, dv, dims", HEADS)
def test_needle_at_the_edges_of_windows(hq, hkv, d, dv, dims, needle, dtype):
    """One key far above all others: seen by the last row that may, and not by the next one; in prompts, portions and decoding."""
    tol = 6e-2 if dtype == "bfloat16" else 1e-3
    for window in (40, 64, 130):
        for lens, past in (([300, 70], [0, 0]), ([1, 1, 1], [needle + window - 1, needle + window, needle + window - 2]),
                           ([2, 3], [needle + window - 1, needle]), ([130, 1], [needle + window - 100, 300])):
            if min(past) >= 0:
                assert cases.attention_case(DEV, DTYPES[dtype], hq, hkv, d, dv, window, dims, lens, past, needle=needle) < tol, (window, lens, past)


DELTA = [(4, 2, 40, 24, 3), (1, 1, 16, 16, 1), (3, 3, 128, 128, 4), (2, 1, 136, 200, 8), (8, 8, 64, 128, 2)]


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("shape", DELTA)
def test_delta_with_head_decays(shape, dtype):
    """Ragged prompts, cut in the middle, in state rows that held other requests; a value written early stays in the memory; decoding."""
    tol = 6e-3 if dtype == "bfloat16" else 2e-5
    run = lambda *a, **k: cases.delta_case(DEV, DTYPES[dtype], *shape, *a, **k)
    assert run([150, 17, 65, 2]) < tol
    assert run([150, 20, 75], past=[71, 18, 74]) < tol
    assert run([90, 90], keep=3) < tol
    assert run([1, 1, 1]) < tol                                                                       # first tokens
    assert run([41, 18, 2], past=[40, 17, 1]) < tol
    if max(shape[2:4]) <= 128:
        assert run([41, 18, 2], past=[40, 17, 1], kernel="walk") < tol


def test_delta_slices():
    """Many (sequence, head) pairs take wider column slices per warp: the same numbers."""
    assert cases.delta_case(DEV, torch.bfloat16, 48, 48, 128, 128, 4, [20] * 4) < 6e-3
    assert cases.delta_case(DEV, torch.float32, 48, 24, 128, 128, 4, [9, 30, 2], past=[4, 20, 1]) < 2e-5


LIGHTNING = [(3, 24, 40), (1, 72, 136), (4, 64, 128), (2, 128, 128), (2, 200, 264), (16, 128, 128)]


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("shape", LIGHTNING)
def test_lightning_prompts(shape, dtype):
    """Ragged prompts and portions; constant, forgetting and everything between; an early row that has to be carried along.  The state is
    fp32 whatever the rows are: it agrees with the plain memory over the same rows."""
    tol = 1e-2 if dtype == "bfloat16" else 2e-5

    def run(*a, **k):
        out, state = cases.lightning_case(DEV, DTYPES[dtype], *shape, *a, **k)
        assert out < tol and state < 2e-5, (a, k, out, state)
    run([150, 17, 300, 2])
    run([150, 20, 275], past=[71, 18, 130])
    run([290, 129], loud=3, decay=[0.999] * shape[0])
    run([140, 260], past=[128, 129], decay=([0.0, 1.0, 0.5, 0.97] * 4)[:shape[0]])


@pytest.mark.parametrize("shape", [s for s in LIGHTNING if s[1] <= 128])
def test_lightning_segments(shape):
    """Long sequences cut into segments that run side by side: the same numbers, also where sequences end inside an early segment."""
    lens, past = [1000, 130, 2, 513], [300, 1, 1, 128]
    for segs in ((1, 8), (8, 1), (4, 2), (3, 3)):
        for kw in (dict(), dict(past=past), dict(loud=3, decay=[0.9995] * shape[0])):
            out, state = cases.lightning_case(DEV, torch.bfloat16, *shape, lens, kernel="chunk", segments=segs, **kw)
            assert out < 1e-2 and state < 2e-5, (segs, kw, out, state)


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("shape", LIGHTNING)
def test_lightning_decoding(shape, dtype):
    tol = 1e-2 if dtype == "bfloat16" else 2e-5
    for lens, past in (([1, 1, 1], None), ([141, 18, 2], [140, 17, 1]), ([30, 18], [15, 17])):
        out, state = cases.lightning_case(DEV, DTYPES[dtype], *shape, lens, past)
        assert out < tol and state < 2e-5, (lens, past, out, state)
    if dtype == "bfloat16":
        assert max(cases.lightning_case(DEV, DTYPES[dtype], *shape, [40, 33], kernel="walk")) < tol


# ---- the model through the runner ---------------------------------------------------------------------------


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(cases.CONFIGS))
def test_prompts_portions_and_decoding(name, dtype, ckpt):
    r = cases.make_runner(ckpt(name), DEV, dtype)
    tol, n = cases.TOL[dtype], 300
    for sizes in ([n], [270, 1], [24, 40, 128], [2, 3, 37]):
        cut = cases.portions(n, sizes) if sizes != [270, 1] else [270] + [1] * 30
        assert cases.replay(r, name, 1.0, {"a": (n, 20)}, [[("a", c)] for c in cut]) < tol, sizes


@pytest.mark.parametrize("name", ["mixed", "wide", "long"])
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
    """Two hundred decoded tokens across page borders and past the windows: captured steps, then the same tokens through one eager step."""
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
