"""Ditenex family on the GPU: every kernel against the plain statement, then whole models in bf16 and in true fp32."""
import pytest
import torch

import ditenex_cases as cases
import ditenex_oracle as oracle

pytestmark = pytest.mark.gpu
DEV = "cuda"
DTYPES = {"bfloat16": torch.bfloat16, "float32": torch.float32}


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
@pytest.mark.parametrize("width", [24, 40, 520, 1032, 2048, 4096, 5120])
def test_stream_norms_and_token_shift(width, dtype):
    """Rows of one portion in several blocks, portions of one and two rows; state rows held other requests."""
    tol = 1e-5 if dtype == "float32" else 8e-3
    for kw in (dict(), dict(top=3), dict(top=2, dense=False), dict(ids=True)):
        for lens, past in (([40, 1, 20], None), ([33, 9, 30], [17, 2, 1]), ([2, 2], [1, 1]), ([7, 100, 3], [6, 99, 2])):
            x, h = cases.sandwich_case(DEV, DTYPES[dtype], width, lens, past, **kw)
            assert x < 1e-5 and h < tol, (kw, lens, x, h)
    x, h = cases.sandwich_case(DEV, DTYPES[dtype], width, [9, 40], shift=False, top=2)
    assert x < 1e-5 and h < tol


def test_stream_long_blocks():
    """Enough rows for longer blocks and for a warp per block, sequences that start inside another one's range."""
    for width in (1024, 1536, 2048, 2056):
        for kw in (dict(), dict(top=5), dict(top=2, dense=False), dict(ids=True), dict(shift=False), dict(shift=False, top=4)):
            x, h = cases.sandwich_case(DEV, torch.bfloat16, width, [1300, 5, 700, 3], [1290, 2, 90, 1], **kw)
            assert x < 1e-5 and h < 8e-3, (width, kw)
            assert cases.sandwich_case(DEV, torch.bfloat16, width, [1300, 5, 700, 3], **kw)[0] < 1e-5
    for n in (900, 5000):
        for kw in (dict(), dict(shift=False)):
            assert max(cases.sandwich_case(DEV, torch.float32, 64, [n, 5, 700, 3], [n - 9, 2, 300, 1], **kw)) < 1e-5
            assert max(cases.sandwich_case(DEV, torch.float32, 64, [n, 5, 700, 3], **kw)) < 1e-5


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_activations(dtype):
    from tensorrt_edge_llm_b200 import ops
    x = (torch.randn(37, 192, generator=torch.Generator().manual_seed(2)) * 4).to(DTYPES[dtype])
    coef = torch.tensor([float(oracle.softplus(torch.tensor(0.7).double())), 0.5 + float(oracle.softplus(torch.tensor(-0.4).double()))])
    want = oracle.xielu(x.double(), torch.tensor(0.7).double(), torch.tensor(-0.4).double())
    tol = 2e-6 if dtype == "float32" else 1e-2
    assert torch.allclose(ops.xielu(x.to(DEV), coef.to(DEV)).cpu().double(), want, atol=tol, rtol=tol)
    g, u = x.double().chunk(2, -1)
    assert torch.allclose(ops.glu(x.to(DEV), "silu").cpu().double(), g * torch.sigmoid(g) * u, atol=tol, rtol=tol)


@pytest.mark.parametrize("experts, top, groups, keep", [(8, 2, 2, 1), (9, 3, 3, 2), (64, 8, 8, 3), (6, 1, 6, 2), (5, 5, 1, 1), (160, 6, 32, 4)])
def test_router(experts, top, groups, keep):
    """Choice scores are negative, so a closed group must count as minus infinity."""
    from tensorrt_edge_llm_b200 import ops
    g = torch.Generator().manual_seed(4)
    z, corr = torch.randn(130, experts, generator=g) * 3, torch.randn(experts, generator=g) * 0.3 - 2.0
    w, idx = ops.moe_route_sigmoid_groups(z.to(DEV), corr.to(DEV), top, groups, keep, 1.7)
    s = torch.sigmoid(z.double())
    for t in range(z.shape[0]):
        want = oracle.chosen_experts(s[t] + corr.double(), top, groups, keep)
        assert idx[t].tolist() == want
        assert torch.allclose(w[t].cpu().double(), s[t, want] * 1.7, rtol=1e-5)


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("tokens", [1, 33, 400])
def test_experts(tokens, dtype):
    from tensorrt_edge_llm_b200.config import ModelConfig
    from tensorrt_edge_llm_b200.models.qwen3_moe import SharedExpertsBlock
    f, d = cases.moe(6, 3, 40, 3, 2, 1.7, 48), 72
    cfg = ModelConfig.from_hf_dict(cases.small_config([(cases.attn(2, 1, 16, 16, 8), f)], width=d))
    cfg.dtype = dtype
    w = {k: v for k, v in cases.random_weights(cases.small_config([(cases.attn(2, 1, 16, 16, 8), f)], width=d), 3).items() if ".mlp." in k}
    block = SharedExpertsBlock(cfg, cfg.layer_specs[0].moe, "m")
    block.router.load_from([{"weight": w["l0.mlp.router"]}])
    block.routed.correction.copy_(w["l0.mlp.correction"].float())
    block.routed.load_checkpoint(lambda n: w["l0.mlp.e{}.{}".format(n.split(".")[2], n.split(".")[3][:-5])])
    block.shared.gate_up_proj.load_from([{"weight": w[f"l0.mlp.shared.{n}"]} for n in ("gate", "up")])
    block.shared.down_proj.load_from([{"weight": w["l0.mlp.shared.down"]}])
    x = torch.randn(tokens, d, generator=torch.Generator().manual_seed(1)).to(DTYPES[dtype])
    shared, routed = block.to(DEV)(x.to(DEV))
    rows = routed.ws.dst_row.view(tokens, -1).long()
    got = shared.double() + (routed.y.double()[rows] * routed.weights.double()[:, :, None]).sum(1)
    want = oracle.feed_forward(x.double(), f, {k: v.double() for k, v in w.items()}, "l0.mlp")
    err = (got.cpu() - want).pow(2).mean(-1).sqrt() / want.std()
    assert float(err.max() if dtype == "float32" else err.quantile(0.9)) < (1e-5 if dtype == "float32" else 2e-2)


HEADS = [(16, 4, 128, 128), (6, 2, 40, 56), (3, 3, 24, 24), (2, 1, 200, 136), (8, 1, 64, 64), (20, 4, 128, 72), (12, 3, 16, 24), (5, 5, 64, 32), (4, 4, 128, 128),
         (33, 1, 100, 128), (2, 2, 128, 16)]


def attention_tol(kv, d, dv, dtype):
    """Prompts of heads with more than 256 key features side by side round their mixed queries once to 16 bits."""
    if dtype == "float32":
        return 1e-4
    return 2e-2 if kv * (64 if max(d, dv) <= 64 else 128 if max(d, dv) <= 128 else 256) <= 256 else 3e-2


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("window", [1, 37, 64, 129, 1000])
@pytest.mark.parametrize("heads, kv, d, dv", HEADS)
def test_mixed_attention(heads, kv, d, dv, window, dtype):
    """Prompts, portions behind a past, single rows far behind the window's start, prompts beside single rows; page and tile borders."""
    tol = attention_tol(kv, d, dv, dtype)
    for lens, past in (([210, 3, 1], [0, 207, 230]), ([1, 1], [400, 64]), ([2, 130], [129, 64]), ([300, 257], [0, 0])):
        assert cases.attention_case(DEV, DTYPES[dtype], heads, kv, d, dv, window, lens, past) < tol, (lens, past)
    assert cases.attention_case(DEV, DTYPES[dtype], heads, kv, d, dv, window, [70, 1], [0, 90], join=False, gate=False) < tol


@pytest.mark.parametrize("heads, kv, d, dv", [h for h in HEADS if max(h[2:]) <= 128])
def test_mixed_attention_kernels_agree(heads, kv, d, dv):
    """Every kernel, tile and number of splits on the same steps."""
    for window in (40, 150):
        for lens, past in (([1, 1, 1], [400, 64, 0]), ([3, 1], [130, 62]), ([9, 30], [120, 0])):
            for kw in (dict(kernel="decode", tile=64, splits=1), dict(kernel="decode", tile=128, splits=1), dict(kernel="decode", tile=64, splits=5),
                       dict(kernel="decode", tile=128, splits=3), dict(kernel="decode", tile=64, splits=33), dict(kernel="simt")):
                assert cases.attention_case(DEV, torch.bfloat16, heads, kv, d, dv, window, lens, past, **kw) < (3e-2 if kw["kernel"] == "simt" else 1.5e-2), (window, lens, kw)
        if kv * (64 if max(d, dv) <= 64 else 128) <= 256:
            for lens, past in (([1, 1, 1], [400, 64, 0]), ([3, 140], [130, 62])):
                assert cases.attention_case(DEV, torch.bfloat16, heads, kv, d, dv, window, lens, past, kernel="prefill") < 1.5e-2


@pytest.mark.parametrize("lens, past", [([1, 2], [200, 100]), ([150, 40], [0, 70])])
def test_mixed_queries_keep_fp32_precision(lens, past):
    """Large scores: one 16-bit rounding of the mixed queries would show."""
    assert cases.attention_case(DEV, torch.bfloat16, 8, 2, 128, 128, 300, lens, past, loud=12.0, gate=False) < 6e-3


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("needle", [0, 63, 64, 127, 200])
@pytest.mark.parametrize("heads, kv, d, dv", HEADS[:8])
def test_needle_at_the_edges_of_windows(heads, kv, d, dv, needle, dtype):
    """One key far above all others: seen by the last row that may, and not by the next one; in prompts, portions and decoding."""
    tol = 10 * attention_tol(kv, d, dv, dtype) if dtype == "float32" else attention_tol(kv, d, dv, dtype)
    for window in (40, 64, 130):
        for lens, past in (([300, 70], [0, 0]), ([1, 1, 1], [needle + window - 1, needle + window, needle + window - 2]),
                           ([2, 3], [needle + window - 1, needle]), ([130, 1], [needle + window - 100, 300])):
            if min(past) >= 0:
                assert cases.attention_case(DEV, DTYPES[dtype], heads, kv, d, dv, window, lens, past, needle=needle) < tol, (window, lens, past)


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
        assert cases.replay(r, name, 4.0, {"a": (150, 2)}, [[("a", c)] for c in cut]) < 3 * cases.TOL["float32"]


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
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_long_decoding_through_graphs(name, dtype, ckpt):
    """Two hundred decoded tokens across page borders and past the windows: captured steps, then the same tokens through one eager step."""
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
        err = cases.row_errors(got, want)
        assert float(err.max() if dtype == "float32" else err.quantile(0.9)) < cases.TOL[dtype]
        lo = len(prompts[n]) - 1
        picked = want[lo:-1].gather(1, torch.tensor(p[lo + 1:])[:, None])[:, 0]
        short = (want[lo:-1].max(-1).values - picked) / want.std()
        assert float(short.max() if dtype == "float32" else short.quantile(0.9)) < 4 * cases.TOL[dtype]     # greedy up to rounding
