"""Configurations and checks of the Dimesun family that the CPU and the GPU tests share: a checkpoint is written to disk, loaded through
the registry and driven through the runner in all kinds of portions and batches, and every logit row is compared with the plain
statement in ``dimesun_oracle``."""
import functools
import json
import os

import torch

import dimesun_oracle as oracle
from dimesun_oracle import attn_mixer, mlstm_mixer, moe, small_config

TOL = {"float32": 2e-4, "bfloat16": 4e-2}


def _cfg_mixed():
    """Uneven sizes: padded heads, value heads unlike key heads, partial rotary, three query heads per KV head, a layer without
    experts, layers with KV sizes of their own, a loop over the middle."""
    return small_config([("mlstm", mlstm_mixer(3, 40, 24, cap=9.0), moe(5, 3, 40, 0.8)),
                         ("attention", attn_mixer(6, 2, 48, 32, size=40, rot=32, base=5000.0, scale=0.2), moe(4, 1, 72, 2.0)),
                         ("mlstm", mlstm_mixer(2, 72, 136, cap=4.0), None),
                         ("attention", attn_mixer(4, 4, 80, size=24), None)], width=72, vocab=101, loop=(1, 3, 2), mult=0.4)


def _cfg_loop_all():
    """The whole stack loops; single heads, as many experts used as there are, a chunk that is a multiple of the page."""
    return small_config([("attention", attn_mixer(2, 1, 64, size=128, base=20000.0), moe(3, 3, 64, 1.0)),
                         ("mlstm", mlstm_mixer(1, 64, 128), moe(7, 2, 24, 5.0))], width=128, vocab=64, loop=(0, 2, 3), mult=0.25, eps=1e-6)


def _cfg_attention_only():
    return small_config([("attention", attn_mixer(8, 2, 128, size=70), moe(4, 2, 32, 1.5)),
                         ("attention", attn_mixer(8, 2, 128, size=200, rot=64), None)], width=96, vocab=80, mult=1.0)


def _cfg_mlstm_only():
    """Heads at the kernels' own sizes and beyond one value tile; one pass of a loop still adds its vector."""
    return small_config([("mlstm", mlstm_mixer(2, 128, 256, cap=6.0), moe(6, 2, 64, 1.0)),
                         ("mlstm", mlstm_mixer(2, 128, 128, cap=20.0), None)], width=64, vocab=72, loop=(1, 2, 1), mult=0.5)


CONFIGS = {"mixed": _cfg_mixed, "loop_all": _cfg_loop_all, "attention_only": _cfg_attention_only, "mlstm_only": _cfg_mlstm_only}


@functools.lru_cache(maxsize=None)
def weights(name: str, sharp: float = 1.0):
    """``sharp`` scales queries and keys of the attention layers: one score per row stands out, so a key that is wrongly seen or
    wrongly hidden moves the logits."""
    cfg = CONFIGS[name]()
    w = oracle.random_weights(cfg, seed=sorted(CONFIGS).index(name) + 1)
    if sharp != 1.0:
        for i, l in enumerate(cfg["layers"]):
            if l["type"] == "attention":
                for k in ("q", "k"):
                    w[f"l{i}.mix.{k}"] = (w[f"l{i}.mix.{k}"].float() * sharp).bfloat16()
    return cfg, w


def save_checkpoint(path, cfg, w):
    from tensorrt_edge_llm_b200.checkpoint.safetensors_io import save_file
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file(w, os.path.join(path, "model.safetensors"))
    return str(path)


@functools.lru_cache(maxsize=None)
def prompt(vocab: int, n: int, seed: int):
    return tuple(torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist())


@functools.lru_cache(maxsize=None)
def expected(name: str, sharp: float, n: int, seed: int):
    cfg, w = weights(name, sharp)
    return oracle.forward(cfg, w, list(prompt(cfg["vocab"], n, seed)))


def make_runner(path, device, dtype, pages=24, seats=4):
    from tensorrt_edge_llm_b200.model import AutoModel
    from tensorrt_edge_llm_b200.runtime.kv_cache import KVCacheManager
    from tensorrt_edge_llm_b200.runtime.runner import ModelRunner
    model = AutoModel.from_pretrained(path, device=device, dtype=dtype)
    kv = KVCacheManager(model.cfg, pages, 64, max_seats=seats, max_pages_per_seq=pages, device=device)
    return ModelRunner(model, kv)


def row_errors(got, want):
    """Per row: root mean square of the difference (means taken off) over the scale of the logits."""
    d = got.double().cpu() - want
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / want.std()


def error(got, want):
    return float(row_errors(got, want).max())


def replay(runner, name, sharp, requests, steps):
    """``requests``: id → (length, seed).  ``steps``: lists of (id, count).  Returns the row error that has to stay below the tolerance: the
    worst one in 32 bits; in 16 bits the upper quartile (rounding flips close router decisions, and the recurrent layers carry a flip on)."""
    cfg, _ = weights(name, sharp)
    errs, at, seat_of, free = [], {}, {}, list(range(runner.kv.max_seats - 1, -1, -1))
    for step in steps:
        seats, toks, want = [], [], []
        for rid, count in step:
            n, seed = requests[rid]
            lo = at.get(rid, 0)
            if lo == 0:
                seat_of[rid] = free.pop()
            seats.append(seat_of[rid])
            toks.append(list(prompt(cfg["vocab"], n, seed)[lo:lo + count]))
            want.append(expected(name, sharp, n, seed)[lo:lo + count])
            at[rid] = lo + count
        errs.append(row_errors(runner.step(seats, toks, logits_all=True), torch.cat(want)))
        for rid, _ in step:
            if at[rid] == requests[rid][0]:
                runner.kv.free(seat_of[rid])
                free.append(seat_of.pop(rid))
    assert not seat_of, "a request was left unfinished"
    errs = torch.cat(errs)
    assert not torch.isnan(errs).any()
    return float(errs.max() if runner.model.cfg.dtype == "float32" else errs.quantile(0.75))


def portions(n, sizes):
    """Cut ``n`` tokens into portions whose sizes cycle through ``sizes``."""
    out, i = [], 0
    while n:
        c = min(n, sizes[i % len(sizes)])
        out.append(c)
        n -= c
        i += 1
    return out
