"""``trtedge trace`` / ``bin/trace_run``: replay a trace of given token ids through a model and write the logits asked for.

Steps arrive on standard input, one JSON object a line::

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

All entries of a step are one batch of the runner (prompt portions beside single tokens), fed from the cache pages and state rows that
earlier steps left; a request takes a seat at its first entry and gives seat and pages back in the step that lists it under ``end``.
``want`` names places among an entry's tokens; their logits go to ``<out>/<step>.f32`` (little-endian fp32, ``[wanted, vocab]``, entries
in order).  ``done <step>`` is printed after every step.  The page pool holds exactly ``--max-tokens`` tokens."""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict, List

PAGE = 64


class TraceReplay:
    """Seats by request id over an ``LLM``'s runner and cache; one call per step."""

    def __init__(self, llm):
        from ..runtime import native as rt
        self.llm, self.runner, self.kv = llm, llm.runner, llm.kv
        self.slots = rt.ResidentSlotPool(self.kv.max_seats)
        self.seat_of: Dict[str, int] = {}

    def step(self, entries: List[dict], end: List[str]):
        """Run one batch; returns the wanted logits ``[wanted, vocab]`` (fp32, host) or ``None`` when nothing is wanted."""
        seats, tokens, rows, r0 = [], [], [], 0
        vocab = self.llm.cfg.vocab_size
        for e in entries:
            ids = [int(t) for t in e["tokens"]]
            want = [int(w) for w in e.get("want", [])]
            if not ids or any(not 0 <= t < vocab for t in ids) or any(not 0 <= w < len(ids) for w in want):
                raise ValueError(f"request {e['id']!r}: token ids inside the vocabulary and places among its tokens are needed")
            rid = str(e["id"])
            if rid not in self.seat_of:
                seat = self.slots.acquire()
                if seat < 0:
                    raise RuntimeError("more live requests than seats")
                self.seat_of[rid] = seat
            if self.seat_of[rid] in seats:
                raise ValueError(f"request {rid!r} appears twice in a step")
            seats.append(self.seat_of[rid])
            tokens.append(ids)
            rows += [r0 + w for w in want]
            r0 += len(ids)
        out = None
        if seats:
            logits = self.runner.step(seats, tokens, logits_rows=rows)
            out = logits.float().cpu() if rows else None
        for rid in end:
            seat = self.seat_of.pop(str(rid))
            self.kv.free(seat)
            self.slots.release(seat)
        return out


def main(argv=None) -> int:
    p = argparse.ArgumentParser(prog="trtedge trace")
    p.add_argument("--model", required=True, help="checkpoint directory")
    p.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float16", "float32"])
    p.add_argument("--out", required=True, help="directory for the logits files")
    p.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at a time (size of the page pool)")
    p.add_argument("--max-requests", type=int, default=4, help="most live requests (seats)")
    p.add_argument("--device", default="cuda", help="cuda (default) or cpu")
    a = p.parse_args(argv)
    from ..build import ensure_built
    from ..config import ModelConfig
    family = ensure_built(ModelConfig.from_pretrained(a.model).model_type)
    import torch
    from ..ops import cuda as cu
    from ..runtime.llm import LLM
    if a.device.startswith("cuda"):
        if not torch.cuda.is_available():
            print("no CUDA device", file=sys.stderr)
            return 2
        cu.KERNEL_FAMILY = family
    pages = (a.max_tokens + PAGE - 1) // PAGE
    llm = LLM(a.model, device=a.device, dtype=a.dtype, max_batch_size=a.max_requests, max_input_len=a.max_tokens,
              max_kv_cache_capacity=pages * PAGE, page_size=PAGE, kv_pages=pages)
    replay = TraceReplay(llm)
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        logits = replay.step(s["entries"], s.get("end", []))
        if logits is not None:
            data = logits.contiguous().numpy().astype("<f4", copy=False).tobytes()
            path = os.path.join(a.out, f"{int(s['step'])}.f32")
            with open(path, "wb") as f:
                f.write(data)
        print(f"done {s['step']}", flush=True)
    if llm.device.type == "cuda":
        cu.Workspace.get(llm.device).check_status()
    return 0


if __name__ == "__main__":
    sys.exit(main())
