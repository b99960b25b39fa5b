"""Replay a trace: feed given token ids through the engine step by step and write the logits asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Standard input holds one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["b"]}

Every step's entries run as one batch through ``EngineBackend.step`` (the serving backend: its page pool, state slots and
kernels); a request is opened at its first entry and released when a step's ``end`` names it.  For a step that wants
something ``DIR/<step>.f32`` receives the logits [wanted, vocab] as little-endian fp32, in the order of the entries and of
their ``want``; after every step ``done <step>`` is printed.  ``--max-tokens``: tokens that live requests hold at most,
each request's count rounded up to whole pages; the page pool is made for exactly these, the state pool for four requests.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

LIVE_REQUESTS = 4
MAX_STEP_TOKENS = 16384


def build_backend(model: str, dtype: str, max_tokens: int):
    import torch

    from ..loader.load import load_engine
    from .backends import EngineBackend
    from .paged import PAGE
    from .state import FIRST_SLOT
    pages = -(-max_tokens // PAGE)
    step_tokens = min(max(PAGE, pages * PAGE), MAX_STEP_TOKENS)
    _, eng = load_engine(model, torch.device("cuda:0"), pages + 1, step_tokens, 64, compute_dtype="f32" if dtype == "float32" else "bf16",
                         state_slots=FIRST_SLOT + 2 * LIVE_REQUESTS)
    return EngineBackend(eng, pages + 1, pages + 1, prefill_chunk=step_tokens, max_decode_rows=LIVE_REQUESTS)


def replay(be, lines, out_dir: str, emit) -> None:
    """Run the steps of ``lines`` on backend ``be``; ``emit(text)`` prints a line."""
    import numpy as np
    from ..ops import kernels as K
    live: dict = {}
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        items = []
        for e in step["entries"]:
            if e["id"] not in live:
                live[e["id"]] = be.open(e["tokens"], cold=True)[0]
            items.append((live[e["id"]], e["tokens"], sorted(set(e["want"]))))
        got = be.step(items)
        if K.read_status():
            raise RuntimeError("a bounded device wait ran out")
        rows = []
        for e, (_, _, places), g in zip(step["entries"], items, got):
            at = {p: k for k, p in enumerate(places)}
            rows += [g[at[p]].numpy() for p in e["want"]]
        if rows:
            np.stack(rows).astype("<f4").tofile(os.path.join(out_dir, f"{step['step']}.f32"))
        for rid in step.get("end", []):
            h = live.pop(rid, None)
            if h is not None:
                be.release(h)
        emit(f"done {step['step']}")


def main(argv: list[str] | None = None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay token-id steps through the engine and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"],
                    help="bfloat16: the serving precisions; float32: every product and activation in 32-bit")
    ap.add_argument("--out", required=True, help="folder the logits of each step are written to")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens live requests hold at any time (whole pages each)")
    a = ap.parse_args(argv)
    from ..loader.snapshot import read_config
    if a.dtype == "float32" and not read_config(a.model)[0].is_hybrid:
        print("trace_run: this model has no 32-bit form", file=sys.stderr)
        return 3
    os.makedirs(a.out, exist_ok=True)

    def emit(text: str) -> None:
        print(text, flush=True)
    import torch
    with torch.inference_mode():
        replay(build_backend(a.model, a.dtype, a.max_tokens), sys.stdin, a.out, emit)
    return 0


if __name__ == "__main__":
    sys.exit(main())
