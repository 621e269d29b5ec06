"""Trace replay: feed given token ids to a model step by step and write the logits it produces.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

One JSON object per input line:

    {"step": 7, "entries": [{"id": "r1", "tokens": [12, 40], "want": [1]}, {"id": "r2", "tokens": [9], "want": []}], "end": ["r2"]}

``entries``: the next tokens of each request and the indices among them whose logits are wanted; ``end``: requests that are
finished after this step. The wanted logits of a step go to ``OUT/<step>.f32`` ([wanted, vocab], little-endian fp32, in the
order of the entries); ``done <step>`` is printed after every step. Nothing is sampled.

The trace runs through ``LLMEngine.feed_step``: the serving engine's scheduler, page pool, state slots, prefill chunks and
captured decode steps. The pool holds ``--max-tokens`` tokens and four requests; pages and slots of ended requests are used
again. Kernels that are not built yet are compiled at the first call.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict, Optional

EXIT_NO_F32 = 3
LIVE_REQUESTS = 4
TOKEN_BUDGET = 8192          # tokens of one engine step (longer portions run as several chunks)


def ensure_built():
    """The kernel library this checkout needs (the host extensions build themselves when they are imported)."""
    from .ops import _native as nv
    if nv.available():
        return
    from . import build
    import fcntl
    build.LIB.mkdir(exist_ok=True)
    with open(build.LIB / ".build.lock", "w") as lock:      # two first calls at once: one builds, the other waits
        fcntl.flock(lock, fcntl.LOCK_EX)
        if not nv.available():
            build.build_kernels()


def make_engine(model_dir: str, dtype_name: str, max_tokens: int, device: Optional[str] = None):
    import torch
    from .engine.executor import EngineConfig, LLMEngine
    from .loader import Loader
    from .models.registry import decoder_class
    dev = torch.device(device or ("cuda" if torch.cuda.is_available() else "cpu"))
    dtype = {"bfloat16": torch.bfloat16, "float32": torch.float32}[dtype_name]
    loaded = Loader.from_source_with_config(model_dir).load()
    cls = decoder_class(loaded.config)
    if dtype == torch.float32 and dev.type == "cuda" and not getattr(cls, "runs_float32", False):
        raise NotImplementedError(f"{cls.__name__} has no 32-bit kernels")
    pages = (max_tokens + 15) // 16
    model = cls(loaded.config, loaded.weights, device=dev, dtype=dtype, max_positions=pages * 16)
    budget = min(TOKEN_BUDGET, max(pages * 16, 64))
    # the pool is exactly the live tokens, so every page may be handed out: no reserve, no pressure or fragmentation limit
    ec = EngineConfig(max_num_seqs=LIVE_REQUESTS, max_model_len=pages * 16, max_batch_tokens=budget, prefill_chunk=budget,
                      num_pages=pages, enable_prefix_cache=False, watermark_pages=0, emergency_pressure=2.0,
                      defrag_threshold=2.0)
    return LLMEngine(model, ec)


def run(engine, lines, out_dir: str, stdout):
    import numpy as np
    ids: Dict[object, int] = {}
    next_id = 0
    for line in lines:
        line = line.strip()
        if not line:
            continue
        step = json.loads(line)
        entries, wanted = [], 0
        for e in step["entries"]:
            if e["id"] not in ids:
                ids[e["id"]] = next_id
                next_id += 1
            entries.append((ids[e["id"]], e["tokens"], e.get("want") or []))
            wanted += len(e.get("want") or [])
        if entries:
            rows = engine.feed_step(entries)
            if wanted:
                data = np.concatenate([r.numpy() for r in rows]).astype("<f4")
                part = os.path.join(out_dir, f".{step['step']}.part")
                data.tofile(part)
                os.replace(part, os.path.join(out_dir, f"{step['step']}.f32"))
        for name in step.get("end") or []:
            engine.feed_end(ids.pop(name))
        print(f"done {step['step']}", file=stdout, flush=True)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(description="Replay a token trace through the engine and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="tokens the live requests hold at any time")
    ap.add_argument("--device", default=None, help="cuda (default when there is one) or cpu")
    a = ap.parse_args(argv)
    import torch
    torch.backends.cuda.matmul.allow_tf32 = False
    if (a.device or "cuda") != "cpu" and torch.cuda.is_available():
        ensure_built()
    try:
        engine = make_engine(a.model, a.dtype, a.max_tokens, a.device)
    except NotImplementedError as e:
        print(f"trace_run: {e}", file=sys.stderr)
        return EXIT_NO_F32
    run(engine, sys.stdin, a.out, sys.stdout)
    return 0


if __name__ == "__main__":
    sys.exit(main())
