"""Trace replay: feed given token ids through a model step by step and write logits. Nothing is sampled.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N
    python -m mojo_b200.cli replay ...              (the same)

Steps are read from standard input, one JSON object a line:
    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}
`entries` holds, per request, its next tokens and the places among them whose logits are wanted; all entries of a step run
as one batch (`LLMEngine.run_tokens`). `end` names the requests that are finished after the step. A step that wants
something writes DIR/<step>.f32, little-endian f32 [wanted, vocab]; every step prints `done <step>` when it is complete.

The engine is the one that serves the model, with a cache for `--max-tokens` tokens (every live request rounded up to 64)
and state for four live requests."""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path

LIVE_REQUESTS = 4
PAGE_SIZE = 128
TOKEN_UNIT = 64        # a request's share of --max-tokens is counted in units of this many tokens


def ensure_built() -> None:
    """Build what the models replayed here need if this checkout has no native extension (one builder at a time)."""
    from . import _ext, build

    if _ext.built():
        return
    import fcntl

    with open(build.ROOT / ".build.lock", "w") as lock:
        fcntl.flock(lock, fcntl.LOCK_EX)
        if not _ext.built():
            build.build(core=True)


def open_engine(model: str, dtype: str, max_tokens: int, device: str | None = None):
    """The serving engine on a checkpoint folder, its cache made for `max_tokens` tokens of live requests."""
    from .pipelines import LLM, PipelineConfig

    # requests rounded up to the page size instead of to 64 tokens: at most one more unit each
    pages = -(-(max_tokens + LIVE_REQUESTS * (PAGE_SIZE - TOKEN_UNIT)) // PAGE_SIZE)
    cfg = PipelineConfig(model=model, dtype=dtype, device=device, page_size=PAGE_SIZE, num_pages=pages, max_num_seqs=LIVE_REQUESTS,
                         state_slots=LIVE_REQUESTS, max_num_batched_tokens=max_tokens, max_model_len=max_tokens)
    return LLM(cfg).engine


def replay(engine, lines, out_dir: Path, write=print) -> None:
    import numpy as np
    import torch

    from . import ops

    ids: dict[str, int] = {}       # live requests
    next_id = 0
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = []
        for e in step["entries"]:
            if e["id"] not in ids:
                ids[e["id"]] = next_id
                next_id += 1
            entries.append((ids[e["id"]], e["tokens"], e.get("want", [])))
        # a later request under a finished one's name is a new one
        logits = engine.run_tokens(entries, [ids.pop(name) for name in step.get("end", [])])
        if logits is not None:
            data = logits.to(torch.float32).cpu().numpy().astype(np.dtype("<f4"))
            (out_dir / f"{step['step']}.f32").write_bytes(data.tobytes())
        if engine.device.type == "cuda":
            ops.check_status(engine.device)
        write(f"done {step['step']}", flush=True)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time, each rounded up to a multiple of 64")
    ap.add_argument("--device", default="cuda")
    a = ap.parse_args(argv)
    if a.max_tokens < 1:
        ap.error("--max-tokens must be positive")
    ensure_built()
    out = Path(a.out)
    out.mkdir(parents=True, exist_ok=True)
    replay(open_engine(a.model, a.dtype, a.max_tokens, a.device), sys.stdin, out)
    return 0
