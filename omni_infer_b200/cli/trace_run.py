"""``bin/trace_run``: replays a trace of token ids through a model, step by step, and writes the logits asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps.jsonl

Every input line is one step: ``{"step": 0, "entries": [{"id": "a", "tokens": [5, 17], "want": [1]}], "end": ["a"]}``.  All
entries of a step are one batch.  ``want`` lists places among the entry's tokens; their logits go to ``OUT/<step>.f32``
(little-endian fp32, [rows, vocab]).  ``end`` lists requests that give their pages and state slot back after the step.
``done <step>`` is printed after each step.  The page pool holds ``--max-tokens`` tokens in pages of 64, and there are state
slots for four live requests.  Kernels are compiled on first use."""
from __future__ import annotations

import argparse
import json
import os
import sys

PAGE = 64
MAX_LIVE = 4


def parse(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True, help="folder with config.json and *.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True,
                    help="most tokens that live requests hold at once, each request's rounded up to a multiple of 64")
    return ap.parse_args(argv)


def build_engine(model: str, dtype: str, max_tokens: int, device=None):
    from ..engine.engine_core import EngineConfig, EngineCore
    pages = (max_tokens + PAGE - 1) // PAGE
    return EngineCore(EngineConfig(model=model, model_overrides={"dtype": dtype}, device=device, block_size=PAGE,
                                   num_kv_blocks=pages + 1, max_num_seqs=MAX_LIVE, max_model_len=pages * PAGE,
                                   max_num_batched_tokens=pages * PAGE, enable_chunked_prefill=True, mixed_batches=True,
                                   enable_prefix_caching=False))


def replay(engine, steps, out_dir: str, report) -> None:
    from ..engine.trace_replay import TraceReplay
    from ..ops import _native as nat
    tr = TraceReplay(engine)
    for line in steps:
        if not line.strip():
            continue
        s = json.loads(line)
        logits = tr.step(s.get("entries") or [], s.get("end") or ())
        if engine.worker.device.type == "cuda":
            nat.check_status()
        if logits is not None:
            logits.numpy().astype("<f4").tofile(os.path.join(out_dir, f"{s['step']}.f32"))
        report(s["step"])


def main(argv=None) -> int:
    a = parse(argv)
    import torch
    if not torch.cuda.is_available():
        print("trace_run needs a CUDA device", file=sys.stderr)
        return 2
    from ..build import ensure_kernels
    from ..models.config import ModelConfig
    from ..ops import _native as nat
    cfg = ModelConfig.from_pretrained(a.model)
    if a.dtype == "float32" and cfg.layers is None:
        print(f"{cfg.architecture} runs in bfloat16 only", file=sys.stderr)
        return 3
    nat.use_library(ensure_kernels(cfg.architecture))
    engine = build_engine(a.model, a.dtype, a.max_tokens)
    replay(engine, sys.stdin, a.out, lambda n: print(f"done {n}", flush=True))
    return 0


if __name__ == "__main__":
    sys.exit(main())
