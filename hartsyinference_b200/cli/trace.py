"""``bin/trace_run``: replay a recorded token stream through a served model and keep the logits.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps.jsonl

Every input line is one engine step as a JSON object, for instance
``{"step": 7, "entries": [{"id": "req1", "tokens": [901, 44, 2], "want": [2]}], "end": []}``: what each request
continues with, at which of these tokens (index from 0) logits are to be kept, and which requests leave
afterwards. Kept logits go to ``<out>/<step>.f32`` (little-endian fp32 [kept, vocab], entry by entry), and
``done <step>`` is printed when the step is through.

The model is loaded and run by the engine that serves it (``LLMEngine.replay``): its page pool holds
``--max-tokens`` tokens, with state slots for ``--max-live`` requests. The kernels library is compiled on
first use in a checkout that has not been built.
"""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path

EXIT_NO_32BIT = 3


def parse(argv=None) -> argparse.Namespace:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n\n")[0])
    ap.add_argument("--model", required=True, help="directory with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16",
                    help="bfloat16: as served; float32: products and caches in 32 bits")
    ap.add_argument("--out", required=True, help="directory of the logits files")
    ap.add_argument("--max-tokens", type=int, required=True, help="size of the page pool in tokens (pages of 16)")
    ap.add_argument("--max-live", type=int, default=4, help="state slots: requests that can be open together")
    ap.add_argument("--device", default="cuda")
    return ap.parse_args(argv)


def make_engine(a: argparse.Namespace):
    import torch
    from ..engine.llm_engine import LLMEngine
    from ..models.llm.loader import load_llm
    model = load_llm(a.model, a.device, dtype=getattr(torch, a.dtype)).model
    page = 16
    tokens = (a.max_tokens + page - 1) // page * page
    return LLMEngine(model, num_pages=tokens // page, page_size=page, max_batch=a.max_live, prefill_chunk=tokens, max_model_len=tokens)


def main(argv=None) -> int:
    a = parse(argv)
    out = Path(a.out)
    out.mkdir(parents=True, exist_ok=True)
    from .. import config, log
    config.set_override("log_level", "warn")
    if a.device.startswith("cuda"):
        from .. import build
        build.ensure("decoder")
    import torch
    if a.device.startswith("cuda") and not torch.cuda.is_available():
        print("trace_run: no CUDA device", file=sys.stderr)
        return 1
    try:
        eng = make_engine(a)
    except ValueError as e:
        if a.dtype == "float32" and "bfloat16" in str(e):
            print(f"trace_run: {e}", file=sys.stderr)
            return EXIT_NO_32BIT
        raise
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = eng.replay([(e["id"], e["tokens"], e.get("want", ())) for e in step.get("entries", ())], step.get("end", ()))
        if logits is not None:
            (out / f"{step['step']}.f32").write_bytes(logits.cpu().contiguous().numpy().astype("<f4", copy=False).tobytes())
        print(f"done {step['step']}", flush=True)
    return 0
