"""Trace replay: feeds given token ids through a model step by step and writes logits.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Reads one JSON object a line from standard input,

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["b"]}

runs all entries of a step as one batch (portions of prompts beside single tokens), writes the logits at the
wanted places to OUT/<step>.f32 (little-endian fp32, [wanted, vocab], in the order of the entries) and prints
"done <step>".  A request is admitted at its first entry and gives its pages and state slot back when a step
lists it under "end".  Nothing is sampled; the engine, its cache, states and kernels are the ones generation
uses (Engine.open / step / close_sequence).  The reference has no counterpart.
"""
from __future__ import annotations

import argparse
import dataclasses
import json
import os
import sys

MAX_LIVE = 4            # state slots of the replay engine
PREFILL_TOKENS = 8192   # most tokens of one launch; longer portions are cut
LOGIT_ROWS = 128


def build_engine(model_dir: str, dtype: str, max_tokens: int, device: str = "cuda:0"):
    """The engine for a model directory, its pages holding `max_tokens` tokens; None if the model cannot run in
    `dtype`."""
    import torch

    from . import model as M
    from . import stack
    from .engine import Engine
    from .executors import PAGE
    cfg = M.config_from_dir(model_dir)
    pages = max(1, -(-max_tokens // PAGE))
    if isinstance(cfg, stack.StackConfig):
        reach = cfg.max_pos if cfg.learned_pos else max(cfg.max_pos, max_tokens)
        cfg = dataclasses.replace(cfg, act_dtype=dtype, max_pos=reach)
    elif dtype != "bfloat16":
        return None
    weights = M.weights_for(cfg).from_safetensors_dir(cfg, model_dir, torch.device(device))
    return Engine(cfg, weights, None, max_model_len=pages * PAGE, max_rows=MAX_LIVE, state_slots=MAX_LIVE,
                  prefill_tokens=min(PREFILL_TOKENS, pages * PAGE), kv_pages=pages, logit_rows=LOGIT_ROWS,
                  enable_prefix_cache=False, device=device)


def replay(engine, lines, out_dir: str, echo=print) -> None:
    live = {}
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        work = []
        for e in step.get("entries", []):
            if e["id"] not in live:
                live[e["id"]] = engine.open()
            work.append((live[e["id"]], e["tokens"], e.get("want", [])))
        if work:
            logits = engine.step(work)
            if logits.shape[0]:
                path = os.path.join(out_dir, f"{step['step']}.f32")
                logits.float().cpu().numpy().astype("<f4").tofile(path)
        for i in step.get("end", []):
            engine.close_sequence(live.pop(i))
        echo(f"done {step['step']}", flush=True)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(description=__doc__.split("\n\n")[0])
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="tokens the cache pool holds")
    a = ap.parse_args(argv)
    from . import build
    build.build()           # compiles the library if this checkout has none yet
    engine = build_engine(a.model, a.dtype, a.max_tokens)
    if engine is None:
        print("this model's kernels run in bfloat16 only", file=sys.stderr)
        return 3
    replay(engine, sys.stdin, a.out)
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
