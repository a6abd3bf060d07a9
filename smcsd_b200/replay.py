"""Trace replay: feeds given token ids through a model of the engine, step by step, and writes the logits asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

Every input line is one step: ``{"step": 0, "entries": [{"id": "a", "tokens": [5, 17], "want": [1]}], "end": []}``.  All
entries of a step are one batch, each continuing the sequence of its id; ``end`` releases sequences after the step.  Wanted
logits go to ``DIR/<step>.f32`` (little-endian fp32, [wanted, vocab]); ``done <step>`` is printed after every step.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

MAX_SEQUENCES = 4


def open_engine(model: str, dtype: str, max_tokens: int, device: str = "auto"):
    """An engine whose page pool holds ``max_tokens`` tokens and whose rows hold MAX_SEQUENCES live sequences."""
    from .engine import SMCEngine
    from .models.config import resolve_config
    cfg = resolve_config(model)
    return SMCEngine(model, model, n_particles=1, gamma=1, dtype=dtype, device=device, max_running_requests=MAX_SEQUENCES,
                     max_total_tokens=max_tokens, context_length=min(cfg.max_position, max_tokens), skip_tokenizer_init=True, in_process=True)


def replay(engine, lines, out_dir: str, reply) -> None:
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = engine.feed([(e["id"], e["tokens"], e.get("want", [])) for e in step["entries"]], step.get("end", []))
        if logits.shape[0]:
            data = logits.float().cpu().contiguous().numpy().astype("<f4").tobytes()
            with open(os.path.join(out_dir, f"{step['step']}.f32"), "wb") as f:
                f.write(data)
        reply(f"done {step['step']}")


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n")[0])
    ap.add_argument("--model", required=True, help="folder with config.json and the weights")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder the logits are written to")
    ap.add_argument("--max-tokens", type=int, required=True, help="tokens the page pool holds")
    ap.add_argument("--device", default="cuda", choices=["cuda", "cpu"], help="cpu: the plain PyTorch reference path")
    ns = ap.parse_args(argv)
    engine = open_engine(ns.model, ns.dtype, ns.max_tokens, ns.device)
    try:
        replay(engine, sys.stdin, ns.out, lambda text: print(text, flush=True))
    finally:
        engine.shutdown()
    return 0


if __name__ == "__main__":
    sys.exit(main())
