"""Replay of a token trace: feed given token ids through a model step by step and write the logits asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps.jsonl

Every line of the input is one step, run as one batch by the engine's step function:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["b"]}

``entries``: for each request its next tokens and the places among them whose logits are wanted (a request is admitted at
its first entry); ``end``: requests that are finished after the step.  The logits of a step go to ``OUT/<step>.f32``
(little-endian fp32, ``[wanted, vocab]``) and ``done <step>`` is printed once it has run.  The cache pool holds
``--max-tokens`` tokens and there are rows for four requests at a time.  Nothing is sampled.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

ROWS = 4
ROUND = 64


def replay(lines, engine, out_dir: str, report) -> None:
    from tah_b200.engine.hybrid import StepEntry
    from tah_b200.ops import cuda as K
    row = {}
    for line in lines:
        if not line.strip():
            continue
        msg = json.loads(line)
        entries = []
        for e in msg["entries"]:
            if e["id"] not in row:
                row[e["id"]] = engine.admit()
            entries.append(StepEntry(row[e["id"]], e["tokens"], e["want"]))
        if entries:
            logits = engine.step(entries)
            host = logits.float().cpu().contiguous()
            K.check_status(engine.device)
            if host.shape[0]:
                with open(os.path.join(out_dir, f"{msg['step']}.f32"), "wb") as fh:
                    fh.write(host.numpy().astype("<f4", copy=False).tobytes())
        for rid in msg.get("end", ()):
            engine.release(row.pop(rid))
        report(f"done {msg['step']}")


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(description="replay a token trace through a model and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at a time")
    a = ap.parse_args(argv)
    import torch
    from tah_b200.models.registry import family_of_config, load_model, make_engine, read_config
    from tah_b200.ops import cuda as K
    family = family_of_config(read_config(a.model))
    if not torch.cuda.is_available():
        raise RuntimeError("trace replay needs a CUDA device")
    if family.sources is not None:
        K.use_group_build(family.sources)
    engine = make_engine(load_model(a.model, getattr(torch, a.dtype), "cuda"), max_rows=ROWS)
    if not hasattr(engine, "step"):
        raise RuntimeError(f"the engine of family {family.name!r} has no step function for token portions")
    engine.open(ROWS, (a.max_tokens + ROUND - 1) // ROUND * ROUND)
    os.makedirs(a.out, exist_ok=True)

    def report(text):
        sys.stdout.write(text + "\n")
        sys.stdout.flush()

    replay(sys.stdin, engine, a.out, report)
    return 0
