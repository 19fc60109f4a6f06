"""Replay of a trace: token ids go through the engine step by step as they come, logits of the wanted places come out.

Standard input has one JSON object per line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["b"]}

A step runs the given tokens of every entry's request (a new id opens one) and writes the logits of the wanted places,
in order, to OUT/<step>.f32 (little-endian fp32 [rows, vocab]) if there are any; requests in "end" are closed; then
``done <step>`` is printed.  Nothing is sampled.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

REFUSED = 3          # exit status: the model does not run in the asked dtype


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Feeds given token ids through a model and writes logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that open requests hold at any time")
    ap.add_argument("--max-requests", type=int, default=16, help="most requests that are open at any time")
    a = ap.parse_args(argv)

    from ..build import build_library
    from ..models.registry import SUPPORTED_MODELS
    from ..models.weight import architecture_of, load_config_dict
    entry = SUPPORTED_MODELS[architecture_of(load_config_dict(a.model))]
    build_library(which=entry.library)           # compiles what this model needs, if it has not been compiled yet
    from .engine import DTYPES, Engine
    if DTYPES[a.dtype] not in entry.dtypes:
        print(f"this model does not run in {a.dtype}", file=sys.stderr)
        return REFUSED
    engine = Engine(a.model, dtype=a.dtype, max_tokens=max(a.max_tokens, 1), max_reqs=a.max_requests)
    open_requests: dict = {}
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = step.get("entries", [])
        for e in entries:
            if e["id"] not in open_requests:
                open_requests[e["id"]] = engine.open()
        if entries:
            logits = engine.step([open_requests[e["id"]] for e in entries], [e["tokens"] for e in entries], [e.get("want", []) for e in entries])
            if logits is not None:
                host = logits.float().cpu().numpy().astype("<f4")
                engine.check_status()
                host.tofile(os.path.join(a.out, f"{int(step['step'])}.f32"))
        for rid in step.get("end", []):
            if rid in open_requests:
                engine.close(open_requests.pop(rid))
        print(f"done {step['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
