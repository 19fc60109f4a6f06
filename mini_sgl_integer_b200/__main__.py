"""Command line: greedy generation of token ids.

    python -m mini_sgl_integer_b200 --model DIR --prompt-ids 5,17,3 [--prompt-ids ...] [--max-new-tokens N]
    python -m mini_sgl_integer_b200 --model DIR < prompts.jsonl        # one list of ids per line

The model class is chosen by DIR/config.json; one line of JSON per prompt is printed.  (Prompts are token ids: this
package has no tokenizer.)
"""
from __future__ import annotations

import argparse
import json
import sys


def main(argv=None) -> int:
    from .models.registry import SUPPORTED_MODELS
    ap = argparse.ArgumentParser(prog="python -m mini_sgl_integer_b200", description=f"Greedy generation. Architectures: {', '.join(SUPPORTED_MODELS.supported_names())}.")
    ap.add_argument("--model", required=True, help="folder with config.json and safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--prompt-ids", action="append", default=[], help="comma-separated token ids; may be given several times")
    ap.add_argument("--max-new-tokens", type=int, default=16)
    ap.add_argument("--stop-ids", default="", help="comma-separated token ids that end a generation")
    ap.add_argument("--max-tokens", type=int, default=65536, help="tokens that running requests hold together")
    ap.add_argument("--max-running", type=int, default=64, help="requests that run at the same time")
    ap.add_argument("--prefill-budget", type=int, default=4096, help="most prompt tokens per step")
    ap.add_argument("--no-cuda-graphs", action="store_true")
    a = ap.parse_args(argv)
    ids = lambda text: [int(t) for t in text.split(",") if t.strip()]
    prompts = [ids(t) for t in a.prompt_ids] or [json.loads(line) for line in sys.stdin if line.strip()]
    if not prompts:
        ap.error("no prompts")
    from .engine import Engine, SamplingParams, Scheduler
    engine = Engine(a.model, dtype=a.dtype, max_tokens=a.max_tokens, max_reqs=a.max_running, max_portion=a.prefill_budget,
                    cuda_graphs=not a.no_cuda_graphs)
    outs = Scheduler(engine).generate(prompts, SamplingParams(a.max_new_tokens, tuple(ids(a.stop_ids))))
    for p, o in zip(prompts, outs):
        print(json.dumps({"prompt": p, "output": o}), flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
