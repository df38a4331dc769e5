"""Replays a trace of token ids through a model, step by step, and writes logits.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps.jsonl

One JSON object a line: {"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}.  A step is one batch of the
engine.  If something is wanted, DIR/<n>.f32 receives the logits (little-endian fp32, [wanted, vocab]); then a line
"done <n>" is printed.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

PAGE = 64           # tokens per cache page
MAX_REQUESTS = 4    # live requests


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.splitlines()[0])
    ap.add_argument("--model", required=True, help="folder with config.json and *.safetensors")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True,
                    help="most tokens that live requests hold, each rounded up to a page")
    ap.add_argument("--device", default="cuda", help=argparse.SUPPRESS)
    a = ap.parse_args(argv)

    from ..llm import LLM
    from ..engine.replay import TokenReplay
    llm = LLM(a.model, dtype=a.dtype, device=a.device, kvcache_block_size=PAGE,
              num_kvcache_blocks=max(1, -(-a.max_tokens // PAGE)), max_model_len=max(a.max_tokens, PAGE),
              max_num_seqs=MAX_REQUESTS, max_num_batched_tokens=max(a.max_tokens, PAGE), prefix_caching=False,
              tokenizer=False)
    replay = TokenReplay(llm)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = replay.step(step.get("entries", []), step.get("end", []))
        if logits.shape[0]:
            with open(os.path.join(a.out, f"{step['step']}.f32"), "wb") as fh:
                fh.write(logits.contiguous().numpy().astype("<f4").tobytes())
        print(f"done {step['step']}", flush=True)
    llm.exit()
    return 0


if __name__ == "__main__":
    sys.exit(main())
