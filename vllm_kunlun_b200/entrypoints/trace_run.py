"""``bin/trace_run``: feed given token ids through a model step by step and write logits.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Reads one JSON object a line from standard input,

    {"step": 0, "entries": [{"id": "req-1", "tokens": [11, 4, 90, 2], "want": [3]}], "end": ["req-1"]}

runs the entries as one batch of the engine, writes the logits at the wanted places to ``DIR/<step>.f32`` (little-endian
fp32 ``[wanted, vocab]``, only when something is wanted) and prints ``done <step>``.  Nothing is sampled."""
from __future__ import annotations

import argparse
import json
import os
import sys


def parse(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.splitlines()[0])
    ap.add_argument("--model", required=True, help="folder with config.json and safetensors")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True,
                    help="tokens that live requests hold at most, each request rounded up to whole cache blocks of 64")
    ap.add_argument("--device", default="cuda", choices=["cuda", "cpu"], help="cpu runs the fp32 reference ops")
    ap.add_argument("--enforce-eager", action="store_true", help="no captured decode steps")
    return ap.parse_args(argv)


def main(argv=None) -> int:
    a = parse(argv)
    if a.device == "cuda":
        from ..build import build
        build()                     # compiles what is missing or out of date, otherwise only compares digests
    from ..engine.replay import ScheduleReplay
    replay = ScheduleReplay(a.model, a.dtype, a.max_tokens, device=a.device, enforce_eager=a.enforce_eager)
    os.makedirs(a.out, exist_ok=True)
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        logits = replay.step(s["entries"], s.get("end", ()))
        if logits.shape[0]:
            logits.contiguous().numpy().astype("<f4", copy=False).tofile(os.path.join(a.out, f"{s['step']}.f32"))
        print(f"done {s['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
