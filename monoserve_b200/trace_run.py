"""Replays a trace of token ids through a model, step by step, and writes the logits it asks for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

A step is one JSON object a line: {"step": n, "entries": [{"id": .., "tokens": [..], "want": [..]}], "end": [..]}.
"""
import argparse
import json
import os
import sys


def main():
    ap = argparse.ArgumentParser(description="Replay token ids through a model and write the logits asked for.")
    ap.add_argument("--model", required=True, help="folder with config.json and safetensors files")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for <step>.f32: float32 [wanted, vocab]")
    ap.add_argument("--max-tokens", type=int, default=4096, help="the most tokens live requests hold at any time")
    args = ap.parse_args()
    from monoserve_b200.build import build
    build()
    from monoserve_b200 import registry
    from monoserve_b200.session import Session
    with Session(registry.load(args.model, args.dtype), args.max_tokens) as session:
        for line in sys.stdin:
            if not line.strip():
                continue
            step = json.loads(line)
            wanted = []
            for entry in step["entries"]:
                logits = session.step(entry["id"], entry["tokens"], entry.get("want", ()))
                wanted.append(logits.tobytes())
            if any(wanted):
                path = os.path.join(args.out, f"{step['step']}.f32")
                with open(path, "wb") as f:
                    f.write(b"".join(wanted))
            for rid in step.get("end", ()):
                session.end(rid)
            print(f"done {step['step']}", flush=True)


if __name__ == "__main__":
    main()
