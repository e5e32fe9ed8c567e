"""Generates tokens with a checkpoint of any family in monoserve_b200/registry.py through the serving loop.

    python -m monoserve_b200.generate --model DIR --prompt 5,17,3 [--prompt 8,1 ...] [--max-tokens 32]
                                      [--temperature 0.0] [--eos 2] [--dtype bfloat16|float32]

Prompts are token ids (the library has no tokenizer).  One JSON line per prompt, in order: the generated ids and why the
request ended.
"""
import argparse
import json


def generate(model, prompts, max_tokens=32, temperature=0.0, eos=(), page=16, max_decode=16, token_budget=None, spare_sms=8,
             timeout_s=600.0):
    """[(tokens, reason)] of each prompt (a list of token ids), batched continuously.  temperature 0 is greedy."""
    import torch

    from monoserve_b200.engine import LOOKAHEAD_PAGES, Engine, PagePool, RequestTable
    from monoserve_b200.fabric import Fabric
    longest = max(len(p) for p in prompts)
    budget = token_budget or max(64, longest)
    bt_stride = -(-(longest + max_tokens + 1) // page) + LOOKAHEAD_PAGES
    slots = max(2, min(2 * max_decode, len(prompts) + max_decode))
    pages = min(slots, len(prompts)) * bt_stride + 1
    workers = torch.cuda.get_device_properties(0).multi_processor_count - spare_sms
    fab = Fabric(num_workers=workers, pool_bytes=512 << 20)
    try:
        fab.set_max_run(timeout_s + 60)
        kv = model.cache(pages, page, slots)
        table = RequestTable(fab, slots, bt_stride)
        eng = Engine(fab, model.cfg, model.weights, kv, table, PagePool(pages), max_decode=max_decode, token_budget=budget,
                     max_len=longest + max_tokens)
        fab.start()
        requests = [(0.0, i, prompt, max_tokens) for i, prompt in enumerate(prompts)]
        records = eng.serve(requests, timeout_s=timeout_s, eos=eos, temperature=temperature)
        error = fab.progress()["error"]
        if error:
            raise RuntimeError(f"monofab: device error {error:#x}")
        return [(records[i]["tokens"], records[i]["reason"]) for i in range(len(prompts))]
    finally:
        fab.stop()
        fab.close()


def main():
    ap = argparse.ArgumentParser(description="Generate tokens with a checkpoint through the serving loop.")
    ap.add_argument("--model", required=True, help="folder with config.json and safetensors files")
    ap.add_argument("--prompt", required=True, action="append", help="token ids separated by commas; may be given several times")
    ap.add_argument("--max-tokens", type=int, default=32)
    ap.add_argument("--temperature", type=float, default=0.0)
    ap.add_argument("--eos", type=int, action="append", default=[])
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    args = ap.parse_args()
    from monoserve_b200 import registry
    prompts = [[int(t) for t in p.split(",")] for p in args.prompt]
    for tokens, reason in generate(registry.load(args.model, args.dtype), prompts, args.max_tokens, args.temperature, args.eos):
        print(json.dumps({"tokens": tokens, "reason": reason}), flush=True)


if __name__ == "__main__":
    main()
