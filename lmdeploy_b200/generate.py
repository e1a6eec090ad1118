"""Command line: generate token ids with a checkpoint folder, through the scheduler.

    python -m lmdeploy_b200.generate --model DIR --ids "1 5 9" [--ids "7 7"] --max-new-tokens 32 [--top-k 40 --top-p 0.8 ...]

The folder decides the model (`--list` prints the known architectures).  Every --ids is one request (token ids, there is no
tokenizer here); requests share the running batch.  One JSON line per request: its number, state and generated tokens.
"""
from __future__ import annotations

import argparse
import json
import sys


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="lmdeploy_b200.generate", description="generate token ids with a checkpoint folder")
    ap.add_argument("--list", action="store_true", help="print the known architectures and leave")
    ap.add_argument("--model", help="checkpoint folder")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--ids", action="append", default=[], help="token ids of one request, separated by spaces or commas")
    ap.add_argument("--max-new-tokens", type=int, default=32)
    ap.add_argument("--session-len", type=int, default=4096)
    ap.add_argument("--max-batch-size", type=int, default=32)
    ap.add_argument("--max-prefill-tokens", type=int, default=0)
    ap.add_argument("--top-k", type=int, default=0)
    ap.add_argument("--top-p", type=float, default=0.0)
    ap.add_argument("--temperature", type=float, default=0.0)
    ap.add_argument("--repetition-penalty", type=float, default=0.0)
    ap.add_argument("--seed", type=int, default=0)
    ap.add_argument("--start-id", type=int, default=1)
    ap.add_argument("--end-id", type=int, default=-1, help="token that ends a request (-1: none)")
    ap.add_argument("--no-graph", action="store_true", help="decode steps as single launches instead of a CUDA graph")
    ap.add_argument("--device", type=int, default=0)
    a = ap.parse_args(argv)

    import torch

    from . import decoder, llama
    if a.list:
        print("\n".join(decoder.architectures()))
        return 0
    if not a.model or not a.ids:
        ap.error("--model and at least one --ids are needed")
    requests = [[int(t) for t in ids.replace(",", " ").split()] for ids in a.ids]
    torch.cuda.set_device(a.device)
    model = decoder.Model.open(a.model, a.dtype, a.max_batch_size, a.session_len, a.max_prefill_tokens, a.device)
    batch = llama.Batch(model, a.max_batch_size, a.start_id, a.end_id)
    rc = 0
    with torch.cuda.stream(torch.cuda.Stream(a.device)):
        for i, ids in enumerate(requests):
            if batch.submit(i, ids, a.max_new_tokens, top_k=a.top_k, top_p=a.top_p, temperature=a.temperature,
                            repetition_penalty=a.repetition_penalty, random_seed=a.seed, ignore_eos=a.end_id < 0) != 0:
                print(f"request {i} was refused", file=sys.stderr)
                rc = 1
        batch.run(use_graph=not a.no_graph)
        model.check_status()
        for i in range(len(requests)):
            tokens, state = batch.output(i)
            rc = rc or int(state != batch.FINISHED)
            print(json.dumps({"request": i, "state": "finished" if state == batch.FINISHED else "failed", "tokens": tokens}))
    batch.close()
    model.close()
    return rc


if __name__ == "__main__":
    sys.exit(main())
