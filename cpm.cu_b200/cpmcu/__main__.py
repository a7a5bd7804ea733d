"""Command line: generate from a checkpoint directory, whatever model class its config.json names.

    python -m cpmcu --model DIR --tokens 5,17,3 --max-new 32          token ids in, token ids out
    python -m cpmcu --model DIR --prompt "..." --max-new 32           with the checkpoint's tokenizer
"""
import argparse
import os
import sys

import torch

from .models import open_model


def main(argv=None):
    ap = argparse.ArgumentParser(prog="cpmcu", description="Generate from a checkpoint directory.")
    ap.add_argument("--model", required=True)
    src = ap.add_mutually_exclusive_group(required=True)
    src.add_argument("--tokens", help="prompt as token ids with commas between them")
    src.add_argument("--prompt", help="prompt text (needs a tokenizer)")
    ap.add_argument("--max-new", type=int, default=32)
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16", help="float32: layered models only")
    ap.add_argument("--temperature", type=float, default=0.0, help="0: greedy")
    ap.add_argument("--seed", type=int, default=None)
    ap.add_argument("--stop", default="", help="token ids that end the generation")
    ap.add_argument("--chunk-length", type=int, default=1024)
    ap.add_argument("--memory-limit", type=float, default=0.8)
    ap.add_argument("--max-tokens", type=int, default=None, help="cap on the tokens the cache holds")
    a = ap.parse_args(argv)
    if a.max_tokens:
        os.environ["CPMCU_MAX_TOKENS"] = str((a.max_tokens + 127) // 128 * 128)
    llm = open_model(a.model, dtype=getattr(torch, a.dtype), temperature=a.temperature, random_seed=a.seed,
                     chunk_length=a.chunk_length, memory_limit=a.memory_limit)
    if a.prompt is not None and llm.tokenizer is None:
        ap.error("this model has no tokenizer: give --tokens")
    ids = [int(t) for t in a.tokens.split(",")] if a.tokens else llm.tokenizer(a.prompt)["input_ids"]
    stop = [int(t) for t in a.stop.split(",") if t]
    out, decode_s, prefill_s = llm.generate(torch.tensor(ids, dtype=torch.int32, device="cuda"), a.max_new, stop)
    if llm.tokenizer is not None:
        print(llm.tokenizer.decode(out))
    print(",".join(map(str, out)))
    print("prefill %.4f s, decode %.4f s, %d tokens" % (prefill_s, decode_s, len(out)), file=sys.stderr)
    return 0


if __name__ == "__main__":
    sys.exit(main())
