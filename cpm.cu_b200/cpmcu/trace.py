"""Trace runner: feeds given token ids through a model, step by step, and writes logits (`bin/trace_run`).

Steps arrive as one JSON object a line on standard input,
    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}
and for a step in which logits are wanted OUT/<step>.f32 receives them as little-endian float32, [wanted, vocab], in the
order of `want`.  `done <step>` on standard output ends a step.  One sequence is live at a time: a request keeps the cache
until it is in `end`.
"""
import argparse
import json
import os
import sys

import torch


class Trace:
    def __init__(self, llm):
        self.llm, self.live, self.length = llm, None, 0

    def step(self, step):
        """Runs one step; returns the wanted logits as a float32 CPU tensor, or None."""
        entries = step["entries"]
        if len(entries) > 1:
            raise ValueError("one request per step: the cache holds a single sequence")
        out = None
        for e in entries:
            if self.live is None:
                self.live, self.length = e["id"], 0
            if e["id"] != self.live:
                raise ValueError("request %r began before %r ended: the cache holds a single sequence" % (e["id"], self.live))
            vocab = self.llm.config.vocab_size
            if any(not 0 <= t < vocab for t in e["tokens"]):
                raise ValueError("token id outside the vocabulary")
            logits = self.llm.extend(e["tokens"], self.length, e["want"])
            self.length += len(e["tokens"])
            if e["want"]:
                out = logits.float().cpu()
        if self.live in step.get("end", []):
            self.live, self.length = None, 0
        return out


def main(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay token ids through a model and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and the weights")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, default=4096, help="most tokens live at any time")
    a = ap.parse_args(argv)
    from .models import open_model
    os.environ["CPMCU_MAX_TOKENS"] = str((max(a.max_tokens, 1) + 127) // 128 * 128)
    try:
        llm = open_model(a.model, dtype=getattr(torch, a.dtype), chunk_length=min(1024, max(64, a.max_tokens)))
    except RuntimeError as e:
        if a.dtype == "float32" and "torch_dtype" in str(e):
            print("trace_run: %s" % e, file=sys.stderr)
            return 3
        raise
    trace = Trace(llm)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        out = trace.step(step)
        if out is not None:
            out.numpy().astype("<f4").tofile(os.path.join(a.out, "%d.f32" % step["step"]))
        print("done %d" % step["step"], flush=True)
    return 0
