"""Replays a trace: given token ids go through a model step by step, and the logits that are asked for go to files.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Standard input has one step a line, {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["a"]}:
the next tokens of a request, the places among them whose logits are wanted, and the requests that are finished after the
step. A step with wanted logits writes OUT/<step>.f32 (little-endian, [wanted, vocab]); every step answers "done <step>" on
standard output. Nothing is sampled; the model, its state and its kernels are those generation uses. A step has one entry,
and a request ends before the next one begins."""

from __future__ import annotations

import argparse
import json
import pathlib
import sys

import numpy as np

MAX_RUN = 2048  # tokens per forward; longer portions go through in several


def replay(model, lines, out: pathlib.Path, reply) -> None:
    live, at = None, 0
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        rows = []
        if len(step["entries"]) > 1:
            raise ValueError("a step has one entry: the model keeps the state of one sequence")
        for e in step["entries"]:
            if live is None:
                live, at = e["id"], 0
            elif live != e["id"]:
                raise ValueError(f"request {e['id']} begins while {live} is not finished")
            want = [int(w) for w in e["want"]]
            got = model.feed(e["tokens"], at, set(want))
            order = {w: i for i, w in enumerate(sorted(set(want)))}
            rows += [got[order[w]] for w in want]
            at += len(e["tokens"])
        if rows:
            np.stack(rows).astype("<f4").tofile(out / f"{step['step']}.f32")
        if live in step["end"]:
            live = None
        reply(f"done {step['step']}")


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Feeds given tokens through a model step by step and writes logits.")
    ap.add_argument("--model", required=True, help="a `.brasa` file, or a folder with config.json and model.safetensors")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, type=pathlib.Path)
    ap.add_argument("--max-tokens", required=True, type=int, help="the most tokens a live request holds")
    ap.add_argument("--device", type=int, default=0)
    a = ap.parse_args(argv)
    from . import Context, model_class
    ctx = Context(a.device)
    run = min(MAX_RUN, a.max_tokens)
    model = model_class(a.model).load_in(ctx, a.model, a.dtype, a.max_tokens, run, max_logit_rows=min(run, 256))
    replay(model, sys.stdin, a.out, lambda text: print(text, flush=True))
    model.free()
    ctx.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
