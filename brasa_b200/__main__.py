"""Command line over token ids (tokenisation is the caller's):

    python -m brasa_b200 info MODEL
    python -m brasa_b200 generate MODEL --prompt 12,7,993 --max-new 64 [--dtype bfloat16|float32] [--temperature T --top-p P --top-k K --seed S]
    python -m brasa_b200 trace --model DIR --dtype D --out DIR --max-tokens N < steps
"""

from __future__ import annotations

import argparse
import sys

from . import Context, Limits, SamplingParams, Session, model_class, model_shape
from . import trace as trace_mod


def info(a) -> int:
    shape, cfg = model_shape(a.model)
    print(f"family {model_class(a.model).__name__}")
    print(f"weights {shape.weight_bytes / 2**20:.1f} MiB")
    for k, v in cfg.items():
        if v:
            print(f"{k} {v}")
    return 0


def generate(a) -> int:
    prompt = [int(t) for t in a.prompt.replace(",", " ").split()]
    ctx = Context(a.device)
    n = a.ctx or len(prompt) + a.max_new + 1
    sess = Session(ctx, a.model, Limits(ctx=n, max_tokens=min(n, 2048), kv=model_class(a.model).kv_type(a.dtype)))
    if a.stop:
        sess.set_stop_ids([int(t) for t in a.stop.split(",")])
    ids, st = sess.generate(prompt, a.max_new, SamplingParams(a.temperature, a.top_k, a.top_p, a.seed))
    print(" ".join(str(int(t)) for t in ids))
    print(f"prompt {st.prompt_tokens} tokens in {st.prefill_ms:.2f} ms, {st.generated} generated, {st.decode_tok_s():.1f} tok/s, stop: {st.stop}", file=sys.stderr)
    sess.free()
    ctx.close()
    return 0


def main(argv=None) -> int:
    argv = sys.argv[1:] if argv is None else argv
    if argv[:1] == ["trace"]:
        return trace_mod.main(argv[1:])
    ap = argparse.ArgumentParser(prog="brasa_b200")
    sub = ap.add_subparsers(dest="cmd", required=True)
    i = sub.add_parser("info", help="family, sizes and weight bytes of a model")
    i.add_argument("model")
    g = sub.add_parser("generate", help="generate from a prompt of token ids")
    g.add_argument("model")
    g.add_argument("--prompt", required=True, help="token ids, separated by commas or spaces")
    g.add_argument("--max-new", type=int, default=64)
    g.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    g.add_argument("--ctx", type=int, default=0)
    g.add_argument("--stop", default="", help="token ids that end the generation")
    g.add_argument("--temperature", type=float, default=0.0)
    g.add_argument("--top-k", type=int, default=0)
    g.add_argument("--top-p", type=float, default=1.0)
    g.add_argument("--seed", type=int, default=0)
    g.add_argument("--device", type=int, default=0)
    sub.add_parser("trace", help="replay a trace of token ids (see bin/trace_run)", add_help=False)
    a = ap.parse_args(argv)
    return info(a) if a.cmd == "info" else generate(a)


if __name__ == "__main__":
    sys.exit(main())
