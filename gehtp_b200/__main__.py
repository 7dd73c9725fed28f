"""Command line of the package:

    python -m gehtp_b200 generate --model DIR --prompt 1,2,3 [--prompt ...] --max-new N   greedy continuations
    python -m gehtp_b200 trace    --model DIR --dtype T --out DIR --max-tokens N          replay of a token trace (stdin)
    python -m gehtp_b200 compile  --model DIR --out FILE.wtop                             runlist + manifest for gehtp_run

DIR is a model folder (config.json, model.safetensors); the model is chosen by its `architecture`.
"""
import argparse
import json
import sys


def parser():
    ap = argparse.ArgumentParser(prog="gehtp_b200")
    sub = ap.add_subparsers(dest="cmd", required=True)

    def common(p):
        p.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
        p.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
        p.add_argument("--max-tokens", type=int, default=2048, help="positions the caches hold")
    g = sub.add_parser("generate", help="greedy continuation of prompts given as token ids")
    common(g)
    g.add_argument("--prompt", action="append", required=True, help="token ids with commas between them")
    g.add_argument("--max-new", type=int, default=16)
    g.add_argument("--stop", default="", help="token ids that end a continuation")
    t = sub.add_parser("trace", help="replay a trace of token ids from standard input")
    common(t)
    t.add_argument("--out", required=True, help="folder the logits are written to")
    c = sub.add_parser("compile", help="write the runlist of a model")
    common(c)
    c.add_argument("--out", required=True, help="blob to write; the manifest goes to <out>.json")
    c.add_argument("--max-rows", type=int, default=2048)
    c.add_argument("--max-sel", type=int, default=64)
    return ap


def ids(text):
    return [int(x) for x in text.split(",") if x.strip()]


def main(argv=None):
    args = parser().parse_args(argv)
    if args.cmd == "trace":
        from . import trace
        return trace.main(args)
    from .registry import load_model
    model = load_model(args.model)
    if args.cmd == "compile":
        blob, man = model.runlist(args.dtype, args.max_tokens, args.max_rows, args.max_sel)
        blob.tofile(args.out)
        with open(args.out + ".json", "w") as f:
            json.dump(man, f, indent=1)
        return 0
    from .session import Request, Scheduler, Session
    session = Session(model, args.dtype, args.max_tokens)
    sched = Scheduler(session)
    for i, p in enumerate(args.prompt):
        sched.submit(Request(i, ids(p), args.max_new, tuple(ids(args.stop))))
    bad = 0
    for r in sched.run():
        print(r.error if r.error else ",".join(map(str, r.tokens)))
        bad += r.error is not None
    session.close()
    return 1 if bad else 0


if __name__ == "__main__":
    sys.exit(main())
