"""Replays a trace of token ids through a model and writes logits: one JSON object per line of standard input,

    {"step": n, "entries": [{"id": ..., "tokens": [...], "want": [...]}], "end": [...]}

runs the tokens of the step's entry from the states earlier steps of that request left, writes the logits at the wanted
places to OUT/<n>.f32 (little-endian fp32, [wanted, vocab]) when there are any, and prints "done <n>". One request is
live at a time; a request named in "end" gives its states back."""
import json
import os
import sys


def replay(session, lines, out_dir, answer):
    live = None
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = step.get("entries", [])
        if len(entries) > 1:
            raise ValueError("step %s has %d entries; one sequence is live at a time" % (step["step"], len(entries)))
        logits = []
        for e in entries:
            if live is None:
                session.reset()
                live = e["id"]
            elif live != e["id"]:
                raise ValueError("request %s begins before %s has ended" % (e["id"], live))
            rows = session.feed(e["tokens"], e.get("want", []))
            if len(rows):
                logits.append(rows)
        if logits:
            path = os.path.join(out_dir, "%d.f32" % step["step"])
            with open(path, "wb") as f:
                for rows in logits:
                    f.write(rows.astype("<f4").tobytes())
        if live in step.get("end", []):
            session.reset()
            live = None
        answer("done %d" % step["step"])


def main(args):
    from .registry import load_model
    from .session import Session
    session = Session(load_model(args.model), args.dtype, args.max_tokens)

    def answer(text):
        sys.stdout.write(text + "\n")
        sys.stdout.flush()
    replay(session, iter(sys.stdin.readline, ""), args.out, answer)
    session.close()
    return 0
