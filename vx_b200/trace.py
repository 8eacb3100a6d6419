"""Replays a trace of token ids through a model, step by step, and writes the
logits that the trace asks for (bin/trace_run).

Steps come on standard input, one JSON object a line:

    {"step": 7, "entries": [{"id": "x9", "tokens": [12, 40, 8], "want": [1]}], "end": ["x9"]}

"want" holds places among the entry's tokens; the logits there go to
<out>/<step>.f32 (little-endian f32, [places, vocab]).  After a step the line
"done <step>" is printed.  A request's tokens may come in any portions; requests
come one after another, and one in "end" gives its cache rows back.
"""
import argparse
import json
import os
import sys

import numpy as np


class Replay:
    """One decoder, and which request its cache belongs to."""

    def __init__(self, decoder):
        self.decoder, self.owner = decoder, None

    def feed(self, request, tokens, want):
        if self.owner is None:
            self.decoder.reset()
            self.owner = request
        elif self.owner != request:
            raise ValueError("request %r begins before %r has ended"
                             % (request, self.owner))
        order = sorted(want)
        if any(not 0 <= w < len(tokens) for w in order):
            raise ValueError("a wanted place is not among the tokens of %r" % request)
        places = sorted(set(order))
        rows = self.decoder.feed(tokens, places)
        at = {w: i for i, w in enumerate(places)}
        return rows[[at[w] for w in want]] if want else rows[:0]

    def step(self, entries, end):
        rows = [self.feed(e["id"], e["tokens"], e.get("want", [])) for e in entries]
        if self.owner in end:
            self.owner = None
        return [r for r in rows if len(r)]


def main(argv=None):
    ap = argparse.ArgumentParser(description=__doc__.split("\n\n")[0])
    ap.add_argument("--model", required=True, help="folder of the model")
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, default=4096,
                    help="the most tokens a request has")
    args = ap.parse_args(argv)

    from . import models
    from .lib import use
    use(models.library(args.model))
    try:
        decoder = models.load(args.model, args.dtype, max(args.max_tokens, 1))
    except models.UnsupportedDtype as e:
        print(e, file=sys.stderr)
        return 3
    replay = Replay(decoder)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        rows = replay.step(step.get("entries", []), step.get("end", []))
        if rows:
            np.concatenate(rows).astype("<f4").tofile(
                os.path.join(args.out, "%d.f32" % step["step"]))
        print("done %d" % step["step"], flush=True)
    decoder.close()
    return 0
