"""Replays a trace of token ids through a model, step by step, and writes logits.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Standard input holds one JSON object a line: {"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}. A step feeds
its entry's tokens to the runner's step call (the call generation uses), writes the logits of the wanted tokens to
DIR/<step>.f32 (little-endian fp32 rows) and prints "done <step>". One request is live at a time; `end` gives back what
it holds in the cache. Exit code 3: the model does not compute in the asked-for number format.
"""
import argparse
import json
import os
import sys

from . import models

MAX_CHUNK = 4096        # tokens per pass through the layers; longer steps run in chunks


class Replay:
    def __init__(self, model):
        self.model, self.live = model, None

    def step(self, entries, end):
        """Runs one step; returns the wanted logits (array('f'), rows of vocab)."""
        if len(entries) > 1:
            raise ValueError("a step carries one request")
        out = None
        for e in entries:
            if self.live is None:
                self.model.reset()
                self.live = e["id"]
            elif self.live != e["id"]:
                raise ValueError("request %r starts while %r is live" % (e["id"], self.live))
            if e["tokens"]:
                out, _ = self.model.step([e["tokens"]], e.get("want", []))
        for i in end:
            if i == self.live:
                self.live = None
                self.model.reset()
        return out


def main(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a trace of token ids through a model and write logits.")
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", required=True, choices=sorted(models.DTYPES))
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, required=True)
    a = ap.parse_args(argv)
    from . import build
    build.build()
    n = max(1, a.max_tokens)
    try:
        model = models.load(a.model, max_batch=1, max_prefill=min(n, MAX_CHUNK), max_ctx=n, dtype=a.dtype)
    except models.UnsupportedDtype as e:
        print(e, file=sys.stderr)
        return 3
    replay = Replay(model)
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        out = replay.step(s.get("entries", []), s.get("end", []))
        if out is not None and len(out):
            if sys.byteorder != "little":
                out.byteswap()
            with open(os.path.join(a.out, "%d.f32" % s["step"]), "wb") as f:
                out.tofile(f)
        print("done %d" % s["step"], flush=True)
    model.close()
    return 0
