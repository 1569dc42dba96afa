"""Command line.

    python -m flexllm_b200 models
    python -m flexllm_b200 generate --model DIR --prompt 12,7,90 [--prompt ...] --n-new 16 [--dtype bfloat16|float32|int8]
                                    [--top-k K --lanes L --seed S] [--max-prefill N] [--no-graph]
"""
import argparse
import json
import random
import sys

from . import models


def main(argv=None):
    ap = argparse.ArgumentParser(prog="flexllm_b200")
    sub = ap.add_subparsers(dest="cmd", required=True)
    sub.add_parser("models", help="list the model registry")
    g = sub.add_parser("generate", help="token ids in, token ids out")
    g.add_argument("--model", required=True, help="folder with config.json and the weights")
    g.add_argument("--prompt", action="append", required=True, help="comma-separated token ids; repeat for a batch of equal lengths")
    g.add_argument("--n-new", type=int, default=16)
    g.add_argument("--dtype")
    g.add_argument("--top-k", type=int, default=0, help="0: greedy")
    g.add_argument("--lanes", type=int, default=1, help="slices of the vocabulary in top-k sampling (must divide it)")
    g.add_argument("--seed", type=int, default=0)
    g.add_argument("--max-prefill", type=int, default=2048)
    g.add_argument("--no-graph", action="store_true")
    a = ap.parse_args(argv)
    if a.cmd == "models":
        for n in sorted(models.REGISTRY):
            e = models.REGISTRY[n]
            print("%s (%s): %s" % (n, ", ".join(e.dtypes), " ".join(e.__doc__.split())))
        return 0
    from . import build
    build.build()
    prompts = [[int(t) for t in p.split(",")] for p in a.prompt]
    B, n = len(prompts), len(prompts[0])
    m = models.load(a.model, max_batch=B, max_prefill=a.max_prefill, max_ctx=n + a.n_new, dtype=a.dtype)
    if a.top_k:
        r = random.Random(a.seed)
        m.set_sampling_host(a.lanes, a.top_k, [r.random() for _ in range(a.n_new * B)], a.n_new, B)
    for row in m.generate(prompts, a.n_new, use_graph=not a.no_graph):
        print(json.dumps(row))
    m.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
