"""Command line: ``python -m rotor_b200 <command>``.

  generate  --model DIR --prompt "1 2 3" [--prompt ...]   token ids in, token ids out
  trace     --model DIR --dtype D --out DIR [--max-tokens N]   replay steps from standard input
  info      [--model DIR]                                 known architectures; a model folder's choice
"""
from __future__ import annotations

import argparse
import json
import sys


def _generate(a):
    from .generation import GreedySampling, TextGenerator, TopKSampling, TopPSampling
    from .registry import load_model
    from .synth import PassThroughTokenizer
    longest = max(len(p.split()) for p in a.prompt) + a.max_new_tokens
    model = load_model(a.model, dtype=a.dtype, max_seq=longest, max_batch=len(a.prompt))
    if len(a.prompt) > 1:
        if a.sampling != "greedy":
            raise SystemExit("several prompts are generated greedily as one batch")
        for row in model.generate_greedy_batch([[int(t) for t in p.split()] for p in a.prompt], a.max_new_tokens):
            print(" ".join(str(int(t)) for t in row))
        return 0
    strategy = {"greedy": GreedySampling, "top-k": lambda: TopKSampling(a.top_k, seed=a.seed),
                "top-p": lambda: TopPSampling(a.top_p, seed=a.seed)}[a.sampling]()
    gen = TextGenerator(model, PassThroughTokenizer(), sampling_strategy=strategy, temperature=a.temperature,
                        max_length=longest)
    text = gen.generate(a.prompt[0], max_new_tokens=a.max_new_tokens, stop_on_eos=False)
    print(" ".join(text.split()[len(a.prompt[0].split()):]))
    return 0


def _trace(a):
    from .registry import UnsupportedDtype, load_model
    from .trace import replay
    try:
        model = load_model(a.model, dtype=a.dtype, max_seq=max(1, a.max_tokens))
    except UnsupportedDtype as e:
        print(e, file=sys.stderr)
        return 3
    replay(model, sys.stdin, a.out, lambda s: print(s, flush=True))
    return 0


def _info(a):
    from .registry import DEFAULT, architectures
    print("architectures: " + ", ".join(architectures()))
    if a.model:
        with open(f"{a.model}/config.json") as f:
            print(f"{a.model}: " + json.load(f).get("architecture", DEFAULT))
    return 0


def main(argv=None):
    ap = argparse.ArgumentParser(prog="rotor_b200")
    sub = ap.add_subparsers(dest="command", required=True)
    g = sub.add_parser("generate", help="token ids in, token ids out")
    g.add_argument("--model", required=True)
    g.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    g.add_argument("--prompt", action="append", required=True, help="token ids separated by spaces; repeat for a batch")
    g.add_argument("--max-new-tokens", type=int, default=32)
    g.add_argument("--sampling", default="greedy", choices=["greedy", "top-k", "top-p"])
    g.add_argument("--top-k", type=int, default=50)
    g.add_argument("--top-p", type=float, default=0.9)
    g.add_argument("--temperature", type=float, default=1.0)
    g.add_argument("--seed", type=int, default=0)
    g.set_defaults(run=_generate)
    t = sub.add_parser("trace", help="replay steps from standard input")
    t.add_argument("--model", required=True)
    t.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    t.add_argument("--out", required=True, help="folder for the logits files")
    t.add_argument("--max-tokens", type=int, default=2048, help="most tokens a live request holds")
    t.set_defaults(run=_trace)
    i = sub.add_parser("info", help="known architectures")
    i.add_argument("--model")
    i.set_defaults(run=_info)
    a = ap.parse_args(argv)
    return a.run(a)


if __name__ == "__main__":
    sys.exit(main())
