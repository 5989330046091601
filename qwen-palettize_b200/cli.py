"""Command line of the framework.

    python cli.py models                                             registered architectures
    python cli.py generate --model DIR --tokens 5,17,3 [--tokens ...] continue token sequences
    python cli.py trace --model DIR --dtype T --out DIR --max-tokens N  replay given tokens from standard input and write logits

A trace is one JSON object per line, {"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}. Each step runs the entries'
tokens from the state earlier steps left, writes the logits at the wanted places to OUT/<n>.f32 (little-endian fp32, [wanted, vocab])
and prints "done <n>".
"""
from __future__ import annotations

import argparse
import json
import os
import sys

_HERE = os.path.dirname(os.path.abspath(__file__))
if _HERE not in sys.path:
    sys.path.insert(0, _HERE)

EXIT_DTYPE = 3


def _load(args):
    import build
    import model_registry as R
    build.build()
    return R.load_model(args.model, args.dtype)


def cmd_models(_args) -> int:
    import model_registry as R
    for name, cls in sorted(R.ARCHITECTURES.items()):
        print(name, ",".join(k for k, t in R.DTYPES.items() if t in cls.DTYPES))
    return 0


def cmd_generate(args) -> int:
    from engine import Engine, SamplingParams
    prompts = [[int(t) for t in p.replace(",", " ").split()] for p in args.tokens]
    params = SamplingParams(args.max_new, args.temperature, args.top_k, args.seed, tuple(args.stop))
    eng = Engine(_load(args), max(len(p) for p in prompts) + args.max_new, args.portion, args.max_live)
    for out in eng.generate(prompts, params):
        print(" ".join(map(str, out)), flush=True)
    return 0


def cmd_trace(args) -> int:
    import numpy as np
    from engine import Engine
    eng = Engine(_load(args), args.max_tokens)
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        parts = []
        for e in s.get("entries", []):
            got = eng.step(e["id"], e["tokens"], e.get("want", []))
            if got is not None:
                parts.append(got.cpu().numpy().astype("<f4"))
        for rid in s.get("end", []):
            eng.end(rid)
        if parts:
            np.concatenate(parts).tofile(os.path.join(args.out, f"{s['step']}.f32"))
        else:
            import torch
            torch.cuda.synchronize()
        print(f"done {s['step']}", flush=True)
    import plz_native
    st = plz_native.device_status()
    if st[0]:
        print(f"device status {st}", file=sys.stderr)
        return 1
    return 0


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="plz", description=__doc__.split("\n")[0])
    sub = ap.add_subparsers(dest="cmd", required=True)
    sub.add_parser("models", help="list the registered architectures").set_defaults(fn=cmd_models)

    def common(p):
        p.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
        p.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])

    g = sub.add_parser("generate", help="continue token sequences")
    common(g)
    g.add_argument("--tokens", action="append", required=True, help="a prompt as token ids, e.g. 5,17,3 (may be repeated)")
    g.add_argument("--max-new", type=int, default=16)
    g.add_argument("--temperature", type=float, default=0.0, help="0: greedy")
    g.add_argument("--top-k", type=int, default=0)
    g.add_argument("--seed", type=int, default=0)
    g.add_argument("--stop", type=int, action="append", default=[], help="token id that ends a sequence")
    g.add_argument("--portion", type=int, default=2048, help="most prompt tokens per step")
    g.add_argument("--max-live", type=int, default=8, help="sequences in flight")
    g.set_defaults(fn=cmd_generate)

    t = sub.add_parser("trace", help="replay tokens from standard input and write logits")
    common(t)
    t.add_argument("--out", required=True)
    t.add_argument("--max-tokens", type=int, required=True)
    t.set_defaults(fn=cmd_trace)
    args = ap.parse_args(argv)
    try:
        if args.cmd != "models":
            import model_registry as R
            R.check_dtype(R.read_config(args.model), args.dtype)
    except R.UnsupportedDtype as e:
        print(e, file=sys.stderr)
        return EXIT_DTYPE
    return args.fn(args)


if __name__ == "__main__":
    sys.exit(main())
