"""Command line: python -m denograd_b200 <generate | info | trace> ...

  generate  continue a prompt of token ids:  --model DIR --tokens 1,2,3 --max-new 32 [--temperature T --top-k K --top-p P]
  info      what a model folder holds, without touching the GPU
  trace     replay a trace of token ids (same options as bin/trace_run)
"""
from __future__ import annotations

import argparse
import json
import sys


def generate(a) -> int:
    import numpy as np

    from . import rand, registry
    if a.text and not a.tokenizer:
        raise SystemExit("--text needs --tokenizer (a vocabulary file)")
    tok = None
    if a.tokenizer:
        from .tokenizer import Tokenizer
        tok = Tokenizer.llama(a.tokenizer)
    prompt = tok.encode(a.text) if a.text else [int(t) for t in a.tokens.replace(",", " ").split()]
    if not prompt:
        raise SystemExit("an empty prompt: give --tokens or --text")
    rand.manual_seed(a.seed)
    llm = registry.load(a.model, a.dtype, max_context=a.max_context or len(prompt) + a.max_new, temperature=a.temperature, top_k=a.top_k,
                        top_p=a.top_p, alpha_f=a.alpha_f, alpha_p=a.alpha_p)
    out = []
    if a.temperature < 1e-6:
        out = llm.generate(np.array(prompt, np.int32), a.max_new, batched=True)[0].tolist()
    else:
        cur = int(llm._prefill(prompt, batched=True).numpy()[0])
        for i in range(a.max_new):
            out.append(cur)
            if i + 1 < a.max_new:
                cur = llm._call(cur)
                llm.start_pos += 1
    print(tok.decode(out) if tok else " ".join(str(t) for t in out))
    return 0


def info(a) -> int:
    from . import registry
    c = registry.read_config(a.model)
    print(json.dumps({"architecture": registry.architecture(c), "config": c}, indent=1))
    return 0


def main(argv=None) -> int:
    argv = list(sys.argv[1:] if argv is None else argv)
    if argv and argv[0] == "trace":
        from .trace import main as trace_main
        return trace_main(argv[1:])
    ap = argparse.ArgumentParser(prog="python -m denograd_b200", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    sub = ap.add_subparsers(dest="cmd", required=True)
    g = sub.add_parser("generate")
    g.add_argument("--model", required=True)
    g.add_argument("--dtype", default=None, help="element type (default: the one the model is served with)")
    g.add_argument("--tokens", default="", help="prompt as token ids")
    g.add_argument("--text", default="", help="prompt as text (needs --tokenizer)")
    g.add_argument("--tokenizer", default="")
    g.add_argument("--max-new", type=int, default=32)
    g.add_argument("--max-context", type=int, default=0)
    g.add_argument("--seed", type=int, default=0)
    g.add_argument("--temperature", type=float, default=0.0)
    g.add_argument("--top-k", type=int, default=0)
    g.add_argument("--top-p", type=float, default=0.0)
    g.add_argument("--alpha-f", type=float, default=0.0)
    g.add_argument("--alpha-p", type=float, default=0.0)
    g.set_defaults(run=generate)
    i = sub.add_parser("info")
    i.add_argument("--model", required=True)
    i.set_defaults(run=info)
    sub.add_parser("trace", help="replay a trace of token ids (see --help of bin/trace_run)")
    a = ap.parse_args(argv)
    return a.run(a)


if __name__ == "__main__":
    sys.exit(main())
