"""Replay of a trace: given token ids go through a model step by step and the logits asked for are written out.

Standard input carries one JSON object per line, {"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}: the next
tokens of each request, the places among them whose logits are wanted, and the requests that are over after the step (their
slots are given back).  OUT/<step>.f32 receives the wanted logits in order, little-endian fp32 [wanted, vocab]; "done <step>"
goes to standard output after every step.  Nothing is sampled.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np


def replay(model, lines, out_dir: str, say) -> None:
    live: dict[str, list] = {}  # request -> [slot, tokens fed so far]
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        rows = []
        for e in step.get("entries", []):
            if e["id"] not in live:
                live[e["id"]] = [model.acquire_slot(), 0]
            slot, at = live[e["id"]]
            want = e.get("want", [])
            logits = model.feed(slot, e["tokens"], at, want)
            live[e["id"]][1] = at + len(e["tokens"])
            if len(want):
                rows.append(logits)
        if rows:
            with open(os.path.join(out_dir, f"{step['step']}.f32"), "wb") as f:
                f.write(np.ascontiguousarray(np.concatenate(rows), "<f4").tobytes())
        for i in step.get("end", []):
            if i in live:
                model.release_slot(live.pop(i)[0])
        say(f"done {step['step']}")


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a trace of token ids through a model and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, default=8192, help="most tokens that live requests hold at any time")
    ap.add_argument("--slots", type=int, default=4, help="most requests that are live at any time")
    a = ap.parse_args(argv)
    from . import registry
    try:
        driver = registry.load(a.model, a.dtype, max_context=max(a.max_tokens, 1) + 64, max_batch=a.slots)
    except registry.UnsupportedDtype as e:
        print(e, file=sys.stderr)
        return 3

    def say(text: str) -> None:
        print(text, flush=True)

    os.makedirs(a.out, exist_ok=True)
    replay(driver.model, sys.stdin, a.out, say)
    return 0


if __name__ == "__main__":
    sys.exit(main())
