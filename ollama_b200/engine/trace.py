"""Replay of a token trace: given ids go through a model step by step and logits come out; nothing is sampled.

Steps arrive on standard input, one JSON object a line: ``{"step": n, "entries": [{"id", "tokens", "want"}, ...], "end": [ids]}``.  The entries of a
step run as one batch; each continues its request, and ``want`` indexes the tokens whose logits go to ``<out>/<step>.f32`` (little-endian
fp32, a row per index).  Requests named in ``end`` give their slot and pages back.  ``done <step>`` on standard output answers each step.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

SLOTS = 4


def replay(backend, lines, out_dir: str, say=print) -> None:
    """Run the steps of ``lines`` on ``backend`` (slots and cache allocated)."""
    import numpy as np
    free = list(range(backend.n_slots - 1, -1, -1))
    live: dict[str, list[int]] = {}            # request -> [slot, tokens so far]
    for line in lines:
        if not line.strip():
            continue
        st = json.loads(line)
        segs, want = [], []
        for e in st["entries"]:
            if e["id"] not in live:
                live[e["id"]] = [free.pop(), 0]
            slot, past = live[e["id"]]
            if not e["tokens"]:
                continue
            segs.append((slot, e["tokens"], past))
            want.append(e.get("want") or [])
            live[e["id"]][1] += len(e["tokens"])
        logits = backend.step(segs, want) if segs else None
        if logits is not None:
            part = os.path.join(out_dir, f"{st['step']}.f32.part")
            logits.float().cpu().numpy().astype(np.dtype("<f4"), copy=False).tofile(part)
            os.replace(part, os.path.join(out_dir, f"{st['step']}.f32"))
        for r in st.get("end") or []:
            if r in live:
                slot, _ = live.pop(r)
                backend.free_slot(slot)
                free.append(slot)
        say(f"done {st['step']}")


def add_arguments(ap: argparse.ArgumentParser) -> None:
    ap.add_argument("--model", required=True, help="checkpoint directory (config.json, model.safetensors) or GGUF file")
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16", help="precision of weights, activations and cache")
    ap.add_argument("--out", required=True, help="directory of the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="size of the page pool: tokens of all open requests together")


def main(argv: list[str] | None = None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a token trace through a model and write logits.")
    add_arguments(ap)
    return run(ap.parse_args(argv))


def run(args: argparse.Namespace) -> int:
    from .backend import make_backend, open_model
    from .cache import PAGE
    from .runner import RunnerOptions
    with open_model(args.model) as g:
        backend = make_backend(g, "cuda", opts=RunnerOptions(dtype=args.dtype))
    if not hasattr(backend, "step"):
        raise SystemExit(f"{backend.cfg.arch} models have no mixed step to replay a trace with")
    pool = -(-args.max_tokens // PAGE) * PAGE        # whole pages
    backend.alloc(SLOTS, pool, pool_tokens=pool)
    replay(backend, sys.stdin, args.out, lambda s: print(s, flush=True))
    backend.close()
    return 0
