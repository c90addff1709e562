"""``trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N``: replay a trace of given tokens through the serving engine
and write the logits it asks for.

Steps come on standard input, one JSON object a line: ``{"step": 0, "entries": [{"id": "a", "tokens": [..], "want": [..]}], "end": [..]}``.
All entries of a step are one batch and continue from the cache and state of earlier steps; ``want`` lists the places among an entry's
tokens whose logits are written, in order, to ``OUT/<step>.f32`` (little-endian f32 ``[wanted, vocab]``; no file when nothing is wanted);
``end`` names the requests that are finished after the step.  ``done <step>`` is printed after every step.  The cache pool holds ``N``
tokens (each request's count rounded up to whole pages) and four live requests.  Exit code 3: the model has no 32-bit path."""
from __future__ import annotations

import argparse
import json
import os
import sys

import torch

LIVE = 4


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run")
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, required=True)
    ap.add_argument("--device", default="cuda", help=argparse.SUPPRESS)
    a = ap.parse_args(argv)
    from .. import _native
    from ..models.registry import family_of, make_engine, open_text_model, read_config
    dtype = getattr(torch, a.dtype)
    if dtype == torch.float32 and a.device.startswith("cuda") and not family_of(read_config(a.model)).f32_on_gpu:
        print("this model has no 32-bit CUDA path", file=sys.stderr)
        return 3
    _native.core()
    model, fam, _ = open_text_model(a.model, a.device, dtype, compile_missing=True)
    eng = make_engine(model, fam, a.max_tokens, LIVE, a.device)
    live: dict[str, int] = {}
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        for e in step["entries"]:
            if e["id"] not in live:
                live[e["id"]] = eng.open_sequence()
        logits = eng.feed([(live[e["id"]], e["tokens"], e.get("want", ())) for e in step["entries"]])
        if logits is not None:
            logits.float().cpu().numpy().astype("<f4").tofile(os.path.join(a.out, f"{step['step']}.f32"))
        if a.device.startswith("cuda"):
            from ..ops import cuda as K
            status = K.last_status()
            if status:
                raise K.KernelError(K._STATUS.get(status, status))
        for rid in step.get("end", ()):
            eng.close_sequence(live.pop(rid))
        print(f"done {step['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
