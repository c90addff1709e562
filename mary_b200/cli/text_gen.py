"""``text_gen --model DIR|PILE (--ids 1,2,3[;4,5,...] | --prompt "...") [--max-new N] [--temperature T --top-k K --top-p P --seed S]``:
continue prompts with any text decoder of the registry, several prompts in one continuous batch.  Without a tokenizer, feed ids and read
ids."""
from __future__ import annotations

import argparse
import sys
import time

import torch


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="text_gen")
    ap.add_argument("--model", required=True, help="a folder with config.json and safetensors, or a pile")
    ap.add_argument("--ids", help="token ids; prompts separated by ';'")
    ap.add_argument("--prompt")
    ap.add_argument("--max-new", type=int, default=32)
    ap.add_argument("--temperature", type=float, default=0.0)
    ap.add_argument("--top-k", type=int, default=0)
    ap.add_argument("--top-p", type=float, default=1.0)
    ap.add_argument("--seed", type=int, default=0)
    ap.add_argument("--max-seqs", type=int, default=64, help="sequences served together")
    ap.add_argument("--prefill-chunk", type=int, default=2048)
    ap.add_argument("--device", default="cuda" if torch.cuda.is_available() else "cpu")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], help="default: bfloat16 on a GPU, float32 on the host")
    a = ap.parse_args(argv)
    if argv is None:                                  # run as a program: fail loudly on any thread
        from ..utils import fatal
        fatal.arm()
    from ..models.registry import make_engine, open_text_model
    from ..ops.sampling import sample
    cuda = a.device.startswith("cuda")
    dtype = getattr(torch, a.dtype or ("bfloat16" if cuda else "float32"))
    t0 = time.time()
    model, fam, tok = open_text_model(a.model, a.device, dtype)
    print(f"loaded {fam.name} in {time.time() - t0:.2f} s", file=sys.stderr)
    if a.prompt is not None:
        if tok is None:
            print("no tokenizer with this model: use --ids", file=sys.stderr)
            return 2
        prompts = [tok.encode(a.prompt, add_special_tokens=False).ids]
    else:
        prompts = [[int(x) for x in p.split(",")] for p in (a.ids or "0").split(";")]
    seqs = min(a.max_seqs, len(prompts))
    page = fam.page_size
    longest = max(len(p) for p in prompts) + a.max_new + 8
    sampler = None
    if a.temperature > 0:
        step = iter(range(1 << 62))
        sampler = lambda logits: sample(logits, a.temperature, a.top_k, a.top_p, a.seed, next(step))  # noqa: E731
    eng = make_engine(model, fam, seqs * ((longest + page - 1) // page) * page, seqs, a.device, prefill_chunk=a.prefill_chunk, sampler=sampler)
    t0 = time.time()
    outs = eng.generate(prompts, a.max_new)
    dt = time.time() - t0
    for o in outs:
        print(tok.decode(o) if a.prompt is not None else ",".join(map(str, o)))
    print(f"{sum(map(len, outs)) / max(dt, 1e-9):.1f} tok/s over {len(prompts)} prompt(s)", file=sys.stderr)
    return 0


if __name__ == "__main__":
    sys.exit(main())
