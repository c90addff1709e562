"""What the tests of the hybrid decoders share: sequences over one shuffled page pool, schedules of unequal portions, weights as a loader or
a checkpoint folder, comparison, a
trace of given tokens."""
from __future__ import annotations

import json
import random

import numpy as np
import torch

from mary_b200.runtime.batch import BatchMeta


def bf16(x):
    return x.to(torch.bfloat16).float()


def prompt(cfg, n, seed=0):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


class Paged:
    """Sequences over one shuffled page pool and shuffled state slots, stepped by hand."""

    def __init__(self, page=16, pages=96, slots=6, device="cpu", seed=0):
        self.rng = random.Random(seed)
        self.page, self.device = page, device
        self.free = list(range(pages))
        self.rng.shuffle(self.free)
        self.slots = list(range(slots))
        self.rng.shuffle(self.slots)
        self.rows, self.len, self.slot = {}, {}, {}

    def step(self, counts: dict):
        for s, n in counts.items():
            if s not in self.rows:
                self.rows[s], self.len[s], self.slot[s] = [], 0, self.slots.pop()
            self.len[s] += n
            while len(self.rows[s]) * self.page < self.len[s]:
                self.rows[s].append(self.free.pop())
        width = max(len(self.rows[s]) for s in counts)
        table = np.array([self.rows[s] + [-1] * (width - len(self.rows[s])) for s in counts], dtype=np.int32)
        return BatchMeta.build(list(counts.values()), [self.len[s] for s in counts], table, self.page, self.device,
                               [self.slot[s] for s in counts])

    def drop(self, s):
        self.free.extend(self.rows.pop(s))
        self.slots.append(self.slot.pop(s))
        del self.len[s]


def schedule(lengths: dict, rng, sizes=(1, 1, 2, 3, 5, 17, 40, 70)):
    """Steps of unequal portions: every step takes a random subset of the unfinished sequences."""
    at = {s: 0 for s in lengths}
    while any(at[s] < n for s, n in lengths.items()):
        live = [s for s in lengths if at[s] < lengths[s]]
        step = {s: min(rng.choice(sizes), lengths[s] - at[s]) for s in live if rng.random() < 0.7} or {live[0]: 1}
        yield {s: (at[s], n) for s, n in step.items()}
        for s, n in step.items():
            at[s] += n


class DictLoader:
    def __init__(self, w):
        self.w = w

    def load_tensor(self, name, dtype=None, device=None):
        t = self.w[name]
        return t if dtype is None else t.to(dtype)

    def shape(self, name):
        return tuple(self.w[name].shape)


def write_folder(path, cfg: dict, w: dict) -> None:
    from mary_b200.format.safetensors import save_file
    bits = {k: v.to(torch.bfloat16).view(torch.int16).numpy().view(np.uint16) for k, v in w.items()}
    save_file(bits, str(path / "model.safetensors"), bf16=set(bits))
    (path / "config.json").write_text(json.dumps(cfg))


def error(got, want) -> float:
    """Largest rms difference of a row relative to the rms of all wanted values."""
    got, want = torch.as_tensor(got).double().cpu(), want.double()
    d = (got - want).flatten(1) if got.dim() > 1 else (got - want)[None]
    return float(d.pow(2).mean(-1).sqrt().max() / want.pow(2).mean().sqrt())


TRACE = [{"step": 0, "entries": [{"id": "a", "tokens": 50, "want": [0, 49]}], "end": []},
         {"step": 1, "entries": [{"id": "b", "tokens": 30, "want": []}], "end": []},
         {"step": 2, "entries": [{"id": "a", "tokens": 1, "want": [0]}, {"id": "c", "tokens": 2, "want": [1]}], "end": ["c"]},
         {"step": 7, "entries": [{"id": "b", "tokens": 25, "want": [3, 24]}, {"id": "d", "tokens": 64, "want": [63]}], "end": ["b"]},
         {"step": 8, "entries": [{"id": "d", "tokens": 1, "want": [0]}, {"id": "a", "tokens": 20, "want": [19]}, {"id": "c", "tokens": 9, "want": [8]}],
          "end": ["a", "c", "d"]}]


def trace_case(cfg, w, run):
    """The trace with tokens filled in and the logits it asks for, by the oracle ``run`` (an id that comes again after its end is a new request)."""
    rng, hist, lines, want = np.random.default_rng(3), {}, [], {}
    for s in TRACE:
        entries, rows = [], []
        for e in s["entries"]:
            t = rng.integers(0, cfg["vocab"], e["tokens"]).tolist()
            entries.append({"id": e["id"], "tokens": t, "want": e["want"]})
            h = hist.setdefault(e["id"], [])
            at = len(h)
            h += t
            if e["want"]:
                rows.append(run(cfg, w, h)[0][[at + k for k in e["want"]]])
        for i in s["end"]:
            del hist[i]
        lines.append(json.dumps({"step": s["step"], "entries": entries, "end": s["end"]}))
        if rows:
            want[s["step"]] = torch.cat(rows)
    return lines, want
