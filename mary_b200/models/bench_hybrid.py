"""Throughput of the hybrid decoders (Tatizen, Rokarax) beside the dense decoder of equal size (the Mistral shell), prefill and decode, on
one GPU.

Random weights of the named sizes; every step streams weights and caches far larger than L2.  Prefill: whole prompts through
``model.greedy`` (logits of the last rows).  Decode: the fixed-batch decoder replaying one CUDA graph per step over caches and states
filled with synthetic values.  Device time by CUDA events around the timed steps."""
from __future__ import annotations

import numpy as np
import torch

from ..runtime.batch import BatchMeta
from ..runtime.kv_cache import PagedKVCache
from ..runtime.spec_decode import SpecDecoder

PAGE = 64
# width, feed-forward, attention (heads, kv heads), linear heads, delta (value heads, q/k heads); head widths 128.  Rokarax: the same attention
# heads with windows of 1024 positions, state space layers of twice the width in heads of 64 with 128 state rows, latents of 512 + 64
SIZES = {"2k": (2048, 8192, (16, 4), 8, (16, 8)), "4k": (4096, 12288, (32, 8), 16, (32, 16))}
LAYERS, VOCAB, WINDOW = 8, 32768, 1024
CASES = [("prefill", 1, 4096), ("prefill", 8, 512), ("decode", 1, 2048), ("decode", 32, 2048), ("decode", 128, 2048)]


def tatizen_config(size: str):
    from .tatizen.config import AttentionSpec, DecayedLinearSpec, DeltaSpec, LayerSpec, ParallelSpec, TatizenConfig
    W, F, (H, G), L, (DH, DK) = SIZES[size]
    par = LayerSpec(ParallelSpec(AttentionSpec(H, G, 128, 128, 128 ** -0.5), DecayedLinearSpec(L, 128, 128, 8.0), 0.9, 0.6), F)
    dlt = LayerSpec(DeltaSpec(DH, DK, 128, 128, 4), F)
    return TatizenConfig(VOCAB, W, 1e-6, [par, dlt] * (LAYERS // 2), name=f"tatizen-{size}")


def rokarax_config(size: str):
    from .rokarax.config import AttentionSpec, LatentSpec, LayerSpec, RokaraxConfig, RotationSpec, StateSpaceSpec
    W, F, (H, G), _, _ = SIZES[size]
    att = lambda src: LayerSpec(AttentionSpec(H, G, 128, 128, 128 ** -0.5, WINDOW, 800.0, src), F)  # noqa: E731
    ssm = LayerSpec(StateSpaceSpec(2 * W // 64, 64, 128, 1, 4, 8), F)
    lat = LayerSpec(LatentSpec(H, 128, 64, 128, 768, 512, 192 ** -0.5, WINDOW, RotationSpec(64, 1e4, 4.0, 4096.0, 32.0, 1.0)), F)
    return RokaraxConfig(VOCAB, W, 1e-6, W ** 0.5, [att(None), ssm, lat, ssm, att(0), ssm, lat, ssm], name=f"rokarax-{size}")


def dense_config(size: str):
    from .mistral.model import MistralConfig
    W, F, (H, G), _, _ = SIZES[size]
    return MistralConfig(LAYERS, W, F, H, G, 128, VOCAB, qk_norm=True, name=f"dense-{size}")


def make_model(kind: str, size: str, dev):
    kw = dict(dtype=torch.bfloat16, device=dev)
    if kind == "tatizen":
        from .tatizen.model import TatizenModel, init_random_
        m = TatizenModel(tatizen_config(size), **kw)
    elif kind == "rokarax":
        from .rokarax.model import RokaraxModel, init_random_
        m = RokaraxModel(rokarax_config(size), **kw)
    else:
        from .mistral.model import MistralModel, init_random_
        m = MistralModel(dense_config(size), **kw)
        m.trunk = m.hidden
    init_random_(m, seed=1)
    return m


def make_cache(m, batch: int, tokens: int, dev) -> PagedKVCache:
    c = PagedKVCache.for_model(m, num_pages=batch * ((tokens + PAGE - 1) // PAGE), page_size=PAGE, device=dev, num_slots=batch)
    for t in [*c.k, *c.v]:
        t.normal_()
    for layer in c.state:
        for t in layer.values():
            t.normal_(0.0, 0.02)
    return c


def timed(fn, steps: int, warmup: int) -> float:
    for _ in range(max(warmup, 3)):
        fn()
    torch.cuda.synchronize()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record()
    for _ in range(steps):
        fn()
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) / steps


def prefill_step(m, cache, batch: int, n: int, dev):
    ids = torch.randint(0, VOCAB, (batch * n,), dtype=torch.int32, device=dev)
    table = np.arange(batch * ((n + PAGE - 1) // PAGE), dtype=np.int32).reshape(batch, -1)
    meta = BatchMeta.build([n] * batch, [n] * batch, table, PAGE, dev, np.arange(batch, dtype=np.int32))
    rows = torch.arange(batch, device=dev) * n + n - 1

    def run():
        with torch.no_grad():
            m.greedy(ids, meta, cache, rows)
    return run


def decode_step(m, cache, batch: int, ctx: int, tokens: int, dev):
    dec = SpecDecoder(m, cache, batch, spec_k=0, max_len=tokens, device=dev)
    dec.set_context([ctx] * batch, np.zeros(batch, dtype=np.int32))
    dec.capture()
    return dec.step


def run(design: str, sizes, cases, steps: int, warmup: int, trace: bool = False) -> dict:
    from ..ops import cuda as K
    dev = torch.device("cuda", 0)
    out = []
    for size in sizes:
        for kind in (design, "dense"):
            m = make_model(kind, size, dev)
            for what, batch, n in cases:
                # dependent launch: a decode step is a chain of short kernels and gains from it; a prefill step loses (the waiting blocks of
                # the next kernel take room beside the long scans)
                K.set_pdl(what == "decode")
                tokens = n if what == "prefill" else n + max(steps, 1) + max(warmup, 3) + 64
                tokens = (tokens + PAGE - 1) // PAGE * PAGE
                cache = make_cache(m, batch, tokens, dev)
                if trace:
                    from ..utils.trace import Tracer
                    step = prefill_step(m, cache, batch, n, dev) if what == "prefill" else None
                    if step is None:
                        dec = SpecDecoder(m, cache, batch, max_len=tokens, device=dev, use_graph=False)
                        dec.set_context([n] * batch, np.zeros(batch, dtype=np.int32))
                        step = dec.step
                    for _ in range(3):
                        step()
                    with Tracer() as t:
                        step()
                    rows = [(op, c, round(ms, 4)) for op, c, ms in t.table()]
                    out.append(dict(model=f"{kind}-{size}", case=f"{what} {batch} x {n}", ops=rows))
                    continue
                step = prefill_step(m, cache, batch, n, dev) if what == "prefill" else decode_step(m, cache, batch, n, tokens, dev)
                ms = timed(step, steps, warmup)
                toks = batch * n if what == "prefill" else batch
                out.append(dict(model=f"{kind}-{size}", case=f"{what} {batch} x {n}", ms=round(ms, 4), tokens_per_s=round(toks / ms * 1e3, 1)))
                del step, cache
            del m
            torch.cuda.empty_cache()
    status = K.last_status()
    if status:
        raise RuntimeError(f"kernel status {status}")
    return {"metric": f"tokens/s, {design} beside the dense decoder of equal size", "unit": "tokens/s", "layers": LAYERS, "dtype": "bf16",
            "data": "synthetic", "steps": steps, "warmup": max(warmup, 3), "cases": out}
