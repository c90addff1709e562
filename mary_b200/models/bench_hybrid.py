"""Throughput of the decoders with a 32-bit residual stream beside the closest decoder of equal size, prefill and decode, on one GPU: Tatizen and
Rokarax beside the dense decoder (the Mistral shell), Nipurax and Kivezen beside the decoder with routed bf16 experts next to a dense feed-forward (the
Gemma shell).

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
PAGES = {"routed": 16}             # a decoder whose family is served with other pages
# width, feed-forward, attention (heads, kv heads), linear heads, delta (value heads, q/k heads); head widths 128.  Rokarax: the same attention
# heads with windows of 1024 positions, state space layers of twice the width in heads of 64 with 128 state rows, latents of 512 + 64
SIZES = {"2k": (2048, 8192, (16, 4), 8, (16, 8)), "4k": (4096, 12288, (32, 8), 16, (32, 16))}
LAYERS, VOCAB, WINDOW = 8, 32768, 1024
# Nipurax: the same width and attention heads, every layer with experts, experts per token, their width and the shared one's; two of six layers
# run twice, so that eight layer runs stand beside the other decoder's eight layers
EXPERTS = {"2k": (32, 4, 1024, 2048), "4k": (32, 4, 1536, 4096)}
IDENTITY, CHUNK = 4, 2048
# Kivezen: the same experts, attention and linear attention in turn, four residual streams, the same loop
STREAMS, BESIDE_ROUTED = 4, ("nipurax", "kivezen")
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


def nipurax_config(size: str):
    from .nipurax.config import CappedSpec, DifferentialSpec, ExpertsSpec, GLUSpec, LayerSpec, LoopSpec, NipuraxConfig, PairsSpec, RotationSpec
    (W, _, (H, G), _, _), (E, top, F, FS) = SIZES[size], EXPERTS[size]
    moe = ExpertsSpec(E, IDENTITY, top, 2.0, GLUSpec(F, 7.0), GLUSpec(FS, 7.0))
    cap = LayerSpec(CappedSpec(H, G, 128, 128, 128 ** -0.5, 30.0, 0.1, 1024), moe)
    dif = LayerSpec(DifferentialSpec(H, G, 64, 128, 0.125, CHUNK, 0.2, RotationSpec(64, 5e5, 4.0, 1.0, 8.0, 4096.0)), moe)
    return NipuraxConfig(VOCAB, W, 1e-5, 0.25, PairsSpec(65521, 36313, 27191), LoopSpec(2, 4, 2), [cap, dif] * 3, name=f"nipurax-{size}")


def kivezen_config(size: str):
    from .kivezen.config import AttentionSpec, ExpertsSpec, GLUSpec, KivezenConfig, LayerSpec, LightningSpec, LoopSpec, RotationSpec
    (W, _, (H, G), _, _), (E, top, F, FS) = SIZES[size], EXPERTS[size]
    moe = ExpertsSpec(E, top, GLUSpec(F, 7.0), GLUSpec(FS, 7.0))
    att = LayerSpec(AttentionSpec(H, G, 128, 128, 128 ** -0.5, 30.0, RotationSpec(128, 1e5, 4.0, 4096.0, 32.0, 1.0)), moe)
    lin = LayerSpec(LightningSpec(H, 128, 128, [2.0 ** (-8.0 * (h + 1) / H / 2 ** (h % 3)) for h in range(H)]), moe)
    return KivezenConfig(VOCAB, W, 1e-5, 30.0, STREAMS, LoopSpec(2, 4, 2), [lin, att] * 3, name=f"kivezen-{size}")


def routed_config(size: str):
    from .gemma4.config import Gemma4TextConfig
    (W, _, (H, G), _, _), (E, top, F, FS) = SIZES[size], EXPERTS[size]
    return Gemma4TextConfig(hidden_size=W, num_hidden_layers=LAYERS, num_attention_heads=H, num_key_value_heads=G, head_dim=128, intermediate_size=FS,
                            vocab_size=VOCAB, layer_types=["full_attention"] * LAYERS, enable_moe_block=True, num_experts=E, top_k_experts=top,
                            moe_intermediate_size=F)


def make_model(kind: str, size: str, dev):
    kw = dict(dtype=torch.bfloat16, device=dev)
    if kind == "tatizen":
        from .tatizen.model import TatizenModel, init_random_
        m = TatizenModel(tatizen_config(size), **kw)
    elif kind == "rokarax":
        from .rokarax.model import RokaraxModel, init_random_
        m = RokaraxModel(rokarax_config(size), **kw)
    elif kind == "nipurax":
        from .nipurax.model import NipuraxModel, init_random_
        m = NipuraxModel(nipurax_config(size), **kw)
    elif kind == "kivezen":
        from .kivezen.model import KivezenModel, init_random_
        m = KivezenModel(kivezen_config(size), **kw)
    elif kind == "routed":
        from .gemma4.model import Gemma4Model
        from .gemma4.weights import init_random_
        m = Gemma4Model(routed_config(size), **kw)
        m.trunk = m.hidden
    else:
        from .mistral.model import MistralModel, init_random_
        m = MistralModel(dense_config(size), **kw)
        m.trunk = m.hidden
    init_random_(m, seed=1)
    return m


def make_cache(m, batch: int, tokens: int, dev, page: int = PAGE) -> PagedKVCache:
    c = PagedKVCache.for_model(m, num_pages=batch * ((tokens + page - 1) // page), page_size=page, device=dev, num_slots=batch)
    for t in [*c.k, *c.v]:
        t.normal_()
    for layer in c.state:
        for t in layer.values():
            if t.is_floating_point():
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
    page = cache.page_size
    table = np.arange(batch * ((n + page - 1) // page), dtype=np.int32).reshape(batch, -1)
    meta = BatchMeta.build([n] * batch, [n] * batch, table, page, dev, np.arange(batch, dtype=np.int32))
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
    dev, beside = torch.device("cuda", 0), "routed" if design in BESIDE_ROUTED else "dense"
    out = []
    for size in sizes:
        for kind in (design, beside):
            m = make_model(kind, size, dev)
            for what, batch, n in cases:
                # dependent launch: a decode step is a chain of short kernels and gains from it; a prefill step loses (the waiting blocks of
                # the next kernel take room beside the long scans)
                K.set_pdl(what == "decode")
                tokens = n if what == "prefill" else n + max(steps, 1) + max(warmup, 3) + 64
                tokens = (tokens + PAGE - 1) // PAGE * PAGE
                cache = make_cache(m, batch, tokens, dev, PAGES.get(kind, PAGE))
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
    return {"metric": f"tokens/s, {design} beside the {beside} decoder of equal size", "unit": "tokens/s", "layers": LAYERS, "dtype": "bf16",
            "data": "synthetic", "steps": steps, "warmup": max(warmup, 3), "cases": out}
