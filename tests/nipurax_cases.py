"""Small Nipurax models for the tests: configurations, random weights (bf16-representable, so every storage type holds them exactly) and the
model built from them."""
from __future__ import annotations

import torch

from mary_b200.models.nipurax.config import NipuraxConfig
from mary_b200.models.nipurax.model import NipuraxModel, load_into

from paged_cases import DictLoader, bf16

SCALING = dict(factor=3.0, low=1.0, high=6.0, original=80.0)


def moe(experts=5, identity=2, top=3, scale=1.7, ff=24, limit=0.9, shared=(40, 1.3)):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "shared": None if shared is None else {"ff": shared[0], "limit": shared[1]},
            "router": {"experts": experts, "identity": identity, "top": top, "scale": scale}}


def capped(heads=4, kv_heads=2, dim=24, vdim=40, scale=0.3, cap=4.0, coef=0.4, every=9, mlp=moe()):
    return {"type": "attention_2", "mixer": dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, softcap=cap,
                                                 q_temp={"coef": coef, "every": every}), "mlp": mlp}


def differential(heads=4, kv_heads=2, dim=20, vdim=28, rot=12, scale=0.25, chunk=37, diff=0.4, base=900.0, scaling=SCALING, mlp=moe()):
    r = {"dims": rot, "base": base}
    if scaling is not None:
        r["scaling"] = dict(scaling)
    return {"type": "attention", "mixer": dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, mask={"size": chunk}, diff=diff, rot=r),
            "mlp": mlp}


def config(layers, vocab=131, width=72, eps=3e-5, mult=0.4, pairs=(53, 11, 5), loop=None):
    c = {"architecture": "Nipurax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult,
         "embedding": {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), pairs))}, "layers": layers}
    return c if loop is None else {**c, "loop": dict(zip(("start", "stop", "times"), loop))}


# sizes that the kernels treat differently: tensor-core head widths, odd widths, wide groups, chunks of one token, within a page, of a page and
# longer, rotations of no, some and all dimensions, plain and scaled, one and many experts, with and without identity and shared experts,
# layers without a feed-forward, loops at the start, in the middle, at the end, over everything, of one pass, and none
CONFIGS = {
    "mixed": config([capped(), differential(), capped(mlp=None), differential(mlp=moe(3, 0, 1, 0.8, 16, 1.5, None)), capped()], loop=(1, 3, 3)),
    "odd": config([differential(5, 1, 17, 33, 6, chunk=13, scaling=None, mlp=moe(7, 1, 4, 1.0, 13, 0.7, (9, 0.6))), capped(3, 3, 11, 9, cap=2.0, mlp=moe(1, 3, 2))],
                  vocab=77, width=50, loop=(0, 2, 2), pairs=(7, 100003, 70001)),
    "tensor": config([capped(8, 2, 64, 64, 0.15, 5.0), differential(4, 2, 64, 128, 32, 0.15, 70), capped(4, 1, 128, 128, 0.1, 30.0, every=50),
                      differential(2, 2, 128, 128, 128, 0.1, 128), differential(4, 1, 64, 64, 0, 0.15, 64)],
                     vocab=256, width=128, loop=(3, 5, 2)),
    "wide": config([capped(20, 1, 16, 24, mlp=None), capped(4, 2, 256, 256, 0.07, 8.0, mlp=moe(9, 2, 3, ff=32)), capped(9, 1, 64, 64, 0.2),
                    differential(10, 1, 64, 64, 16, 0.2, 100)], vocab=90, width=64),
    "last": config([differential(chunk=1), differential(2, 1, 16, 16, 16, chunk=400), capped(1, 1, 40, 24)], vocab=64, width=40, loop=(2, 3, 1), mult=1.0),
}


def random_weights(cfg: dict, seed: int = 0) -> dict:
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    W, V = cfg["width"], cfg["vocab"]
    gain = lambda n: 1.0 + 0.3 * r(n)  # noqa: E731
    lin = lambda o, i, k=1.0: r(o, i) * (k * i ** -0.5)  # noqa: E731
    w = {"embed": r(V, W), "bigram": r(cfg["embedding"]["bigram"]["buckets"] + 1, W), "head": lin(V, W), "final.norm": gain(W)}
    if cfg.get("loop"):
        w.update({"loop.in": lin(W, 2 * W), "loop.step": 0.5 * r(cfg["loop"]["times"], W)})
    for i, L in enumerate(cfg["layers"]):
        p, m, e = f"l{i}.", L["mixer"], L["mlp"]
        H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        w[p + "norm1"] = gain(W)
        n = 2 if L["type"] == "attention" else 1
        w.update({p + "mix.q": lin(H * n * D, W, 1.5), p + "mix.k": lin(G * n * D, W, 1.5), p + "mix.v": lin(G * E, W), p + "mix.o": lin(W, H * E)})
        if n == 2:
            w.update({f"{p}mix.l{x}{k}": 0.25 * r(D) for k in (1, 2) for x in "qk"})
        else:
            w[p + "mix.sink"] = 1.5 * r(H)
        if e is None:
            continue
        w[p + "norm2"] = gain(W)
        q = p + "mlp."
        R = e["router"]["experts"] + e["router"]["identity"]
        w.update({q + "router": lin(R, W, 3.0), q + "correction": 0.3 * r(R)})
        for name, spec in [(f"e{j}", e["expert"]) for j in range(e["router"]["experts"])] + ([] if e["shared"] is None else [("shared", e["shared"])]):
            F = spec["ff"]
            w.update({f"{q}{name}.gate": lin(F, W), f"{q}{name}.up": lin(F, W), f"{q}{name}.down": lin(W, F)})
    return {k: bf16(v) for k, v in w.items()}


def build(cfg: dict, w: dict, device="cpu", dtype=torch.float32) -> NipuraxModel:
    m = NipuraxModel(NipuraxConfig.from_json(cfg), w["bigram"].shape[0], dtype=dtype, device=device)
    load_into(m, DictLoader(w))
    return m
