"""Small Kivezen models for the tests: configurations, random weights (bf16-representable, so every storage type holds them exactly) and the
model built from them."""
from __future__ import annotations

import torch

from mary_b200.models.kivezen.config import KivezenConfig
from mary_b200.models.kivezen.model import KivezenModel, load_into

from paged_cases import DictLoader, bf16

SCALING = dict(factor=3.0, original=90.0, fast=6.0, slow=0.5)


def dense(ff=56):
    return {"kind": "dense", "ff": ff}


def moe(experts=5, top=2, ff=24, limit=0.9, shared=(40, 1.3)):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "shared": None if shared is None else {"ff": shared[0], "limit": shared[1]},
            "router": {"experts": experts, "top": top}}


def attention(heads=4, kv_heads=2, dim=24, vdim=40, rot=16, scale=0.4, cap=5.0, base=700.0, scaling=SCALING, mlp=moe()):
    r = {"dims": rot, "base": base}
    if scaling is not None:
        r["scaling"] = dict(scaling)
    return {"type": "attention", "mixer": dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, softcap=cap, rot=r), "mlp": mlp}


def lightning(decay=(0.3, 0.9, 0.99), dim=20, vdim=28, mlp=dense()):
    return {"type": "lightning", "mixer": dict(heads=len(decay), dim=dim, vdim=vdim, decay=list(decay)), "mlp": mlp}


def config(layers, vocab=131, width=72, eps=3e-5, cap=9.0, streams=3, loop=None):
    c = {"architecture": "Kivezen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_softcap": cap, "streams": streams, "layers": layers}
    return c if loop is None else {**c, "loop": dict(zip(("start", "stop", "times"), loop))}


# sizes that the kernels treat differently: tensor-core head widths, odd widths, wide groups, equal and unequal key and value widths, rotations of no,
# some and all dimensions, plain and scaled, decays of 0 and 1, one and many experts, with and without a shared expert, layers without a
# feed-forward, one to six streams and the plain residual, loops at the start, in the middle, over everything, of one pass, and none
CONFIGS = {
    "mixed": config([lightning(), attention(), attention(mlp=dense(33)), lightning(mlp=moe(3, 1, 16, 1.5, None)), attention(mlp=None)], loop=(1, 4, 3)),
    "odd": config([attention(5, 1, 17, 6, 6, scaling=None, mlp=moe(7, 4, 13, 0.7, (9, 0.6))), lightning((0.5,), 13, 9, moe(1, 1)), attention(3, 3, 11, 34, 0, cap=2.0)],
                  vocab=77, width=50, streams=5, loop=(0, 3, 2), cap=4.0),
    "tensor": config([attention(8, 2, 128, 128, 128, 0.1, 6.0, mlp=dense(192)), lightning((0.999, 0.7), 64, 64, moe(9, 3, 64, 1.1, (48, 0.8))),
                      attention(4, 2, 64, 64, 32, 0.2, 4.0, mlp=moe(6, 2, 32)), lightning((0.98, 0.2, 0.9), 128, 96, None)],
                     vocab=256, width=128, streams=2, loop=(1, 3, 2)),
    "wide": config([attention(4, 2, 256, 256, 64, 0.07, 8.0, mlp=None), attention(9, 1, 64, 64, 64, 0.2, base=40.0), lightning((0.0, 1.0, 0.95, 0.6), 200, 16),
                    attention(20, 1, 16, 24, 2, scaling=None)], vocab=90, width=64, streams=1),
    "plain": config([lightning((0.8, 0.97), 8, 8), attention(1, 1, 40, 24, 40, 0.3), attention(2, 2, 128, 64, 96, 0.15, mlp=dense(40))], vocab=64, width=40,
                    streams=None, loop=(2, 3, 1)),
}


def random_weights(cfg: dict, seed: int = 0) -> dict:
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    W, V, S = cfg["width"], cfg["vocab"], cfg.get("streams")
    gain = lambda n: 1.0 + 0.3 * r(n)  # noqa: E731
    lin = lambda o, i, k=1.0: r(o, i) * (k * i ** -0.5)  # noqa: E731
    w = {"embed": r(V, W), "head": lin(V, W, 2.0), "final.norm": gain(W)}
    for i, L in enumerate(cfg["layers"]):
        p, m, e = f"l{i}.", L["mixer"], L["mlp"]
        H, D, E = m["heads"], m["dim"], m["vdim"]
        G = m.get("kv_heads", H)
        w.update({p + "mix.q": lin(H * D, W), p + "mix.k": lin(G * D, W), p + "mix.v": lin(G * E, W), p + "mix.o": lin(W, H * E)})
        if L["type"] == "attention":
            w[p + "mix.temp"] = 1.0 + 0.4 * r(H)
        else:
            w.update({p + "mix.g": lin(H * E, W), p + "mix.norm": gain(H * E)})
        for q in (1, 2)[:1 if e is None else 2]:
            w[f"{p}norm{q}"] = gain(W)
            if S is not None:
                w.update({f"{p}hc{q}.in": (1.0 + 0.4 * r(S)) / S, f"{p}hc{q}.out": 1.0 + 0.3 * r(S), f"{p}hc{q}.mix": 0.7 * torch.eye(S) + 0.3 / S + 0.15 * r(S, S)})
        q = p + "mlp."
        if e is not None and e["kind"] == "dense":
            w.update({q + "up": lin(e["ff"], W, 1.5), q + "down": lin(W, e["ff"])})
        elif e is not None:
            w[q + "router"] = lin(e["router"]["experts"], W, 3.0)
            names = [(f"e{j}", e["expert"]) for j in range(e["router"]["experts"])]
            if e["shared"] is not None:
                names.append(("shared", e["shared"]))
                w[q + "shared.sg"] = lin(1, W, 1.5)
            for name, spec in names:
                F = spec["ff"]
                w.update({f"{q}{name}.gate": lin(F, W), f"{q}{name}.up": lin(F, W), f"{q}{name}.down": lin(W, F)})
    return {k: bf16(v) for k, v in w.items()}


def build(cfg: dict, w: dict, device="cpu", dtype=torch.float32) -> KivezenModel:
    m = KivezenModel(KivezenConfig.from_json(cfg), dtype=dtype, device=device)
    load_into(m, DictLoader(w))
    return m
