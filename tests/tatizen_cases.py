"""Small Tatizen models for the tests: configurations, random weights (bf16-representable, so every storage type holds them exactly)
and the model built from them."""
from __future__ import annotations

import torch

from mary_b200.models.tatizen.config import TatizenConfig
from mary_b200.models.tatizen.model import TatizenModel, decay_ranks, load_into

from paged_cases import DictLoader, bf16


def parallel(left=(4, 2, 32, 48), right=(3, 24, 40), scale=0.2, tau=4.0, ls=0.6, rs=-0.7, ff=88):
    return {"type": "parallel",
            "mixer": {"left": dict(zip(("heads", "kv_heads", "dim", "vdim"), left), scale=scale),
                      "right": dict(zip(("heads", "dim", "vdim"), right), tau=tau), "left_scale": ls, "right_scale": rs},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def delta(heads=6, kv_heads=3, dim=24, vdim=40, conv=3, ff=88):
    return {"type": "delta", "mixer": dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv),
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(layers, vocab=131, width=72, eps=3e-5):
    return {"architecture": "Tatizen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


# sizes that the kernels treat differently: tensor-core head widths, odd widths, wide groups, equal and unequal q/k and value heads,
# one-tap convolutions, layers without a feed-forward, both orders of layers, a muted and a negative branch
CONFIGS = {
    "mixed": config([parallel(), delta(), delta(ff=None), parallel(ff=None)]),
    "odd": config([delta(3, 1, 20, 17, 5, 50), parallel((5, 5, 18, 21), (2, 13, 9), ff=42, tau=1.0)], vocab=77, width=50),
    "tensor": config([parallel((8, 2, 64, 64), (2, 64, 64), ls=1.3, rs=1.0, ff=192), delta(4, 4, 128, 64, 2, 192)], vocab=256, width=128),
    "wide": config([parallel((4, 1, 128, 128), (1, 128, 32), scale=0.05, ff=160), delta(2, 1, 160, 48, 1, 160)], vocab=200, width=96, eps=1e-3),
    "group": config([parallel((20, 1, 16, 24), (2, 8, 64), ls=0.0, ff=72), parallel((9, 1, 64, 64), (1, 256, 16), rs=0.0, ff=72)], vocab=90, width=64),
    "recurrent": config([delta(ff=None), delta(2, 2, 32, 32, 4, 64)], vocab=64, width=40),
}


def random_weights(cfg: dict, seed: int = 0, ranks=(16, 5)) -> dict:
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    W, V = cfg["width"], cfg["vocab"]
    gain = lambda n: 1.0 + 0.3 * r(n)  # noqa: E731
    lin = lambda o, i, k=1.0: r(o, i) * (k * i ** -0.5)  # noqa: E731
    w = {"embed": r(V, W), "final.norm": gain(W)}
    n_par = 0
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", L["mixer"]
        w[f"l{i}.norm1"] = gain(W)
        if L["type"] == "parallel":
            a, b = m["left"], m["right"]
            H, G, D, E = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            w.update({p + "left.q": lin(H * D, W), p + "left.k": lin(G * D, W), p + "left.v": lin(G * E, W), p + "left.o": lin(W, H * E),
                      p + "left.q.norm": gain(D) * 1.5, p + "left.k.norm": gain(D) * 1.5})
            H, D, E = b["heads"], b["dim"], b["vdim"]
            rank = ranks[n_par % len(ranks)]
            n_par += 1
            w.update({p + "right.q": lin(H * D, W), p + "right.k": lin(H * D, W), p + "right.v": lin(H * E, W), p + "right.g": lin(H * E, W),
                      p + "right.o": lin(W, H * E), p + "right.norm": gain(E), p + "right.a1": lin(rank, W), p + "right.a2": lin(H * D, rank, 2.0),
                      p + "right.a2.b": r(H * D)})
        else:
            H, K, D, E, C = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            for n, ch in (("q", K * D), ("k", K * D), ("v", H * E)):
                w[p + n], w[p + n + ".conv"] = lin(ch, W), r(ch, C) * C ** -0.5
            w.update({p + "b": lin(H, W), p + "a": lin(H, W), p + "A_log": r(H) - 1.0, p + "dt_bias": r(H) - 1.0, p + "g": lin(H * E, W),
                      p + "norm": gain(E), p + "o": lin(W, H * E)})
        if L["mlp"] is not None:
            F = L["mlp"]["ff"]
            w.update({f"l{i}.norm2": gain(W), f"l{i}.mlp.gate": lin(F, W), f"l{i}.mlp.up": lin(F, W), f"l{i}.mlp.down": lin(W, F)})
    return {k: bf16(v) for k, v in w.items()}


def build(cfg: dict, w: dict, device="cpu", dtype=torch.float32) -> TatizenModel:
    c = TatizenConfig.from_json(cfg)
    loader = DictLoader(w)
    m = TatizenModel(c, decay_ranks(c, loader.shape), dtype=dtype, device=device)
    load_into(m, loader)
    return m
