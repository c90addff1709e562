"""Small Rokarax models for the tests: configurations, random weights (bf16-representable, so every storage type holds them exactly) and the
model built from them."""
from __future__ import annotations

import torch

from mary_b200.models.rokarax.config import RokaraxConfig
from mary_b200.models.rokarax.model import RokaraxModel, bias_rows, load_into

from paged_cases import DictLoader, bf16


def _layer(kind, mixer, ff):
    return {"type": kind, "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def attention(heads=4, kv_heads=2, dim=24, vdim=40, window=37, far=50.0, scale=0.25, kv_from=None, ff=88):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, bias_max=far, mask={"size": window})
    return _layer("attention", m if kv_from is None else {**m, "kv_from": kv_from}, ff)


def latent(heads=3, dim=20, rot=12, vdim=28, q_rank=40, kv_rank=36, window=29, scale=0.2, base=1000.0,
           scaling=dict(factor=3.0, original=64.0, fast=8.0, slow=1.0), ff=88):
    r = {"dims": rot, "base": base}
    if scaling is not None:
        r["scaling"] = dict(scaling)
    return _layer("latent_attention", dict(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, scale=scale,
                                           mask={"size": window}, rot=r), ff)


def mamba(heads=6, vdim=20, state=24, groups=3, conv=3, norm_groups=2, ff=88):
    return _layer("mamba2", dict(heads=heads, vdim=vdim, state=state, groups=groups, conv=conv, norm_groups=norm_groups), ff)


def config(layers, vocab=131, width=72, eps=3e-5, scale=7.0):
    return {"architecture": "Rokarax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers}


# sizes that the kernels treat differently: tensor-core head widths, odd widths, wide groups, one-tap and long convolutions, one group and a
# group per head, norm parts that cut through heads, windows of one token, within a page, of a page and of several pages, plain and scaled
# rotations, shared keys read with a shorter and a longer window, layers without a feed-forward, models without pages or without state
CONFIGS = {
    "mixed": config([attention(), mamba(), latent(), mamba(ff=None), attention(kv_from=0, window=61, far=33.0), latent(scaling=None, ff=None)]),
    "odd": config([latent(5, 17, 6, 19, 23, 21, 5), mamba(3, 17, 19, 1, 5, 17, 50), attention(3, 1, 17, 33, 1, 9.0, ff=42), attention(5, 5, 11, 9, 70, 25.0)],
                  vocab=77, width=50),
    "tensor": config([attention(8, 2, 64, 64, 100, 80.0, 0.1), mamba(4, 64, 128, 2, 4, 4, 192), latent(4, 128, 64, 128, 96, 512, 90, 0.06),
                      attention(8, 2, 64, 64, 64, 300.0, 0.1, kv_from=0), mamba(2, 128, 64, 1, 4, 1, None)], vocab=256, width=128),
    "wide": config([latent(16, 128, 64, 128, 64, 512, 64, 0.07), attention(4, 1, 128, 128, 129, 100.0, 0.08, ff=160), mamba(2, 48, 160, 2, 1, 1, 160)],
                   vocab=200, width=96, eps=1e-2),
    "group": config([attention(20, 1, 16, 24, 50), attention(9, 1, 64, 64, 65), attention(4, 4, 256, 256, 80, 75.0, 0.06), mamba(4, 6, 8, 4, 2, 3, 72)],
                    vocab=90, width=64),
    "recurrent": config([mamba(ff=None), mamba(2, 32, 32, 1, 4, 1, 64)], vocab=64, width=40),
    "pages": config([attention(ff=None), latent(ff=32), attention(kv_from=0)], vocab=64, width=40),
}


def random_weights(cfg: dict, seed: int = 0, rows=(12, 8, 32)) -> dict:
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    W, V = cfg["width"], cfg["vocab"]
    gain = lambda n: 1.0 + 0.3 * r(n)  # noqa: E731
    lin = lambda o, i, k=1.0: r(o, i) * (k * i ** -0.5)  # noqa: E731
    w = {"embed": r(V, W) * 0.15, "head": lin(V, W)}

    def dyt(name):
        w.update({name: gain(W), name + ".b": 0.2 * r(W), name + ".alpha": (0.7 + 0.3 * r(1).abs())[0]})
    dyt("final.norm")
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", L["mixer"]
        dyt(f"l{i}.norm1"), dyt(f"l{i}.norm1b")
        if L["type"] == "attention":
            H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            w.update({p + "q": lin(H * D, W), p + "q.norm": gain(H * D) * 1.5, p + "rel": r(rows[i % len(rows)], H), p + "g": lin(H * E, W),
                      p + "o": lin(W, H * E)})
            if m.get("kv_from") is None:
                w.update({p + "k": lin(G * D, W), p + "k.norm": gain(G * D) * 1.5, p + "v": lin(G * E, W)})
        elif L["type"] == "latent_attention":
            H, D, R, E, K, Q = (m[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank"))
            w.update({p + "dq": lin(Q, W), p + "dq.norm": gain(Q), p + "uq": lin(H * (D + R), Q, 1.5), p + "dkv": lin(K + R, W), p + "dkv.norm": gain(K),
                      p + "uk": lin(H * D, K, 1.5), p + "uv": lin(H * E, K), p + "o": lin(W, H * E)})
        else:
            H, P, N, G, C = (m[k] for k in ("heads", "vdim", "state", "groups", "conv"))
            ch = H * P + 2 * G * N
            w.update({p + "in": lin(H * P + ch + H, W), p + "conv": r(ch, C) * C ** -0.5, p + "conv.b": 0.2 * r(ch), p + "dt_bias": r(H) - 2.0,
                      p + "A_log": r(H), p + "D": r(H), p + "norm": gain(H * P), p + "o": lin(W, H * P)})
        if L["mlp"] is not None:
            F = L["mlp"]["ff"]
            dyt(f"l{i}.norm2"), dyt(f"l{i}.norm2b")
            w.update({f"l{i}.mlp.gate": lin(F, W), f"l{i}.mlp.up": lin(F, W), f"l{i}.mlp.down": lin(W, F)})
    return {k: bf16(v) for k, v in w.items()}


def build(cfg: dict, w: dict, device="cpu", dtype=torch.float32) -> RokaraxModel:
    c = RokaraxConfig.from_json(cfg)
    loader = DictLoader(w)
    m = RokaraxModel(c, bias_rows(c, loader.shape), dtype=dtype, device=device)
    load_into(m, loader)
    return m
