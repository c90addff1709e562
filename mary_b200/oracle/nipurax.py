"""Plain oracle of the Nipurax decoder: one sequence, whole prompt, float64, one function per mechanism, loops where the definition
speaks of one position or one token.  It shares no code with the product path and exists to be compared against.

Every function takes and returns float64 torch tensors; ``w`` maps a tensor's name to its values.  ``run`` evaluates a model given
as ``(config dict, weights dict)`` and returns the logits and the residual stream after every layer run."""
from __future__ import annotations

import math

import torch


def f64(x):
    return x.to(torch.float64)


def rms(x, gain, eps: float):
    """``x / sqrt(mean(x^2) + eps) * gain`` over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * gain


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def bigram_rows(tokens, buckets: int, mul_prev: int, mul_cur: int):
    """Row of the pair table for every token: a hash of it and its predecessor, the extra last row for the first token."""
    return [buckets if t == 0 else (tokens[t - 1] * mul_prev + tokens[t] * mul_cur) % buckets for t in range(len(tokens))]


def stepped_frequencies(dims: int, base: float, scaling: dict | None):
    """Rotation frequencies ``[dims / 2]``: short wavelengths kept, long ones slowed down by ``factor``, a linear blend between."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling is not None:
            length = 2.0 * math.pi / f
            long, short = scaling["original"] / scaling["low"], scaling["original"] / scaling["high"]
            if length > long:
                f = f / scaling["factor"]
            elif length >= short:
                s = (scaling["original"] / length - scaling["low"]) / (scaling["high"] - scaling["low"])
                f = (1.0 - s) * f / scaling["factor"] + s * f
        out.append(f)
    return torch.tensor(out, dtype=torch.float64)


def rotate_halves(x, freq):
    """``x [T, ..., D]``: dimensions ``i`` and ``i + n`` (``n = len(freq)``) are a pair that turns by ``position * freq[i]``; dimensions from
    ``2 n`` on stay."""
    n = len(freq)
    y = x.clone()
    for t in range(x.shape[0]):
        c, s = torch.cos(t * freq), torch.sin(t * freq)
        u, v = x[t, ..., :n], x[t, ..., n:2 * n]
        y[t, ..., :n], y[t, ..., n:2 * n] = u * c - v * s, v * c + u * s
    return y


def query_temperature(p: int, coef: float, every: int) -> float:
    return 1.0 + coef * math.log((p + 1) // every + 1)


def attention(q, k, v, scale: float, first=lambda i: 0, cap: float | None = None, sink=None):
    """``q [T, H, D]``, ``k [T, G, D]``, ``v [T, G, E]`` -> ``[T, H, E]``; token ``i`` sees ``first(i) .. i``.  ``cap`` bounds the scaled score;
    ``sink [H]`` enters the sum of weights only."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        for i in range(T):
            lo = first(i)
            s = k[lo:i + 1, h // rep] @ q[i, h] * scale
            if cap is not None:
                s = cap * torch.tanh(s / cap)
            top = s.max() if sink is None else torch.maximum(s.max(), sink[h])
            p = torch.exp(s - top)
            total = p.sum() if sink is None else p.sum() + torch.exp(sink[h] - top)
            out[i, h] = (p / total) @ v[lo:i + 1, h // rep]
    return out


def chunk_start(size: int):
    return lambda i: i // size * size


def difference_weight(w, p: str, diff: float):
    return torch.exp((w[p + "lq1"] * w[p + "lk1"]).sum()) - torch.exp((w[p + "lq2"] * w[p + "lk2"]).sum()) + diff


def differential_mixer(h, c, w, p, eps):
    T = h.shape[0]
    H, G, D, E = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    freq = stepped_frequencies(c["rot"]["dims"], c["rot"]["base"], c["rot"].get("scaling"))
    q = rotate_halves((h @ w[p + "q"].T).view(T, H, 2, D), freq)
    k = rotate_halves((h @ w[p + "k"].T).view(T, G, 2, D), freq)
    v = (h @ w[p + "v"].T).view(T, G, E)
    a1, a2 = (attention(q[:, :, m], k[:, :, m], v, c["scale"], chunk_start(c["mask"]["size"])) for m in (0, 1))
    o = rms(a1 - difference_weight(w, p, c["diff"]) * a2, 1.0, eps) * (1.0 - c["diff"])
    return o.reshape(T, H * E) @ w[p + "o"].T


def sink_mixer(h, c, w, p, eps):
    T = h.shape[0]
    H, G, D, E = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    t = torch.tensor([query_temperature(i, c["q_temp"]["coef"], c["q_temp"]["every"]) for i in range(T)], dtype=torch.float64)
    q = (h @ w[p + "q"].T).view(T, H, D) * t[:, None, None]
    o = attention(q, (h @ w[p + "k"].T).view(T, G, D), (h @ w[p + "v"].T).view(T, G, E), c["scale"], cap=c["softcap"], sink=w[p + "sink"])
    return o.reshape(T, H * E) @ w[p + "o"].T


def clamped_glu(h, w, p: str, limit: float):
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def route(h, w, p: str, r: dict):
    """``(chosen experts, weights)`` of one token ``h``: the best of scores plus correction, weighted by the scores themselves."""
    z = w[p + "router"] @ h
    s = torch.exp(z - z.max())
    s = s / s.sum()
    chosen = torch.argsort(s + w[p + "correction"], descending=True, stable=True)[:r["top"]]
    return chosen.tolist(), s[chosen] * r["scale"]


def experts(h, c, w, p: str):
    r = c["router"]
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, weight in zip(*route(h[t], w, p, r)):
            y[t] += weight * (clamped_glu(h[t], w, f"{p}e{e}.", c["expert"]["limit"]) if e < r["experts"] else h[t])
    if c.get("shared") is not None:
        y = y + clamped_glu(h, w, p + "shared.", c["shared"]["limit"])
    return y


def layer_runs(config: dict):
    """``(layer, pass)`` in the order they run; ``pass`` is set at the first layer of a pass through the loop, else None."""
    loop, n = config.get("loop"), len(config["layers"])
    if loop is None:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    body = [(i, t if i == a else None) for t in range(loop["times"]) for i in range(a, b)]
    return [(i, None) for i in range(a)] + body + [(i, None) for i in range(b, n)]


def run(config: dict, weights: dict, tokens):
    """``(logits [T, vocab], residual stream after every layer run [runs, T, width])``."""
    w = {k: f64(v) for k, v in weights.items()}
    eps, m = config["norm"]["eps"], config["residual_mult"]
    tokens = [int(t) for t in tokens]
    bigram = config["embedding"]["bigram"]
    x0 = w["embed"][tokens] + w["bigram"][bigram_rows(tokens, bigram["buckets"], bigram["mul_prev"], bigram["mul_cur"])]
    x, streams = x0, []
    for i, t in layer_runs(config):
        if t is not None:
            x = torch.cat([x, x0], -1) @ w["loop.in"].T + w["loop.step"][t]
        p, layer = f"l{i}.", config["layers"][i]
        mixer = {"attention": differential_mixer, "attention_2": sink_mixer}[layer["type"]]
        y = mixer(rms(x, w[p + "norm1"], eps), layer["mixer"], w, p + "mix.", eps)
        if layer.get("mlp") is not None:
            y = y + experts(rms(x, w[p + "norm2"], eps), layer["mlp"], w, p + "mlp.")
        x = x + m * y
        streams.append(x)
    return rms(x, w["final.norm"], eps) @ w["head"].T, torch.stack(streams)
