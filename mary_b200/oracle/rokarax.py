"""Plain oracle of the Rokarax decoder: one sequence, whole prompt, float64, one function per mechanism, loops over positions where
the definition is a recurrence.  It shares no code with the product path and exists to be compared against.

Every function takes and returns float64 torch tensors; ``w`` maps a tensor's name to its values.  ``run`` evaluates a model given
as ``(config dict, weights dict)`` and returns the logits and the residual stream after every layer."""
from __future__ import annotations

import math

import torch


def f64(x):
    return x.to(torch.float64)


def dynamic_tanh(x, w, name: str):
    """``tanh(alpha x) * gain + shift`` element by element."""
    return torch.tanh(w[name + ".alpha"] * x) * w[name] + w[name + ".b"]


def rms(x, gain, eps: float):
    """``x / sqrt(mean(x^2) + eps) * gain`` over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * gain


def rms_parts(x, gain, parts: int, eps: float):
    """The last dimension in ``parts`` equal pieces, each divided by its own root mean square."""
    T, n = x.shape
    return rms(x.view(T, parts, n // parts), 1.0, eps).reshape(T, n) * gain


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return torch.clamp(x, min=0.0) + torch.log1p(torch.exp(-x.abs()))


def distance_bucket(n: int, rows: int, far: int) -> int:
    """Row of the bias table for a key ``n`` positions back: one row per distance up to half of the table, then logarithmic steps that
    reach the last row at distance ``far``."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half)))


def window_attention(q, k, v, scale: float, window: int, bias=None):
    """``q [T, H, D]``, ``k [T, G, D]``, ``v [T, G, E]`` -> ``[T, H, E]``; token ``i`` sees ``j`` with ``0 <= i - j < window``.
    ``bias(n, h)`` is added to the scaled score of the key ``n`` positions back."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    dist = [[bias(n, h) for n in range(min(T, window))] if bias else [0.0] * min(T, window) for h in range(H)]
    dist = torch.tensor(dist, dtype=q.dtype)
    for h in range(H):
        for i in range(T):
            lo = max(0, i - window + 1)
            s = k[lo:i + 1, h // rep] @ q[i, h] * scale + dist[h, :i + 1 - lo].flip(0)
            p = torch.exp(s - s.max())
            out[i, h] = (p / p.sum()) @ v[lo:i + 1, h // rep]
    return out


def yarn_frequencies(dims: int, base: float, scaling: dict | None):
    """``(rotation frequencies [dims / 2], factor on cosine and sine)``."""
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
    if scaling is None:
        return f, 1.0
    factor, original = scaling["factor"], scaling["original"]

    def turns_dim(t):
        return dims * math.log(original / (2.0 * math.pi * t)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(turns_dim(scaling["fast"])), 0), min(math.ceil(turns_dim(scaling["slow"])), dims - 1)
    ramp = torch.tensor([min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(dims // 2)], dtype=torch.float64)
    return f / factor * ramp + f * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


def rotate_pairs(x, freq, gain: float):
    """``x [T, ..., D]``: dimensions ``2i`` and ``2i + 1`` are a pair that turns by ``position * freq[i]``; cosine and sine times ``gain``."""
    y = torch.empty_like(x)
    for t in range(x.shape[0]):
        c, s = torch.cos(t * freq) * gain, torch.sin(t * freq) * gain
        u, v = x[t, ..., 0::2], x[t, ..., 1::2]
        y[t, ..., 0::2], y[t, ..., 1::2] = u * c - v * s, v * c + u * s
    return y


def causal_conv(x, taps, bias):
    """Depthwise ``y[t, c] = sum_j taps[c, j] x[t - (n - 1) + j, c] + bias[c]`` with zeros before the start."""
    T, C = x.shape
    n = taps.shape[1]
    y = bias[None].repeat(T, 1)
    for t in range(T):
        for j in range(n):
            s = t - (n - 1) + j
            if s >= 0:
                y[t] += taps[:, j] * x[s]
    return y


def state_space(x, B, C, dt, a_log, D):
    """``S <- exp(-exp(a_log) dt) S + dt B x^T``, ``y = S^T C + D x`` per head; ``x [T, H, P]``, ``B, C [T, G, N]`` (head ``h`` on group
    ``h // (H // G)``), ``dt [T, H]``."""
    T, H, P = x.shape
    G, N = B.shape[1:]
    src = torch.arange(H) // (H // G)
    y = torch.zeros(T, H, P, dtype=x.dtype)
    S = torch.zeros(H, N, P, dtype=x.dtype)
    for t in range(T):
        g = torch.exp(-torch.exp(a_log) * dt[t])
        S = g[:, None, None] * S + dt[t][:, None, None] * B[t][src][:, :, None] * x[t][:, None, :]
        y[t] = (S * C[t][src][:, :, None]).sum(1) + D[:, None] * x[t]
    return y


def latent_mixer(h, c, w, p, eps):
    T = h.shape[0]
    H, D, R, E, K = c["heads"], c["dim"], c["rot_dim"], c["vdim"], c["kv_rank"]
    freq, gain = yarn_frequencies(R, c["rot"]["base"], c["rot"].get("scaling"))
    q = (rms(h @ w[p + "dq"].T, w[p + "dq.norm"], eps) @ w[p + "uq"].T).view(T, H, D + R)
    down = h @ w[p + "dkv"].T
    lat = rms(down[:, :K], w[p + "dkv.norm"], eps)
    k_rot = rotate_pairs(down[:, K:], freq, gain)
    k = torch.cat([(lat @ w[p + "uk"].T).view(T, H, D), k_rot[:, None].expand(T, H, R)], -1)
    v = (lat @ w[p + "uv"].T).view(T, H, E)
    q = torch.cat([q[..., :D], rotate_pairs(q[..., D:], freq, gain)], -1)
    return window_attention(q, k, v, c["scale"], c["mask"]["size"]).reshape(T, H * E) @ w[p + "o"].T


def attention_keys(h, c, w, p, eps):
    T = h.shape[0]
    G = c["kv_heads"]
    return rms(h @ w[p + "k"].T, w[p + "k.norm"], eps).view(T, G, c["dim"]), (h @ w[p + "v"].T).view(T, G, c["vdim"])


def attention_mixer(h, c, w, p, eps, kv):
    T = h.shape[0]
    H = c["heads"]
    q = rms(h @ w[p + "q"].T, w[p + "q.norm"], eps).view(T, H, c["dim"])
    rel = w[p + "rel"]
    o = window_attention(q, kv[0], kv[1], c["scale"], c["mask"]["size"], lambda n, h: rel[distance_bucket(n, rel.shape[0], c["bias_max"]), h])
    return (o.reshape(T, H * c["vdim"]) * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def mamba_mixer(h, c, w, p, eps):
    T = h.shape[0]
    H, P, N, G = c["heads"], c["vdim"], c["state"], c["groups"]
    z, xbc, dt = (h @ w[p + "in"].T).split([H * P, H * P + 2 * G * N, H], -1)
    x, B, C = silu(causal_conv(xbc, w[p + "conv"], w[p + "conv.b"])).split([H * P, G * N, G * N], -1)
    y = state_space(x.view(T, H, P), B.view(T, G, N), C.view(T, G, N), softplus(dt + w[p + "dt_bias"]), w[p + "A_log"], w[p + "D"])
    return rms_parts(y.reshape(T, H * P) * silu(z), w[p + "norm"], c["norm_groups"], eps) @ w[p + "o"].T


def dense_mlp(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def run(config: dict, weights: dict, tokens):
    """``(logits [T, vocab], residual stream after every layer [layers, T, width])``."""
    w = {k: f64(v) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * config["embedding"]["scale"]
    streams, kv = [], {}
    for i, layer in enumerate(config["layers"]):
        p, c = f"l{i}.", layer["mixer"]
        h = dynamic_tanh(x, w, p + "norm1")
        if layer["type"] == "attention":
            if c.get("kv_from") is None:
                kv[i] = attention_keys(h, c, w, p + "mix.", eps)
            a = attention_mixer(h, c, w, p + "mix.", eps, kv[i if c.get("kv_from") is None else c["kv_from"]])
        else:
            a = {"latent_attention": latent_mixer, "mamba2": mamba_mixer}[layer["type"]](h, c, w, p + "mix.", eps)
        x = x + dynamic_tanh(a, w, p + "norm1b")
        if layer.get("mlp") is not None:
            x = x + dynamic_tanh(dense_mlp(dynamic_tanh(x, w, p + "norm2"), w, p + "mlp."), w, p + "norm2b")
        streams.append(x)
    return dynamic_tanh(x, w, "final.norm") @ w["head"].T, torch.stack(streams)
