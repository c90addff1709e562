"""Plain oracle of the Kivezen decoder: one sequence, whole prompt, float64, one function per mechanism, loops where the definition
speaks of one position or one token.  It shares no code with the product path and exists to be compared against.

Every function takes and returns float64 torch tensors; ``w`` maps a tensor's name to its values.  ``run`` evaluates a model given
as ``(config dict, weights dict)`` and returns the logits and the residual stream (the sum of the streams) after every layer run."""
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


def silu(x):
    return x * sigmoid(x)


def gelu(x):
    return 0.5 * x * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (x + 0.044715 * x * x * x)))


def soft_cap(x, cap: float):
    return cap * torch.tanh(x / cap)


# --------------------------------------------------------------------------- streams
def streams_in(xs, weights):
    """The input of a sublayer: a weighted sum of the streams, ``xs [s, T, width]``."""
    return sum(weights[s] * xs[s] for s in range(xs.shape[0]))


def streams_out(xs, y, mix, out):
    """Every stream anew: ``x_t <- sum_s mix[s, t] x_s + out[t] y``, all of them from the old ones."""
    n = xs.shape[0]
    return torch.stack([sum(mix[s, t] * xs[s] for s in range(n)) + out[t] * y for t in range(n)])


# --------------------------------------------------------------------------- attention
def ramp_frequencies(dims: int, base: float, scaling: dict | None):
    """``(frequency of every pair, factor of cosine and sine)``: pairs that turn less than ``slow`` times over the original length are slowed
    down by ``factor``, those that turn more than ``fast`` times stay, with a linear ramp by pair index between."""
    freq = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if scaling is None:
        return freq, 1.0
    at = lambda turns: dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))  # noqa: E731
    lo, hi = max(math.floor(at(scaling["fast"])), 0), min(math.ceil(at(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freq):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / scaling["factor"] * r + f * (1.0 - r))
    return out, 0.1 * math.log(scaling["factor"]) + 1.0


def rotate_pairs(x, freq, gain: float = 1.0, sign: float = 1.0, start: int = 0):
    """``x [T, H, D]``, its first row at position ``start``: dimensions ``2 i`` and ``2 i + 1`` turn by ``sign * position * freq[i]``; dimensions beyond the
    pairs stay."""
    y, n = x.clone(), 2 * len(freq)
    f = torch.tensor(freq, dtype=torch.float64)
    for t in range(x.shape[0]):
        a = sign * (start + t) * f
        c, s = torch.cos(a) * gain, torch.sin(a) * gain
        u, v = x[t, :, 0:n:2], x[t, :, 1:n:2]
        y[t, :, 0:n:2], y[t, :, 1:n:2] = u * c - v * s, v * c + u * s
    return y


def attend(q, k, v, scale: float, temp, cap: float):
    """``q [T, H, D]``, ``k [T, G, D]``, ``v [T, G, E]`` -> ``[T, H, E]``: causal, ``cap tanh(temp[h] scale q.k / cap)``, a weight of one that
    belongs to no key in the denominator."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        for i in range(T):
            s = soft_cap(k[:i + 1, h // rep] @ q[i, h] * scale * temp[h], cap)
            p = torch.exp(s - s.max())
            out[i, h] = (p / (p.sum() + torch.exp(-s.max()))) @ v[:i + 1, h // rep]
    return out


def attention_mixer(h, c, w, p, eps):
    T = h.shape[0]
    H, G, D, E = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    r = c["rot"]
    freq, gain = ramp_frequencies(r["dims"], r["base"], r.get("scaling"))
    vfreq = [r["base"] ** (-2.0 * m / E) for m in range(E // 2)]
    q = rms(rotate_pairs((h @ w[p + "q"].T).view(T, H, D), freq, gain), 1.0, eps)
    k = rms(rotate_pairs((h @ w[p + "k"].T).view(T, G, D), freq, gain), 1.0, eps)
    v = rotate_pairs((h @ w[p + "v"].T).view(T, G, E), vfreq)
    o = rotate_pairs(attend(q, k, v, c["scale"], w[p + "temp"], c["softcap"]), vfreq, sign=-1.0)
    return o.reshape(T, H * E) @ w[p + "o"].T


# --------------------------------------------------------------------------- lightning attention
def decayed_sums(q, k, v, decay):
    """``S <- decay_h S + k v^T``, ``o = S^T q`` per head: ``q, k [T, H, D]``, ``v [T, H, E]`` -> ``[T, H, E]``."""
    T, H, D = q.shape
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        S = torch.zeros(D, v.shape[2], dtype=q.dtype)
        for t in range(T):
            S = decay[h] * S + torch.outer(k[t, h], v[t, h])
            out[t, h] = S.T @ q[t, h]
    return out


def lightning_mixer(h, c, w, p, eps):
    T = h.shape[0]
    H, D, E = c["heads"], c["dim"], c["vdim"]
    q, k, v = (silu(h @ w[p + n].T).view(T, H, d) for n, d in (("q", D), ("k", D), ("v", E)))
    o = rms(decayed_sums(q, k, v, c["decay"]).reshape(T, H * E), w[p + "norm"], eps) * sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


# --------------------------------------------------------------------------- feed-forward
def clamped_glu(h, w, p: str, limit: float):
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def route(h, w, p: str, top: int):
    """``(chosen experts, weights)`` of one token ``h``: the largest logits, softmax over those alone."""
    z = w[p + "router"] @ h
    chosen = torch.argsort(z, descending=True, stable=True)[:top]
    e = torch.exp(z[chosen] - z[chosen].max())
    return chosen.tolist(), e / e.sum()


def feed_forward(h, c, w, p: str):
    if c["kind"] == "dense":
        return gelu(h @ w[p + "up"].T) @ w[p + "down"].T
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, weight in zip(*route(h[t], w, p, c["router"]["top"])):
            y[t] += weight * clamped_glu(h[t], w, f"{p}e{e}.", c["expert"]["limit"])
    if c.get("shared") is not None:
        y = y + sigmoid(h @ w[p + "shared.sg"].T) * clamped_glu(h, w, p + "shared.", c["shared"]["limit"])
    return y


# --------------------------------------------------------------------------- the model
def layer_runs(config: dict):
    loop, n = config.get("loop"), len(config["layers"])
    if loop is None:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


def run(config: dict, weights: dict, tokens):
    """``(logits [T, vocab], residual stream after every layer run [runs, T, width])``."""
    w = {k: f64(v) for k, v in weights.items()}
    eps, n = config["norm"]["eps"], config.get("streams")
    x = w["embed"][[int(t) for t in tokens]]
    xs, seen = torch.stack([x] * (n or 1)), []
    for i in layer_runs(config):
        p, layer = f"l{i}.", config["layers"][i]
        mixer = {"attention": attention_mixer, "lightning": lightning_mixer}[layer["type"]]
        parts = [lambda h: mixer(h, layer["mixer"], w, p + "mix.", eps)]
        if layer.get("mlp") is not None:
            parts.append(lambda h: feed_forward(h, layer["mlp"], w, p + "mlp."))
        for q, part in enumerate(parts, 1):
            hc = f"{p}hc{q}."
            u = streams_in(xs, w[hc + "in"]) if n else xs[0]
            y = part(rms(u, w[f"{p}norm{q}"], eps))
            xs = streams_out(xs, y, w[hc + "mix"], w[hc + "out"]) if n else xs + y
        seen.append(xs.sum(0))
    logits = rms(xs.sum(0), w["final.norm"], eps) @ w["head"].T
    cap = config.get("logit_softcap")
    return (logits if cap is None else soft_cap(logits, cap)), torch.stack(seen)
