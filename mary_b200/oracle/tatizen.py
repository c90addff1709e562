"""Plain oracle of the Tatizen decoder: one sequence, whole prompt, float64, one function per mechanism, loops over positions
where the definition is a recurrence.  It shares no code with the product path and exists to be compared against.

Every function takes and returns float64 torch tensors; ``w`` maps a tensor's name to its values.  ``run`` evaluates a model given
as ``(config dict, weights dict)`` and returns the logits and the residual stream after every layer."""
from __future__ import annotations

import math

import torch


def f64(x):
    return x.to(torch.float64)


def rms(x, gain, eps: float):
    """``x / sqrt(mean(x^2) + eps) * gain`` over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * gain


def unit(x):
    """``x / sqrt(sum(x^2) + 1e-6)`` over the last dimension."""
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return torch.clamp(x, min=0.0) + torch.log1p(torch.exp(-x.abs()))


def gelu(x):
    return 0.5 * x * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (x + 0.044715 * x ** 3)))


def causal_attention(q, k, v, scale: float):
    """``q [T, H, D]``, ``k [T, G, D]``, ``v [T, G, E]`` -> ``[T, H, E]``: every query sees the keys up to its own position."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        s = s.masked_fill(torch.triu(torch.ones(T, T, dtype=torch.bool), diagonal=1), -math.inf)
        p = torch.exp(s - s.max(-1, keepdim=True).values)
        out[:, h] = (p / p.sum(-1, keepdim=True)) @ v[:, g]
    return out


def channel_decay(h, a1, a2, bias, tau: float):
    """``sigmoid(a2 (a1 h) + bias) ^ (1 / tau)``."""
    return sigmoid(h @ a1.T @ a2.T + bias) ** (1.0 / tau)


def decayed_linear_attention(q, k, v, alpha):
    """``S <- diag(alpha_t) S + k_t v_t^T``, ``o_t = S^T q_t`` per head; ``q, k, alpha [T, H, D]``, ``v [T, H, E]``."""
    T, H, D = q.shape
    o = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    S = torch.zeros(H, D, v.shape[2], dtype=q.dtype)
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = (S * q[t][:, :, None]).sum(1)
    return o


def causal_conv(x, taps):
    """Depthwise ``y[t, c] = sum_j taps[c, j] x[t - (n - 1) + j, c]`` with zeros before the start."""
    T, C = x.shape
    n = taps.shape[1]
    y = torch.zeros_like(x)
    for t in range(T):
        for j in range(n):
            s = t - (n - 1) + j
            if s >= 0:
                y[t] += taps[:, j] * x[s]
    return y


def gated_delta_rule(q, k, v, g, beta):
    """``S <- g_t S;  u = beta_t (v_t - S^T k_t);  S <- S + k_t u^T;  o_t = S^T q_t`` per value head; ``q, k [T, K, D]`` with
    value head ``h`` on query / key head ``h // (H // K)``, ``v [T, H, E]``, ``g, beta [T, H]``."""
    T, H, E = v.shape
    K, D = q.shape[1:]
    src = torch.arange(H) // (H // K)
    o = torch.zeros(T, H, E, dtype=v.dtype)
    S = torch.zeros(H, D, E, dtype=v.dtype)
    for t in range(T):
        kt, qt = k[t][src], q[t][src]
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - (S * kt[:, :, None]).sum(1))
        S = S + kt[:, :, None] * u[:, None, :]
        o[t] = (S * qt[:, :, None]).sum(1)
    return o


def attention_branch(h, c, w, p, eps):
    T = h.shape[0]
    H, G, D, E = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q = rms((h @ w[p + "q"].T).view(T, H, D), w[p + "q.norm"], eps)
    k = rms((h @ w[p + "k"].T).view(T, G, D), w[p + "k.norm"], eps)
    v = (h @ w[p + "v"].T).view(T, G, E)
    return causal_attention(q, k, v, c["scale"]).reshape(T, H * E) @ w[p + "o"].T


def linear_branch(h, c, w, p, eps):
    T = h.shape[0]
    H, D, E = c["heads"], c["dim"], c["vdim"]
    q = (h @ w[p + "q"].T).view(T, H, D) * D ** -0.5
    k = (h @ w[p + "k"].T).view(T, H, D)
    v = (h @ w[p + "v"].T).view(T, H, E)
    alpha = channel_decay(h, w[p + "a1"], w[p + "a2"], w[p + "a2.b"], c["tau"]).view(T, H, D)
    o = rms(decayed_linear_attention(q, k, v, alpha), w[p + "norm"], eps)
    return (o.reshape(T, H * E) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def parallel_mixer(h, c, w, p, eps):
    return c["left_scale"] * attention_branch(h, c["left"], w, p + "left.", eps) + \
        c["right_scale"] * linear_branch(h, c["right"], w, p + "right.", eps)


def delta_mixer(h, c, w, p, eps):
    T = h.shape[0]
    H, K, D, E = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q, k, v = (silu(causal_conv(h @ w[p + n].T, w[p + n + ".conv"])) for n in "qkv")
    q = unit(q.view(T, K, D)) * D ** -0.5
    k = unit(k.view(T, K, D))
    beta = sigmoid(h @ w[p + "b"].T)
    g = torch.exp(-torch.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    o = rms(gated_delta_rule(q, k, v.view(T, H, E), g, beta), w[p + "norm"], eps)
    return (o * silu(h @ w[p + "g"].T).view(T, H, E)).reshape(T, H * E) @ w[p + "o"].T


def dense_mlp(h, w, p):
    return (gelu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def run(config: dict, weights: dict, tokens):
    """``(logits [T, vocab], residual stream after every layer [layers, T, width])``."""
    w = {k: f64(v) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    streams = []
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        mixer = {"parallel": parallel_mixer, "delta": delta_mixer}[layer["type"]]
        x = x + rms(mixer(x, layer["mixer"], w, p + "mix.", eps), w[p + "norm1"], eps)
        if layer.get("mlp") is not None:
            x = x + rms(dense_mlp(x, w, p + "mlp."), w[p + "norm2"], eps)
        streams.append(x)
    return rms(x, w["final.norm"], eps) @ w["embed"].T, torch.stack(streams)
