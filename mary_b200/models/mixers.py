"""Sequence mixers and the dense feed-forward that decoder layers are assembled from.

Every mixer is a module over the flattened ragged batch: ``mixer(x, meta, cache) -> [T, width]`` in f32 (what a post-norm consumes), with
its input projections fused into one product and its sizes and constants as constructor arguments.  Mixers with an attention part
declare their cache pages through ``kv_spec()`` and are given their layer index in the cache as ``kv_index``; mixers with a recurrent part
declare their per-sequence state through ``state_spec(dtype)`` (``{name: (shape, dtype)}``) and get ``state_index``."""
from __future__ import annotations

import torch
from torch import nn

from .. import ops


def param(*shape, dtype, device):
    return nn.Parameter(torch.empty(*shape, dtype=dtype, device=device), requires_grad=False)


def pad8(n: int) -> int:
    return (n + 7) // 8 * 8


class FusedProjection:
    """Row blocks of several projections of the same input stacked into one weight; every block starts at a multiple of 8 rows (the
    rows between are zero), so the blocks of an output row stay 16-byte aligned."""

    def __init__(self, blocks: dict[str, int]):
        self.at, n = {}, 0
        for name, rows in blocks.items():
            self.at[name] = (n, rows)
            n += pad8(rows)
        self.rows = n

    def fill(self, weight, name: str, value) -> None:
        a, n = self.at[name]
        weight.data[a:a + n].copy_(value)

    def part(self, y, name: str):
        a, n = self.at[name]
        return y[:, a:a + n]


class DenseGLU(nn.Module):
    """``down(act(gate x) * (up x))`` as f32."""

    def __init__(self, width: int, ff: int, act: str, dtype, device):
        super().__init__()
        self.act, self.ff = act, ff
        self.w_gu, self.w_down = param(2 * ff, width, dtype=dtype, device=device), param(width, ff, dtype=dtype, device=device)

    def forward(self, x):
        return ops.linear_f32(ops.linear_glu(x, self.w_gu, self.act), self.w_down)


def state_shape(heads: int, dk: int, dv: int):
    """One column of key channels (padded to whole 16-byte vectors) per head and value channel."""
    return heads, dv, (dk + 3) // 4 * 4


class AttentionLinearMixer(nn.Module):
    """Softmax attention (grouped query heads, per-head query / key norm, no rotation) and decayed linear attention side by side on the
    same input; result ``a_scale * attention + l_scale * linear``.  One input projection; the two read-outs share one output projection:
    ``a_scale [o_a | (l_scale / a_scale) o_l] [W_a | W_l]^T``, the ratio applied in 32 bits before ``o_l`` is rounded."""

    def __init__(self, width, heads, kv_heads, dk, dv, scale, a_scale, l_heads, l_dk, l_dv, tau, rank, l_scale, eps, dtype, device):
        super().__init__()
        if l_dk > 256 or dk > 512 or dv > 512:
            raise ValueError(f"head widths {dk}/{dv} (attention) and {l_dk} (recurrent keys) exceed what the kernels hold (512/512 and 256)")
        self.heads, self.kv_heads, self.dk, self.dv, self.scale, self.eps = heads, kv_heads, dk, dv, scale, eps
        self.l_heads, self.l_dk, self.l_dv, self.inv_tau = l_heads, l_dk, l_dv, 1.0 / tau
        self.alpha, self.l_ratio = (a_scale, l_scale / a_scale) if a_scale != 0.0 else (1.0, l_scale)
        self.drop_attention = a_scale == 0.0
        kw = dict(dtype=dtype, device=device)
        self.proj = FusedProjection(dict(q=heads * dk, k=kv_heads * dk, v=kv_heads * dv, lq=l_heads * l_dk, lk=l_heads * l_dk, lv=l_heads * l_dv,
                                         lg=l_heads * l_dv, low=rank))
        self.k_att, self.k_lin = heads * dv, l_heads * l_dv
        self.w_in = param(self.proj.rows, width, **kw)
        self.w_out = param(width, self.k_att + self.k_lin, **kw)
        self.q_gain, self.k_gain, self.l_gain = param(dk, **kw), param(dk, **kw), param(l_dv, **kw)
        self.w_decay, self.b_decay = param(l_heads * l_dk, rank, **kw), param(l_heads * l_dk, **kw)
        self.kv_index = self.state_index = -1

    def kv_spec(self):
        return self.kv_heads, self.dk, self.dv

    def state_spec(self, dtype):
        return {"S": (state_shape(self.l_heads, self.l_dk, self.l_dv), torch.float32)}

    def forward(self, x, meta, cache):
        y = ops.linear(x, self.w_in)
        part = lambda n: self.proj.part(y, n)  # noqa: E731
        kc, vc = cache.k[self.kv_index], cache.v[self.kv_index]
        o = ops.rows_buffer(x.shape[0], self.k_att + self.k_lin, x)
        q = ops.qk_norm_append(part("q"), part("k"), part("v"), self.heads, self.kv_heads, self.dk, self.dv, self.q_gain, self.k_gain, meta, kc, vc,
                               self.eps)
        ops.attention_exact(q, kc, vc, meta, self.scale, out=o[:, :self.k_att])
        ops.decayed_linear_attention(part("lq"), part("lk"), part("lv"), part("lg"), part("low"), self.w_decay, self.b_decay, self.inv_tau,
                                     self.l_gain, cache.state[self.state_index]["S"], meta, self.l_heads, self.l_dk, self.l_dv, self.eps,
                                     self.l_ratio, o[:, self.k_att:])
        return ops.linear_f32(o, self.w_out, alpha=self.alpha)

    def load(self, get, p: str) -> None:
        """``get(name)`` returns a tensor of the checkpoint; ``p`` is the mixer's prefix."""
        for mine, theirs in dict(q="left.q", k="left.k", v="left.v", lq="right.q", lk="right.k", lv="right.v", lg="right.g", low="right.a1").items():
            self.proj.fill(self.w_in, mine, get(p + theirs))
        w_a = get(p + "left.o")
        self.w_out.data[:, :self.k_att].copy_(torch.zeros_like(w_a) if self.drop_attention else w_a)
        self.w_out.data[:, self.k_att:].copy_(get(p + "right.o"))
        for mine, theirs in ((self.q_gain, "left.q.norm"), (self.k_gain, "left.k.norm"), (self.l_gain, "right.norm"), (self.w_decay, "right.a2"),
                             (self.b_decay, "right.a2.b")):
            mine.data.copy_(get(p + theirs))


class GatedDeltaMixer(nn.Module):
    """Gated delta rule with short convolutions on q, k, v, unit-norm queries and keys (grouped value heads), one decay and one write
    strength per value head, gated norm of the read-out."""

    def __init__(self, width, heads, kv_heads, dk, dv, taps, eps, dtype, device):
        super().__init__()
        if dk > 256:
            raise ValueError(f"recurrent key width {dk} exceeds what the kernels hold (256)")
        self.heads, self.kv_heads, self.dk, self.dv, self.taps, self.eps = heads, kv_heads, dk, dv, taps, eps
        kw = dict(dtype=dtype, device=device)
        self.channels = 2 * kv_heads * dk + heads * dv
        self.proj = FusedProjection(dict(qkv=self.channels, g=heads * dv, b=heads, a=heads))
        self.w_in, self.w_out = param(self.proj.rows, width, **kw), param(width, heads * dv, **kw)
        self.w_taps, self.gain = param(self.channels, taps, **kw), param(dv, **kw)
        self.a_log, self.dt_bias = param(heads, dtype=torch.float32, device=device), param(heads, dtype=torch.float32, device=device)
        self.kv_index = self.state_index = -1

    def kv_spec(self):
        return None

    def state_spec(self, dtype):
        return {"S": (state_shape(self.heads, self.dk, self.dv), torch.float32), "conv": ((self.taps, self.channels), dtype)}

    def forward(self, x, meta, cache):
        y = ops.linear(x, self.w_in)
        part = lambda n: self.proj.part(y, n)  # noqa: E731
        st = cache.state[self.state_index]
        o = ops.rows_buffer(x.shape[0], self.heads * self.dv, x)
        ops.gated_delta_attention(part("qkv"), self.w_taps, part("b"), part("a"), self.a_log, self.dt_bias, part("g"), self.gain, st["conv"], st["S"],
                                  meta, self.kv_heads, self.heads, self.dk, self.dv, self.eps, 1.0, o)
        return ops.linear_f32(o, self.w_out)

    def load(self, get, p: str) -> None:
        self.proj.fill(self.w_in, "qkv", torch.cat([get(p + n) for n in "qkv"], 0))
        for n in "gba":
            self.proj.fill(self.w_in, n, get(p + n))
        self.w_taps.data.copy_(torch.cat([get(p + n + ".conv") for n in "qkv"], 0))
        for mine, theirs in ((self.w_out, "o"), (self.gain, "norm"), (self.a_log, "A_log"), (self.dt_bias, "dt_bias")):
            mine.data.copy_(get(p + theirs))
