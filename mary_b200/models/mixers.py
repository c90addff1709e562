"""Sequence mixers and the dense feed-forward that decoder layers are assembled from.

Every mixer is a module over the flattened ragged batch: ``mixer(x, meta, cache) -> [T, width]`` in f32 (what a post-norm consumes), with
its input projections fused into one product and its sizes and constants as constructor arguments.  Mixers with an attention part
declare their cache pages through ``kv_spec()`` and are given their layer index in the cache as ``kv_index``; mixers with a recurrent part
declare their per-sequence state through ``state_spec(dtype)`` (``{name: (shape, dtype)}``) and get ``state_index``."""
from __future__ import annotations

import math

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

    def load(self, get, p: str) -> None:
        self.w_gu.data[:self.ff].copy_(get(p + "gate"))
        self.w_gu.data[self.ff:].copy_(get(p + "up"))
        self.w_down.data.copy_(get(p + "down"))


class DynamicTanh(nn.Module):
    """``tanh(alpha x) * w + b``: the elementwise stand-in for a norm.  Applied by the op that produces or consumes the residual stream."""

    def __init__(self, width: int, dtype, device):
        super().__init__()
        self.w, self.b = param(width, dtype=dtype, device=device), param(width, dtype=dtype, device=device)
        self.alpha = param(1, dtype=torch.float32, device=device)

    def load(self, get, name: str) -> None:
        self.w.data.copy_(get(name))
        self.b.data.copy_(get(name + ".b"))
        self.alpha.data.copy_(get(name + ".alpha").reshape(1))


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


def distance_buckets(window: int, rows: int, far: float):
    """Row of a bias table with ``rows`` rows for the distances ``0 .. window - 1``: one row each up to half of the table, from there
    logarithmic steps that reach the last row at distance ``far``."""
    half = rows // 2
    if window > half and (rows < 2 or far <= half):
        raise ValueError(f"a table of {rows} rows cannot reach to distance {far}")
    step = math.log(far / half)
    return torch.tensor([n if n < half else min(rows - 1, half + math.floor(math.log(n / half) / step * (rows - half))) for n in range(window)])


def yarn_frequencies(dims: int, base: float, factor: float | None = None, original: float = 0.0, fast: float = 0.0, slow: float = 0.0):
    """``(rotation frequencies [dims / 2] in f64, gain of cosine and sine)``.  With a ``factor``, dimensions that turn fewer than ``slow``
    times over ``original`` positions are slowed down by it, those that turn more than ``fast`` times are kept, with a ramp between."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    f = base ** (-2.0 * i / dims)
    if factor is None:
        return f, 1.0
    turn = lambda t: dims * math.log(original / (2.0 * math.pi * t)) / (2.0 * math.log(base))  # noqa: E731
    lo, hi = max(math.floor(turn(fast)), 0), min(math.ceil(turn(slow)), dims - 1)
    ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return f / factor * ramp + f * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


class BiasedAttentionMixer(nn.Module):
    """Sliding-window attention without rotation: queries and keys normed over their whole projection, a learned bias by distance added to the
    scaled score, the heads' output multiplied by a sigmoid gate of the input before the output projection.  ``kv_from``: the layer whose
    cached keys and values are read instead of own ones."""

    def __init__(self, width, heads, kv_heads, dk, dv, scale, window, bias_rows, bias_far, kv_from, eps, dtype, device):
        super().__init__()
        if dk > 640 or dv > 512:
            raise ValueError(f"head widths {dk}/{dv} exceed what the kernels hold (640/512)")
        self.heads, self.kv_heads, self.dk, self.dv, self.scale, self.window, self.eps = heads, kv_heads, dk, dv, scale, window, eps
        self.kv_from, self.bias_far = kv_from, bias_far
        kw = dict(dtype=dtype, device=device)
        own = dict(k=kv_heads * dk, v=kv_heads * dv) if kv_from is None else {}
        self.proj = FusedProjection(dict(q=heads * dk, **own, g=heads * dv))
        self.w_in, self.w_out = param(self.proj.rows, width, **kw), param(width, heads * dv, **kw)
        self.q_gain = param(heads * dk, **kw)
        self.k_gain = param(kv_heads * dk, **kw) if kv_from is None else None
        self.rel = param(bias_rows, heads, dtype=torch.float32, device=device)
        self.register_buffer("bias", torch.zeros(heads, window, dtype=torch.float32, device=device), persistent=False)      # by distance
        self.kv_index = self.state_index = -1

    def kv_spec(self):
        return (self.kv_heads, self.dk, self.dv) if self.kv_from is None else None

    def state_spec(self, dtype):
        return None

    def finish(self) -> None:
        """Spread the bias table over the distances of the window (after the parameters have been set)."""
        at = distance_buckets(self.window, self.rel.shape[0], self.bias_far).to(self.rel.device)
        self.bias.copy_(self.rel.data[at].T)

    def forward(self, x, meta, cache):
        y = ops.linear(x, self.w_in)
        part = lambda n: self.proj.part(y, n)  # noqa: E731
        kc, vc = cache.k[self.kv_index], cache.v[self.kv_index]
        k, v = (part("k"), part("v")) if self.kv_from is None else (None, None)
        q = ops.row_norm_append(part("q"), k, v, self.heads, self.kv_heads, self.dk, self.dv, self.q_gain, self.k_gain, meta, kc, vc, self.eps)
        o = ops.rows_buffer(x.shape[0], self.heads * self.dv, x)
        ops.attention_exact(q, kc, vc, meta, self.scale, out=o, window=self.window, bias=self.bias, gate=part("g"))
        return ops.linear_f32(o, self.w_out)

    def load(self, get, p: str) -> None:
        for n in self.proj.at:
            self.proj.fill(self.w_in, n, get(p + n))
        for mine, theirs in ((self.w_out, "o"), (self.q_gain, "q.norm"), (self.k_gain, "k.norm"), (self.rel, "rel")):
            if mine is not None:
                mine.data.copy_(get(p + theirs))


class LatentAttentionMixer(nn.Module):
    """Sliding-window attention over a latent: the cache row of a token is ``[normed latent | rotated key part shared by all heads]``; per-head
    keys and values are linear in the latent, so one-token steps attend in latent space (the key matrix applied to the query, the value
    matrix to the read-out) and prompts attend over expanded keys and values where that is the smaller work."""

    kv_from = None

    def __init__(self, width, heads, dim, rot, dv, q_rank, rank, scale, window, freq, rot_gain, eps, dtype, device):
        super().__init__()
        if rank + rot > 640 or rank > 512:
            raise ValueError(f"latent width {rank} + {rot} exceeds what the kernels hold (512, 640 with the rotated part)")
        self.heads, self.dim, self.rot, self.dv, self.rank, self.q_rank = heads, dim, rot, dv, rank, q_rank
        self.scale, self.window, self.rot_gain, self.eps = scale, window, rot_gain, eps
        kw = dict(dtype=dtype, device=device)
        self.proj = FusedProjection(dict(dq=q_rank, dkv=rank + rot))
        self.w_in, self.w_out = param(self.proj.rows, width, **kw), param(width, heads * dv, **kw)
        self.q_gain, self.kv_gain = param(q_rank, **kw), param(rank, **kw)
        self.w_q, self.w_k, self.w_v = param(heads * (dim + rot), q_rank, **kw), param(heads * dim, rank, **kw), param(heads * dv, rank, **kw)
        self.register_buffer("w_k_t", torch.zeros(heads, rank, dim, **kw), persistent=False)      # the key matrices, applied to queries
        self.register_buffer("freq", freq.to(torch.float32).to(device), persistent=False)
        self.kv_index = self.state_index = -1

    def kv_spec(self):
        return 1, self.rank + self.rot, 0           # the values are part of the key row

    def state_spec(self, dtype):
        return None

    def finish(self) -> None:
        self.w_k_t.copy_(self.w_k.data.view(self.heads, self.dim, self.rank).transpose(1, 2))

    def forward(self, x, meta, cache):
        y = ops.linear(x, self.w_in)
        rows = cache.k[self.kv_index]
        c = ops.latent_prep(self.proj.part(y, "dq"), self.proj.part(y, "dkv"), self.q_gain, self.kv_gain, self.freq, self.rot_gain, meta, rows, self.eps)
        o = ops.latent_attention(ops.linear(c, self.w_q), rows, meta, self)
        return ops.linear_f32(o, self.w_out)

    def load(self, get, p: str) -> None:
        for n in self.proj.at:
            self.proj.fill(self.w_in, n, get(p + n))
        for mine, theirs in ((self.w_out, "o"), (self.q_gain, "dq.norm"), (self.kv_gain, "dkv.norm"), (self.w_q, "uq"), (self.w_k, "uk"), (self.w_v, "uv")):
            mine.data.copy_(get(p + theirs))


class StateSpaceMixer(nn.Module):
    """Mamba-2 (state-space duality): short convolutions with bias on ``x``, ``B``, ``C``, one step size and decay per head, ``B`` and ``C``
    shared by the heads of a group, a skip per head, the read-out gated and then normed in equal parts."""

    kv_from = None

    def __init__(self, width, heads, dv, state, groups, taps, norm_parts, eps, dtype, device):
        super().__init__()
        if state > 256:
            raise ValueError(f"state width {state} exceeds what the kernels hold (256)")
        self.heads, self.dv, self.state, self.groups, self.taps, self.norm_parts, self.eps = heads, dv, state, groups, taps, norm_parts, eps
        kw, f32 = dict(dtype=dtype, device=device), dict(dtype=torch.float32, device=device)
        self.inner = heads * dv
        self.channels = self.inner + 2 * groups * state
        self.proj = FusedProjection(dict(z=self.inner, xbc=self.channels, dt=heads))
        self.w_in, self.w_out = param(self.proj.rows, width, **kw), param(width, self.inner, **kw)
        self.w_taps, self.b_taps, self.gain = param(self.channels, taps, **kw), param(self.channels, **kw), param(self.inner, **kw)
        self.a_log, self.dt_bias, self.skip = param(heads, **f32), param(heads, **f32), param(heads, **f32)
        self.kv_index = self.state_index = -1

    def kv_spec(self):
        return None

    def state_spec(self, dtype):
        return {"S": (state_shape(self.heads, self.state, self.dv), torch.float32), "conv": ((self.taps, self.channels), dtype)}

    def finish(self) -> None:
        pass

    def forward(self, x, meta, cache):
        y = ops.linear(x, self.w_in)
        part = lambda n: self.proj.part(y, n)  # noqa: E731
        st = cache.state[self.state_index]
        o = ops.rows_buffer(x.shape[0], self.inner, x)
        ops.state_space(part("xbc"), self.w_taps, self.b_taps, part("dt"), self.dt_bias, self.a_log, self.skip, part("z"), self.gain, self.norm_parts,
                        st["conv"], st["S"], meta, self.groups, self.heads, self.state, self.dv, self.eps, o)
        return ops.linear_f32(o, self.w_out)

    def load(self, get, p: str) -> None:
        w, at = get(p + "in"), 0
        for n, (_, rows) in self.proj.at.items():
            self.proj.fill(self.w_in, n, w[at:at + rows])
            at += rows
        for mine, theirs in ((self.w_out, "o"), (self.w_taps, "conv"), (self.b_taps, "conv.b"), (self.gain, "norm"), (self.a_log, "A_log"),
                             (self.dt_bias, "dt_bias"), (self.skip, "D")):
            mine.data.copy_(get(p + theirs))


def stepped_frequencies(dims: int, base: float, factor: float | None = None, low: float = 0.0, high: float = 0.0, original: float = 0.0):
    """Rotation frequencies ``[dims / 2]`` in f64.  With a ``factor``: wavelengths below ``original / high`` stay, those above ``original / low`` grow by
    the factor, between them the two frequencies are blended linearly in ``original / wavelength``."""
    f = base ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims)
    if factor is None:
        return f
    turns = original * f / (2.0 * math.pi)
    s = ((turns - low) / (high - low)) if high != low else torch.zeros_like(f)
    return torch.where(turns > high, f, torch.where(turns < low, f / factor, (1.0 - s) * f / factor + s * f))


class JoinedColumns:
    """Several inputs side by side, every block from a multiple of 8 columns on, for one product with a matrix whose columns are laid out alike
    (``[b0 | b1 | ..] [W0 | W1 | ..]^T``, the sum of the blocks' products); columns between blocks are zero on both sides."""

    def __init__(self, blocks: dict[str, int]):
        self.at, n = {}, 0
        for name, cols in blocks.items():
            self.at[name] = (n, cols)
            n += pad8(cols)
        self.cols, self.gaps = n, any(c % 8 for c in blocks.values())

    def fill(self, weight, name: str, value) -> None:
        a, n = self.at[name]
        weight.data[:, a:a + n].copy_(value)

    def buffer(self, rows: int, like):
        return (torch.zeros if self.gaps else torch.empty)(rows, self.cols, dtype=like.dtype, device=like.device)

    def part(self, buf, name: str):
        a, n = self.at[name]
        return buf[:, a:a + n]


class CappedAttentionMixer(nn.Module):
    """Causal attention without rotation: the query scaled by a temperature that grows with the logarithm of the position, the score capped by a
    hyperbolic tangent, a learned sink per head in the sum of the weights.  Writes the heads' outputs; the output projection is the caller's."""

    def __init__(self, width, heads, kv_heads, dk, dv, scale, cap, temperature, dtype, device):
        super().__init__()
        if dk > 640 or dv > 512:
            raise ValueError(f"head widths {dk}/{dv} exceed what the kernels hold (640/512)")
        self.heads, self.kv_heads, self.dk, self.dv, self.scale, self.cap, self.temperature = heads, kv_heads, dk, dv, scale, cap, temperature
        self.proj = FusedProjection(dict(q=heads * dk, k=kv_heads * dk, v=kv_heads * dv))
        self.w_in = param(self.proj.rows, width, dtype=dtype, device=device)
        self.sink = param(heads, dtype=torch.float32, device=device)

    @property
    def out_width(self) -> int:
        return self.heads * self.dv

    def kv_spec(self):
        return self.kv_heads, self.dk, self.dv

    def finish(self) -> None:
        self.form = ops.AttentionForm(cap=self.cap, sink=self.sink.data, temperature=self.temperature)

    def forward(self, x, meta, kc, vc, out):
        y = ops.linear(x, self.w_in)
        part = lambda n: self.proj.part(y, n)  # noqa: E731
        ops.rotate_append(None, part("k"), part("v"), self.heads, self.kv_heads, self.dk, None, meta, kc, vc)
        ops.attention_exact(part("q").unflatten(1, (self.heads, self.dk)), kc, vc, meta, self.scale, out=out, form=self.form)

    def load(self, get, p: str) -> None:
        for n in "qkv":
            self.proj.fill(self.w_in, n, get(p + n))
        self.sink.data.copy_(get(p + "sink"))


class DifferentialAttentionMixer(nn.Module):
    """Attention within chunks of the sequence as the difference of two softmax maps over the same values: query and key heads hold the maps side
    by side (split-half rotation on the first dimensions of each), the second map enters with a learned weight, the result is normed per head.
    Writes the heads' outputs; the output projection is the caller's."""

    def __init__(self, width, heads, kv_heads, dk, dv, scale, chunk, freq, diff, eps, dtype, device):
        super().__init__()
        if dk > 640 or dv > 512:
            raise ValueError(f"head widths {dk}/{dv} exceed what the kernels hold (640/512)")
        self.heads, self.kv_heads, self.dk, self.dv, self.scale, self.chunk, self.diff, self.eps = heads, kv_heads, dk, dv, scale, chunk, diff, eps
        self.proj = FusedProjection(dict(q=2 * heads * dk, k=2 * kv_heads * dk, v=kv_heads * dv))
        self.w_in = param(self.proj.rows, width, dtype=dtype, device=device)
        self.mix = nn.ParameterDict({n: param(dk, dtype=torch.float32, device=device) for n in ("lq1", "lk1", "lq2", "lk2")})
        self.register_buffer("freq", freq.to(torch.float64).to(device), persistent=False)

    @property
    def out_width(self) -> int:
        return self.heads * self.dv

    def kv_spec(self):
        return self.kv_heads, 2 * self.dk, self.dv

    def finish(self) -> None:
        dot = lambda i: float((self.mix[f"lq{i}"].double() * self.mix[f"lk{i}"].double()).sum())  # noqa: E731
        mix = math.exp(dot(1)) - math.exp(dot(2)) + self.diff
        self.form = ops.AttentionForm(chunk=self.chunk, difference=(mix, 1.0 - self.diff, self.eps))

    def forward(self, x, meta, kc, vc, out):
        y = ops.linear(x, self.w_in)
        part = lambda n: self.proj.part(y, n)  # noqa: E731
        q = part("q")
        ops.rotate_append(q, part("k"), part("v"), 2 * self.heads, 2 * self.kv_heads, self.dk, self.freq, meta, kc, vc)
        ops.attention_exact(q.unflatten(1, (self.heads, 2 * self.dk)), kc, vc, meta, self.scale, out=out, form=self.form)

    def load(self, get, p: str) -> None:
        for n in "qkv":
            self.proj.fill(self.w_in, n, get(p + n))
        for n, v in self.mix.items():
            v.data.copy_(get(p + n))


class TurnedAttentionMixer(nn.Module):
    """Causal attention in which values are rotated as well: queries and keys turned by neighbouring pairs on their first dimensions and then divided by
    their root mean square, a learned temperature per head, scores capped by a hyperbolic tangent, a sink of score 0 without a value; values enter the
    cache turned by their position, and the result is turned back by the query's.  Writes the heads' outputs; the output projection is the
    caller's."""

    def __init__(self, width, heads, kv_heads, dk, dv, scale, cap, freq, gain, vfreq, eps, dtype, device):
        """``freq`` (f64) and ``gain``: as ``yarn_frequencies`` gives them; ``vfreq``: frequencies of the value pairs."""
        super().__init__()
        if dk > 640 or dv > 512 or 2 * vfreq.numel() != dv:
            raise ValueError(f"head widths {dk}/{dv}: the kernels hold 640/512, and values are turned in pairs")
        self.heads, self.kv_heads, self.dk, self.dv, self.scale, self.cap, self.gain, self.eps = heads, kv_heads, dk, dv, scale, cap, gain, eps
        self.proj = FusedProjection(dict(q=heads * dk, k=kv_heads * dk, v=kv_heads * dv))
        self.w_in = param(self.proj.rows, width, dtype=dtype, device=device)
        self.temp = param(heads, dtype=torch.float32, device=device)
        for name, f in (("freq", freq), ("vfreq", vfreq)):
            self.register_buffer(name, f.to(torch.float64).to(device), persistent=False)
        self.register_buffer("sink", torch.zeros(heads, dtype=torch.float32, device=device), persistent=False)
        self.table_key = (tuple(freq.tolist()), gain, tuple(vfreq.tolist()))

    @property
    def out_width(self) -> int:
        return self.heads * self.dv

    def kv_spec(self):
        return self.kv_heads, self.dk, self.dv

    def tables(self, meta):
        """Cosines and sines of the batch's positions for queries and keys and for values; the same for every mixer with this ``table_key``."""
        return ops.turn_table(meta.positions, self.freq, self.gain) if self.freq.numel() else None, ops.turn_table(meta.positions, self.vfreq)

    def forward(self, x, meta, kc, vc, tables, out):
        y = ops.linear(x, self.w_in)
        part = lambda n: self.proj.part(y, n)  # noqa: E731
        q, (turn, vturn) = part("q"), tables
        ops.turn_norm_append(q, part("k"), part("v"), self.heads, self.kv_heads, self.dk, turn, vturn, self.temp, meta, kc, vc, self.eps)
        ops.attention_exact(q.unflatten(1, (self.heads, self.dk)), kc, vc, meta, self.scale, out=out,
                            form=ops.AttentionForm(cap=self.cap, sink=self.sink, turn=vturn))

    def load(self, get, p: str) -> None:
        for n in "qkv":
            self.proj.fill(self.w_in, n, get(p + n))
        self.temp.data.copy_(get(p + "temp"))


class HeadDecays(nn.Module):
    """One constant decay per head in the forms that the kernels take: ``head [H]``, ``channel [H * dk]`` and, for chunks of 64 tokens, ``chunk [4, H, 64]``: a step
    size of one, log2 of ``d ** 1 .. d ** 64`` as two floats, a skip of zero."""

    def __init__(self, decays, dk: int, device):
        super().__init__()
        d = torch.tensor(decays, dtype=torch.float64)
        if bool((d < 0.0).any()) or bool((d > 1.0).any()):
            raise ValueError(f"decays {list(decays)} outside 0 .. 1")
        c = torch.log2(d).clamp(min=-1e4)[:, None] * torch.arange(1, 65, dtype=torch.float64)       # 2 ** -1e4 is zero in 32 bits
        hi = c.float()
        chunk = torch.stack([torch.ones_like(hi), hi, (c - hi.double()).float(), torch.zeros_like(hi)])
        for name, t in (("head", d.float()), ("channel", d.float().repeat_interleave(dk)), ("chunk", chunk)):
            self.register_buffer(name, t.contiguous().to(device), persistent=False)


class LightningMixer(nn.Module):
    """Linear attention with one constant decay per head, SiLU on queries, keys and values; the read-out of all heads normed together and gated by a
    logistic function of the input.  Writes the gated row; the output projection is the caller's."""

    def __init__(self, width, heads, dk, dv, decays, eps, dtype, device):
        super().__init__()
        if dk > 256 or dv > 4096:
            raise ValueError(f"recurrent widths {dk}/{dv} exceed what the kernels hold (256/4096)")
        if len(decays) != heads:
            raise ValueError(f"{len(decays)} decays for {heads} heads")
        self.heads, self.dk, self.dv, self.eps = heads, dk, dv, eps
        self.proj = FusedProjection(dict(v=heads * dv, k=heads * dk, q=heads * dk, g=heads * dv))
        self.w_in = param(self.proj.rows, width, dtype=dtype, device=device)
        self.norm = param(heads * dv, dtype=dtype, device=device)
        self.decays = HeadDecays(decays, dk, device)

    @property
    def out_width(self) -> int:
        return self.heads * self.dv

    def state_spec(self):
        return {"S": (state_shape(self.heads, self.dk, self.dv), torch.float32)}

    def forward(self, x, meta, state, out):
        y = ops.linear_act(x, self.w_in, "silu", cols=self.proj.at["g"][0])
        part = lambda n: self.proj.part(y, n)  # noqa: E731
        ops.lightning_attention(y, part("q"), part("k"), part("v"), part("g"), self.decays, self.norm, state["S"], meta, self.heads, self.dk, self.dv,
                                self.eps, out)

    def load(self, get, p: str) -> None:
        for n in self.proj.at:
            self.proj.fill(self.w_in, n, get(p + n))
        self.norm.data.copy_(get(p + "norm"))


class DenseMLP(nn.Module):
    """``down(act(up x))`` as f32."""

    def __init__(self, width: int, ff: int, act: str, dtype, device):
        super().__init__()
        self.act = act
        self.w_up, self.w_down = param(ff, width, dtype=dtype, device=device), param(width, ff, dtype=dtype, device=device)

    def forward(self, x):
        return ops.linear_f32(ops.linear_act(x, self.w_up, self.act), self.w_down)

    def load(self, get, p: str) -> None:
        self.w_up.data.copy_(get(p + "up"))
        self.w_down.data.copy_(get(p + "down"))


class StreamWeights(nn.Module):
    """How one sublayer reads from and writes to ``n`` residual streams: its input ``sum_s read[s] x_s``, then ``x_t <- sum_s mix[s, t] x_s + write[t] y``.
    A single stream without weights of its own is the plain residual sum."""

    def __init__(self, n: int, device):
        super().__init__()
        self.read, self.write, self.mix = (param(*shape, dtype=torch.float32, device=device) for shape in ((n,), (n,), (n, n)))

    def plain(self) -> None:
        for p in (self.read, self.write, self.mix):
            p.data.fill_(1.0)

    def load(self, get, p: str) -> None:
        for mine, theirs in ((self.read, "in"), (self.write, "out"), (self.mix, "mix")):
            mine.data.copy_(get(p + theirs))


class RoutedExperts(nn.Module):
    """A mixture of GLU experts: softmax scores over all of them, the ``top`` best by score plus a correction (``correction`` False: by score), weighted by
    ``scale`` times the score, or with ``renorm`` by the softmax over the chosen ones.  The last ``identity`` scores stand for the input itself; ``extra`` more
    router rows give logits of their own.  The result goes to ``ops.stream_step`` or ``ops.mix_streams``, which sums it up."""

    def __init__(self, width, experts, identity, ff, top, scale, act, limit, dtype, device, renorm: bool = False, correction: bool = True, extra: int = 0):
        super().__init__()
        if experts + identity > 512 or not 1 <= top <= min(32, experts + identity):
            raise ValueError(f"{top} of {experts} + {identity} experts: the router holds 512 and chooses up to 32")
        self.experts, self.identity, self.ff, self.top, self.scale, self.act, self.limit = experts, identity, ff, top, scale, act, limit
        kw = dict(dtype=dtype, device=device)
        self.renorm, self.scores = renorm, experts + identity
        self.w_router = param(experts + identity + extra, width, **kw)
        self.correction = param(experts + identity, dtype=torch.float32, device=device) if correction else None
        self.w_gu, self.w_down = param(experts, 2 * ff, width, **kw), param(experts, width, ff, **kw)

    def forward(self, x, z=None):
        """``z``: the router's logits where the caller has them already."""
        z = ops.linear_f32(x, self.w_router) if z is None else z
        idx, w = ops.router_topk(z[:, :self.scores], self.top, "softmax", self.correction, scale=self.scale, renorm=self.renorm)
        return ops.expert_outputs(x, idx, w, self.w_gu, self.w_down, self.act, self.limit)

    def load(self, get, p: str) -> None:
        self.w_router.data[:self.scores].copy_(get(p + "router"))
        if self.correction is not None:
            self.correction.data.copy_(get(p + "correction"))
        for e in range(self.experts):
            self.w_gu.data[e, :self.ff].copy_(get(f"{p}e{e}.gate"))
            self.w_gu.data[e, self.ff:].copy_(get(f"{p}e{e}.up"))
            self.w_down.data[e].copy_(get(f"{p}e{e}.down"))


class SharedRoutedExperts(nn.Module):
    """Routed experts weighted by the softmax over the chosen ones, beside a shared expert that a logistic gate per token (its logit is one more row of
    the router) multiplies.  The shared expert may be absent."""

    def __init__(self, width, experts, ff, top, act, limit, shared_ff, shared_limit, dtype, device):
        super().__init__()
        self.act, self.shared_ff, self.shared_limit = act, shared_ff, shared_limit
        self.routed = RoutedExperts(width, experts, 0, ff, top, 1.0, act, limit, dtype, device, renorm=True, correction=False, extra=1 if shared_ff else 0)
        self.w_shared = self.w_down = None
        if shared_ff:
            self.w_shared, self.w_down = param(2 * shared_ff, width, dtype=dtype, device=device), param(width, shared_ff, dtype=dtype, device=device)

    def forward(self, x):
        """``(shared expert's output f32 or None, its gate's logits [T] or None, routed experts)`` as ``ops.mix_streams`` takes them."""
        z = ops.linear_f32(x, self.routed.w_router)
        routed = self.routed(x, z)
        if self.w_shared is None:
            return None, None, routed
        return ops.linear_f32(ops.linear_glu(x, self.w_shared, self.act, self.shared_limit), self.w_down), z[:, self.routed.scores], routed

    def load(self, get, p: str) -> None:
        self.routed.load(get, p)
        if self.w_shared is not None:
            self.routed.w_router.data[self.routed.scores:].copy_(get(p + "shared.sg"))
            self.w_shared.data[:self.shared_ff].copy_(get(p + "shared.gate"))
            self.w_shared.data[self.shared_ff:].copy_(get(p + "shared.up"))
            self.w_down.data.copy_(get(p + "shared.down"))
