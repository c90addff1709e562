"""Nipurax: a decoder with parallel sublayers around a 32-bit residual stream, part of which is a loop over the same layers.

Layer: ``h += m (mixer(n1(h)) + ff(n2(h)))``, RMS norms of the same ``h``; the feed-forward is a mixture of experts beside a shared one, or
absent.  A mixer is capped attention with sinks or differential attention within chunks (``models/mixers.py``).  The embedding adds a row per
token pair.  Layers ``start .. stop - 1`` run several times with the same weights, each pass with a cache of its own, and before each pass
the stream is replaced by a product of itself and the embedding output plus a vector of the pass.

What is fused: the mixer's output projection and the shared expert's down projection are one product; the residual step sums the routed
experts, adds and norms in one pass (``ops.stream_step``).  The model runs over the flattened ragged batch with the paged cache, the newest
token of every sequence in the cache's state slots; bf16 or 32-bit activations."""
from __future__ import annotations

import torch
from torch import nn

from ... import ops
from ..mixers import CappedAttentionMixer, DifferentialAttentionMixer, JoinedColumns, RoutedExperts, param, stepped_frequencies
from .config import CappedSpec, NipuraxConfig


def _mixer(cfg: NipuraxConfig, s, dtype, device):
    if isinstance(s, CappedSpec):
        return CappedAttentionMixer(cfg.width, s.heads, s.kv_heads, s.dim, s.vdim, s.scale, s.softcap, (s.temp_coef, s.temp_every), dtype, device)
    r = s.rot
    return DifferentialAttentionMixer(cfg.width, s.heads, s.kv_heads, s.dim, s.vdim, s.scale, s.chunk,
                                      stepped_frequencies(r.dims, r.base, r.factor, r.low, r.high, r.original), s.diff, cfg.eps, dtype, device)


class NipuraxLayer(nn.Module):
    def __init__(self, cfg: NipuraxConfig, i: int, dtype, device):
        super().__init__()
        spec, kw = cfg.layers[i], dict(dtype=dtype, device=device)
        e = spec.mlp
        self.mixer = _mixer(cfg, spec.mixer, dtype, device)
        self.norm1 = param(cfg.width, **kw)
        self.norm2 = self.experts = self.w_shared = None
        blocks = {"mixer": self.mixer.out_width}
        if e is not None:
            self.norm2 = param(cfg.width, **kw)
            self.experts = RoutedExperts(cfg.width, e.experts, e.identity, e.expert.ff, e.top, e.scale, "clamped", e.expert.limit, dtype, device)
            if e.shared is not None:
                self.shared = e.shared
                self.w_shared = param(2 * e.shared.ff, cfg.width, **kw)
                blocks["shared"] = e.shared.ff
        self.joined = JoinedColumns(blocks)
        self.w_out = param(cfg.width, self.joined.cols, **kw)

    @property
    def gains(self):
        return (self.norm1,) if self.norm2 is None else (self.norm1, self.norm2)

    def forward(self, xs, meta, kc, vc):
        """``xs``: the stream through this layer's norms.  Returns the mixer's plus the shared expert's output (f32) and the routed experts'."""
        o = self.joined.buffer(xs[0].shape[0], xs[0])
        self.mixer(xs[0], meta, kc, vc, self.joined.part(o, "mixer"))
        if self.w_shared is not None:
            ops.linear_glu(xs[1], self.w_shared, "clamped", self.shared.limit, out=self.joined.part(o, "shared"))
        return ops.linear_f32(o, self.w_out), None if self.experts is None else self.experts(xs[1])

    def load(self, get, p: str) -> None:
        self.norm1.data.copy_(get(p + "norm1"))
        self.mixer.load(get, p + "mix.")
        self.mixer.finish()
        self.joined.fill(self.w_out, "mixer", get(p + "mix.o"))
        if self.experts is not None:
            self.norm2.data.copy_(get(p + "norm2"))
            self.experts.load(get, p + "mlp.")
        if self.w_shared is not None:
            ff = self.shared.ff
            self.w_shared.data[:ff].copy_(get(p + "mlp.shared.gate"))
            self.w_shared.data[ff:].copy_(get(p + "mlp.shared.up"))
            self.joined.fill(self.w_out, "shared", get(p + "mlp.shared.down"))


class NipuraxModel(nn.Module):
    def __init__(self, cfg: NipuraxConfig, pair_rows: int | None = None, dtype=torch.float32, device="cpu"):
        """``pair_rows``: rows of the pair table in the checkpoint, the configuration's buckets and the row of first tokens when not given."""
        super().__init__()
        self.cfg, self.dtype = cfg, dtype
        kw = dict(dtype=dtype, device=device)
        if pair_rows is not None and pair_rows != cfg.pairs.buckets + 1:
            raise ValueError(f"a pair table of {pair_rows} rows for {cfg.pairs.buckets} buckets and the row of first tokens")
        self.embed, self.head = param(cfg.vocab, cfg.width, **kw), param(cfg.vocab, cfg.width, **kw)
        self.pairs = param(cfg.pairs.buckets + 1, cfg.width, **kw)
        self.layers = nn.ModuleList([NipuraxLayer(cfg, i, dtype, device) for i in range(len(cfg.layers))])
        self.norm = param(cfg.width, **kw)
        self.runs = cfg.runs()
        self.joined = self.w_loop = self.loop_step = None
        if cfg.loop is not None:
            self.joined = JoinedColumns(dict(x=cfg.width, x0=cfg.width))
            self.w_loop, self.loop_step = param(cfg.width, self.joined.cols, **kw), param(cfg.loop.times, cfg.width, **kw)

    def kv_spec(self):
        specs = [self.layers[i].mixer.kv_spec() for i, _ in self.runs]          # every pass has pages of its own
        return dict(num_layers=len(specs), kv_heads=[s[0] for s in specs], head_dim=[s[1] for s in specs], v_head_dim=[s[2] for s in specs])

    def state_spec(self):
        return [{"last": ((1,), torch.int32)}]

    def head_weight(self):
        return self.head

    def _layers(self, ids, meta, cache):
        """Goes through the layer runs one by one: yields ``(stream, normed inputs of what follows)`` before the first and after each."""
        c, eps = self.cfg, self.cfg.eps
        loop = x = x0 = None
        if self.joined is not None:
            loop = self.joined.buffer(ids.shape[0], self.embed)
            x, x0 = self.joined.part(loop, "x"), self.joined.part(loop, "x0")

        def follow(j):
            """What the residual step leaves for run ``j``: the stream itself where a pass begins, else its normed inputs."""
            if j == len(self.runs):
                return dict(gains=(self.norm,), eps=eps)
            i, t = self.runs[j]
            return dict(gains=self.layers[i].gains, eps=eps) if t is None else dict(copy=x)
        enters = self.runs[0][1] is not None
        h = ops.embed_pairs(ids, self.embed, self.pairs, c.pairs.mul_prev, c.pairs.mul_cur, cache.state[0]["last"], meta, x0, x if enters else None)
        xs = [] if enters else ops.stream_step(h, **follow(0))
        yield h, xs
        for j, (i, t) in enumerate(self.runs):
            layer = self.layers[i]
            if t is not None:
                xs = ops.stream_step(h, ops.linear_f32(loop, self.w_loop), vec=self.loop_step[t], keep=False, gains=layer.gains, eps=eps)
            a, routed = layer(xs, meta, cache.k[j], cache.v[j])
            xs = ops.stream_step(h, a, c.residual_mult, routed, **follow(j + 1))
            yield h, xs

    def hidden(self, ids, meta, cache):
        xs = None
        for _, xs in self._layers(ids, meta, cache):
            pass
        return xs[0]

    trunk = hidden

    def layer_states(self, ids, meta, cache):
        """The residual stream after every layer run ``[runs, T, width]`` (runs the batch like ``hidden``)."""
        return torch.stack([h.clone() for h, _ in self._layers(ids, meta, cache)][1:])

    def forward(self, ids, meta, cache, rows=None):
        x = self.hidden(ids, meta, cache)
        if rows is not None:
            x = x[rows]
        return ops.linear_f32(x, self.head)

    def greedy(self, ids, meta, cache, rows):
        tok, _ = ops.lm_head_argmax(self.hidden(ids, meta, cache)[rows], self.head)
        return tok


def init_random_(model: NipuraxModel, seed: int = 0, std: float = 0.02) -> None:
    g = torch.Generator(device=model.embed.device).manual_seed(seed)
    for n, p in model.named_parameters():
        leaf = n.rpartition(".")[2]
        if leaf in ("norm", "norm1", "norm2"):
            p.data.fill_(1.0)
        elif leaf == "correction":
            p.data.zero_()
        else:
            scale = 1.0 if leaf == "sink" else 0.1 if p.dim() == 1 else std
            for part in (p.data if p.dim() == 3 else [p.data]):           # expert by expert: no f32 copy of all of them
                part.copy_(torch.randn(part.shape, generator=g, device=p.device) * scale)
    for layer in model.layers:
        layer.mixer.finish()


def load_into(model: NipuraxModel, loader) -> None:
    """Fill the model from a ``WeightLoader`` with tensors ``embed``, ``bigram``, ``head``, ``final.norm``, ``loop.*``, ``l<i>.norm*``, ``l<i>.mix.*``,
    ``l<i>.mlp.*``."""
    def get(name):
        return loader.load_tensor(name)
    for p in model.parameters():
        p.data.zero_()                     # rows and columns between the blocks of fused projections
    for mine, theirs in ((model.embed, "embed"), (model.pairs, "bigram"), (model.head, "head"), (model.norm, "final.norm")):
        mine.data.copy_(get(theirs))
    if model.w_loop is not None:
        w = get("loop.in")
        model.joined.fill(model.w_loop, "x", w[:, :model.cfg.width])
        model.joined.fill(model.w_loop, "x0", w[:, model.cfg.width:])
        model.loop_step.data.copy_(get("loop.step"))
    for i, layer in enumerate(model.layers):
        layer.load(get, f"l{i}.")
