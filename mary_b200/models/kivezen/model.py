"""Kivezen: a pre-norm decoder whose residual is several 32-bit streams, part of whose layers run several times.

Layer: ``y = mixer(n1(sum_s in1[s] x_s))``, all streams anew as ``sum_s mix1[s, t] x_s + out1[t] y``; the same for the feed-forward with weights of its
own.  A mixer is attention with turned values and capped scores or linear attention with constant decays (``models/mixers.py``); the feed-forward is
dense, a mixture of experts beside a gated shared one, or absent.  The logits are capped.  Layers ``start .. stop - 1`` run several times with the
same weights, each pass with a cache or state of its own.

What is fused: the update of the streams after a sublayer sums the routed experts, gates the shared one and forms the next sublayer's normed input
(``ops.mix_streams``); activations are applied in the products' epilogues; attention turns its result back.  The rotation tables of a batch are made once
for all layers.  The model runs over the flattened ragged batch with the paged cache, recurrent states in the cache's slots; bf16 or 32-bit
activations."""
from __future__ import annotations

import torch
from torch import nn

from ... import ops
from ..mixers import DenseMLP, LightningMixer, SharedRoutedExperts, StreamWeights, TurnedAttentionMixer, param, yarn_frequencies
from .config import AttentionSpec, DenseSpec, KivezenConfig


def _mixer(cfg: KivezenConfig, s, dtype, device):
    if not isinstance(s, AttentionSpec):
        return LightningMixer(cfg.width, s.heads, s.dim, s.vdim, s.decay, cfg.eps, dtype, device)
    r = s.rot
    freq, gain = yarn_frequencies(r.dims, r.base, r.factor, r.original, r.fast, r.slow)
    return TurnedAttentionMixer(cfg.width, s.heads, s.kv_heads, s.dim, s.vdim, s.scale, s.softcap, freq, gain, yarn_frequencies(s.vdim, r.base)[0], cfg.eps,
                                dtype, device)


def _feed_forward(cfg: KivezenConfig, e, dtype, device):
    if e is None:
        return None
    if isinstance(e, DenseSpec):
        return DenseMLP(cfg.width, e.ff, "gelu", dtype, device)
    shared = (e.shared.ff, e.shared.limit) if e.shared is not None else (0, 0.0)
    return SharedRoutedExperts(cfg.width, e.experts, e.expert.ff, e.top, "clamped", e.expert.limit, *shared, dtype, device)


class KivezenLayer(nn.Module):
    def __init__(self, cfg: KivezenConfig, i: int, dtype, device):
        super().__init__()
        spec, kw = cfg.layers[i], dict(dtype=dtype, device=device)
        self.mixer = _mixer(cfg, spec.mixer, dtype, device)
        self.w_out = param(cfg.width, self.mixer.out_width, **kw)
        self.mlp = _feed_forward(cfg, spec.mlp, dtype, device)
        n = 1 if self.mlp is None else 2
        self.norms = nn.ParameterList([param(cfg.width, **kw) for _ in range(n)])
        self.streams = nn.ModuleList([StreamWeights(cfg.streams or 1, device) for _ in range(n)])

    @property
    def recurrent(self) -> bool:
        return isinstance(self.mixer, LightningMixer)

    def mix(self, x, meta, pages, state, tables):
        """The mixer's output in f32."""
        o = ops.rows_buffer(x.shape[0], self.mixer.out_width, x)
        if self.recurrent:
            self.mixer(x, meta, state, o)
        else:
            self.mixer(x, meta, *pages, tables, o)
        return ops.linear_f32(o, self.w_out)

    def feed(self, x):
        """The feed-forward's output as ``(rows, gate logits, routed experts)``."""
        return (self.mlp(x), None, None) if isinstance(self.mlp, DenseMLP) else self.mlp(x)

    def load(self, get, p: str, plain: bool) -> None:
        self.mixer.load(get, p + "mix.")
        self.w_out.data.copy_(get(p + "mix.o"))
        if self.mlp is not None:
            self.mlp.load(get, p + "mlp.")
        for q, (norm, w) in enumerate(zip(self.norms, self.streams), 1):
            norm.data.copy_(get(f"{p}norm{q}"))
            w.plain() if plain else w.load(get, f"{p}hc{q}.")


class KivezenModel(nn.Module):
    def __init__(self, cfg: KivezenConfig, dtype=torch.float32, device="cpu"):
        super().__init__()
        self.cfg, self.dtype = cfg, dtype
        kw = dict(dtype=dtype, device=device)
        self.embed, self.head = param(cfg.vocab, cfg.width, **kw), param(cfg.vocab, cfg.width, **kw)
        self.layers = nn.ModuleList([KivezenLayer(cfg, i, dtype, device) for i in range(len(cfg.layers))])
        self.norm = param(cfg.width, **kw)
        self.register_buffer("total", torch.ones(cfg.streams or 1, dtype=torch.float32, device=device), persistent=False)      # the sum of the streams
        self.runs = cfg.runs()                     # every run has pages or a state of its own: (layer, its place among them)
        n = {True: 0, False: 0}
        self.places = []
        for i in self.runs:
            r = self.layers[i].recurrent
            self.places.append(n[r])
            n[r] += 1

    def kv_spec(self):
        specs = [self.layers[i].mixer.kv_spec() for i in self.runs if not self.layers[i].recurrent]
        return dict(num_layers=len(specs), kv_heads=[s[0] for s in specs], head_dim=[s[1] for s in specs], v_head_dim=[s[2] for s in specs])

    def state_spec(self):
        return [self.layers[i].mixer.state_spec() for i in self.runs if self.layers[i].recurrent]

    def head_weight(self):
        return self.head

    def _layers(self, ids, meta, cache, keep: bool):
        """Goes through the layer runs one by one: yields ``(streams, normed input of what follows)`` after each.  ``keep``: the streams after the last
        run are wanted too."""
        eps, layers, tables = self.cfg.eps, [self.layers[i] for i in self.runs], {}
        reads = [(w.read, norm) for layer in layers for w, norm in zip(layer.streams, layer.norms)] + [(self.total, self.norm)]
        xs, x = ops.embed_streams(ids, self.embed, self.total.numel(), *reads[0], eps)
        at = 0
        for j, (layer, place) in enumerate(zip(layers, self.places)):
            pages = state = table = None
            if layer.recurrent:
                state = cache.state[place]
            else:
                pages, key = (cache.k[place], cache.v[place]), layer.mixer.table_key
                if key not in tables:
                    tables[key] = layer.mixer.tables(meta)
                table = tables[key]
            for q, w in enumerate(layer.streams):
                y = (layer.mix(x, meta, pages, state, table), None, None) if q == 0 else layer.feed(x)
                at += 1
                x = ops.mix_streams(xs, w.mix, w.write, *y, *reads[at], eps, keep=keep or at + 1 < len(reads))
            yield xs, x
        if not layers:
            yield xs, x

    def hidden(self, ids, meta, cache):
        x = None
        for _, x in self._layers(ids, meta, cache, keep=False):
            pass
        return x

    trunk = hidden

    def layer_states(self, ids, meta, cache):
        """The residual stream (the sum of the streams) after every layer run ``[runs, T, width]`` (runs the batch like ``hidden``)."""
        return torch.stack([xs.sum(1) for xs, _ in self._layers(ids, meta, cache, keep=True)])

    def forward(self, ids, meta, cache, rows=None):
        x = self.hidden(ids, meta, cache)
        if rows is not None:
            x = x[rows]
        z = ops.linear_f32(x, self.head)
        return ops.soft_cap(z, self.cfg.logit_softcap) if self.cfg.logit_softcap > 0 else z

    def greedy(self, ids, meta, cache, rows):
        tok, _ = ops.lm_head_argmax(self.hidden(ids, meta, cache)[rows], self.head)       # the cap keeps the order
        return tok


def init_random_(model: KivezenModel, seed: int = 0, std: float = 0.02) -> None:
    g = torch.Generator(device=model.embed.device).manual_seed(seed)
    n = model.total.numel()
    gains = {id(p) for layer in model.layers for p in layer.norms} | {id(model.norm)}
    for name, p in model.named_parameters():
        leaf = name.rpartition(".")[2]
        if id(p) in gains or leaf in ("norm", "temp", "write"):
            p.data.fill_(1.0)
        elif leaf == "read":
            p.data.fill_(1.0 / n)
        elif leaf == "mix":
            p.data.copy_(torch.eye(n))
        else:
            for part in (p.data if p.dim() == 3 else [p.data]):           # expert by expert: no f32 copy of all of them
                part.copy_(torch.randn(part.shape, generator=g, device=p.device) * std)


def load_into(model: KivezenModel, loader) -> None:
    """Fill the model from a ``WeightLoader`` with tensors ``embed``, ``head``, ``final.norm``, ``l<i>.norm*``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``l<i>.hc*.*``."""
    def get(name):
        return loader.load_tensor(name)
    for p in model.parameters():
        p.data.zero_()                     # rows between the blocks of fused projections
    for mine, theirs in ((model.embed, "embed"), (model.head, "head"), (model.norm, "final.norm")):
        mine.data.copy_(get(theirs))
    for i, layer in enumerate(model.layers):
        layer.load(get, f"l{i}.", plain=model.cfg.streams is None)
