"""Rokarax: a decoder with dynamic tanh before and after every sublayer and a residual stream in 32 bits.

Layer: ``h += n1b(mixer(n1(h)))``; ``h += n2b(ff(n2(h)))`` (the second half is absent in a layer without a feed-forward), every ``n`` a
dynamic tanh.  A mixer is latent attention, a Mamba-2 state space or grouped attention with a learned distance bias and an output gate,
which may read another layer's keys and values (``models/mixers.py``).  Embedding and head are separate tables.  The model runs over the
flattened ragged batch with the paged cache, recurrent state in the cache's slots; bf16 or 32-bit activations."""
from __future__ import annotations

import torch
from torch import nn

from ... import ops
from ..mixers import BiasedAttentionMixer, DenseGLU, DynamicTanh, LatentAttentionMixer, StateSpaceMixer, param, yarn_frequencies
from .config import AttentionSpec, LatentSpec, RokaraxConfig


def _mixer(cfg: RokaraxConfig, s, rows: int, dtype, device):
    if isinstance(s, LatentSpec):
        r = s.rot
        freq, gain = yarn_frequencies(r.dims, r.base, r.factor, r.original, r.fast, r.slow)
        return LatentAttentionMixer(cfg.width, s.heads, s.dim, s.rot_dim, s.vdim, s.q_rank, s.kv_rank, s.scale, s.window, freq, gain, cfg.eps, dtype,
                                    device)
    if isinstance(s, AttentionSpec):
        return BiasedAttentionMixer(cfg.width, s.heads, s.kv_heads, s.dim, s.vdim, s.scale, s.window, rows, s.bias_max, s.kv_from, cfg.eps, dtype, device)
    return StateSpaceMixer(cfg.width, s.heads, s.vdim, s.state, s.groups, s.conv, s.norm_groups, cfg.eps, dtype, device)


class RokaraxLayer(nn.Module):
    def __init__(self, cfg: RokaraxConfig, i: int, bias_rows: int, dtype, device):
        super().__init__()
        spec = cfg.layers[i]
        norm = lambda: DynamicTanh(cfg.width, dtype, device)  # noqa: E731
        self.mixer = _mixer(cfg, spec.mixer, bias_rows, dtype, device)
        self.norm1, self.norm1b = norm(), norm()
        self.mlp = self.norm2 = self.norm2b = None
        if spec.ff is not None:
            self.mlp = DenseGLU(cfg.width, spec.ff, "swiglu", dtype, device)
            self.norm2, self.norm2b = norm(), norm()

    def forward(self, x, h, meta, cache, following):
        """``x``: the normed input of the mixer, ``h``: the stream (f32, updated in place), ``following``: the norm of whatever comes next.
        Returns the next normed input."""
        a = self.mixer(x, meta, cache)
        if self.mlp is None:
            return ops.dyt_add(a, self.norm1b, h, following)
        x = ops.dyt_add(a, self.norm1b, h, self.norm2)
        return ops.dyt_add(self.mlp(x), self.norm2b, h, following)


class RokaraxModel(nn.Module):
    def __init__(self, cfg: RokaraxConfig, bias_rows=None, dtype=torch.float32, device="cpu"):
        """``bias_rows``: rows of every layer's distance-bias table (a property of the checkpoint's tensors; entries of layers without one are
        ignored), 32 when not given."""
        super().__init__()
        self.cfg, self.dtype = cfg, dtype
        rows = bias_rows or [32] * len(cfg.layers)
        self.embed, self.head = param(cfg.vocab, cfg.width, dtype=dtype, device=device), param(cfg.vocab, cfg.width, dtype=dtype, device=device)
        self.layers = nn.ModuleList([RokaraxLayer(cfg, i, rows[i], dtype, device) for i in range(len(cfg.layers))])
        self.norm = DynamicTanh(cfg.width, dtype, device)
        kv = st = 0
        for layer in self.layers:
            m = layer.mixer
            if m.kv_spec() is not None:
                m.kv_index, kv = kv, kv + 1
            elif m.kv_from is not None:
                m.kv_index = self.layers[m.kv_from].mixer.kv_index
            if m.state_spec(dtype) is not None:
                m.state_index, st = st, st + 1

    def kv_spec(self):
        specs = [s for s in (layer.mixer.kv_spec() for layer in self.layers) if s is not None]
        return dict(num_layers=len(specs), kv_heads=[s[0] for s in specs], head_dim=[s[1] for s in specs], v_head_dim=[s[2] for s in specs])

    def state_spec(self):
        return [s for s in (layer.mixer.state_spec(self.dtype) for layer in self.layers) if s is not None]

    def head_weight(self):
        return self.head

    def _layers(self, ids, meta, cache):
        """Runs the layers one by one: yields ``(stream, next normed input)`` after each."""
        norms = [layer.norm1 for layer in self.layers] + [self.norm]
        h, x = ops.embed_dyt(ids, self.embed, self.cfg.embed_scale, norms[0])
        yield h, x
        for layer, following in zip(self.layers, norms[1:]):
            x = layer(x, h, meta, cache, following)
            yield h, x

    def hidden(self, ids, meta, cache):
        x = None
        for _, x in self._layers(ids, meta, cache):
            pass
        return x

    trunk = hidden

    def layer_states(self, ids, meta, cache):
        """The residual stream after every layer ``[layers, T, width]`` (runs the batch like ``hidden``)."""
        return torch.stack([h.clone() for h, _ in self._layers(ids, meta, cache)][1:])

    def forward(self, ids, meta, cache, rows=None):
        x = self.hidden(ids, meta, cache)
        if rows is not None:
            x = x[rows]
        return ops.linear_f32(x, self.head)

    def greedy(self, ids, meta, cache, rows):
        tok, _ = ops.lm_head_argmax(self.hidden(ids, meta, cache)[rows], self.head)
        return tok


def init_random_(model: RokaraxModel, seed: int = 0, std: float = 0.02) -> None:
    g = torch.Generator(device=model.embed.device).manual_seed(seed)
    for n, p in model.named_parameters():
        leaf = n.rpartition(".")[2]
        r = torch.randn(p.shape, generator=g, device=p.device)
        if leaf in ("a_log", "dt_bias"):
            p.data.copy_(r - 1.0)
        elif leaf == "w_taps":
            p.data.copy_(r * p.shape[1] ** -0.5)
        elif leaf in ("b", "b_taps", "rel"):
            p.data.copy_(r * 0.1)
        elif p.dim() == 1:
            p.data.fill_(1.0)
        else:
            p.data.copy_(r * std)
    for layer in model.layers:
        layer.mixer.finish()


def bias_rows(cfg: RokaraxConfig, shape_of) -> list[int]:
    """Rows of the distance-bias tables from the checkpoint's tensor shapes."""
    return [shape_of(f"l{i}.mix.rel")[0] if isinstance(s.mixer, AttentionSpec) else 0 for i, s in enumerate(cfg.layers)]


def load_into(model: RokaraxModel, loader) -> None:
    """Fill the model from a ``WeightLoader`` with tensors ``embed``, ``head``, ``final.norm*``, ``l<i>.norm*``, ``l<i>.mix.*``, ``l<i>.mlp.*``."""
    def get(name):
        return loader.load_tensor(name)
    for p in model.parameters():
        p.data.zero_()                     # rows between the blocks of a fused projection
    model.embed.data.copy_(get("embed"))
    model.head.data.copy_(get("head"))
    model.norm.load(get, "final.norm")
    for i, layer in enumerate(model.layers):
        layer.norm1.load(get, f"l{i}.norm1")
        layer.norm1b.load(get, f"l{i}.norm1b")
        layer.mixer.load(get, f"l{i}.mix.")
        layer.mixer.finish()
        if layer.mlp is not None:
            layer.norm2.load(get, f"l{i}.norm2")
            layer.norm2b.load(get, f"l{i}.norm2b")
            layer.mlp.load(get, f"l{i}.mlp.")
