"""Tatizen: a decoder that norms the OUTPUT of its sublayers and keeps its residual stream in 32 bits.

Layer: ``h += rms(mixer(h)) w1``; ``h += rms(ff(h)) w2`` (the second half is absent in a layer without a feed-forward).  A mixer is either
softmax attention beside decayed linear attention or a gated delta rule (``models/mixers.py``); the head is tied to the embedding.  The
model runs over the flattened ragged batch with the paged cache, recurrent state in the cache's slots; bf16 or 32-bit activations."""
from __future__ import annotations

import torch
from torch import nn

from ... import ops
from ..mixers import AttentionLinearMixer, DenseGLU, GatedDeltaMixer, param
from .config import ParallelSpec, TatizenConfig


def _mixer(cfg: TatizenConfig, s, rank: int, dtype, device):
    if isinstance(s, ParallelSpec):
        a, r = s.left, s.right
        return AttentionLinearMixer(cfg.width, a.heads, a.kv_heads, a.dim, a.vdim, a.scale, s.left_scale, r.heads, r.dim, r.vdim, r.tau, rank,
                                    s.right_scale, cfg.eps, dtype, device)
    return GatedDeltaMixer(cfg.width, s.heads, s.kv_heads, s.dim, s.vdim, s.conv, cfg.eps, dtype, device)


class TatizenLayer(nn.Module):
    def __init__(self, cfg: TatizenConfig, i: int, rank: int, dtype, device):
        super().__init__()
        spec = cfg.layers[i]
        self.eps = cfg.eps
        self.mixer = _mixer(cfg, spec.mixer, rank, dtype, device)
        self.norm1 = param(cfg.width, dtype=dtype, device=device)
        self.mlp = self.norm2 = None
        if spec.ff is not None:
            self.mlp = DenseGLU(cfg.width, spec.ff, "geglu", dtype, device)
            self.norm2 = param(cfg.width, dtype=dtype, device=device)

    def forward(self, x, h, meta, cache, final_norm=None):
        """``x``: the stream in the activation type, ``h``: the stream (f32, updated in place).  Returns the next ``x``, normed with
        ``final_norm`` when given."""
        a = self.mixer(x, meta, cache)
        if self.mlp is None:
            return ops.post_norm_add(a, self.norm1, h, final_norm, self.eps)
        x = ops.post_norm_add(a, self.norm1, h, None, self.eps)
        return ops.post_norm_add(self.mlp(x), self.norm2, h, final_norm, self.eps)


class TatizenModel(nn.Module):
    def __init__(self, cfg: TatizenConfig, decay_ranks=None, dtype=torch.float32, device="cpu"):
        """``decay_ranks``: inner width of the low-rank decay projection of every layer (a property of the checkpoint's tensors; entries of
        layers without one are ignored), 16 when not given."""
        super().__init__()
        self.cfg, self.dtype = cfg, dtype
        ranks = decay_ranks or [16] * len(cfg.layers)
        self.embed = param(cfg.vocab, cfg.width, dtype=dtype, device=device)
        self.layers = nn.ModuleList([TatizenLayer(cfg, i, ranks[i], dtype, device) for i in range(len(cfg.layers))])
        self.norm = param(cfg.width, dtype=dtype, device=device)
        kv = st = 0
        for layer in self.layers:
            m = layer.mixer
            if m.kv_spec() is not None:
                m.kv_index, kv = kv, kv + 1
            m.state_index, st = st, st + 1

    def kv_spec(self):
        specs = [layer.mixer.kv_spec() for layer in self.layers if layer.mixer.kv_spec() is not None]
        return dict(num_layers=len(specs), kv_heads=[s[0] for s in specs], head_dim=[s[1] for s in specs], v_head_dim=[s[2] for s in specs])

    def state_spec(self):
        return [layer.mixer.state_spec(self.dtype) for layer in self.layers]

    def head_weight(self):
        return self.embed

    def hidden(self, ids, meta, cache):
        h, x = ops.embed32(ids, self.embed)
        n = len(self.layers)
        if n == 0:
            return ops.rmsnorm32(h, self.norm, self.cfg.eps)
        for i, layer in enumerate(self.layers):
            x = layer(x, h, meta, cache, self.norm if i + 1 == n else None)
        return x

    trunk = hidden

    def layer_states(self, ids, meta, cache):
        """The residual stream after every layer ``[layers, T, width]`` (runs the batch like ``hidden``)."""
        h, x = ops.embed32(ids, self.embed)
        out = []
        for layer in self.layers:
            x = layer(x, h, meta, cache)
            out.append(h.clone())
        return torch.stack(out)

    def forward(self, ids, meta, cache, rows=None):
        x = self.hidden(ids, meta, cache)
        if rows is not None:
            x = x[rows]
        return ops.linear_f32(x, self.embed)

    def greedy(self, ids, meta, cache, rows):
        tok, _ = ops.lm_head_argmax(self.hidden(ids, meta, cache)[rows], self.embed)
        return tok


def init_random_(model: TatizenModel, seed: int = 0, std: float = 0.02) -> None:
    g = torch.Generator(device=model.embed.device).manual_seed(seed)
    for n, p in model.named_parameters():
        leaf = n.rpartition(".")[2]
        if leaf in ("a_log", "dt_bias", "b_decay"):
            p.data.copy_(torch.rand(p.shape, generator=g, device=p.device))
        elif leaf == "w_taps":
            p.data.copy_(torch.randn(p.shape, generator=g, device=p.device) * p.shape[1] ** -0.5)
        elif p.dim() == 1:
            p.data.fill_(1.0)
        else:
            p.data.copy_(torch.randn(p.shape, generator=g, device=p.device) * std)


def decay_ranks(cfg: TatizenConfig, shape_of) -> list[int]:
    """Inner widths of the low-rank decay projections from the checkpoint's tensor shapes."""
    return [shape_of(f"l{i}.mix.right.a1")[0] if isinstance(s.mixer, ParallelSpec) else 0 for i, s in enumerate(cfg.layers)]


def load_into(model: TatizenModel, loader) -> None:
    """Fill the model from a ``WeightLoader`` with tensors ``embed``, ``final.norm``, ``l<i>.norm1``, ``l<i>.mix.*``, ``l<i>.mlp.*``."""
    def get(name):
        return loader.load_tensor(name)
    for p in model.parameters():
        p.data.zero_()                     # rows between the blocks of a fused projection
    model.embed.data.copy_(get("embed"))
    model.norm.data.copy_(get("final.norm"))
    for i, layer in enumerate(model.layers):
        layer.norm1.data.copy_(get(f"l{i}.norm1"))
        layer.mixer.load(get, f"l{i}.mix.")
        if layer.mlp is not None:
            layer.norm2.data.copy_(get(f"l{i}.norm2"))
            layer.mlp.load(get, f"l{i}.mlp.")
