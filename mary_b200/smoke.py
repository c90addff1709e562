"""One tiny end-to-end pass on ``cuda:0`` through the hand-written kernels (used by ``__graft_entry__.smoke``):
the flagship decoder (MLA attention, NVFP4 routed experts, MTP speculative decoding), the continuous-batching engine on a
Gemma-4 decoder, and one LoRA forward + backward + fused AdamW step."""
from __future__ import annotations

import numpy as np
import torch


def _flagship(dev):
    from .models.moe import MoEDecoder, init_random_, tiny_moe_config
    from .runtime.kv_cache import PagedKVCache
    from .runtime.spec_decode import SpecDecoder
    cfg = tiny_moe_config("mla")
    m = MoEDecoder(cfg, dtype=torch.bfloat16, device=dev)
    init_random_(m, 0)
    spec = m.kv_spec()
    B = 4
    cache = PagedKVCache(spec["num_layers"], B * 8 + 2, 16, spec["kv_heads"], spec["head_dim"], dtype=torch.bfloat16, device=dev,
                         latent_dim=spec.get("latent_dim"))
    dec = SpecDecoder(m, cache, B, spec_k=2, max_len=128, device=dev, use_graph=True)
    dec.prefill(np.random.default_rng(0).integers(0, cfg.vocab_size, (B, 21)), chunk=16)
    dec.capture()
    n = 0
    for _ in range(4):
        dec.step()
        n += int(dec.n_emitted.sum())
    assert n >= 4 * B
    return n


def _gemma_engine(dev):
    from .models.gemma4 import Gemma4Model, Gemma4TextConfig
    from .models.gemma4.weights import init_random_
    from .runtime.engine import Engine
    from .runtime.kv_cache import PagedKVCache
    cfg = Gemma4TextConfig(hidden_size=512, num_hidden_layers=2, num_attention_heads=8, num_key_value_heads=2, head_dim=64,
                           intermediate_size=1024, vocab_size=2048, sliding_window=32)
    m = Gemma4Model(cfg, dtype=torch.bfloat16, device=dev)
    init_random_(m, 0)
    spec = m.kv_spec()
    cache = PagedKVCache(spec["num_layers"], 64, 16, spec["kv_heads"], spec["head_dim"], dtype=torch.bfloat16, device=dev)
    e = Engine(m, cache, max_tokens=256, max_seqs=4, device=dev)
    out = e.generate([[1, 2, 3, 4, 5, 6, 7], [9, 8, 7]], 4)
    assert all(len(o) == 4 for o in out)
    return m, out


def _recurrent_engine(dev):
    """A Tatizen decoder (attention beside decayed linear attention, gated delta rule) generating through the scheduler, two sequences."""
    from .models.registry import family_of, make_engine
    from .models.tatizen import TatizenConfig, TatizenModel, init_random_
    layers = [{"type": "parallel", "mlp": {"kind": "dense", "ff": 512}, "mixer": {
        "left": dict(heads=8, kv_heads=2, dim=64, vdim=64, scale=0.1), "right": dict(heads=4, dim=64, vdim=64, tau=8.0),
        "left_scale": 0.9, "right_scale": 0.7}},
        {"type": "delta", "mlp": {"kind": "dense", "ff": 512}, "mixer": dict(heads=4, kv_heads=2, dim=64, vdim=64, conv=4)}]
    d = {"architecture": "Tatizen", "vocab": 1024, "width": 512, "norm": {"eps": 1e-6}, "layers": layers}
    m = TatizenModel(TatizenConfig.from_json(d), dtype=torch.bfloat16, device=dev)
    init_random_(m, 0)
    out = make_engine(m, family_of(d), 512, 2, dev).generate([list(range(90)), [5, 4, 3]], 4)
    assert all(len(o) == 4 for o in out)
    return out


def _state_space_engine(dev):
    """A Rokarax decoder (attention with a distance bias, state space, latent attention, a layer with shared keys) generating through the
    scheduler, two sequences."""
    from .models.registry import family_of, make_engine
    from .models.rokarax import RokaraxConfig, RokaraxModel, init_random_
    mlp = {"kind": "dense", "ff": 512}
    att = dict(heads=8, kv_heads=2, dim=64, vdim=64, scale=0.1, bias_max=100.0, mask={"size": 70})
    layers = [{"type": "attention", "mlp": mlp, "mixer": att},
              {"type": "mamba2", "mlp": None, "mixer": dict(heads=8, vdim=64, state=128, groups=2, conv=4, norm_groups=2)},
              {"type": "latent_attention", "mlp": mlp, "mixer": dict(
                  heads=4, dim=128, rot_dim=64, vdim=128, q_rank=128, kv_rank=512, scale=0.07, mask={"size": 50},
                  rot={"dims": 64, "base": 10000.0, "scaling": dict(factor=2.0, original=1024.0, fast=32.0, slow=1.0)})},
              {"type": "attention", "mlp": mlp, "mixer": {**att, "kv_from": 0}}]
    d = {"architecture": "Rokarax", "vocab": 1024, "width": 512, "norm": {"eps": 1e-6}, "embedding": {"scale": 8.0}, "layers": layers}
    m = RokaraxModel(RokaraxConfig.from_json(d), dtype=torch.bfloat16, device=dev)
    init_random_(m, 0)
    out = make_engine(m, family_of(d), 512, 2, dev).generate([list(range(90)), [5, 4, 3]], 4)
    assert all(len(o) == 4 for o in out)
    return out


def _routed_engine(dev):
    """A Nipurax decoder (capped attention with sinks, differential attention, routed experts, a loop over two layers) generating through the
    scheduler, two sequences."""
    from .models.nipurax import NipuraxConfig, NipuraxModel, init_random_
    from .models.registry import family_of, make_engine
    mlp = {"kind": "moe", "expert": {"ff": 256, "limit": 2.0}, "shared": {"ff": 384, "limit": 2.0},
           "router": {"experts": 8, "identity": 2, "top": 3, "scale": 2.0}}
    cap = {"type": "attention_2", "mlp": mlp, "mixer": dict(heads=8, kv_heads=2, dim=128, vdim=128, scale=0.09, softcap=30.0,
                                                            q_temp={"coef": 0.2, "every": 32})}
    dif = {"type": "attention", "mlp": mlp, "mixer": dict(heads=4, kv_heads=2, dim=64, vdim=128, scale=0.12, mask={"size": 48}, diff=0.3, rot={
        "dims": 32, "base": 10000.0, "scaling": dict(factor=4.0, low=1.0, high=4.0, original=1024.0)})}
    d = {"architecture": "Nipurax", "vocab": 1024, "width": 512, "norm": {"eps": 1e-6}, "residual_mult": 0.5, "layers": [cap, dif, cap],
         "embedding": {"bigram": {"buckets": 1021, "mul_prev": 17, "mul_cur": 3}}, "loop": {"start": 0, "stop": 2, "times": 2}}
    m = NipuraxModel(NipuraxConfig.from_json(d), dtype=torch.bfloat16, device=dev)
    init_random_(m, 0)
    out = make_engine(m, family_of(d), 512, 2, dev).generate([list(range(90)), [5, 4, 3]], 4)
    assert all(len(o) == 4 for o in out)
    return out


def _streams_engine(dev):
    """A Kivezen decoder (four residual streams, lightning attention, attention with turned values, gated shared expert, a loop over two layers) generating
    through the scheduler, two sequences."""
    from .models.kivezen import KivezenConfig, KivezenModel, init_random_
    from .models.registry import family_of, make_engine
    moe = {"kind": "moe", "expert": {"ff": 256, "limit": 2.0}, "shared": {"ff": 384, "limit": 1.5}, "router": {"experts": 8, "top": 2}}
    lin = {"type": "lightning", "mlp": {"kind": "dense", "ff": 768}, "mixer": dict(heads=4, dim=128, vdim=64, decay=[0.5, 0.9, 0.97, 0.995])}
    att = {"type": "attention", "mlp": moe, "mixer": dict(heads=8, kv_heads=2, dim=128, vdim=128, scale=0.09, softcap=20.0, rot={
        "dims": 96, "base": 50000.0, "scaling": dict(factor=4.0, original=1024.0, fast=32.0, slow=1.0)})}
    d = {"architecture": "Kivezen", "vocab": 1024, "width": 512, "norm": {"eps": 1e-6}, "logit_softcap": 20.0, "streams": 4, "layers": [lin, att, lin],
         "loop": {"start": 0, "stop": 2, "times": 2}}
    m = KivezenModel(KivezenConfig.from_json(d), dtype=torch.bfloat16, device=dev)
    init_random_(m, 0)
    out = make_engine(m, family_of(d), 512, 2, dev).generate([list(range(90)), [5, 4, 3]], 4)
    assert all(len(o) == 4 for o in out)
    return out


def _lora_step(m, dev):
    from .train.trainer import LoraTrainer
    tr = LoraTrainer(m, rank=8, alpha=16.0, lr=1e-3)
    ids = torch.randint(0, 2048, (2, 32), device=dev)
    l0 = tr.step(ids)
    l1 = tr.step(ids)
    assert np.isfinite(l0) and np.isfinite(l1)
    return l0, l1


def run_smoke() -> None:
    from .ops import cuda
    cuda.lib()                                       # fails loudly when the kernel library is missing
    dev = "cuda:0"
    torch.cuda.set_device(0)
    n = _flagship(dev)
    m, out = _gemma_engine(dev)
    rec = _recurrent_engine(dev)
    ssm = _state_space_engine(dev)
    moe = _routed_engine(dev)
    hyper = _streams_engine(dev)
    losses = _lora_step(m, dev)
    torch.cuda.synchronize()
    st = cuda.last_status()
    assert st == 0, f"kernel status {st}"
    print(f"smoke ok: flagship emitted {n} tokens in 4 speculative steps; gemma {out}; tatizen {rec}; rokarax {ssm}; nipurax {moe}; kivezen {hyper}; lora loss {losses[0]:.3f} -> {losses[1]:.3f}; "
          f"{cuda.LAUNCHES} kernel launches")
