"""Micro-benchmarks of the kernels of decoders with recurrent layers, beside the like kernels of the dense decoders
(``python -m mary_b200.ops.bench_kernels hybrid``).  Fractions: bytes against the measured copy bandwidth, tensor-core products against
the measured cuBLAS rate, the recurrences (32-bit multiply-adds on the CUDA cores) against the nominal 128 multiply-adds per SM and clock."""
from __future__ import annotations

import numpy as np
import torch

F32_TFLOPS = 148 * 128 * 2 * 1.965e9 / 1e12


def _meta(B, q, ctx, page=64):
    from ..runtime.batch import BatchMeta
    n = (ctx + page - 1) // page
    return BatchMeta.build([q] * B, [ctx] * B, np.arange(B * n, dtype=np.int32).reshape(B, n), page, "cuda", np.arange(B, dtype=np.int32))


def run(width: int = 4096, heads: int = 32, kv_heads: int = 8, l_heads: int = 16, d_heads: int = 32, d_kv: int = 16, D: int = 128) -> list[dict]:
    from . import cuda as K
    from . import cuda_hybrid as H
    from .bench_kernels import peaks, time_op
    hbm, tf, tag = peaks()
    bf = dict(dtype=torch.bfloat16, device="cuda")
    rows: list[dict] = []

    def add(name, case, fn, flops=0.0, peak=None, nbytes=0.0, like=None):
        us = time_op(fn) * 1e3
        frac = max(flops / us / 1e6 / peak if peak else 0.0, nbytes / us / 1e3 / hbm)
        rows.append(dict(kernel=name, case=case, us=round(us, 1), tflops=round(flops / us / 1e6, 1), gbs=round(nbytes / us / 1e3), frac=round(frac, 3),
                         like=like))
        print(f"{name:<28}{case:<18}{us:>9.1f} us {flops / us / 1e6:>8.1f} TFLOP/s {nbytes / us / 1e3:>7.0f} GB/s  {frac:.3f} {tag}" + (f"  (like: {like})" if like else ""))

    for B, q in ((1, 4096), (8, 512)):
        case, T = f"{B} x {q} tokens", B * q
        m = _meta(B, q, q)
        kc = torch.randn(m.page_table.numel(), 64, kv_heads, D, **bf)
        vc, Q = torch.randn_like(kc), torch.randn(T, heads, D, **bf)
        fl = 4.0 * heads * D * T * (q + 1) / 2
        add("attention_prefill", case, lambda: K.attention_prefill(Q, kc, vc, m, 0.1), fl, tf, like="dense decoder")
        add("attention_prefill split_p", case, lambda: H.attention_exact(Q, kc, vc, m, 0.1), fl, tf)
        # projection row of an attention-linear layer
        C, E = l_heads * D, D
        y = torch.randn(T, 4 * C + 16, **bf)
        lq, lk, lv, lg, low = y.split([C, C, C, C, 16], 1)
        a2, b2, gain = torch.randn(C, 16, **bf), torch.randn(C, **bf), torch.ones(E, **bf)
        S = torch.zeros(B, l_heads, E, D, device="cuda")
        out = torch.empty(T, C, **bf)
        dec = H.channel_decay(low, a2, b2, 1 / 16)
        o = H.decay_scan(lq, lk, lv, dec, S, m, l_heads, D, E, D ** -0.5)
        add("channel_decay", case, lambda: H.channel_decay(low, a2, b2, 1 / 16), nbytes=T * (C * 4 + 32))
        add("decay_scan", case, lambda: H.decay_scan(lq, lk, lv, dec, S, m, l_heads, D, E, D ** -0.5), 5.0 * T * l_heads * D * E, F32_TFLOPS,
            T * C * (2 + 2 + 2 + 4 + 4))
        add("gated_head_norm", case, lambda: H.gated_head_norm(o, lg, gain, 1e-5, 1.0, out), nbytes=T * C * 8)
        del y, lq, lk, lv, lg, low, dec, o
        # projection row of a delta layer
        C = 2 * d_kv * D + d_heads * E
        ld = C + d_heads * E + 2 * d_heads
        y = torch.randn(T, ld, **bf)
        x, b, a = y[:, :C], y[:, ld - 2 * d_heads:ld - d_heads], y[:, ld - d_heads:]
        w, z = torch.randn(C, 4, **bf), torch.zeros(d_heads, device="cuda")
        S, ring = torch.zeros(B, d_heads, E, D, device="cuda"), torch.zeros(B, 4, C, **bf)
        pre = H.delta_prep(x, w, ring, b, a, z, z, m, d_kv, d_heads, D, E)
        add("delta_prep", case, lambda: H.delta_prep(x, w, ring, b, a, z, z, m, d_kv, d_heads, D, E), nbytes=T * C * 6)
        add("delta_scan", case, lambda: H.delta_scan(*pre, S, m, d_kv, d_heads, D, E), 7.0 * T * d_heads * D * E, F32_TFLOPS, T * (C + d_heads * E) * 4)
        del y, x, a, b, pre
        n_in = (heads + 2 * kv_heads) * D
        y, g = torch.randn(T, n_in, **bf), torch.ones(D, **bf)
        parts = y.split([heads * D, kv_heads * D, kv_heads * D], 1)
        inv = torch.ones(D // 2, device="cuda")
        add("qk_norm_rope_append", case, lambda: K.qk_norm_rope_append(y, heads, kv_heads, D, g, g, False, inv, m, kc, vc, 1e-5), nbytes=T * n_in * 4,
            like="dense decoder")
        add("qk_norm_append", case, lambda: H.qk_norm_append(*parts, heads, kv_heads, D, D, g, g, m, kc, vc, 1e-5), nbytes=T * n_in * 4)
        ar, h, hb = torch.randn(T, width, device="cuda"), torch.randn(T, width, device="cuda"), torch.randn(T, width, **bf)
        gw, xb = torch.ones(width, **bf), torch.randn(T, width, **bf)
        add("add_rmsnorm", case, lambda: K.add_rmsnorm(xb, hb, gw, 1e-5), nbytes=T * width * 8, like="dense decoder")
        add("post_norm_add", case, lambda: H.post_norm_add(ar, gw, h, None, 1e-5), nbytes=T * width * 14)
    for B in (1, 32, 128):
        case, ctx = f"{B} x 1 token", 2048
        m = _meta(B, 1, ctx)
        kc = torch.randn(m.page_table.numel(), 64, kv_heads, D, **bf)
        vc, Q = torch.randn_like(kc), torch.randn(B, heads, D, **bf)
        nb = 2.0 * B * ctx * kv_heads * D * 2
        add("paged_attention_decode", case, lambda: H.attention_exact(Q, kc, vc, m, 0.1), nbytes=nb, like="both decoders")
        C = l_heads * D
        y = torch.randn(B, 4 * C + 16, **bf)
        lq, lk, lv, lg, low = y.split([C, C, C, C, 16], 1)
        S, out = torch.zeros(B, l_heads, D, D, device="cuda"), torch.empty(B, C, **bf)
        a2, b2, gain = torch.randn(C, 16, **bf), torch.randn(C, **bf), torch.ones(D, **bf)
        add("decay_step", case, lambda: H.decayed_linear_attention(lq, lk, lv, lg, low, a2, b2, 1 / 16, gain, S, m, l_heads, D, D, 1e-5, 1.0, out),
            nbytes=B * l_heads * D * D * 8.0)
        C = 2 * d_kv * D + d_heads * D
        ld = C + d_heads * D + 2 * d_heads
        y = torch.randn(B, ld, **bf)
        w, z = torch.randn(C, 4, **bf), torch.zeros(d_heads, device="cuda")
        S, ring, out = torch.zeros(B, d_heads, D, D, device="cuda"), torch.zeros(B, 4, C, **bf), torch.empty(B, d_heads * D, **bf)
        add("delta_step", case, lambda: H.gated_delta_attention(y[:, :C], w, y[:, ld - 2 * d_heads:ld - d_heads], y[:, ld - d_heads:], z, z,
                                                                y[:, C:C + d_heads * D], gain, ring, S, m, d_kv, d_heads, D, D, 1e-5, 1.0, out),
            nbytes=B * d_heads * D * D * 8.0)
    for T in (4096, 32):
        case = f"{T} rows"
        for name, N, Kd in (("gemm in (bf16 out)", 3 * width, width), ("gemm out (f32 out)", width, width + l_heads * D), ("gemm down (f32 out)", width, 3 * width)):
            x, w = torch.randn(T, Kd, **bf), torch.randn(N, Kd, **bf)
            fn = (lambda: K.linear(x, w)) if "bf16" in name else (lambda: K.linear_f32(x, w))
            add(name, case, fn, 2.0 * T * N * Kd, tf, 2.0 * (N * Kd + T * Kd + T * N))
    assert K.last_status() == 0
    return rows
