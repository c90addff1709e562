"""Micro-benchmarks of the kernels of decoders with recurrent layers, beside the like kernels of the dense decoders
(``python -m mary_b200.ops.bench_kernels hybrid``, ``rokarax``, ``nipurax`` and ``kivezen``).  Fractions: bytes against the measured copy bandwidth, tensor-core products against
the measured cuBLAS rate, the recurrences (32-bit multiply-adds on the CUDA cores) against the nominal 128 multiply-adds per SM and clock."""
from __future__ import annotations

import numpy as np
import torch

F32_TFLOPS = 148 * 128 * 2 * 1.965e9 / 1e12


def _meta(B, q, ctx, page=64):
    from ..runtime.batch import BatchMeta
    n = (ctx + page - 1) // page
    return BatchMeta.build([q] * B, [ctx] * B, np.arange(B * n, dtype=np.int32).reshape(B, n), page, "cuda", np.arange(B, dtype=np.int32))


class _Table:
    """Times calls and prints them against the measured peaks."""

    def __init__(self):
        from .bench_kernels import peaks
        self.hbm, self.tf, self.tag = peaks()
        self.rows: list[dict] = []

    def __call__(self, name, case, fn, flops=0.0, peak=None, nbytes=0.0, like=None):
        from .bench_kernels import time_op
        us = time_op(fn) * 1e3
        frac = max(flops / us / 1e6 / peak if peak else 0.0, nbytes / us / 1e3 / self.hbm)
        self.rows.append(dict(kernel=name, case=case, us=round(us, 1), tflops=round(flops / us / 1e6, 1), gbs=round(nbytes / us / 1e3), frac=round(frac, 3),
                              like=like))
        print(f"{name:<30}{case:<18}{us:>9.1f} us {flops / us / 1e6:>8.1f} TFLOP/s {nbytes / us / 1e3:>7.0f} GB/s  {frac:.3f} {self.tag}"
              + (f"  (like: {like})" if like else ""))


def run(width: int = 4096, heads: int = 32, kv_heads: int = 8, l_heads: int = 16, d_heads: int = 32, d_kv: int = 16, D: int = 128) -> list[dict]:
    from . import cuda as K
    from . import cuda_hybrid as H
    add = _Table()
    tf, rows = add.tf, add.rows
    bf = dict(dtype=torch.bfloat16, device="cuda")

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


def run_rokarax(width: int = 4096, heads: int = 32, kv_heads: int = 8, window: int = 1024) -> list[dict]:
    """The kernels of the Rokarax decoder: attention with a distance bias, a window and a gate beside the dense decoder's, latent attention
    beside the expanded and the absorbed form without a window, the state space layer, the row kernels."""
    from types import SimpleNamespace

    from . import cuda as K
    from . import cuda_hybrid as H
    add = _Table()
    tf = add.tf
    bf = dict(dtype=torch.bfloat16, device="cuda")
    D, P, N, G, taps = 128, 64, 128, 1, 4
    SH = 2 * width // P
    inner = SH * P
    C = inner + 2 * G * N
    bias = torch.randn(heads, window, device="cuda")
    lat = SimpleNamespace(heads=heads, dim=128, rot=64, dv=128, rank=512, scale=0.07, window=window, rot_gain=1.0, freq=torch.rand(32, device="cuda"),
                          w_k=torch.randn(heads * 128, 512, **bf) * 0.04, w_v=torch.randn(heads * 128, 512, **bf) * 0.04)
    lat.w_k_t = lat.w_k.view(heads, 128, 512).transpose(1, 2).contiguous()
    w, wb, gain = torch.randn(C, taps, **bf), torch.randn(C, **bf), torch.ones(inner, **bf)
    one = torch.ones(SH, device="cuda")
    norm = SimpleNamespace(w=torch.ones(width, **bf), b=torch.ones(width, **bf), alpha=torch.ones(1, device="cuda"))
    pad = (SH + 7) // 8 * 8
    for B, q in ((1, 4096), (8, 512)):
        case, T = f"{B} x {q} tokens", B * q
        m = _meta(B, q, q)
        kc = torch.randn(m.page_table.numel(), 64, kv_heads, D, **bf)
        vc, Q, gate = torch.randn_like(kc), torch.randn(T, heads, D, **bf), torch.randn(T, heads * D, **bf)
        out = torch.empty(T, heads * D, **bf)
        keys = sum(min(i + 1, window) for i in range(q)) / q
        add("attention_prefill", case, lambda: K.attention_prefill(Q, kc, vc, m, 0.1), 4.0 * heads * D * T * (q + 1) / 2, tf, like="dense decoder")
        fl = 4.0 * heads * D * T * keys
        add("  windowed", case, lambda: K.attention_prefill(Q, kc, vc, m, 0.1, window), fl, tf, like="dense decoder")
        add("  windowed split_p", case, lambda: H.attention_exact(Q, kc, vc, m, 0.1, out=out, window=window), fl, tf)
        add("  windowed split_p bias gate", case, lambda: H.attention_exact(Q, kc, vc, m, 0.1, out=out, window=window, bias=bias, gate=gate), fl, tf)
        cache = torch.randn(m.page_table.numel(), 64, 1, 576, **bf) * 0.1
        ql = torch.randn(T, heads * 192, **bf)
        k, v = H.expand_latent(cache.view(-1, 576), lat)
        k, v = k.view(-1, 64, heads, 192), v.view(-1, 64, heads, 128)
        fl = 2.0 * heads * (192 + 128) * T * keys
        add("attention 192/128 windowed", case, lambda: K.attention_prefill(ql.view(T, heads, 192), k, v, m, 0.1, window), fl, tf, like="latent decoder")
        add("  split_p", case, lambda: K.attention_prefill(ql.view(T, heads, 192), k, v, m, 0.1, window, split_p=True), fl, tf)
        add("expand_latent", case, lambda: H.expand_latent(cache.view(-1, 576), lat), 2.0 * T * heads * 256 * 512, tf, T * heads * 320 * 2)
        add("latent_attention (all)", case, lambda: H.latent_attention(ql, cache, m, lat), fl + 2.0 * T * heads * 256 * 512, tf)
        del k, v, ql, Q, kc, vc
        y = torch.randn(T, inner + C + pad, **bf)
        z, xbc, dt = y[:, :inner], y[:, inner:inner + C], y[:, inner + C:inner + C + SH]
        S, ring, o = torch.zeros(B, SH, P, N, device="cuda"), torch.zeros(B, taps, C, **bf), torch.empty(T, inner, **bf)
        pre = H.ssd_chunk_prep(xbc, w, wb, ring, dt, one, one, m, SH)
        yy = H.ssd_chunk(*pre, one, S, m, G, SH, N, P)
        add("ss_conv_decay", case, lambda: H.ssd_chunk_prep(xbc, w, wb, ring, dt, one, one, m, SH), nbytes=T * C * 4)
        # 64-token chunks: products of the chunk (lower half), read and update of the state
        add("ssd_chunk", case, lambda: H.ssd_chunk(*pre, one, S, m, G, SH, N, P), 2.0 * T * SH * (32 * P + 32 * N + 2 * N * P), tf, T * (C * 2 + inner * 4))
        add("gated_part_norm", case, lambda: H.gated_part_norm(yy, z, gain, 8, 1e-5, o), nbytes=T * inner * 8)
        sp = H.ss_prep(xbc, w, wb, ring, dt, one, one, m, G, SH, N, P)
        add("ss_prep (32-bit models)", case, lambda: H.ss_prep(xbc, w, wb, ring, dt, one, one, m, G, SH, N, P), nbytes=T * C * 6)
        add("head_decay_scan (32-bit)", case, lambda: H.head_decay_scan(*sp, one, S, m, G, SH, N, P), 5.0 * T * SH * N * P, F32_TFLOPS)
        del y, z, xbc, dt, pre, yy, sp
        kc = torch.randn(m.page_table.numel(), 64, kv_heads, D, **bf)
        vc = torch.randn_like(kc)
        n_in = (heads + 2 * kv_heads) * D
        y, g1 = torch.randn(T, n_in, **bf), torch.ones(D, **bf)
        parts = y.split([heads * D, kv_heads * D, kv_heads * D], 1)
        gq, gk = torch.ones(heads * D, **bf), torch.ones(kv_heads * D, **bf)
        inv = torch.ones(D // 2, device="cuda")
        add("qk_norm_rope_append", case, lambda: K.qk_norm_rope_append(y, heads, kv_heads, D, g1, g1, False, inv, m, kc, vc, 1e-5), nbytes=T * n_in * 4,
            like="dense decoder")
        add("row_norm_append", case, lambda: H.row_norm_append(*parts, heads, kv_heads, D, D, gq, gk, m, kc, vc, 1e-5), nbytes=T * n_in * 4)
        yl = torch.randn(T, 768 + 576, **bf)
        add("latent_prep", case, lambda: H.latent_prep(yl[:, :768], yl[:, 768:], torch.ones(768, **bf), torch.ones(512, **bf), lat.freq, 1.0, m, cache, 1e-5),
            nbytes=T * 1344 * 4)
        ar, h, hb, xb = torch.randn(T, width, device="cuda"), torch.randn(T, width, device="cuda"), torch.randn(T, width, **bf), torch.randn(T, width, **bf)
        add("add_rmsnorm", case, lambda: K.add_rmsnorm(xb, hb, norm.w, 1e-5), nbytes=T * width * 8, like="dense decoder")
        add("dyt_add", case, lambda: H.dyt_add(ar, norm, h, norm), nbytes=T * width * 14)
    for B in (1, 32, 128):
        case, ctx = f"{B} x 1 token", 2048
        m = _meta(B, 1, ctx)
        kc = torch.randn(m.page_table.numel(), 64, kv_heads, D, **bf)
        vc, Q, gate = torch.randn_like(kc), torch.randn(B, heads, D, **bf), torch.randn(B, heads * D, **bf)
        out = torch.empty(B, heads * D, **bf)
        add("paged_attention_decode", case, lambda: H.attention_exact(Q, kc, vc, m, 0.1), nbytes=2.0 * B * ctx * kv_heads * D * 2, like="dense decoder")
        nb = 2.0 * B * window * kv_heads * D * 2
        add("  windowed", case, lambda: H.attention_exact(Q, kc, vc, m, 0.1, window=window), nbytes=nb, like="dense decoder")
        add("  windowed bias gate", case, lambda: H.attention_exact(Q, kc, vc, m, 0.1, out=out, window=window, bias=bias, gate=gate), nbytes=nb)
        cache = torch.randn(m.page_table.numel(), 64, 1, 576, **bf) * 0.1
        qf, ql = torch.randn(B, heads, 576, **bf), torch.randn(B, heads * 192, **bf)
        cv = cache.view(-1, 64, 576)
        add("mla_attention", case, lambda: K.mla_attention(qf, cv, m, 0.1), 2.0 * B * ctx * heads * 1088, tf, B * ctx * 1152.0, like="latent decoder")
        fl, nb = 2.0 * B * window * heads * 1088, B * window * 1152.0
        add("  windowed", case, lambda: K.mla_attention(qf, cv, m, 0.1, window=window), fl, tf, nb, like="latent decoder")
        add("  windowed split_p", case, lambda: K.mla_attention(qf, cv, m, 0.1, window=window, split_p=True), fl, tf, nb)
        add("latent_attention (all)", case, lambda: H.latent_attention(ql, cache, m, lat), fl, tf, nb + heads * 256 * 512 * 2)
        y = torch.randn(B, inner + C + pad, **bf)
        S, ring, o = torch.zeros(B, SH, P, N, device="cuda"), torch.zeros(B, taps, C, **bf), torch.empty(B, inner, **bf)
        add("ss_step", case, lambda: H.state_space(y[:, inner:inner + C], w, wb, y[:, inner + C:inner + C + SH], one, one, one, y[:, :inner], gain, 8, ring, S, m,
                                                   G, SH, N, P, 1e-5, o), nbytes=B * SH * P * N * 8.0)
        ar, h, hb, xb = torch.randn(B, width, device="cuda"), torch.randn(B, width, device="cuda"), torch.randn(B, width, **bf), torch.randn(B, width, **bf)
        add("add_rmsnorm", case, lambda: K.add_rmsnorm(xb, hb, norm.w, 1e-5), nbytes=B * width * 8, like="dense decoder")
        add("dyt_add", case, lambda: H.dyt_add(ar, norm, h, norm), nbytes=B * width * 14)
    assert K.last_status() == 0
    return add.rows


def run_nipurax(width: int = 2048, heads: int = 16, kv_heads: int = 4, experts: int = 32, top: int = 4, ff: int = 1024, chunk: int = 2048) -> list[dict]:
    """The kernels of the Nipurax decoder: capped attention with a sink and differential attention beside the plain ones, routed experts with the
    clamped GLU beside those of the decoder with a GEGLU, the row kernels."""
    from ..models.mixers import stepped_frequencies
    from . import AttentionForm
    from . import cuda as K
    from . import cuda_hybrid as H
    from . import cuda_moe as M
    from . import cuda_parallel as P
    add = _Table()
    tf = add.tf
    bf = dict(dtype=torch.bfloat16, device="cuda")
    D = 128
    cap = AttentionForm(cap=30.0, sink=torch.zeros(heads, device="cuda"), temperature=(0.1, 1024))
    dif = AttentionForm(chunk=chunk, difference=(0.4, 0.7, 1e-5))
    freq = stepped_frequencies(64, 5e5, 4.0, 1.0, 8.0, 4096.0).cuda()
    gu, down = torch.randn(experts, 2 * ff, width, **bf) * 0.02, torch.randn(experts, width, ff, **bf) * 0.02
    gain, vec = torch.ones(width, **bf), torch.ones(width, **bf)

    def rows(T, case):
        x = torch.randn(T, width, **bf)
        lg = torch.randn(T, experts + 4, device="cuda")
        corr = torch.zeros(experts + 4, device="cuda")
        idx, w = K.router_topk(lg[:, :experts].contiguous(), top, "softmax")
        add("router_topk", case, lambda: K.router_topk(lg, top, "softmax", corr, scale=2.0, renorm=False), nbytes=T * (experts + 4) * 4.0)
        n = T * top
        used = min(n, experts) if n < experts else experts
        wb, fl = used * 3.0 * ff * width * 2, 6.0 * n * ff * width
        add("experts, decoder with GEGLU", case, lambda: M.experts_forward_bf16(x, idx, w, gu, down, "geglu"), fl, tf, wb, like="routed decoder")
        add("experts, clamped", case, lambda: P.expert_outputs(x, idx, w, gu, down, "clamped", 7.0), fl, tf, wb)
        r = P.expert_outputs(x, idx, w, gu, down, "clamped", 7.0)
        a, h, hb = torch.randn(T, width, device="cuda"), torch.randn(T, width, device="cuda"), torch.randn(T, width, **bf)
        add("add_rmsnorm", case, lambda: K.add_rmsnorm(x, hb, gain, 1e-5), nbytes=T * width * 8, like="routed decoder")
        add("norm_add_norm", case, lambda: K.norm_add_norm(a, gain, hb, gain, 1e-5), nbytes=T * width * 10, like="routed decoder")
        per = 4 if r.sum is not None else 2 * top
        add("stream_step, experts", case, lambda: P.stream_step(h, a, 0.3, r, None, True, (gain, gain), 1e-5, None), nbytes=T * width * (16.0 + per))
        add("stream_step, pass", case, lambda: P.stream_step(h, a, 1.0, None, vec, False, (gain, gain), 1e-5, None), nbytes=T * width * 12.0)

    for B, q in ((1, 4096), (8, 512)):
        case, T = f"{B} x {q} tokens", B * q
        m = _meta(B, q, q)
        n_in = (heads + 2 * kv_heads) * D
        y = torch.randn(T, n_in, **bf)
        pq, pk, pv = y.split([heads * D, kv_heads * D, kv_heads * D], 1)
        kc = torch.randn(m.page_table.numel(), 64, kv_heads, D, **bf)
        vc, out = torch.randn_like(kc), torch.empty(T, heads * D, **bf)
        Q = torch.randn(T, heads, D, **bf)
        fl = 4.0 * heads * D * T * (q + 1) / 2
        add("attention_prefill", case, lambda: K.attention_prefill(Q, kc, vc, m, 0.05), fl, tf, like="routed decoder")
        add("  split_p", case, lambda: H.attention_exact(Q, kc, vc, m, 0.05, out=out), fl, tf)
        add("  capped, sink, temperature", case, lambda: H.attention_exact(Q, kc, vc, m, 0.05, out=out, form=cap), fl, tf)
        keys = sum(i % chunk + 1 for i in range(q)) / q
        add("difference of maps (64 / 128)", case, lambda: H.attention_exact(Q, kc, vc, m, 0.05, out=out, form=dif), heads * T * keys * (4.0 * 64 + 4.0 * 128), tf)
        inv, g = torch.ones(D // 2, device="cuda"), torch.ones(D, **bf)
        add("qk_norm_rope_append", case, lambda: K.qk_norm_rope_append(y, heads, kv_heads, D, g, g, False, inv, m, kc, vc, 1e-5), nbytes=T * n_in * 4,
            like="routed decoder")
        add("rotate_append", case, lambda: P.rotate_append(pq, pk, pv, 2 * heads, 2 * kv_heads, 64, freq, m, kc, vc), nbytes=T * n_in * 4)
        add("append", case, lambda: P.rotate_append(None, pk, pv, heads, kv_heads, D, None, m, kc, vc), nbytes=T * 2 * kv_heads * D * 4)
        rows(T, case)
    for B in (1, 32, 128):
        case, ctx = f"{B} x 1 token", 2048
        m = _meta(B, 1, ctx)
        n_in = (heads + 2 * kv_heads) * D
        y = torch.randn(B, n_in, **bf)
        pq, pk, pv = y.split([heads * D, kv_heads * D, kv_heads * D], 1)
        kc = torch.randn(m.page_table.numel(), 64, kv_heads, D, **bf)
        vc, Q = torch.randn_like(kc), torch.randn(B, heads, D, **bf)
        out = torch.empty(B, heads * D, **bf)
        nb = 2.0 * B * ctx * kv_heads * D * 2
        m16, k16, v16 = _meta(B, 1, ctx, 16), kc.view(-1, 16, kv_heads, D), vc.view(-1, 16, kv_heads, D)
        add("gqa_decode_tc", case, lambda: K.gqa_decode_tc(Q, k16, v16, m16, 0.1), nbytes=nb, like="routed decoder")
        add("paged_attention_decode", case, lambda: H.attention_exact(Q, kc, vc, m, 0.1), nbytes=nb)
        add("  capped, sink, temperature", case, lambda: H.attention_exact(Q, kc, vc, m, 0.1, out=out, form=cap), nbytes=nb)
        add("difference of maps (64 / 128)", case, lambda: H.attention_exact(Q, kc, vc, m, 0.1, out=out, form=dif), nbytes=nb)
        inv, g = torch.ones(D // 2, device="cuda"), torch.ones(D, **bf)
        add("qk_norm_rope_append", case, lambda: K.qk_norm_rope_append(y, heads, kv_heads, D, g, g, False, inv, m, kc, vc, 1e-5), nbytes=B * n_in * 4,
            like="routed decoder")
        add("rotate_append", case, lambda: P.rotate_append(pq, pk, pv, 2 * heads, 2 * kv_heads, 64, freq, m, kc, vc), nbytes=B * n_in * 4)
        rows(B, case)
    assert K.last_status() == 0
    return add.rows


def run_kivezen(width: int = 2048, heads: int = 16, kv_heads: int = 4, experts: int = 32, top: int = 4, ff: int = 1024, streams: int = 4) -> list[dict]:
    """The kernels of the Kivezen decoder: attention with a cap and turned values beside the plain one, lightning attention beside the Mamba-2 chunks and
    steps and the decayed linear attention, the mixing of the residual streams beside the row kernels of the routed decoder, products with an
    activation beside plain ones."""
    from ..models.mixers import HeadDecays, state_shape, yarn_frequencies
    from . import AttentionForm
    from . import cuda as K
    from . import cuda_hybrid as H
    from . import cuda_moe as M
    from . import cuda_parallel as P
    add = _Table()
    tf = add.tf
    bf = dict(dtype=torch.bfloat16, device="cuda")
    D = 128
    C = heads * D
    sink = torch.zeros(heads, device="cuda")
    freq = yarn_frequencies(D, 1e5, 4.0, 4096.0, 32.0, 1.0)[0].cuda()
    gu, down = torch.randn(experts, 2 * ff, width, **bf) * 0.02, torch.randn(experts, width, ff, **bf) * 0.02
    gain, row_gain = torch.ones(width, **bf), torch.ones(C, **bf)
    read, mix = torch.ones(streams, device="cuda"), torch.eye(streams, device="cuda")
    decays = HeadDecays([1.0 - 2.0 ** -(4 + h % 8) for h in range(heads)], D, "cuda")
    # the like recurrence of Rokarax at the same width: heads of 64 with 128 state rows shared by all
    SH = C // 64
    ones = torch.ones(SH, device="cuda")

    def rows(T, case):
        x = torch.randn(T, width, **bf)
        z = torch.randn(T, experts + 1, device="cuda")
        idx, w = K.router_topk(z[:, :experts], top, "softmax")
        n = T * top
        used = min(n, experts)
        wb, fl = used * 3.0 * ff * width * 2, 6.0 * n * ff * width
        add("experts, decoder with GEGLU", case, lambda: M.experts_forward_bf16(x, idx, w, gu, down, "geglu"), fl, tf, wb, like="routed decoder")
        add("experts, clamped", case, lambda: P.expert_outputs(x, idx, w, gu, down, "clamped", 7.0), fl, tf, wb)
        r = P.expert_outputs(x, idx, w, gu, down, "clamped", 7.0)
        a, hb, xs = torch.randn(T, width, device="cuda"), torch.randn(T, width, **bf), torch.randn(T, streams, width, device="cuda")
        add("add_rmsnorm", case, lambda: K.add_rmsnorm(x, hb, gain, 1e-5), nbytes=T * width * 8, like="routed decoder")
        add("norm_add_norm", case, lambda: K.norm_add_norm(a, gain, hb, gain, 1e-5), nbytes=T * width * 10, like="routed decoder")
        add("mix_streams", case, lambda: P.mix_streams(xs, mix, read, a, None, None, read, gain, 1e-5, True), nbytes=T * width * (8.0 * streams + 6))
        per = 4 if r.sum is not None else 2 * top
        add("mix_streams, experts", case, lambda: P.mix_streams(xs, mix, read, a, z[:, experts], r, read, gain, 1e-5, True),
            nbytes=T * width * (8.0 * streams + 6 + per))
        w_up, w_in = torch.randn(4 * width, width, **bf) * 0.02, torch.randn(4 * C, width, **bf) * 0.02
        for name, wt, fn, like in (("linear", w_up, lambda: K.linear(x, w_up), "both decoders"), ("linear, gelu", w_up, lambda: K.linear_act(x, w_up, "gelu", 4 * width), None),
                                   ("linear, silu on 3 of 4 parts", w_in, lambda: K.linear_act(x, w_in, "silu", 3 * C), None)):
            add(name, case, fn, 2.0 * T * wt.numel(), tf, 2.0 * (wt.numel() + T * width + T * wt.shape[0]), like=like)

    for B, q in ((1, 4096), (8, 512)):
        case, T = f"{B} x {q} tokens", B * q
        m = _meta(B, q, q)
        n_in = (heads + 2 * kv_heads) * D
        y = torch.randn(T, n_in, **bf)
        pq, pk, pv = y.split([heads * D, kv_heads * D, kv_heads * D], 1)
        kc = torch.randn(m.page_table.numel(), 64, kv_heads, D, **bf)
        vc, out = torch.randn_like(kc), torch.empty(T, C, **bf)
        Q = torch.randn(T, heads, D, **bf)
        turn = P.turn_table(m.positions, freq, 1.0)
        fl = 4.0 * heads * D * T * (q + 1) / 2
        add("attention_prefill", case, lambda: K.attention_prefill(Q, kc, vc, m, 0.05), fl, tf, like="routed decoder")
        add("  capped, sink", case, lambda: H.attention_exact(Q, kc, vc, m, 0.05, out=out, form=AttentionForm(cap=30.0, sink=sink)), fl, tf)
        add("  capped, sink, turned", case, lambda: H.attention_exact(Q, kc, vc, m, 0.05, out=out, form=AttentionForm(cap=30.0, sink=sink, turn=turn)), fl, tf)
        half, half_turn = vc.view(-1, 64, kv_heads, D // 2)[:kc.shape[0]].contiguous(), turn[:, :D // 4].contiguous()
        add("  .., values of 64", case, lambda: H.attention_exact(Q, kc, half, m, 0.05, out=out[:, :C // 2], form=AttentionForm(cap=30.0, sink=sink, turn=half_turn)),
            0.75 * fl, tf)
        inv, g = torch.ones(D // 2, device="cuda"), torch.ones(D, **bf)
        add("qk_norm_rope_append", case, lambda: K.qk_norm_rope_append(y, heads, kv_heads, D, g, g, False, inv, m, kc, vc, 1e-5), nbytes=T * n_in * 4,
            like="routed decoder")
        add("turn_table", case, lambda: P.turn_table(m.positions, freq, 1.0), nbytes=T * D * 4.0)
        add("turn_norm_append", case, lambda: P.turn_norm_append(pq, pk, pv, heads, kv_heads, D, turn, turn, sink, m, kc, vc, 1e-5), nbytes=T * (n_in * 4 + D * 8.0))
        yl = torch.randn(T, 4 * C, **bf)
        pv, pk, pq, pg = yl.split([C] * 4, 1)
        S = torch.zeros(B, *state_shape(heads, D, D), device="cuda")
        fl = 2.0 * T * heads * (2 * D * D + 64 * D + 32 * D)
        add("lightning_chunk", case, lambda: H.lightning_chunk(yl, decays, S, m, heads, D, D), fl, tf, T * C * 10.0)
        o = H.lightning_chunk(yl, decays, S, m, heads, D, D)
        add("norm, gate", case, lambda: H.gated_part_norm(o, pg, row_gain, 1, 1e-5, out, norm_first=True), nbytes=T * C * 8.0)
        xbc = torch.randn(T, C + 256, **bf)
        S2 = torch.zeros(B, *state_shape(SH, 128, 64), device="cuda")
        hi = (-0.02 * (torch.arange(T, device="cuda") % 64 + 1.0)).expand(SH, T).contiguous()
        dt, lo = torch.ones_like(hi), torch.zeros_like(hi)
        add("ssd_chunk (Mamba-2)", case, lambda: H.ssd_chunk(xbc, dt, hi, lo, ones, S2, m, 1, SH, 128, 64), 2.0 * T * SH * (2 * 128 * 64 + 32 * 64) + 2.0 * T * 64 * 128, tf,
            T * (C * 6.0 + 512), like="rokarax")
        add("decay_scan", case, lambda: H.decay_scan(pq, pk, pv, decays.channel, S, m, heads, D, D, 1.0), 5.0 * T * C * D, F32_TFLOPS, T * C * 10.0, like="tatizen")
        rows(T, case)
    for B in (1, 32, 128):
        case, ctx = f"{B} x 1 token", 2048
        m = _meta(B, 1, ctx)
        n_in = (heads + 2 * kv_heads) * D
        y = torch.randn(B, n_in, **bf)
        pq, pk, pv = y.split([heads * D, kv_heads * D, kv_heads * D], 1)
        kc = torch.randn(m.page_table.numel(), 64, kv_heads, D, **bf)
        vc, Q = torch.randn_like(kc), torch.randn(B, heads, D, **bf)
        out = torch.empty(B, C, **bf)
        turn = P.turn_table(m.positions, freq, 1.0)
        nb = 2.0 * B * ctx * kv_heads * D * 2
        m16, k16, v16 = _meta(B, 1, ctx, 16), kc.view(-1, 16, kv_heads, D), vc.view(-1, 16, kv_heads, D)
        add("gqa_decode_tc", case, lambda: K.gqa_decode_tc(Q, k16, v16, m16, 0.1), nbytes=nb, like="routed decoder")
        add("  capped, sink, turned", case, lambda: H.attention_exact(Q, kc, vc, m, 0.05, out=out, form=AttentionForm(cap=30.0, sink=sink, turn=turn)), nbytes=nb)
        half, half_turn = vc.view(-1, 64, kv_heads, D // 2)[:kc.shape[0]].contiguous(), turn[:, :D // 4].contiguous()
        add("  .., values of 64", case, lambda: H.attention_exact(Q, kc, half, m, 0.05, out=out[:, :C // 2], form=AttentionForm(cap=30.0, sink=sink, turn=half_turn)),
            nbytes=0.75 * nb)
        inv, g = torch.ones(D // 2, device="cuda"), torch.ones(D, **bf)
        add("qk_norm_rope_append", case, lambda: K.qk_norm_rope_append(y, heads, kv_heads, D, g, g, False, inv, m, kc, vc, 1e-5), nbytes=B * n_in * 4,
            like="routed decoder")
        add("turn_table", case, lambda: P.turn_table(m.positions, freq, 1.0), nbytes=B * D * 4.0)
        add("turn_norm_append", case, lambda: P.turn_norm_append(pq, pk, pv, heads, kv_heads, D, turn, turn, sink, m, kc, vc, 1e-5), nbytes=B * (n_in * 4 + D * 8.0))
        yl = torch.randn(B, 4 * C, **bf)
        pv, pk, pq, pg = yl.split([C] * 4, 1)
        S = torch.zeros(B, *state_shape(heads, D, D), device="cuda")
        add("lightning_step", case, lambda: H.lightning_attention(yl, pq, pk, pv, pg, decays, row_gain, S, m, heads, D, D, 1e-5, out), nbytes=B * C * D * 8.0)
        a2, b2, hg = torch.randn(C, 16, **bf), torch.randn(C, **bf), torch.ones(D, **bf)
        yd = torch.randn(B, 4 * C + 16, **bf)
        dq, dk, dv, dg, low = yd.split([C, C, C, C, 16], 1)
        add("decay_step", case, lambda: H.decayed_linear_attention(dq, dk, dv, dg, low, a2, b2, 1 / 16, hg, S, m, heads, D, D, 1e-5, 1.0, out),
            nbytes=B * C * D * 8.0, like="tatizen")
        rows(B, case)
    assert K.last_status() == 0
    return add.rows
