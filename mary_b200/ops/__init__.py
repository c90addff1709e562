"""Op entry points.  A CUDA tensor runs the hand-written sm_100a kernel (``ops.cuda``; a missing kernel
library is an error, never a silent fallback); a CPU tensor runs the PyTorch reference (``ops.reference``),
which is also the oracle the kernels are tested against."""
from __future__ import annotations

import torch

from . import reference as ref
from .attention_form import AttentionForm  # noqa: F401


def _cuda(x) -> bool:
    return isinstance(x, torch.Tensor) and x.is_cuda


def _k():
    from . import cuda
    return cuda


def rmsnorm(x, weight=None, eps=1e-6):
    return _k().rmsnorm(x, weight, eps) if _cuda(x) else ref.rmsnorm(x, weight, eps)


def add_rmsnorm(x, residual, weight, eps=1e-6):
    return _k().add_rmsnorm(x, residual, weight, eps) if _cuda(x) else ref.add_rmsnorm(x, residual, weight, eps)


def norm_add_norm(a, w_post, h, w_next, eps=1e-6, scalar: float = 1.0):
    """Gemma sandwich step: ``h' = (h + rms(a, w_post)) * scalar``; ``x = rms(h', w_next)``.  Returns ``(x, h')``;
    ``w_next=None`` skips the second norm and returns ``(None, h')``."""
    if _cuda(a):
        return _k().norm_add_norm(a, w_post, h, w_next, eps, scalar)
    hn = (h.float() + ref.rmsnorm(a, w_post, eps).float()) * scalar
    hn = hn.to(h.dtype)
    return (ref.rmsnorm(hn, w_next, eps) if w_next is not None else None), hn


def linear(x, w, bias=None):
    return _k().linear(x, w, bias) if _cuda(x) else ref.linear(x, w, bias)


def linear_f32(x, w, alpha: float = 1.0):
    """``alpha * x @ w^T`` with an f32 result (router logits, row-parallel partial sums, inputs of a post-norm)."""
    if _cuda(x):
        return _k().linear_f32(x, w, alpha=alpha)
    y = ref.linear(x.float(), w.float())
    return y if alpha == 1.0 else y * alpha


def qk_norm_rope_append(qkv, n_q, n_kv, head_dim, q_norm, k_norm, v_norm: bool, inv_freq, meta, kcache, vcache, eps):
    """Split ``qkv[T, (n_q+2 n_kv) D]``; per-head RMSNorm on q and k (learned gains) and optionally a weightless
    norm on v; split-half RoPE on q and k at ``meta.positions``; append k, v to the paged cache.
    Returns ``q[T, n_q, D]``."""
    if _is_q8(kcache):
        # 8-bit cache: norm and rotate into a bf16 staging row per token (the same kernel, slots 0..T-1), then quantise the rows
        # into their pages
        from types import SimpleNamespace
        T = qkv.shape[0]
        stage_k = torch.empty(T, 1, n_kv, head_dim, dtype=qkv.dtype, device=qkv.device)
        stage_v = torch.empty_like(stage_k)
        flat = SimpleNamespace(positions=meta.positions, slot_mapping=torch.arange(T, dtype=torch.int64, device=qkv.device))
        q = qk_norm_rope_append(qkv, n_q, n_kv, head_dim, q_norm, k_norm, v_norm, inv_freq, flat, stage_k, stage_v, eps)
        kv_quant_append(stage_k[:, 0], meta.slot_mapping, kcache)
        kv_quant_append(stage_v[:, 0], meta.slot_mapping, vcache)
        return q
    if _cuda(qkv):
        return _k().qk_norm_rope_append(qkv, n_q, n_kv, head_dim, q_norm, k_norm, v_norm, inv_freq, meta, kcache, vcache, eps)
    T = qkv.shape[0]
    q, k, v = qkv.split([n_q * head_dim, n_kv * head_dim, n_kv * head_dim], dim=-1)
    q, k, v = q.reshape(T, n_q, head_dim), k.reshape(T, n_kv, head_dim), v.reshape(T, n_kv, head_dim)
    if n_kv == 0:                                  # queries only (a layer that reads another layer's cache)
        q = ref.rmsnorm(q, q_norm, eps) if q_norm is not None else q
        return ref.rope(q, meta.positions, inv_freq) if inv_freq is not None else q
    if q_norm is not None:
        q = ref.rmsnorm(q, q_norm, eps)
    if k_norm is not None:
        k = ref.rmsnorm(k, k_norm, eps)
    if v_norm:
        v = ref.rmsnorm(v, None, eps)
    if inv_freq is not None:
        q, k = ref.rope(q, meta.positions, inv_freq), ref.rope(k, meta.positions, inv_freq)
    ref.kv_append(k, v, kcache, vcache, meta.slot_mapping)
    return q


def _is_q8(cache) -> bool:
    from ..runtime.kv_cache import Q8Pages
    return isinstance(cache, Q8Pages)


def kv_quant_append(rows, slots, pages) -> None:
    """Quantise ``rows [T, Hkv, D]`` to 8-bit codes with a (scale, zero) pair per (token, head) and store them at the flat cache
    slots ``slots [T]`` of ``pages`` (a ``runtime.kv_cache.Q8Pages``)."""
    if _cuda(rows):
        return _k().kv_quant_append(rows, slots, pages)
    pages.append(rows, slots)


def paged_attention(q, kcache, vcache, meta, scale, window=0, softcap=0.0, rel_bias=None):
    """``rel_bias [T, Hq, extent]`` (f32): an additive bias on the scaled score of the key ``dist`` positions back, for ``dist < extent``.
    With an 8-bit cache, decode-shaped batches run the dequantising kernel; everything else dequantises the pages of the batch."""
    if _is_q8(kcache):
        if _cuda(q) and rel_bias is None and _k().decode_q8_supported(q, kcache, meta):
            return _k().paged_attention_decode_q8(q, kcache, vcache, meta, scale, window, softcap)
        import dataclasses
        need = (meta.kv_len.long() + meta.page_size - 1) // meta.page_size
        cols = torch.arange(meta.page_table.shape[1], device=need.device)[None]
        used = (cols < need[:, None])
        pages = torch.unique(meta.page_table[used].long())
        remap = torch.zeros(kcache.shape[0], dtype=torch.int32, device=pages.device)
        remap[pages] = torch.arange(pages.numel(), dtype=torch.int32, device=pages.device)
        m2 = dataclasses.replace(meta, page_table=torch.where(used, remap[meta.page_table.long()], 0).to(torch.int32).contiguous())
        return paged_attention(q, kcache.dequantize(pages, q.dtype), vcache.dequantize(pages, q.dtype), m2, scale, window, softcap, rel_bias)
    if _cuda(q):
        return _k().paged_attention(q, kcache, vcache, meta, scale, window, softcap, rel_bias=rel_bias)
    return ref.paged_attention(q, kcache, vcache, meta, scale, window, softcap, rel_bias=rel_bias)


def mla_attention(q, cache, meta, scale):
    """Latent attention: ``q[T, Hq, 576]`` against the latent cache ``[pages, page, 576]`` (keys = all 576 dims,
    values = the first 512).  Returns ``[T, Hq, 512]``."""
    if _cuda(q):
        return _k().mla_attention(q, cache, meta, scale)
    return ref.paged_attention(q, cache, cache, meta, scale, dv=512)


def mla_expand_kv(rows, w_uk_t, w_uv, H):
    """GPU only (the host path concatenates): see ``ops.cuda.mla_expand_kv``."""
    return _k().mla_expand_kv(rows, w_uk_t, w_uv, H)


def mla_q_rope_inplace(qb, inv_freq, meta, H):
    return _k().mla_q_rope_inplace(qb, inv_freq, meta, H)


def mla_prep(qakv, q_lora, w_qa, w_kv, inv_freq, meta, cache, eps):
    """Norm the q_a part, norm the latent, rotate the carried rope dims and append ``[c_kv | k_rope]`` to the cache."""
    if _cuda(qakv):
        return _k().mla_prep(qakv, q_lora, w_qa, w_kv, inv_freq, meta, cache, eps)
    qa = ref.rmsnorm(qakv[:, :q_lora], w_qa, eps)
    ckv = ref.rmsnorm(qakv[:, q_lora:q_lora + 512], w_kv, eps)
    kr = qakv[:, q_lora + 512:q_lora + 576]
    if inv_freq is not None:
        kr = ref.rope(kr[:, None, :], meta.positions, inv_freq)[:, 0]
    cache.view(-1, 576)[meta.slot_mapping] = torch.cat([ckv, kr], -1).to(cache.dtype)
    return qa


def mla_absorb_q(qb, w_uk, inv_freq, meta, H):
    if _cuda(qb):
        return _k().mla_absorb_q(qb, w_uk, inv_freq, meta, H)
    T = qb.shape[0]
    q = qb.view(T, H, 192)
    lat = torch.einsum("thd,hnd->thn", q[..., :128].float(), w_uk.float()).to(qb.dtype)
    qr = q[..., 128:]
    if inv_freq is not None:
        qr = ref.rope(qr, meta.positions, inv_freq)
    return torch.cat([lat, qr], -1)


def mla_unabsorb_o(o_lat, w_uv, H):
    if _cuda(o_lat):
        return _k().mla_unabsorb_o(o_lat, w_uv, H)
    return torch.einsum("thk,hnk->thn", o_lat.float(), w_uv.float()).to(o_lat.dtype).reshape(o_lat.shape[0], H * 128)


def glu(gate_up, act: str = "geglu"):
    """``act(gate) * up`` over ``gate_up[T, 2F] = [gate | up]``."""
    if _cuda(gate_up):
        return _k().glu(gate_up, act)
    F = gate_up.shape[-1] // 2
    return {"geglu": ref.geglu, "swiglu": ref.swiglu, "situ": ref.situ}[act](gate_up[..., :F], gate_up[..., F:])


def linear_act(x, w, act: str, cols: int | None = None):
    """``act(x @ w^T)``, the activation (``gelu``: tanh form, or ``silu``) on the first ``cols`` outputs only (None: all of them)."""
    cols = w.shape[0] if cols is None else cols
    return _k().linear_act(x, w, act, cols) if _cuda(x) else ref.linear_act(x, w, act, cols)


def soft_cap(x, cap: float):
    """``cap * tanh(x / cap)`` of f32 values, in place."""
    return _h().soft_cap(x, cap) if _cuda(x) else x.copy_(cap * torch.tanh(x / cap))


def linear_glu(x, w_gu, act: str = "geglu", limit: float = 0.0, out=None):
    """``act(x @ gate^T) * (x @ up^T)`` with ``w_gu = [gate; up]``; fused into the GEMM epilogue on the GPU.  ``clamped``: gate at most
    ``limit``, up within it, ``g * sigmoid(1.702 g) * (u + 1)``.  ``out``: a row view that receives the result."""
    if _cuda(x):
        return _k().linear_glu(x, w_gu, act, limit, out)
    y = ref.linear(x, w_gu)
    F = y.shape[-1] // 2
    y = ref.clamped_glu(y[..., :F], y[..., F:], limit).to(x.dtype) if act == "clamped" else glu(y, act)
    return y if out is None else out.copy_(y)


def embed(ids, table, scale=1.0):
    return _k().embed(ids, table, scale) if _cuda(table) else ref.embed(ids, table, scale)


def lm_head_argmax(h, table, softcap=0.0, vocab_limit: int | None = None):
    """``argmax(softcap(h @ table^T))`` per row (first maximum wins) and the max logit.  Returns ``(ids, logit)``."""
    if _cuda(h):
        return _k().lm_head_argmax(h, table, softcap, vocab_limit)
    logits = ref.softcap(ref.linear(h, table).float(), softcap)
    if vocab_limit:
        logits = logits[:, :vocab_limit]
    ids = ref.argmax_first(logits)
    return ids, logits.gather(-1, ids[:, None])[:, 0]


def router_topk(logits, k, mode="softmax", bias=None, n_group=1, topk_group=1, scale=1.0, renorm=True):
    if _cuda(logits):
        return _k().router_topk(logits, k, mode, bias, n_group, topk_group, scale, renorm)
    if mode == "softmax":
        return ref.router_softmax_topk(logits, k, renorm, bias, scale)
    return ref.router_sigmoid_topk(logits, bias, k, n_group, topk_group, scale, renorm)


def bf16_experts(x, idx, w, gate_up, down, e0: int = 0, act: str = "geglu"):
    """``sum_k w[t,k] * down[e] (act(gate[e] x_t) * up[e] x_t)`` over the experts ``e0 .. e0 + len(gate_up)`` held here, with
    unquantised expert weights ``gate_up[E, 2F, H]`` / ``down[E, H, F]`` (src/models/inkling/moegroup.rs:556-719, the grouped bf16
    lane; src/models/gemma/gemma4/layers.rs:328-418).  GPU: routing plan + grouped tensor-core GEMMs.  CPU: entries grouped by
    expert, one GLU MLP per expert on its rows, weighted rows summed per token in f32."""
    if _cuda(x):
        from . import cuda_moe
        return cuda_moe.experts_forward_bf16(x, idx, w, gate_up, down, act, e0)
    T, k = idx.shape
    out = torch.zeros(T, x.shape[1], dtype=torch.float32, device=x.device)
    flat = idx.reshape(-1).long()
    order = torch.argsort(flat, stable=True)
    counts = torch.bincount(flat, minlength=e0 + gate_up.shape[0]).tolist()
    start = sum(counts[:e0])
    for e in range(gate_up.shape[0]):
        n = counts[e0 + e]
        if n == 0:
            continue
        ent = order[start:start + n]
        start += n
        tok = ent // k
        y = linear(linear_glu(x[tok].contiguous(), gate_up[e], act), down[e])
        out.index_add_(0, tok, y.float() * w.reshape(-1)[ent].float()[:, None])
    return out.to(x.dtype)


def quantize_nvfp4(x):
    return _k().quantize_nvfp4(x) if _cuda(x) else ref.quantize_nvfp4(x)


def short_conv(x, w, history=None):
    return _k().short_conv(x, w, history) if _cuda(x) else ref.short_conv(x, w, history)


# --------------------------------------------------------------------------- 32-bit residual stream, exact attention, recurrent layers
def _h():
    from . import cuda_hybrid
    return cuda_hybrid


def rows_buffer(T: int, n: int, like):
    """An uninitialised ``[T, n]`` row view whose pitch keeps every row 16-byte aligned."""
    return torch.empty(T, (n + 7) // 8 * 8, dtype=like.dtype, device=like.device)[:, :n]


def embed32(ids, table, scale=1.0):
    """Rows of the embedding table as ``(residual stream f32, activations)``."""
    return _h().embed32(ids, table, scale) if _cuda(table) else ref.embed32(ids, table, scale)


def post_norm_add(a, w_post, h, w_next, eps):
    """Post-norm residual step on a 32-bit stream: ``h += rms(a) * w_post`` in place; returns the next sublayer's input in the
    activation type: ``rms(h) * w_next``, or ``h`` itself with ``w_next=None``."""
    return _h().post_norm_add(a, w_post, h, w_next, eps) if _cuda(h) else ref.post_norm_add(a, w_post, h, w_next, eps)


def rmsnorm32(h, w, eps):
    """RMS norm of a 32-bit stream into the activation type."""
    return _h().rmsnorm32(h, w, eps) if _cuda(h) else ref.rmsnorm32(h, w, eps)


def qk_norm_append(q, k, v, n_q, n_kv, dk, dv, q_gain, k_gain, meta, kcache, vcache, eps):
    """Per-head RMS norm of queries and keys (no rotation), keys and values appended to the cache; ``q``, ``k``, ``v`` are row views of
    one projection, keys ``dk`` and values ``dv`` wide.  Returns ``q [T, n_q, dk]``."""
    f = _h().qk_norm_append if _cuda(q) else ref.qk_norm_append
    return f(q, k, v, n_q, n_kv, dk, dv, q_gain, k_gain, meta, kcache, vcache, eps)


def attention_exact(q, kcache, vcache, meta, scale, out=None, window: int = 0, bias=None, gate=None, form=None):
    """Causal paged attention whose scores, softmax weights and sums stay in 32 bits, for any head widths: ``[T, Hq * DV]``.  ``window``: keys
    at most ``window - 1`` positions back (0: all); ``bias [Hq, window]`` f32 is added to the scaled score by distance; ``gate [T, Hq * DV]``
    multiplies the result by its logistic function before it is rounded.  ``form`` (an ``AttentionForm``; no window, bias or gate then): chunks,
    capped scores, sinks, query temperature, the difference of two maps, a rotation of the result; ``q`` may be a row view of a projection."""
    if _cuda(q):
        return _h().attention_exact(q, kcache, vcache, meta, scale, out, window, bias, gate, form)
    o = ref.attention_exact(q, kcache, vcache, meta, scale, window, bias, gate, form)
    if out is None:
        return o
    out.copy_(o)
    return out


def embed_dyt(ids, table, scale, norm):
    """Scaled rows of the embedding table as the 32-bit residual stream, and the stream through the dynamic tanh ``norm``: ``(h, x)``."""
    return _h().embed_dyt(ids, table, scale, norm) if _cuda(table) else ref.embed_dyt(ids, table, scale, norm)


def dyt_add(a, post, h, following):
    """Residual step between dynamic tanhs (objects with ``w``, ``b``, ``alpha``): ``h += post(a)`` in place; returns ``following(h)`` in the
    activation type."""
    return _h().dyt_add(a, post, h, following) if _cuda(h) else ref.dyt_add(a, post, h, following)


def row_norm_append(q, k, v, n_q, n_kv, dk, dv, q_gain, k_gain, meta, kcache, vcache, eps):
    """RMS norm over the whole query row and the whole key row (gains of those sizes), keys and values appended to the cache; ``k`` and ``v``
    are None for a layer that reads another layer's cache.  Returns ``q [T, n_q, dk]``."""
    f = _h().row_norm_append if _cuda(q) else ref.row_norm_append
    return f(q, k, v, n_q, n_kv, dk, dv, q_gain, k_gain, meta, kcache, vcache, eps)


def latent_prep(y_q, y_kv, q_gain, kv_gain, freq, rot_gain, meta, cache, eps):
    """RMS norm of the query latent (returned) and of the key/value latent, rotation of the shared key part (pairs ``2i, 2i + 1``, cosine and
    sine times ``rot_gain``); ``[latent | rotated part]`` goes to the cache."""
    f = _h().latent_prep if _cuda(y_q) else ref.latent_prep
    return f(y_q, y_kv, q_gain, kv_gain, freq, rot_gain, meta, cache, eps)


def latent_attention(q, cache, meta, m):
    """Sliding-window latent attention of ``q [T, heads * (dim + rot)]`` (not yet rotated) over cached rows ``[latent | rotated part]``;
    ``m``: a ``LatentAttentionMixer``.  Returns ``[T, heads * dv]``."""
    return (_h() if _cuda(q) else ref).latent_attention(q, cache, meta, m)


def state_space(xbc, taps_w, taps_b, dt_in, dt_bias, a_log, skip, z, gain, norm_parts, ring, state, meta, G, H, N, P, eps, out):
    """Mamba-2 mixer between its projections: ``silu(conv(xbc) + taps_b) = [x [H, P] | B [G, N] | C [G, N]]``, ``dt = softplus(dt_in + dt_bias)``,
    ``S <- exp(-exp(a_log) dt) S + dt B x^T``, ``y = S^T C + skip x``; then ``y * silu(z)`` normed in ``norm_parts`` equal parts times ``gain``
    into ``out [T, H * P]``.  ``ring`` and ``state`` as above."""
    f = _h().state_space if _cuda(xbc) else ref.state_space
    return f(xbc, taps_w, taps_b, dt_in, dt_bias, a_log, skip, z, gain, norm_parts, ring, state, meta, G, H, N, P, eps, out)


def lightning_attention(y, q, k, v, gate, decays, gain, state, meta, H, dk, dv, eps, out):
    """``S <- d_h S + k v^T``, ``o = S^T q`` per head with constant decays (``models.mixers.HeadDecays``); then ``rms(o) * gain * sigmoid(gate)``, the
    norm over the whole row, into ``out [T, H * dv]``.  ``q``, ``k``, ``v``, ``gate``: columns of the projection rows ``y``.  ``state`` as below."""
    f = _h().lightning_attention if _cuda(q) else ref.lightning_attention
    return f(y, q, k, v, gate, decays, gain, state, meta, H, dk, dv, eps, out)


def decayed_linear_attention(q, k, v, gate, low, a2, a2_bias, inv_tau, gain, state, meta, H, dk, dv, eps, out_scale, out):
    """``S <- diag(alpha) S + k v^T``, ``o = S^T q`` per head with ``alpha = sigmoid(low a2^T + a2_bias) ** inv_tau`` per key channel and
    ``q`` scaled by ``dk ** -0.5``; then ``rms(o) * gain * silu(gate) * out_scale`` into ``out [T, H * dv]``.  Continues from and updates
    ``state [slots, H, dv, pitch]`` (f32, one column of key channels per value channel)."""
    f = _h().decayed_linear_attention if _cuda(q) else ref.decayed_linear_attention
    return f(q, k, v, gate, low, a2, a2_bias, inv_tau, gain, state, meta, H, dk, dv, eps, out_scale, out)


def gated_delta_attention(x, taps_w, b_in, a_in, a_log, dt_bias, gate, gain, ring, state, meta, HK, H, dk, dv, eps, out_scale, out):
    """Gated delta rule with short convolutions: ``x [T, 2 HK dk + H dv]`` holds the q, k, v inputs; ``silu(conv(x))``, unit q and k per
    head, ``beta = sigmoid(b_in)``, ``g = exp(-exp(a_log) softplus(a_in + dt_bias))``; ``S <- g S``, ``S <- S + k (beta (v - S^T k))^T``,
    ``o = S^T q``; then ``rms(o) * gain * silu(gate) * out_scale`` into ``out``.  ``ring [slots, taps, channels]`` keeps the last inputs of
    the convolutions by absolute position, ``state`` is laid out as above."""
    f = _h().gated_delta_attention if _cuda(x) else ref.gated_delta_attention
    return f(x, taps_w, b_in, a_in, a_log, dt_bias, gate, gain, ring, state, meta, HK, H, dk, dv, eps, out_scale, out)


# --------------------------------------------------------------------------- parallel sublayers, routed experts, token pairs
def _pl():
    from . import cuda_parallel
    return cuda_parallel


def embed_pairs(ids, table, pairs, mul_prev: int, mul_cur: int, last, meta, x0=None, x1=None):
    """Residual stream ``table[id] + pairs[(previous id * mul_prev + id * mul_cur) mod (len(pairs) - 1)]`` in f32, the last row of ``pairs`` for a
    sequence's first token.  ``last [slots, 1]`` int32 keeps a sequence's newest token between steps; ``x0``, ``x1``: row views that receive
    copies in the activation type."""
    f = _pl().embed_pairs if _cuda(table) else ref.embed_pairs
    return f(ids, table, pairs, mul_prev, mul_cur, last, meta, x0, x1)


def rotate_append(q, k, v, n_q, n_kv, dk, freq, meta, kcache, vcache) -> None:
    """Rotate ``q`` (row views of one projection: ``n_q`` heads of ``dk``) in place and ``k`` (``n_kv`` heads) into the cache, ``v`` into the cache.
    ``freq``: f64 frequencies of the pairs ``(i, i + len(freq))``, ``None`` for no rotation (then ``q`` may be None)."""
    f = _pl().rotate_append if _cuda(k) else ref.rotate_append
    return f(q, k, v, n_q, n_kv, dk, freq, meta, kcache, vcache)


def turn_table(positions, freq, gain: float = 1.0):
    """Cosine and sine of ``positions[t] * freq[i]`` times ``gain``: f32 ``[T, n, 2]`` (``freq``: f64, angles reduced in 64 bits)."""
    return _pl().turn_table(positions, freq, gain) if _cuda(positions) else ref.turn_table(positions, freq, gain)


def turn_norm_append(q, k, v, n_q, n_kv, dk, turn, vturn, temp, meta, kcache, vcache, eps) -> None:
    """Queries (``n_q`` heads of ``dk``) in place and keys (``n_kv`` heads) into the cache, their pairs ``2 i, 2 i + 1`` turned by the table ``turn`` (dimensions
    beyond it stay), then divided by their root mean square per head (``eps`` None: not), queries times ``temp [n_q]`` (or None); values turned by ``vturn`` (or
    None) into the cache.  ``q``, ``k``, ``v``: row views of one projection."""
    f = _pl().turn_norm_append if _cuda(k) else ref.turn_norm_append
    return f(q, k, v, n_q, n_kv, dk, turn, vturn, temp, meta, kcache, vcache, eps)


def embed_streams(ids, table, n: int, weights, gain, eps):
    """``n`` residual streams that all start as the token's row of the embedding table, and the first sublayer's input: ``(xs [T, n, width] f32,
    rms(sum_s weights[s] xs[s]) * gain)``."""
    return (_pl() if _cuda(table) else ref).embed_streams(ids, table, n, weights, gain, eps)


def mix_streams(xs, mix, out, a, gate, routed, weights, gain, eps, keep: bool = True):
    """The step between two sublayers of a residual of several streams: ``y = a * sigmoid(gate) + routed experts`` (``a``: f32 rows or None, ``gate [T]`` f32
    or None, ``routed``: from ``expert_outputs`` or None), ``xs[t] <- sum_s mix[s, t] xs[s] + out[t] y`` in place (``keep`` False: left undefined); returns
    ``rms(sum_t weights[t] xs[t]) * gain`` in the activation type."""
    return (_pl() if _cuda(xs) else ref).mix_streams(xs, mix, out, a, gate, routed, weights, gain, eps, keep)


def expert_outputs(x, idx, w, gate_up, down, act: str, limit: float = 0.0):
    """The routed experts of a batch (``gate_up [E, 2 F, W]``, ``down [E, W, F]``; entries with an index of ``E`` or more stand for ``x`` itself) in
    the form that ``stream_step`` sums up."""
    f = _pl().expert_outputs if _cuda(x) else ref.expert_outputs
    return f(x, idx, w, gate_up, down, act, limit)


def stream_step(h, a=None, m: float = 1.0, routed=None, vec=None, keep: bool = True, gains=(), eps: float = 0.0, copy=None):
    """``h <- keep h + m (a + sum of the routed experts) + vec`` on a 32-bit stream, in place; returns ``rms(h) * gain`` in the activation type for
    every one of ``gains`` (at most two).  ``copy``: a row view that receives ``h``."""
    f = _pl().stream_step if _cuda(h) else ref.stream_step
    return f(h, a, m, routed, vec, keep, gains, eps, copy)
