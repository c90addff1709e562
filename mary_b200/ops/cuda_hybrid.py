"""CUDA wrappers of the ops that decoders with a 32-bit residual stream, exact attention and recurrent layers are made of.

Each wrapper serves bf16 and 32-bit activations (the kernels are instantiated for both): the storage type follows the tensors it is
given.  Nothing here converts a 32-bit product to a reduced-precision mode."""
from __future__ import annotations

import numpy as np
import torch

from ..utils.canary import empty as _empty
from . import cuda as K
from .cuda import _p, _stream, check, declare, lib

declare("mary_gemm_simt", "pppiiilllfiiis")
declare("mary_embed32", "ppppiifiis")
declare("mary_post_norm_add", "plppppiifis")
declare("mary_rmsnorm32", "pppiifis")
declare("mary_glu_any", "ppiiifis")
declare("mary_act_rows", "pliiiis")
declare("mary_soft_cap", "plfs")
declare("mary_lightning_chunk", "pl" + "ppppppp" + "ppp" + "iiiiiis")
declare("mary_lightning_step", "pppplpppl" + "ppp" + "ppp" + "iiiifis")
declare("mary_qk_norm_append", "ppp" + "liiii" + "pppppp" + "fil" + "is")
declare("mary_attention_general", "ppppppppp" + "iii" + "lllll" + "iiiiiii" + "fpplppis")
declare("mary_map_difference", "pplpiiifffis")
declare("mary_attention_general_rows", "i")
declare("mary_attention_general_scratch_floats", "iiiii", ret64=True)
declare("mary_channel_decay", "pli" + "ppp" + "iifis")
declare("mary_delta_prep", "pl" + "pppppp" + "ppp" + "pppppp" + "iiiiiii" + "is")
declare("mary_conv_history", "plpppp" + "iiiis")
declare("mary_gated_head_norm", "pplppl" + "iiiffis")
declare("mary_decay_scan", "pppplpp" + "ppp" + "illl" + "iiifis")
declare("mary_delta_scan", "pppppppp" + "ppp" + "illl" + "iiiifs")
declare("mary_decay_step", "ppppp" + "li" + "ppfp" + "plfp" + "ppp" + "iiiiffis")
declare("mary_delta_step", "plppi" + "pppppp" + "plp" + "ppp" + "iiiiiffis")


declare("mary_gemm_simt_batched", "pppiiilll" + "illl" + "fiiis")
declare("mary_embed_dyt", "ppppiif" + "ppp" + "iis")
declare("mary_dyt_add", "pl" + "ppp" + "p" + "ppp" + "piiis")
declare("mary_row_norm_append", "ppp" + "liii" + "pppppp" + "filis")
declare("mary_latent_prep", "pp" + "liii" + "ppp" + "f" + "pppp" + "filis")
declare("mary_rotate_heads", "pppfp" + "iiiiii" + "is")
declare("mary_fill_shared_part", "pliplii" + "iis")
declare("mary_ss_prep", "pl" + "pppppp" + "ppp" + "pppppp" + "iiiiiii" + "is")
declare("mary_ss_conv_decay", "pl" + "pppppp" + "ppp" + "pppp" + "iiiiiis")
declare("mary_ssd_chunk", "pppppppp" + "ppp" + "iiiiiiis")
declare("mary_ssd_chunk_scratch_floats", "iiiiiii", ret64=True)
declare("mary_ssd_chunk_supported", "ii")
declare("mary_head_decay_scan", "pppppppp" + "p" + "ppp" + "illl" + "iiiis")
declare("mary_gated_part_norm", "pplppl" + "iiifiis")
declare("mary_ss_step", "plppp" + "pppp" + "pp" + "ipl" + "ppp" + "ppp" + "iiiiiifis")


def _f32(t) -> int:
    if t.dtype not in (torch.float32, torch.bfloat16):
        raise TypeError(f"expected a bf16 or f32 tensor, got {t.dtype}")
    return int(t.dtype == torch.float32)


def _rows(t):
    """``(tensor, pitch)`` of a row view ``[T, n]`` whose last dimension is contiguous."""
    assert t.dim() == 2 and t.stride(1) == 1
    return _p(t), t.stride(0)


def tensor_core_ok(x, w) -> bool:
    """Whether the TMA-fed tensor-core GEMM can address ``x [M, K]`` and ``w [N, K]``."""
    return (x.dtype == torch.bfloat16 and w.dtype == torch.bfloat16 and x.shape[1] % 8 == 0 and x.stride(0) % 8 == 0 and w.stride(0) % 8 == 0
            and x.data_ptr() % 16 == 0 and w.data_ptr() % 16 == 0)


def gemm_simt(x, w, out=None, alpha: float = 1.0, accumulate: bool = False, out_f32: bool = False):
    """``alpha * x @ w^T`` (added to ``out`` when ``accumulate``) with 32-bit products and sums, any shape."""
    M, Kd = x.shape
    N = w.shape[0]
    assert x.dtype == w.dtype and w.shape[1] == Kd and x.stride(1) == 1 and w.stride(1) == 1
    if out is None:
        out = _empty(M, N, dtype=torch.float32 if out_f32 else x.dtype, device=x.device)
    check(lib().mary_gemm_simt(_p(x), _p(w), _p(out), M, N, Kd, x.stride(0), w.stride(0), out.stride(0), alpha, int(accumulate), _f32(x), _f32(out),
                               _stream()), "gemm_simt")
    return out


def embed32(ids, table, scale: float = 1.0):
    """``(h f32, x)``: the rows of the embedding table as the residual stream and in the activation type."""
    ids = ids.to(torch.int32)
    T, H = ids.shape[0], table.shape[1]
    h = _empty(T, H, dtype=torch.float32, device=table.device)
    x = _empty(T, H, dtype=table.dtype, device=table.device)
    check(lib().mary_embed32(_p(ids), _p(table), _p(h), _p(x), T, H, scale, table.shape[0], _f32(table), _stream()), "embed32")
    return h, x


def post_norm_add(a, w_post, h, w_next, eps):
    x = _empty(h.shape, dtype=w_post.dtype, device=h.device)
    pa, lda = _rows(a)
    assert a.dtype == torch.float32 and h.dtype == torch.float32 and h.is_contiguous()
    check(lib().mary_post_norm_add(pa, lda, _p(w_post), _p(h), _p(w_next), _p(x), h.shape[0], h.shape[1], eps, _f32(w_post), _stream()), "post_norm_add")
    return x


def rmsnorm32(h, w, eps):
    y = _empty(h.shape, dtype=w.dtype, device=h.device)
    check(lib().mary_rmsnorm32(_p(h), _p(w), _p(y), h.shape[0], h.shape[1], eps, _f32(w), _stream()), "rmsnorm32")
    return y


def glu_any(gate_up, act: str, limit: float = 0.0):
    T, F2 = gate_up.shape
    out = _empty(T, F2 // 2, dtype=gate_up.dtype, device=gate_up.device)
    check(lib().mary_glu_any(_p(gate_up.contiguous()), _p(out), T, F2 // 2, {"geglu": 0, "swiglu": 1, "clamped": 3}[act], limit, _f32(gate_up),
                             _stream()), "glu_any")
    return out


def act_rows(y, act: str, cols: int):
    """The activation in place on the first ``cols`` columns."""
    py, ld = _rows(y)
    check(lib().mary_act_rows(py, ld, y.shape[0], cols, {"gelu": 0, "silu": 1}[act], _f32(y), _stream()), "act_rows")
    return y


def soft_cap(x, cap: float):
    assert x.dtype == torch.float32 and x.is_contiguous()
    check(lib().mary_soft_cap(_p(x), x.numel(), cap, _stream()), "soft_cap")
    return x


def qk_norm_append(q, k, v, n_q, n_kv, dk, dv, q_gain, k_gain, meta, kcache, vcache, eps):
    T = q.shape[0]
    qo = _empty(T, n_q, dk, dtype=q.dtype, device=q.device)
    (pq, ld), (pk, l2), (pv, l3) = _rows(q), _rows(k), _rows(v)
    assert ld == l2 == l3 and kcache.is_contiguous() and vcache.is_contiguous() and kcache.dtype == q.dtype
    check(lib().mary_qk_norm_append(pq, pk, pv, ld, n_q, n_kv, dk, dv, _p(q_gain), _p(k_gain), _p(meta.slot_mapping), _p(qo), _p(kcache), _p(vcache),
                                    eps, T, kcache.shape[0] * kcache.shape[1], _f32(q), _stream()), "qk_norm_append")
    return qo


# --------------------------------------------------------------------------- exact attention
DECODE_ROWS = K.DECODE_GROUP_ROWS         # sequences with at most this many query tokens take the decode kernel, the others the prefill kernel


def attention_general(q, kcache, vcache, meta, scale, out, group=None, nsplit=None, window: int = 0, bias=None, gate=None, form=None):
    """Any head widths, group size and storage type; ``group`` restricts the call to ``"prefill"`` or ``"decode"`` sequences.  ``bias``,
    ``gate``, ``form``: see ``ops.attention_exact``."""
    T, Hq, DK = q.shape
    Hkv, DV = kcache.shape[2], vcache.shape[3]
    G = Hq // Hkv
    fs, result = K.form_struct(form, q), out
    if form is not None and form.maps == 2:           # the kernel counts (head, map) pairs and leaves both maps' outputs in 32 bits
        Hq, Hkv, DK = 2 * Hq, 2 * Hkv, DK // 2
        out = _empty(T, Hq * DV, dtype=torch.float32, device=q.device)
    rq = max(1, min(lib().mary_attention_general_rows(G), meta.max_q_len))
    blk_seq, blk_q0, NB = K._q_blocks(meta, rq, group)
    if NB == 0:
        return out
    if nsplit is None:
        want = max(1, 296 // max(1, NB * Hkv * ((G + 15) // 16)))
        span = meta.max_kv_len if window <= 0 else min(meta.max_kv_len, window + rq)
        nsplit = max(1, min(want, 32, span // 128))
    scratch = None
    if nsplit > 1:
        scratch = _empty(lib().mary_attention_general_scratch_floats(NB, Hq, Hkv, nsplit, DV), dtype=torch.float32, device=q.device)
    check(lib().mary_attention_general(_p(q), _p(kcache), _p(vcache), _p(out), _p(meta.page_table), _p(meta.kv_len), _p(meta.q_start), _p(blk_seq),
                                       _p(blk_q0), NB, meta.page_table.shape[1], meta.page_size, kcache.stride(1), kcache.stride(0), vcache.stride(1),
                                       vcache.stride(0), out.stride(0), Hq, Hkv, DK, DV, rq, nsplit, window, scale, _p(bias), *K._gate(gate), _p(scratch),
                                       K._form_p(fs), _f32(q), _stream()), "attention_general")
    if out is not result:
        rows = None if group is None else _group_rows(meta, group)
        check(lib().mary_map_difference(_p(out), _p(result), result.stride(0), _p(rows), T if rows is None else rows.numel(), Hq // 2, DV,
                                        *form.difference, _f32(q), _stream()), "map_difference")
    return result


def _group_rows(meta, group: str):
    """The rows of the batch that belong to a group of sequences (int32, memoised)."""
    memo = meta.__dict__.setdefault("_cache", {})
    key = ("rows", group)
    if key not in memo:
        q = meta.q_lens_host
        pick = np.repeat((q > DECODE_ROWS) == (group == "prefill"), q)
        memo[key] = torch.from_numpy(np.nonzero(pick)[0].astype(np.int32)).to(meta.positions.device, non_blocking=True)
    return memo[key]


def attention_exact(q, kcache, vcache, meta, scale, out=None, window: int = 0, bias=None, gate=None, form=None):
    """Causal attention with scores, softmax weights and sums in 32 bits: the tensor-core prefill kernel with two-term weights for
    sequences that bring more than ``DECODE_ROWS`` tokens, the bandwidth-oriented decode kernel for the others (its tensor-core twin where that takes
    the ``form``), the general kernel for 32-bit tensors and for head shapes those have no instantiation for.  ``out`` may be a row view ``[T, Hq * DV]``."""
    T, Hq, DK = q.shape
    Hkv, DV = kcache.shape[2], vcache.shape[3]
    assert (q.is_contiguous() or form is not None) and kcache.is_contiguous() and vcache.stride(3) == 1 and kcache.shape[1] == meta.page_size
    assert bias is None or (bias.is_contiguous() and bias.shape == (Hq, window) and bias.dtype == torch.float32)
    assert gate is None or gate.dtype == q.dtype
    if out is None:
        out = _empty(T, Hq * DV, dtype=q.dtype, device=q.device)
    assert out.stride(1) == 1
    kw = dict(window=window, bias=bias, gate=gate, form=form)
    aligned = all(t is None or (t.stride(0) % 8 == 0 and t.data_ptr() % 16 == 0) for t in (out, gate, q))
    bf16 = q.dtype == torch.bfloat16 and vcache.is_contiguous()
    if form is not None and form.maps == 2:
        bf16 = bf16 and bool(lib().mary_attention_prefill_maps_supported(DK // 2, DV))
        fast_prefill = bf16 and meta.page_size in (16, 64) and aligned
        fast_decode = bf16 and Hq // Hkv <= 4 and aligned
    else:
        equal = DK == DV and DK in (64, 128, 256)
        fast_prefill = bf16 and (bool(lib().mary_attention_prefill_form_supported(DK, DV)) if form is not None else equal) and meta.page_size in (16, 64) and aligned
        fast_decode = bf16 and equal and Hq // Hkv <= (4 if DK == 256 else 8) and (q.is_contiguous() or aligned)
    tc_decode = form is not None and aligned and window == 0 and bias is None and gate is None and K.gqa_tc_form_supported(q, kcache, vcache, meta, form)
    fast_decode = fast_decode or tc_decode
    if not (fast_prefill or fast_decode):
        return attention_general(q, kcache, vcache, meta, scale, out, **kw)
    if meta.max_q_len > DECODE_ROWS:
        if fast_prefill:
            K.attention_prefill(q, kcache, vcache, meta, scale, out=out, split_p=True, group="prefill", **kw)
        else:
            attention_general(q, kcache, vcache, meta, scale, out, "prefill", **kw)
    if K._q_blocks(meta, 1, "decode")[2]:
        if tc_decode:
            K.gqa_decode_tc(q, kcache, vcache, meta, scale, out=out, group="decode", form=form)
        elif fast_decode:
            K._paged_attention_decode(q, kcache, vcache, meta, scale, window, 0.0, None, out=out, group="decode", bias=bias, gate=gate, form=form)
        else:
            attention_general(q, kcache, vcache, meta, scale, out, "decode", **kw)
    return out


# --------------------------------------------------------------------------- recurrent layers
def channel_decay(low, a2, bias, inv_tau: float):
    """``sigmoid(low @ a2^T + bias) ** inv_tau`` in f32 ``[T, C]``."""
    T, C = low.shape[0], a2.shape[0]
    out = _empty(T, C, dtype=torch.float32, device=low.device)
    pl, ld = _rows(low)
    assert a2.is_contiguous() and a2.dtype == low.dtype
    check(lib().mary_channel_decay(pl, ld, a2.shape[1], _p(a2), _p(bias), _p(out), T, C, inv_tau, _f32(low), _stream()), "channel_decay")
    return out


def decay_scan(q, k, v, decay, state, meta, H, dk, dv, q_scale):
    """Decayed linear attention over the portions of a batch; the state of every sequence's slot is read and updated.  f32 ``[T, H, dv]``.  ``decay``: a
    row of channel decays per token, or a single one for all of them."""
    T = q.shape[0]
    out = _empty(T, H, dv, dtype=torch.float32, device=q.device)
    (pq, lq), (pk, lk), (pv, lv) = _rows(q), _rows(k), _rows(v)
    lda = 0 if decay.dim() == 1 else decay.stride(0)
    check(lib().mary_decay_scan(pq, pk, pv, _p(decay), lda, _p(out), _p(state), _p(meta.q_start), _p(meta.kv_len), _p(meta.state_slots), meta.num_seqs,
                                lq, lk, lv, H, dk, dv, q_scale, _f32(q), _stream()), "decay_scan")
    return out


def delta_prep(x, taps_w, ring, b_in, a_in, a_log, dt_bias, meta, HK, H, dk, dv):
    """Short convolutions, unit norms and gates of a gated-delta-rule layer: f32 ``q, k [T, HK * dk]``, ``v [T, H * dv]``, ``g, beta [T, H]``
    and the products ``pairs [T, HK, 8]`` of every four tokens' keys with their keys and queries (what ``delta_scan`` takes)."""
    T = x.shape[0]
    f = dict(dtype=torch.float32, device=x.device)
    q, k, v = _empty(T, HK * dk, **f), _empty(T, HK * dk, **f), _empty(T, H * dv, **f)
    g, beta, pairs = _empty(T, H, **f), _empty(T, H, **f), _empty(T, HK, 8, **f)
    px, ldx = _rows(x)
    assert b_in.stride(0) == ldx and a_in.stride(0) == ldx
    check(lib().mary_delta_prep(px, ldx, _p(taps_w), _p(ring), _p(b_in), _p(a_in), _p(a_log), _p(dt_bias), _p(meta.q_start), _p(meta.kv_len),
                                _p(meta.state_slots), _p(q), _p(k), _p(v), _p(g), _p(beta), _p(pairs), meta.num_seqs, meta.max_q_len, HK, H, dk, dv,
                                taps_w.shape[1], _f32(x), _stream()), "delta_prep")
    return q, k, v, g, beta, pairs


def conv_history(x, ring, meta, taps, C):
    px, ldx = _rows(x)
    check(lib().mary_conv_history(px, ldx, _p(ring), _p(meta.q_start), _p(meta.kv_len), _p(meta.state_slots), meta.num_seqs, taps, C, _f32(x),
                                  _stream()), "conv_history")


def delta_scan(q, k, v, g, beta, pairs, state, meta, HK, H, dk, dv, q_scale: float = 1.0):
    T = q.shape[0]
    out = _empty(T, H, dv, dtype=torch.float32, device=q.device)
    (pq, lq), (pk, lk), (pv, lv) = _rows(q), _rows(k), _rows(v)
    check(lib().mary_delta_scan(pq, pk, pv, _p(g), _p(beta), _p(pairs), _p(out), _p(state), _p(meta.q_start), _p(meta.kv_len), _p(meta.state_slots),
                                meta.num_seqs, lq, lk, lv, HK, H, dk, dv, q_scale, _stream()), "delta_scan")
    return out


def gated_head_norm(o, gate, gain, eps, scale, out):
    T, H, dv = o.shape
    (pg, ldg), (po, ldo) = _rows(gate), _rows(out)
    check(lib().mary_gated_head_norm(_p(o), pg, ldg, _p(gain), po, ldo, T, H, dv, eps, scale, _f32(gate), _stream()), "gated_head_norm")
    return out


def decayed_linear_attention(q, k, v, gate, low, a2, a2_bias, inv_tau, gain, state, meta, H, dk, dv, eps, out_scale, out):
    q_scale = dk ** -0.5
    if meta.max_q_len == 1:
        po, ldo = _rows(out)
        ld = q.stride(0)
        assert all(t.stride(0) == ld for t in (k, v, gate, low)) and a2.is_contiguous()
        check(lib().mary_decay_step(_p(q), _p(k), _p(v), _p(gate), _p(low), ld, a2.shape[1], _p(a2), _p(a2_bias), inv_tau, _p(gain), po, ldo, q_scale,
                                    _p(state), _p(meta.q_start), _p(meta.positions), _p(meta.state_slots), meta.num_seqs, H, dk, dv, eps, out_scale,
                                    _f32(q), _stream()), "decay_step")
        return out
    o = decay_scan(q, k, v, channel_decay(low, a2, a2_bias, inv_tau), state, meta, H, dk, dv, q_scale)
    return gated_head_norm(o, gate, gain, eps, out_scale, out)


def gated_delta_attention(x, taps_w, b_in, a_in, a_log, dt_bias, gate, gain, ring, state, meta, HK, H, dk, dv, eps, out_scale, out):
    taps = taps_w.shape[1]
    if meta.max_q_len == 1:
        (px, ldx), (po, ldo) = _rows(x), _rows(out)
        assert b_in.stride(0) == ldx and a_in.stride(0) == ldx and gate.stride(0) == ldx
        check(lib().mary_delta_step(px, ldx, _p(taps_w), _p(ring), taps, _p(b_in), _p(a_in), _p(a_log), _p(dt_bias), _p(gate), _p(gain), po, ldo,
                                    _p(state), _p(meta.q_start), _p(meta.positions), _p(meta.state_slots), meta.num_seqs, HK, H, dk, dv, eps,
                                    out_scale, _f32(x), _stream()), "delta_step")
        return out
    q, k, v, g, beta, pairs = delta_prep(x, taps_w, ring, b_in, a_in, a_log, dt_bias, meta, HK, H, dk, dv)
    conv_history(x, ring, meta, taps, taps_w.shape[0])
    o = delta_scan(q, k, v, g, beta, pairs, state, meta, HK, H, dk, dv)
    return gated_head_norm(o, gate, gain, eps, out_scale, out)


# --------------------------------------------------------------------------- dynamic tanh around the stream, whole-row norms
def embed_dyt(ids, table, scale, norm):
    ids = ids.to(torch.int32)
    T, H = ids.shape[0], table.shape[1]
    h = _empty(T, H, dtype=torch.float32, device=table.device)
    x = _empty(T, H, dtype=table.dtype, device=table.device)
    check(lib().mary_embed_dyt(_p(ids), _p(table), _p(h), _p(x), T, H, scale, _p(norm.w), _p(norm.b), _p(norm.alpha), table.shape[0], _f32(table),
                               _stream()), "embed_dyt")
    return h, x


def dyt_add(a, post, h, following):
    x = _empty(h.shape, dtype=post.w.dtype, device=h.device)
    pa, lda = _rows(a)
    assert a.dtype == torch.float32 and h.dtype == torch.float32 and h.is_contiguous()
    check(lib().mary_dyt_add(pa, lda, _p(post.w), _p(post.b), _p(post.alpha), _p(h), _p(following.w), _p(following.b), _p(following.alpha), _p(x),
                             h.shape[0], h.shape[1], _f32(x), _stream()), "dyt_add")
    return x


def row_norm_append(q, k, v, n_q, n_kv, dk, dv, q_gain, k_gain, meta, kcache, vcache, eps):
    T = q.shape[0]
    qo = _empty(T, n_q, dk, dtype=q.dtype, device=q.device)
    pq, ld = _rows(q)
    pk = pv = None
    if k is not None:
        (pk, l2), (pv, l3) = _rows(k), _rows(v)
        assert ld == l2 == l3 and kcache.is_contiguous() and vcache.is_contiguous() and kcache.dtype == q.dtype
    check(lib().mary_row_norm_append(pq, pk, pv, ld, n_q * dk, n_kv * dk, n_kv * dv, _p(q_gain), _p(k_gain), _p(meta.slot_mapping), _p(qo), _p(kcache),
                                     _p(vcache), eps, T, kcache.shape[0] * kcache.shape[1], _f32(q), _stream()), "row_norm_append")
    return qo


# --------------------------------------------------------------------------- latent attention
def latent_prep(y_q, y_kv, q_gain, kv_gain, freq, rot_gain, meta, cache, eps):
    T, rank = y_q.shape[0], kv_gain.shape[0]
    (pq, ld), (pk, l2) = _rows(y_q), _rows(y_kv)
    assert ld == l2 and cache.is_contiguous() and cache.dtype == y_q.dtype
    c = _empty(T, q_gain.shape[0], dtype=y_q.dtype, device=y_q.device)
    check(lib().mary_latent_prep(pq, pk, ld, q_gain.shape[0], rank, cache.shape[-1] - rank, _p(q_gain), _p(kv_gain), _p(freq), rot_gain,
                                 _p(meta.positions), _p(meta.slot_mapping), _p(c), _p(cache), eps, T, cache.shape[0] * cache.shape[1], _f32(y_q),
                                 _stream()), "latent_prep")
    return c


def rotate_heads(src, dst, dst_off, rot, freq, rot_gain, meta):
    """The last ``rot`` values of every head of ``src [T, H, w]`` rotated into ``dst [T, H, w']`` from ``dst_off`` on (``src`` itself allowed)."""
    T, H, w = src.shape
    check(lib().mary_rotate_heads(_p(src), _p(dst), _p(freq), rot_gain, _p(meta.positions), T, H, w, dst.shape[2], dst_off, rot, _f32(src), _stream()),
          "rotate_heads")
    return dst


def head_matmul(x, w, out):
    """Per head ``out[t, h] = w[h] x[t, h]``: ``x [T, H, k]``, ``out [T, H, n]`` (views whose rows may be wider), ``w [H, n, k]``."""
    T, H, k = x.shape
    n = w.shape[1]
    (ldx, bx), (ldo, bo) = x.stride()[:2], out.stride()[:2]
    if x.dtype == torch.bfloat16 and k % 8 == 0 and n % 8 == 0 and ldx % 8 == 0 and bx % 8 == 0 and x.data_ptr() % 16 == 0 and bo % 8 == 0 and ldo % 8 == 0:
        with K.static_weights:
            return K.gemm_batched(x, w, out, T, n, k, ldx, k, ldo, H, bx, n * k, bo)
    check(lib().mary_gemm_simt_batched(_p(x), _p(w), _p(out), T, n, k, ldx, k, ldo, H, bx, n * k, bo, 1.0, 0, _f32(x), _f32(out), _stream()),
          "gemm_simt_batched")
    return out


EXPAND_ROWS = DECODE_ROWS        # sequences with more query tokens than this attend over expanded keys and values


def _visible_pages(meta, window: int):
    """The pages that the sequences with a prompt portion can see, as a cache of their own: ``(pick, meta2)`` where ``cache[pick]`` holds them
    and ``meta2`` addresses them, positions shifted by whole pages (only differences of positions enter the masks).  Memoised: every layer
    with the same window asks for the same."""
    import dataclasses
    memo = meta.__dict__.setdefault("_cache", {})
    key = ("visible", window)
    if key not in memo:
        ps = meta.page_size
        shift, spans = [0] * meta.num_seqs, []
        for s, (n, kv) in enumerate(zip(meta.q_lens_host.tolist(), meta.kv_lens_host.tolist())):
            lo = max(0, kv - n - window + 1) // ps
            spans.append((lo, (kv + ps - 1) // ps) if n > EXPAND_ROWS else (0, 0))
            shift[s] = spans[-1][0] * ps
        dev = meta.page_table.device
        width = max(b - a for a, b in spans)
        table, at, picks = torch.zeros(meta.num_seqs, width, dtype=torch.int32), 0, []
        for s, (a, b) in enumerate(spans):
            table[s, :b - a] = torch.arange(at, at + b - a, dtype=torch.int32)
            at += b - a
            picks.append(meta.page_table[s, a:b])
        host = meta.kv_lens_host - torch.tensor(shift).numpy().astype(meta.kv_lens_host.dtype)
        memo[key] = (torch.cat(picks).long(), dataclasses.replace(meta, page_table=table.to(dev, non_blocking=True), kv_lens_host=host,
                                                                  kv_len=torch.from_numpy(host).to(dev, non_blocking=True)))
    return memo[key]


def expand_latent(rows, m):
    """Keys ``[N, H, dim + rot]`` and values ``[N, H, dv]`` of cache rows ``[N, rank + rot]``, written straight into their final layout."""
    N, H, w = rows.shape[0], m.heads, m.dim + m.rot
    k = _empty(N, H, w, dtype=rows.dtype, device=rows.device)
    with K.static_weights:
        K.gemm_batched(rows, m.w_k, k, N, m.dim, m.rank, rows.stride(0), m.rank, H * w, H, 0, m.dim * m.rank, w)
        v = K.gemm(rows[:, :m.rank], m.w_v)
    check(lib().mary_fill_shared_part(_p(rows), rows.stride(0), m.rank, _p(k), N, H, m.dim, m.rot, _f32(rows), _stream()), "fill_shared_part")
    return k, v.view(N, H, m.dv)


def _latent_prompts(q, cache, meta, m, out):
    """Sequences with a prompt portion: keys and values expanded from the visible rows, then ordinary attention, a third of the arithmetic of
    attending in latent space."""
    T, H, ps = q.shape[0], m.heads, meta.page_size
    pick, meta2 = _visible_pages(meta, m.window)
    rows = cache[pick].view(-1, m.rank + m.rot)
    k, v = expand_latent(rows, m)
    q = rotate_heads(q, q, m.dim, m.rot, m.freq, m.rot_gain, meta)
    K.attention_prefill(q, k.view(-1, ps, H, m.dim + m.rot), v.view(-1, ps, H, m.dv), meta2, m.scale, m.window, out=out, split_p=True, group="prefill")


def latent_attention(q, cache, meta, m):
    T, H = q.shape[0], m.heads
    q = q.view(T, H, m.dim + m.rot)
    out = _empty(T, H * m.dv, dtype=q.dtype, device=q.device)
    bf16 = q.dtype == torch.bfloat16
    group = None
    if (bf16 and meta.max_q_len > EXPAND_ROWS and meta.page_size == 64 and m.rank % 8 == 0 and m.rot % 8 == 0
            and lib().mary_attention_prefill_supported(m.dim + m.rot, m.dv)):
        decoded = bool((meta.q_lens_host <= EXPAND_ROWS).any())
        _latent_prompts(q.clone() if decoded else q, cache, meta, m, out)
        if not decoded:
            return out
        group = "decode"
    prompts = out
    qf = _empty(T, H, m.rank + m.rot, dtype=q.dtype, device=q.device)
    head_matmul(q[..., :m.dim], m.w_k_t, qf[..., :m.rank])
    rotate_heads(q, qf, m.rank, m.rot, m.freq, m.rot_gain, meta)
    if bf16 and (m.rank, m.rot) == (512, 64) and meta.page_size in (16, 32, 64):
        lat = K.mla_attention(qf, cache.view(cache.shape[0], meta.page_size, 576), meta, m.scale, window=m.window, split_p=True, group=group)
    else:
        lat = _empty(T, H * m.rank, dtype=q.dtype, device=q.device)
        attention_general(qf, cache, cache[..., :m.rank], meta, m.scale, lat, group, window=m.window)
    out = _empty(T, H * m.dv, dtype=q.dtype, device=q.device) if group else prompts
    head_matmul(lat.view(T, H, m.rank), m.w_v.view(H, m.dv, m.rank), out.view(T, H, m.dv))
    if group:                                  # rows of the prompt portions keep what the expanded attention gave
        rows = torch.from_numpy(meta.q_lens_host > EXPAND_ROWS).to(q.device).repeat_interleave(torch.from_numpy(meta.q_lens_host).to(q.device).long())
        out = torch.where(rows[:, None], prompts, out)
    return out


# --------------------------------------------------------------------------- state space layers
_ARRIVED: dict = {}


def _arrival_counters(dev, n: int):
    """Counters of the one-token kernel, zero between launches; never freed, since a captured graph may hold them."""
    pool = _ARRIVED.setdefault(dev, [])
    if not pool or pool[-1].numel() < n:
        pool.append(torch.zeros(max(n, 4096), dtype=torch.int32, device=dev))
    return pool[-1]


def ss_prep(xbc, taps_w, taps_b, ring, dt_in, dt_bias, a_log, meta, G, H, N, P):
    """Convolutions, step sizes and decays of a Mamba-2 layer: f32 ``x [T, H * P]``, ``B, C [T, G * N]``, ``dt, decay [T, H]`` and the products
    ``pairs [T, G, 4]`` of every four tokens' ``B`` and ``C`` (what ``head_decay_scan`` takes)."""
    T = xbc.shape[0]
    f = dict(dtype=torch.float32, device=xbc.device)
    x, b, c, dt, decay, pairs = _empty(T, H * P, **f), _empty(T, G * N, **f), _empty(T, G * N, **f), _empty(T, H, **f), _empty(T, H, **f), _empty(T, G, 4, **f)
    px, ldx = _rows(xbc)
    assert dt_in.stride(0) == ldx
    check(lib().mary_ss_prep(px, ldx, _p(taps_w), _p(taps_b), _p(ring), _p(dt_in), _p(dt_bias), _p(a_log), _p(meta.q_start), _p(meta.kv_len),
                             _p(meta.state_slots), _p(x), _p(b), _p(c), _p(dt), _p(decay), _p(pairs), meta.num_seqs, meta.max_q_len, G, H, N, P,
                             taps_w.shape[1], _f32(xbc), _stream()), "ss_prep")
    return x, b, c, dt, decay, pairs


def head_decay_scan(x, b, c, dt, decay, pairs, skip, state, meta, G, H, N, P):
    out = _empty(x.shape[0], H * P, dtype=torch.float32, device=x.device)
    check(lib().mary_head_decay_scan(_p(c), _p(b), _p(x), _p(decay), _p(dt), _p(pairs), _p(skip), _p(out), _p(state), _p(meta.q_start), _p(meta.kv_len),
                                     _p(meta.state_slots), meta.num_seqs, c.stride(0), b.stride(0), x.stride(0), G, H, N, P, _stream()), "head_decay_scan")
    return out


def ssd_chunk_prep(xbc, taps_w, taps_b, ring, dt_in, dt_bias, a_log, meta, H):
    """bf16 models: convolved rows ``[T, C]`` and, per head and token, step size and summed log2 decay of the chunk as two floats."""
    T, C = xbc.shape
    rows = _empty(T, C, dtype=xbc.dtype, device=xbc.device)
    dt, hi, lo = (_empty(H, T, dtype=torch.float32, device=xbc.device) for _ in range(3))
    px, ldx = _rows(xbc)
    assert dt_in.stride(0) == ldx
    check(lib().mary_ss_conv_decay(px, ldx, _p(taps_w), _p(taps_b), _p(ring), _p(dt_in), _p(dt_bias), _p(a_log), _p(meta.q_start), _p(meta.kv_len),
                                   _p(meta.state_slots), _p(rows), _p(dt), _p(hi), _p(lo), meta.num_seqs, meta.max_q_len, T, H, C, taps_w.shape[1],
                                   _stream()), "ss_conv_decay")
    return rows, dt, hi, lo


def ssd_chunk(rows, dt, hi, lo, skip, state, meta, G, H, N, P):
    """The recurrence on the tensor cores, 64 tokens at a time: f32 ``[T, H * P]``."""
    T = rows.shape[0]
    y = _empty(T, H * P, dtype=torch.float32, device=rows.device)
    scratch = _empty(lib().mary_ssd_chunk_scratch_floats(T, meta.num_seqs, meta.max_q_len, G, H, N, P), dtype=torch.float32, device=rows.device)
    check(lib().mary_ssd_chunk(_p(rows), _p(dt), _p(hi), _p(lo), _p(skip), _p(y), _p(state), _p(scratch), _p(meta.q_start), _p(meta.kv_len),
                               _p(meta.state_slots), meta.num_seqs, meta.max_q_len, T, G, H, N, P, _stream()), "ssd_chunk")
    return y


def gated_part_norm(y, z, gain, parts, eps, out, norm_first: bool = False):
    (pz, ldz), (po, ldo) = _rows(z), _rows(out)
    check(lib().mary_gated_part_norm(_p(y), pz, ldz, _p(gain), po, ldo, y.shape[0], y.shape[1], parts, eps, int(norm_first), _f32(z), _stream()),
          "gated_part_norm")
    return out


def state_space(xbc, taps_w, taps_b, dt_in, dt_bias, a_log, skip, z, gain, norm_parts, ring, state, meta, G, H, N, P, eps, out):
    taps = taps_w.shape[1]
    if meta.max_q_len == 1:
        (px, ldx), (po, ldo) = _rows(xbc), _rows(out)
        assert dt_in.stride(0) == ldx and z.stride(0) == ldx
        S = meta.num_seqs
        row = _empty(S, H * P, dtype=torch.float32, device=xbc.device)
        cnt = _arrival_counters(xbc.device, S * norm_parts)
        check(lib().mary_ss_step(px, ldx, _p(taps_w), _p(taps_b), _p(ring), _p(dt_in), _p(dt_bias), _p(a_log), _p(skip), _p(z), _p(gain), norm_parts, po, ldo,
                                 _p(state), _p(row), _p(cnt), _p(meta.q_start), _p(meta.positions), _p(meta.state_slots), S, G, H, N, P, taps, eps,
                                 _f32(xbc), _stream()), "ss_step")
        return out
    if (xbc.dtype == torch.bfloat16 and lib().mary_ssd_chunk_supported(N, P) and xbc.stride(0) % 4 == 0
            and all(t.data_ptr() % 8 == 0 for t in (xbc, taps_w, ring))):
        pre = ssd_chunk_prep(xbc, taps_w, taps_b, ring, dt_in, dt_bias, a_log, meta, H)
        conv_history(xbc, ring, meta, taps, taps_w.shape[0])
        return gated_part_norm(ssd_chunk(*pre, skip, state, meta, G, H, N, P), z, gain, norm_parts, eps, out)
    x, b, c, dt, decay, pairs = ss_prep(xbc, taps_w, taps_b, ring, dt_in, dt_bias, a_log, meta, G, H, N, P)
    conv_history(xbc, ring, meta, taps, taps_w.shape[0])
    return gated_part_norm(head_decay_scan(x, b, c, dt, decay, pairs, skip, state, meta, G, H, N, P), z, gain, norm_parts, eps, out)


# --------------------------------------------------------------------------- linear attention with one constant decay per head
def lightning_chunk(y_in, decays, state, meta, H, dk, dv):
    """The recurrence on the tensor cores, 64 tokens at a time, over projection rows that start with ``[v | k | q]``: f32 ``[T, H * dv]``."""
    T = y_in.shape[0]
    o = _empty(T, H * dv, dtype=torch.float32, device=y_in.device)
    scratch = _empty(lib().mary_ssd_chunk_scratch_floats(T, meta.num_seqs, meta.max_q_len, H, H, dk, dv), dtype=torch.float32, device=y_in.device)
    one, hi, lo, zero = (_p(t) for t in decays.chunk)
    py, ld = _rows(y_in)
    check(lib().mary_lightning_chunk(py, ld, one, hi, lo, zero, _p(o), _p(state), _p(scratch), _p(meta.q_start), _p(meta.kv_len), _p(meta.state_slots),
                                     meta.num_seqs, meta.max_q_len, T, H, dk, dv, _stream()), "lightning_chunk")
    return o


def lightning_attention(y_in, q, k, v, gate, decays, gain, state, meta, H, dk, dv, eps, out):
    (pq, ld), (po, ldo) = _rows(q), _rows(out)
    assert all(t.stride(0) == ld for t in (k, v, gate))
    if meta.max_q_len == 1:
        S = meta.num_seqs
        rows = _empty(S, H * dv, dtype=torch.float32, device=q.device)
        check(lib().mary_lightning_step(pq, _p(k), _p(v), _p(gate), ld, _p(decays.head), _p(gain), po, ldo, _p(state), _p(rows),
                                        _p(_arrival_counters(q.device, S)), _p(meta.q_start), _p(meta.positions), _p(meta.state_slots), S, H, dk, dv, eps,
                                        _f32(q), _stream()), "lightning_step")
        return out
    if (q.dtype == torch.bfloat16 and lib().mary_ssd_chunk_supported(dk, dv) and ld % 8 == 0 and y_in.data_ptr() % 16 == 0
            and v.data_ptr() == y_in.data_ptr() and k.data_ptr() == v.data_ptr() + H * dv * 2 and q.data_ptr() == k.data_ptr() + H * dk * 2):
        o = lightning_chunk(y_in, decays, state, meta, H, dk, dv)
    else:
        o = decay_scan(q, k, v, decays.channel, state, meta, H, dk, dv, 1.0).view(-1, H * dv)
    return gated_part_norm(o, gate, gain, 1, eps, out, norm_first=True)
