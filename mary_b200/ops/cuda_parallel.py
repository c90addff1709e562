"""CUDA wrappers of the ops that decoders with parallel sublayers, routed experts and a 32-bit residual stream are made of, for bf16 and
for 32-bit activations."""
from __future__ import annotations

from dataclasses import dataclass

import torch

from ..utils.canary import empty as _empty
from . import cuda as K
from .cuda import _p, _stream, check, declare, lib
from .cuda_hybrid import _f32, _rows, glu_any
from .cuda_moe import grouped_gemm_bf16, moe_plan

declare("mary_embed_pairs", "ppp" + "llip" + "pppp" + "ppp" + "liiiis")
declare("mary_rotate_append", "ppp" + "liiiii" + "ppp" + "pp" + "ilis")
declare("mary_stream_step", "plf" + "plp" + "pppp" + "ii" + "ppi" + "ppppp" + "liifis")
declare("mary_mix_streams", "ppi" + "plpl" + "plpppppii" + "ppp" + "ii" + "ppp" + "iifis")
declare("mary_turn_table", "ppifpis")
declare("mary_turn_norm_append", "ppp" + "liiii" + "pipip" + "ppp" + "filis")
declare("mary_gather_rows", "plpiipis")
declare("mary_expert_glu", "plpiiiplpiiifs")
declare("mary_expert_down", "pppiiiplpiis")
declare("mary_gemm_simt_grouped", "ppp" + "ii" + "lll" + "il" + "pp" + "iis")


def embed_pairs(ids, table, pairs, mul_prev: int, mul_cur: int, last, meta, x0=None, x1=None):
    ids = ids.to(torch.int32)
    T, H = ids.shape[0], table.shape[1]
    h = _empty(T, H, dtype=torch.float32, device=table.device)
    views = [v for v in (x0, x1) if v is not None]
    assert all(v.stride(1) == 1 and v.stride(0) == views[0].stride(0) and v.dtype == table.dtype for v in views) and last.dtype == torch.int32
    check(lib().mary_embed_pairs(_p(ids), _p(table), _p(pairs), mul_prev, mul_cur, pairs.shape[0] - 1, _p(last), _p(meta.q_start), _p(meta.seq_index),
                                 _p(meta.positions), _p(meta.state_slots), _p(h), _p(x0), _p(x1), views[0].stride(0) if views else 0, T, H,
                                 table.shape[0], _f32(table), _stream()), "embed_pairs")
    return h


def rotate_append(q, k, v, n_q, n_kv, dk, freq, meta, kcache, vcache):
    (pk, ld), (pv, l2) = _rows(k), _rows(v)
    assert ld == l2 and (q is None or q.stride(0) == ld) and kcache.is_contiguous() and vcache.is_contiguous() and kcache.dtype == k.dtype
    n = 0 if freq is None else freq.numel()
    assert freq is None or freq.dtype == torch.float64
    check(lib().mary_rotate_append(_p(q), pk, pv, ld, n_q, n_kv, dk, v.shape[1], n, _p(freq), _p(meta.positions), _p(meta.slot_mapping), _p(kcache),
                                   _p(vcache), k.shape[0], kcache.shape[0] * kcache.shape[1], _f32(k), _stream()), "rotate_append")


def turn_table(positions, freq, gain: float):
    T, n = positions.shape[0], freq.numel()
    assert freq.dtype == torch.float64 and positions.dtype == torch.int32
    out = _empty(T, n, 2, dtype=torch.float32, device=positions.device)
    check(lib().mary_turn_table(_p(positions), _p(freq), n, gain, _p(out), T, _stream()), "turn_table")
    return out


def turn_norm_append(q, k, v, n_q, n_kv, dk, turn, vturn, temp, meta, kcache, vcache, eps):
    T = q.shape[0]
    (pq, ld), (pk, l2), (pv, l3) = _rows(q), _rows(k), _rows(v)
    assert ld == l2 == l3 and kcache.is_contiguous() and vcache.is_contiguous() and kcache.dtype == q.dtype
    table = lambda t: (None, 0) if t is None else (_p(t), t.shape[1])  # noqa: E731
    assert all(t is None or (t.is_contiguous() and t.dtype == torch.float32 and t.shape[0] == T) for t in (turn, vturn))
    check(lib().mary_turn_norm_append(pq, pk, pv, ld, n_q, n_kv, dk, vcache.shape[3], *table(turn), *table(vturn), _p(temp), _p(meta.slot_mapping),
                                      _p(kcache), _p(vcache), -1.0 if eps is None else eps, T, kcache.shape[0] * kcache.shape[1], _f32(q), _stream()),
          "turn_norm_append")


# --------------------------------------------------------------------------- routed experts
@dataclass
class RoutedOutputs:
    """Outputs of a batch's routed experts before they are weighted and summed: padded rows ``y`` with ``row_of`` (or their finished sum), and
    what the entries with an expert index of ``n_experts`` or more stand for, the input ``x``."""
    idx: torch.Tensor
    w: torch.Tensor
    x: torch.Tensor
    n_experts: int
    y: torch.Tensor | None = None
    row_of: torch.Tensor | None = None
    sum: torch.Tensor | None = None


# entries per batch up to which experts run entry by entry (each streams its expert's matrices) instead of through a routing plan
STEP_ENTRIES_PER_EXPERT, STEP_ENTRIES_MIN, STEP_ENTRIES_MAX = 1.0, 16, 512


def gather_rows(x, plan, k: int):
    out = _empty(plan.max_rows, x.shape[1], dtype=x.dtype, device=x.device)
    b = x.element_size()
    check(lib().mary_gather_rows(_p(x), x.stride(0) * b, _p(plan.row_of), x.shape[0], k, _p(out), x.shape[1] * b, _stream()), "gather_rows")
    return out


def _grouped_simt(x, w, plan):
    E, N, Kd = w.shape
    out = _empty(plan.max_rows, N, dtype=x.dtype, device=x.device)
    check(lib().mary_gemm_simt_grouped(_p(x), _p(w), _p(out), N, Kd, x.stride(0), w.stride(1), N, E, w.stride(0), _p(plan.tiles), _p(plan.meta),
                                       plan.max_rows // plan.nt, _f32(x), _stream()), "gemm_simt_grouped")
    return out


def _experts_step(x, idx, w, gate_up, down, act, limit):
    T, k = idx.shape
    E, F2, W = gate_up.shape
    code = {"geglu": 0, "swiglu": 1, "situ": 2, "clamped": 3}[act]
    h = _empty(T * k, F2 // 2, dtype=x.dtype, device=x.device)
    out = _empty(T, down.shape[1], dtype=torch.float32, device=x.device)
    check(lib().mary_expert_glu(_p(x), x.stride(0), _p(idx), T, k, E, _p(gate_up), gate_up.stride(0), _p(h), F2 // 2, W, code, limit, _stream()), "expert_glu")
    check(lib().mary_expert_down(_p(h), _p(idx), _p(w), T, k, E, _p(down), down.stride(0), _p(out), down.shape[1], F2 // 2, _stream()), "expert_down")
    return out


def expert_outputs(x, idx, w, gate_up, down, act: str, limit: float = 0.0) -> RoutedOutputs:
    """Entries with an index of ``len(gate_up)`` or more are not computed.  No host synchronisation."""
    T, k = idx.shape
    E, F2, W = gate_up.shape
    assert idx.dtype == torch.int32 and w.dtype == torch.float32 and idx.is_contiguous() and w.is_contiguous()
    out = RoutedOutputs(idx, w, x, E)
    fast = x.dtype == torch.bfloat16 and W % 8 == 0 and F2 % 16 == 0 and x.stride(0) % 8 == 0
    n = T * k
    if fast and n <= STEP_ENTRIES_MAX and n <= max(STEP_ENTRIES_MIN, STEP_ENTRIES_PER_EXPERT * E) and k * F2 // 2 <= 49152 and W <= 16384:
        out.sum = _experts_step(x, idx, w, gate_up, down, act, limit)
        return out
    if not fast:
        plan = moe_plan(idx, E, 64)
        h = glu_any(_grouped_simt(gather_rows(x, plan, k), gate_up, plan), act, limit)
        out.y = _grouped_simt(h, down, plan)
    else:
        nt = 32 if n <= 32 * E else (64 if n <= 64 * E else 128)
        plan = moe_plan(idx, E, nt)
        xg = gather_rows(x, plan, k)
        if nt == 128 and n >= 256 * E:
            h = K.glu(grouped_gemm_bf16(xg, gate_up, plan, F2, None, swap=False), act, limit)
            out.y = grouped_gemm_bf16(h, down, plan, down.shape[1], None, swap=False)
        else:
            h = grouped_gemm_bf16(xg, gate_up, plan, F2 // 2, act, limit=limit)
            out.y = grouped_gemm_bf16(h, down, plan, down.shape[1], None)
    out.row_of = plan.row_of
    return out


# --------------------------------------------------------------------------- the residual step
def _routed_args(r, like):
    """The arguments that describe routed experts to a kernel (see ``csrc/kernels/routed.cuh``)."""
    if r is None:
        return None, 0, None, None, None, None, None, 0, 0
    assert r.x.is_contiguous() and r.x.dtype == like.dtype and (r.y is None or r.y.dtype == like.dtype)
    return (_p(r.y), 0 if r.y is None else r.y.stride(0), _p(r.row_of), _p(r.sum), _p(r.idx), _p(r.w), _p(r.x), r.idx.shape[1], r.n_experts)


def embed_streams(ids, table, n: int, weights, gain, eps):
    ids = ids.to(torch.int32)
    T, H = ids.shape[0], table.shape[1]
    xs = _empty(T, n, H, dtype=torch.float32, device=table.device)
    x = _empty(T, H, dtype=table.dtype, device=table.device)
    check(lib().mary_mix_streams(_p(ids), _p(table), table.shape[0], None, 0, None, 0, *_routed_args(None, x), None, None, _p(xs), n, 1, _p(weights),
                                 _p(gain), _p(x), T, H, eps, _f32(table), _stream()), "embed_streams")
    return xs, x


def mix_streams(xs, mix, out, a, gate, routed, weights, gain, eps, keep: bool):
    T, n, H = xs.shape
    x = _empty(T, H, dtype=gain.dtype, device=xs.device)
    pa, lda = (None, 0) if a is None else _rows(a)
    assert xs.dtype == torch.float32 and xs.is_contiguous() and (a is None or a.dtype == torch.float32)
    assert gate is None or (gate.dtype == torch.float32 and gate.dim() == 1 and gate.shape[0] == T)
    assert all(t.dtype == torch.float32 and t.is_contiguous() for t in (mix, out, weights)) and mix.shape == (n, n)
    check(lib().mary_mix_streams(None, None, 0, pa, lda, _p(gate), 0 if gate is None else gate.stride(0), *_routed_args(routed, x), _p(mix), _p(out), _p(xs), n,
                                 int(keep), _p(weights), _p(gain), _p(x), T, H, eps, _f32(x), _stream()), "mix_streams")
    return x


def stream_step(h, a, m, routed, vec, keep, gains, eps, copy):
    T, H = h.shape
    like = next(t for t in (*gains, copy) if t is not None)
    f32 = _f32(like)
    xs = [_empty(T, H, dtype=like.dtype, device=h.device) for _ in gains]
    pa, lda = (None, 0) if a is None else _rows(a)
    assert h.dtype == torch.float32 and h.is_contiguous() and (a is None or a.dtype == torch.float32) and len(gains) <= 2
    pc, ldc = (None, 0) if copy is None else _rows(copy)
    g = list(gains) + [None] * (2 - len(gains))
    x = xs + [None] * (2 - len(gains))
    check(lib().mary_stream_step(pa, lda, m, *_routed_args(routed, like),
                                 _p(vec), _p(h), int(keep), _p(g[0]), _p(x[0]), _p(g[1]), _p(x[1]), pc, ldc, T, H, eps, f32, _stream()), "stream_step")
    return xs
