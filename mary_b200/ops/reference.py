"""Plain PyTorch implementations of every op.

They serve three purposes: the CPU execution path (the tiny-decoder configuration runs on CPU in f32), the fp32
oracle each CUDA kernel is tested against, and the "NCCL + library" baseline arm of the benchmarks.
All of them accept any device and dtype; reductions are done in float32."""
from __future__ import annotations

import math

import torch
import torch.nn.functional as F


def rmsnorm(x, weight=None, eps: float = 1e-6):
    xf = x.float()
    y = xf * torch.rsqrt(xf.pow(2).mean(-1, keepdim=True) + eps)
    if weight is not None:
        y = y * weight.float()
    return y.to(x.dtype)


def add_rmsnorm(x, residual, weight, eps: float = 1e-6):
    """``residual += x`` (one rounding to the storage dtype, src/models/inkling/resid.rs:180-270) then norm."""
    r = (residual.float() + x.float()).to(residual.dtype)
    return rmsnorm(r, weight, eps), r


def rope_inv_freq(head_dim: int, theta: float, partial_rotary_factor: float = 1.0, device="cpu"):
    """``theta^(-2j/D)`` computed in f64 then cast to f32; a partial rotation zeroes the tail of inv_freq
    (src/models/gemma/rope.rs:68-99)."""
    j = torch.arange(head_dim // 2, dtype=torch.float64)
    inv = theta ** (-2.0 * j / head_dim)
    rot = int(head_dim // 2 * partial_rotary_factor)
    inv[rot:] = 0.0
    return inv.to(torch.float32).to(device)


def rope(x, positions, inv_freq):
    """Split-half (NeoX) rotation of ``x[T, heads, D]`` (src/models/gemma/rope.rs:190-217)."""
    ang = positions.float()[:, None] * inv_freq[None, :]
    cos, sin = ang.cos()[:, None, :], ang.sin()[:, None, :]
    d = x.shape[-1] // 2
    x1, x2 = x[..., :d].float(), x[..., d:].float()
    return torch.cat([x1 * cos - x2 * sin, x1 * sin + x2 * cos], dim=-1).to(x.dtype)


def kv_append(k, v, kcache, vcache, slot_mapping):
    """Write rows ``k[T, Hkv, D]`` / ``v`` into page slots ``slot_mapping[T]``."""
    kc = kcache.view(-1, *kcache.shape[2:])
    kc[slot_mapping] = k.to(kc.dtype)
    if v is not None and vcache is not None and vcache is not kcache:
        vc = vcache.view(-1, *vcache.shape[2:])
        vc[slot_mapping] = v.to(vc.dtype)


def gather_pages(cache, page_row, kv_len: int):
    """Dense ``[kv_len, ...]`` view of one sequence's pages."""
    ps = cache.shape[1]
    n = (kv_len + ps - 1) // ps
    return cache[page_row[:n].long()].reshape(n * ps, *cache.shape[2:])[:kv_len]


def paged_attention(q, kcache, vcache, meta, scale: float, window: int = 0, softcap: float = 0.0, dv: int | None = None, rel_bias=None):
    """Causal (optionally sliding-window) attention of the flattened batch over the paged cache.
    ``q[T, Hq, D]``; caches ``[pages, page, Hkv, D]``; GQA by index; softmax in f32.  A latent cache
    (``[pages, page, D]``, one shared kv head) passes ``vcache is kcache`` and ``dv`` = value width (the first ``dv`` dims)."""
    T, Hq, D = q.shape
    if kcache.dim() == 3:
        kcache = kcache.unsqueeze(2)
        vcache = vcache.unsqueeze(2)
    if dv is not None:
        vcache = vcache[..., :dv]
    Hkv = kcache.shape[2]
    g = Hq // Hkv
    out = torch.empty(T, Hq, vcache.shape[-1], dtype=q.dtype, device=q.device)
    qs = meta.q_start.tolist()
    kl = meta.kv_len.tolist()
    for s in range(meta.num_seqs):
        a, b = qs[s], qs[s + 1]
        if a == b:
            continue
        K = gather_pages(kcache, meta.page_table[s], kl[s]).float()      # [L, Hkv, D]
        V = gather_pages(vcache, meta.page_table[s], kl[s]).float()
        Q = q[a:b].float()                                               # [n, Hq, D]
        qpos = meta.positions[a:b].long()
        kpos = torch.arange(kl[s], device=q.device)
        Kh = K.repeat_interleave(g, dim=1)
        Vh = V.repeat_interleave(g, dim=1)
        sc = torch.einsum("nhd,lhd->hnl", Q, Kh) * scale
        if rel_bias is not None:                 # rel_bias[row, head, dist] for keys dist positions back, zero outside the extent
            dist = qpos[:, None] - kpos[None, :]
            ext = rel_bias.shape[-1]
            inside = (dist >= 0) & (dist < ext)
            rb = rel_bias[a:b].float().permute(1, 0, 2)                       # [Hq, n, ext]
            sc = sc + torch.gather(rb, 2, dist.clamp(0, ext - 1)[None].expand(Hq, -1, -1)) * inside[None]
        if softcap > 0:
            sc = softcap * torch.tanh(sc / softcap)
        mask = kpos[None, :] <= qpos[:, None]
        if window > 0:
            mask &= (qpos[:, None] - kpos[None, :]) < window
        sc = sc.masked_fill(~mask[None], float("-inf"))
        p = torch.softmax(sc, dim=-1)
        out[a:b] = torch.einsum("hnl,lhd->nhd", p, Vh).to(q.dtype)
    return out


def linear(x, w, bias=None):
    return F.linear(x, w, bias)


def gelu_tanh(x):
    return F.gelu(x.float(), approximate="tanh").to(x.dtype)


def geglu(gate, up):
    return (F.gelu(gate.float(), approximate="tanh") * up.float()).to(gate.dtype)


def swiglu(gate, up):
    return (F.silu(gate.float()) * up.float()).to(gate.dtype)


def situ(gate, up, beta: float = 4.0, linear_beta: float = 25.0):
    """``beta*tanh(g/beta)*sigmoid(g) * lb*tanh(u/lb)`` (src/models/k3/situ.rs:54-145)."""
    g, u = gate.float(), up.float()
    return (beta * torch.tanh(g / beta) * torch.sigmoid(g) * (linear_beta * torch.tanh(u / linear_beta))).to(gate.dtype)


def softcap(x, cap: float):
    return (cap * torch.tanh(x.float() / cap)).to(x.dtype) if cap and cap > 0 else x


def embed(ids, table, scale: float = 1.0):
    e = table[ids.long()]
    return e if scale == 1.0 else (e.float() * scale).to(e.dtype)


def argmax_first(logits):
    """Greedy pick, first maximum wins (src/models/gemma/gemma4/lm.rs:22-32)."""
    m = logits.max(dim=-1, keepdim=True).values
    idx = torch.arange(logits.shape[-1], device=logits.device).expand_as(logits)
    return torch.where(logits == m, idx, logits.shape[-1]).min(dim=-1).values


# --------------------------------------------------------------------------- MoE
def router_softmax_topk(logits, k: int, renorm: bool = True, bias=None, scale: float = 1.0):
    """Softmax router: probabilities over all experts, top-k of them plus ``bias`` (ties -> lower index), weights without it, renormalised."""
    p = torch.softmax(logits.float(), dim=-1)
    idx = topk_first(p if bias is None else p + bias.float(), k)[1]
    w = p.gather(-1, idx.long())
    if renorm:
        w = w / w.sum(-1, keepdim=True)
    return idx.int(), w * scale


def topk_first(scores, k: int):
    """top-k where equal scores resolve to the lower index, returned in selection order."""
    s = scores.clone()
    vals, idxs = [], []
    for _ in range(k):
        i = argmax_first(s)
        vals.append(s.gather(-1, i[:, None]))
        idxs.append(i[:, None])
        s.scatter_(-1, i[:, None], float("-inf"))
    return torch.cat(vals, -1), torch.cat(idxs, -1)


def router_sigmoid_topk(logits, bias, k: int, n_group: int = 1, topk_group: int = 1, scale: float = 1.0,
                        renorm: bool = True):
    """Sigmoid router with selection bias (``noaux_tc``, src/models/k3/router.rs:9-15): pick top-k of
    ``sigmoid(l)+bias`` — optionally restricted to the ``topk_group`` best of ``n_group`` expert groups, a group's
    score being the sum of its two best biased scores — and weight with the UNBIASED scores renormalised by
    ``sum + 1e-20`` times ``scale``."""
    s = torch.sigmoid(logits.float())
    sel = s + (bias.float() if bias is not None else 0.0)
    T, E = sel.shape
    if n_group > 1:
        gs = sel.view(T, n_group, E // n_group)
        top2, _ = topk_first(gs.reshape(T * n_group, -1), 2)
        gscore = top2.sum(-1).view(T, n_group)
        _, gi = topk_first(gscore, topk_group)
        gmask = torch.zeros(T, n_group, dtype=torch.bool, device=sel.device).scatter_(1, gi, True)
        sel = sel.masked_fill(~gmask[:, :, None].expand(T, n_group, E // n_group).reshape(T, E), float("-inf"))
    _, idx = topk_first(sel, k)
    w = s.gather(-1, idx)
    if renorm:
        w = w / (w.sum(-1, keepdim=True) + 1e-20)
    return idx.int(), w * scale


def moe_experts_dense(x, idx, w, w13, w2, act="swiglu"):
    """Reference expert MLP: ``sum_j w[t,j] * w2[e] (act(w13[e] x))`` with ``w13[e] = [gate; up]`` stacked
    (halved layout).  Weights are dense float tensors ``w13[E, 2F, H]``, ``w2[E, H, F]``."""
    T, H = x.shape
    out = torch.zeros(T, H, dtype=torch.float32, device=x.device)
    Fdim = w2.shape[-1]
    actf = {"swiglu": swiglu, "geglu": geglu, "situ": situ}[act]
    for e in idx.unique().tolist():
        t, j = (idx == e).nonzero(as_tuple=True)
        h = x[t].float() @ w13[e].float().T
        h = actf(h[:, :Fdim], h[:, Fdim:])
        y = h @ w2[e].float().T
        out.index_add_(0, t, y * w[t, j][:, None].float())
    return out.to(x.dtype)


# --------------------------------------------------------------------------- NVFP4 (torch twins of nn/fp4.py)
_E2M1 = torch.tensor([0.0, 0.5, 1.0, 1.5, 2.0, 3.0, 4.0, 6.0])


def quantize_nvfp4(x):
    """Activation quantiser, bit-exact twin of :func:`mary_b200.nn.fp4.quantize_act_nvfp4`.
    Returns ``(codes uint8[rows, k/2], scales uint8[rows, k/16])`` with E4M3 scale bytes."""
    rows, k = x.shape
    blk = x.float().reshape(rows, k // 16, 16)
    amax = blk.abs().amax(-1)
    sf = torch.clamp(amax / 6.0, max=448.0)
    sb = sf.to(torch.float8_e4m3fn)
    s = sb.float()
    y = blk / torch.where(s > 0, s, torch.ones_like(s))[..., None]
    mag = y.abs()
    code = torch.zeros_like(mag, dtype=torch.uint8)
    for t in (0.25, 0.75, 1.25, 1.75, 2.5, 3.5, 5.0):
        code += (mag >= t).to(torch.uint8)
    code = torch.where(torch.signbit(y), code | 8, code)
    code = torch.where((s == 0)[..., None], torch.zeros_like(code), code).reshape(rows, k)
    return (code[:, 0::2] | (code[:, 1::2] << 4)).contiguous(), sb.view(torch.uint8).contiguous()


def dequantize_nvfp4(codes, scales, scale2: float = 1.0):
    rows = codes.shape[0]
    c = torch.stack([codes & 0xF, codes >> 4], dim=-1).reshape(rows, -1).long()
    tab = torch.cat([_E2M1, -_E2M1]).to(codes.device)
    v = tab[c]
    s = scales.view(torch.float8_e4m3fn).float().repeat_interleave(16, dim=-1)
    return v * s * scale2


def short_conv(x, w, history=None):
    """``y = x + depthwise_causal_conv(x)`` with kernel ``w[D, k]`` (tap k-1 = current); ``history`` holds the
    previous ``k-1`` pre-conv rows (zeros at sequence start).  Returns ``(y, new_history)``
    (src/models/inkling/block.rs:48-127)."""
    T, D = x.shape
    k = w.shape[1]
    h = history if history is not None else torch.zeros(k - 1, D, dtype=x.dtype, device=x.device)
    xp = torch.cat([h, x], 0).float()
    y = x.float().clone()
    for j in range(k):
        y += xp[j:j + T] * w[:, j].float()[None, :]
    return y.to(x.dtype), xp[-(k - 1):].to(x.dtype)


# --------------------------------------------------------------------------- 32-bit residual stream, exact attention, recurrent layers
def embed32(ids, table, scale: float = 1.0):
    h = table[ids.long()].float() * scale
    return h, h.to(table.dtype, copy=True)


def post_norm_add(a, w_post, h, w_next, eps: float):
    """``h += rms(a) * w_post`` (in place, f32); returns ``rms(h) * w_next``, or a copy of ``h``, in the weights' type."""
    af = a.float()
    h += af / torch.sqrt(af.pow(2).mean(-1, keepdim=True) + eps) * w_post.float()
    return rmsnorm32(h, w_next, eps) if w_next is not None else h.to(w_post.dtype, copy=True)


def rmsnorm32(h, w, eps: float):
    return (h / torch.sqrt(h.pow(2).mean(-1, keepdim=True) + eps) * w.float()).to(w.dtype)


def qk_norm_append(q, k, v, n_q, n_kv, dk, dv, q_gain, k_gain, meta, kcache, vcache, eps):
    T = q.shape[0]
    q, k = q.reshape(T, n_q, dk), k.reshape(T, n_kv, dk)
    q = rmsnorm(q, q_gain, eps) if q_gain is not None else q
    k = rmsnorm(k, k_gain, eps) if k_gain is not None else k
    kv_append(k, v.reshape(T, n_kv, dv), kcache, vcache, meta.slot_mapping)
    return q


def _portions(meta):
    """``(rows, state slot, position of the first row)`` of every sequence of the batch."""
    qs, kl, sl = meta.q_start.tolist(), meta.kv_len.tolist(), meta.state_slots.tolist()
    return [(slice(qs[s], qs[s + 1]), sl[s], kl[s] - (qs[s + 1] - qs[s])) for s in range(meta.num_seqs)]


def head_norm_gate(o, gate, gain, eps: float, scale: float):
    """``rms(o) * gain * silu(gate) * scale`` for ``o [T, H, dv]`` f32, ``gate [T, H * dv]``."""
    T, H, dv = o.shape
    y = o / torch.sqrt(o.pow(2).mean(-1, keepdim=True) + eps) * gain.float() * F.silu(gate.float()).view(T, H, dv) * scale
    return y.reshape(T, H * dv).to(gate.dtype)


def decayed_linear_attention(q, k, v, gate, low, a2, a2_bias, inv_tau, gain, state, meta, H, dk, dv, eps, out_scale, out):
    T = q.shape[0]
    qf, kf, vf = q.float().view(T, H, dk) * dk ** -0.5, k.float().view(T, H, dk), v.float().view(T, H, dv)
    alpha = torch.exp(F.logsigmoid(low.float() @ a2.float().T + a2_bias.float()) * inv_tau).view(T, H, dk)
    o = torch.empty(T, H, dv)
    for rows, slot, pos in _portions(meta):
        S = state[slot, :, :, :dk] * (0.0 if pos == 0 else 1.0)                 # [H, dv, dk]
        for t in range(rows.start, rows.stop):
            S = S * alpha[t][:, None, :] + vf[t][:, :, None] * kf[t][:, None, :]
            o[t] = (S * qf[t][:, None, :]).sum(-1)
        state[slot, :, :, :dk] = S
    out.copy_(head_norm_gate(o, gate, gain, eps, out_scale))
    return out


def _causal_conv(x, taps_w, bias, ring, meta):
    """Depthwise convolution of every sequence's rows, continued from and recorded in its history ring."""
    taps, w = taps_w.shape[1], taps_w.float()
    y = torch.empty(x.shape[0], taps_w.shape[0])
    for rows, slot, pos in _portions(meta):
        n = rows.stop - rows.start
        hist = [ring[slot, (pos - d) % taps].float() if pos - d >= 0 else torch.zeros(w.shape[0]) for d in range(taps - 1, 0, -1)]
        ext = torch.cat([torch.stack(hist), x[rows].float()]) if hist else x[rows].float()
        y[rows] = sum(ext[j:j + n] * w[:, j] for j in range(taps))
        for d in range(min(taps, n)):
            ring[slot, (pos + n - 1 - d) % taps] = x[rows.stop - 1 - d].to(ring.dtype)
    return y if bias is None else y + bias.float()


def gated_delta_attention(x, taps_w, b_in, a_in, a_log, dt_bias, gate, gain, ring, state, meta, HK, H, dk, dv, eps, out_scale, out):
    T = x.shape[0]
    y = F.silu(_causal_conv(x, taps_w, None, ring, meta))
    q, k, v = y.split([HK * dk, HK * dk, H * dv], -1)
    unit = lambda z: z / torch.sqrt(z.pow(2).sum(-1, keepdim=True) + 1e-6)  # noqa: E731
    rep = H // HK
    q = (unit(q.view(T, HK, dk)) * dk ** -0.5).repeat_interleave(rep, 1)
    k = unit(k.view(T, HK, dk)).repeat_interleave(rep, 1)
    v = v.view(T, H, dv)
    beta = torch.sigmoid(b_in.float())
    g = torch.exp(-torch.exp(a_log) * F.softplus(a_in.float() + dt_bias))
    o = torch.empty(T, H, dv)
    for rows, slot, pos in _portions(meta):
        S = state[slot, :, :, :dk] * (0.0 if pos == 0 else 1.0)
        for t in range(rows.start, rows.stop):
            S = S * g[t][:, None, None]
            u = beta[t][:, None] * (v[t] - (S * k[t][:, None, :]).sum(-1))
            S = S + u[:, :, None] * k[t][:, None, :]
            o[t] = (S * q[t][:, None, :]).sum(-1)
        state[slot, :, :, :dk] = S
    out.copy_(head_norm_gate(o, gate, gain, eps, out_scale))
    return out


def _attention_form(q, kcache, vcache, meta, scale, f):
    """One map of ``attention_exact`` with an ``AttentionForm``: f32 ``[T, Hq, DV]``."""
    T, Hq, _ = q.shape
    G = Hq // kcache.shape[2]
    out = torch.empty(T, Hq, vcache.shape[3])
    qs, kl = meta.q_start.tolist(), meta.kv_len.tolist()
    for s in range(meta.num_seqs):
        rows = slice(qs[s], qs[s + 1])
        K = gather_pages(kcache, meta.page_table[s], kl[s]).float().repeat_interleave(G, 1)
        V = gather_pages(vcache, meta.page_table[s], kl[s]).float().repeat_interleave(G, 1)
        pos, kpos = meta.positions[rows].long(), torch.arange(kl[s])
        Q = q[rows].float()
        if f.temperature is not None:
            Q = Q * (1.0 + f.temperature[0] * torch.log((pos + 1).div(f.temperature[1], rounding_mode="floor").float() + 1.0))[:, None, None]
        sc = torch.einsum("nhd,lhd->hnl", Q, K) * scale
        if f.cap > 0:
            sc = f.cap * torch.tanh(sc / f.cap)
        seen = kpos[None] <= pos[:, None]
        if f.chunk > 0:
            seen &= kpos[None] >= (pos // f.chunk * f.chunk)[:, None]
        sc = sc.masked_fill(~seen[None], float("-inf"))
        if f.sink is not None:
            sc = torch.cat([sc, f.sink.float()[:, None, None].expand(-1, sc.shape[1], 1)], -1)
        out[rows] = torch.einsum("hnl,lhd->nhd", torch.softmax(sc, -1)[..., :kl[s]], V)
    return out if f.turn is None else _turn_pairs(out, f.turn, -1.0)


def attention_exact(q, kcache, vcache, meta, scale, window: int = 0, bias=None, gate=None, form=None):
    if form is not None:
        assert window == 0 and bias is None and gate is None
        d = q.shape[2] // form.maps
        o = [_attention_form(q[..., m * d:(m + 1) * d], kcache[..., m * d:(m + 1) * d], vcache, meta, scale, form) for m in range(form.maps)]
        y = o[0]
        if form.difference is not None:
            mix, post, eps = form.difference
            y = y - mix * o[1]
            y = y / torch.sqrt(y.pow(2).mean(-1, keepdim=True) + eps) * post
        return y.reshape(q.shape[0], -1).to(q.dtype)
    rel = None if bias is None else bias[None].expand(q.shape[0], -1, -1)
    o = paged_attention(q.float(), kcache, vcache, meta, scale, window, rel_bias=rel).reshape(q.shape[0], -1)
    return (o if gate is None else o * torch.sigmoid(gate.float())).to(q.dtype)


def _dyt(x, norm):
    return torch.tanh(norm.alpha * x) * norm.w.float() + norm.b.float()


def embed_dyt(ids, table, scale: float, norm):
    h = table[ids.long()].float() * scale
    return h, _dyt(h, norm).to(table.dtype)


def dyt_add(a, post, h, following):
    h += _dyt(a.float(), post)
    return _dyt(h, following).to(following.w.dtype)


def row_norm_append(q, k, v, n_q, n_kv, dk, dv, q_gain, k_gain, meta, kcache, vcache, eps):
    T = q.shape[0]
    if k is not None:
        kv_append(rmsnorm(k, k_gain, eps).reshape(T, n_kv, dk), v.reshape(T, n_kv, dv), kcache, vcache, meta.slot_mapping)
    return rmsnorm(q, q_gain, eps).reshape(T, n_q, dk)


def rotate_pairs(x, positions, freq, gain: float):
    """``x [T, ..., D]``: the pair ``(2i, 2i + 1)`` turns by ``position * freq[i]``; cosine and sine times ``gain``."""
    ang = (positions.float()[:, None] * freq[None]).view(x.shape[0], *[1] * (x.dim() - 2), -1)
    c, s = ang.cos() * gain, ang.sin() * gain
    u, v = x[..., 0::2].float(), x[..., 1::2].float()
    return torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2).to(x.dtype)


def latent_prep(y_q, y_kv, q_gain, kv_gain, freq, rot_gain, meta, cache, eps):
    rank = kv_gain.shape[0]
    row = torch.cat([rmsnorm(y_kv[:, :rank], kv_gain, eps), rotate_pairs(y_kv[:, rank:], meta.positions, freq, rot_gain)], -1)
    cache.view(-1, cache.shape[-1])[meta.slot_mapping] = row.to(cache.dtype)
    return rmsnorm(y_q, q_gain, eps)


def latent_attention(q, cache, meta, m):
    T = q.shape[0]
    q = q.view(T, m.heads, m.dim + m.rot)
    lat = torch.einsum("thd,hrd->thr", q[..., :m.dim].float(), m.w_k_t.float()).to(q.dtype)
    qf = torch.cat([lat, rotate_pairs(q[..., m.dim:], meta.positions, m.freq, m.rot_gain)], -1)
    o = attention_exact(qf, cache, cache[..., :m.rank], meta, m.scale, m.window).view(T, m.heads, m.rank)
    return torch.einsum("thr,hvr->thv", o.float(), m.w_v.view(m.heads, m.dv, m.rank).float()).to(q.dtype).reshape(T, -1)


def state_space(xbc, taps_w, taps_b, dt_in, dt_bias, a_log, skip, z, gain, norm_parts, ring, state, meta, G, H, N, P, eps, out):
    T = xbc.shape[0]
    x, B, C = F.silu(_causal_conv(xbc, taps_w, taps_b, ring, meta)).split([H * P, G * N, G * N], -1)
    x = x.view(T, H, P)
    B, C = (v.view(T, G, N).repeat_interleave(H // G, 1) for v in (B, C))
    dt = F.softplus(dt_in.float() + dt_bias)
    g = torch.exp(-torch.exp(a_log) * dt)
    y = torch.empty(T, H, P)
    for rows, slot, pos in _portions(meta):
        S = state[slot, :, :, :N] * (0.0 if pos == 0 else 1.0)                  # [H, P, N]
        for t in range(rows.start, rows.stop):
            S = S * g[t][:, None, None] + (dt[t][:, None] * x[t])[:, :, None] * B[t][:, None, :]
            y[t] = (S * C[t][:, None, :]).sum(-1)
        state[slot, :, :, :N] = S
    y = ((y + skip[:, None] * x).reshape(T, H * P) * F.silu(z.float())).view(T, norm_parts, -1)
    out.copy_((y / torch.sqrt(y.pow(2).mean(-1, keepdim=True) + eps)).reshape(T, H * P) * gain.float())
    return out


# --------------------------------------------------------------------------- parallel sublayers, routed experts, token pairs
def embed_pairs(ids, table, pairs, mul_prev: int, mul_cur: int, last, meta, x0=None, x1=None):
    ids, buckets = ids.long(), pairs.shape[0] - 1
    row = torch.empty_like(ids)
    for rows, slot, pos in _portions(meta):
        t = ids[rows]
        prev = torch.cat([last[slot].long().view(1), t[:-1]])
        row[rows] = (prev * mul_prev + t * mul_cur) % buckets
        if pos == 0:
            row[rows.start] = buckets
        last[slot] = t[-1].to(torch.int32)
    h = table[ids].float() + pairs[row].float()
    for x in (x0, x1):
        if x is not None:
            x.copy_(h)
    return h


def rotate_halves(x, positions, freq):
    """``x [T, H, D]``: dimensions ``i`` and ``i + n`` turn by ``position * freq[i]`` (``n`` f64 frequencies), the others stay."""
    n = freq.numel()
    ang = (positions.double()[:, None] * freq.double()[None])[:, None]
    c, s = ang.cos().float(), ang.sin().float()
    u, v = x[..., :n].float(), x[..., n:2 * n].float()
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * n:].float()], -1).to(x.dtype)


def rotate_append(q, k, v, n_q, n_kv, dk, freq, meta, kcache, vcache):
    T = k.shape[0]
    k = k.reshape(T, n_kv, dk)
    if freq is not None:
        q.copy_(rotate_halves(q.reshape(T, n_q, dk), meta.positions, freq).reshape(T, -1))
        k = rotate_halves(k, meta.positions, freq)
    kv_append(k.reshape(T, *kcache.shape[2:]), v.reshape(T, *vcache.shape[2:]), kcache, vcache, meta.slot_mapping)


def turn_table(positions, freq, gain: float):
    a = positions.double()[:, None] * freq.double()[None]
    return (torch.stack([a.cos(), a.sin()], -1).float() * gain).contiguous()


def _turn_pairs(x, turn, sign: float = 1.0):
    """``x [T, H, D]`` f32: the pair ``2 i, 2 i + 1`` turned by entry ``i`` of the table ``[T, n, 2]``, backwards with ``sign`` -1; the other dimensions stay."""
    n = turn.shape[1]
    c, s = turn[:, None, :, 0], sign * turn[:, None, :, 1]
    u, v = x[..., 0:2 * n:2], x[..., 1:2 * n:2]
    return torch.cat([torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2), x[..., 2 * n:]], -1)


def turn_norm_append(q, k, v, n_q, n_kv, dk, turn, vturn, temp, meta, kcache, vcache, eps):
    T = k.shape[0]
    y = []
    for z, n in ((q, n_q), (k, n_kv)):
        z = z.reshape(T, n, dk).float()
        z = z if turn is None else _turn_pairs(z, turn)
        y.append(z if eps is None else z / torch.sqrt(z.pow(2).mean(-1, keepdim=True) + eps))
    vv = v.reshape(T, n_kv, -1).float()
    vv = vv if vturn is None else _turn_pairs(vv, vturn)
    q.copy_((y[0] if temp is None else y[0] * temp.float()[:, None]).reshape(T, -1))
    kv_append(y[1].to(kcache.dtype), vv.to(vcache.dtype), kcache, vcache, meta.slot_mapping)


def linear_act(x, w, act: str, cols: int):
    y = linear(x, w).float()
    y[:, :cols] = F.gelu(y[:, :cols], approximate="tanh") if act == "gelu" else F.silu(y[:, :cols])
    return y.to(x.dtype)


def embed_streams(ids, table, n: int, weights, gain, eps):
    e = table[ids.long()].float()
    return e[:, None].repeat(1, n, 1), rmsnorm32(e * weights.sum(), gain, eps)


def mix_streams(xs, mix, out, a, gate, routed, weights, gain, eps, keep):
    y = 0.0
    if a is not None:
        y = a.float() if gate is None else a.float() * torch.sigmoid(gate)[:, None]
    if routed is not None:
        y = y + routed
    xs.copy_(torch.einsum("tsw,so->tow", xs, mix) + out[:, None] * y[:, None])
    return rmsnorm32(torch.einsum("tsw,s->tw", xs, weights), gain, eps)


def lightning_attention(y, q, k, v, gate, decays, gain, state, meta, H, dk, dv, eps, out):
    T = q.shape[0]
    q, k, v = q.reshape(T, H, dk).float(), k.reshape(T, H, dk).float(), v.reshape(T, H, dv).float()
    o = torch.empty(T, H, dv)
    for rows, slot, pos in _portions(meta):
        S = state[slot, :, :, :dk] * (0.0 if pos == 0 else 1.0)                  # [H, dv, dk]
        for t in range(rows.start, rows.stop):
            S = S * decays.head[:, None, None] + v[t][:, :, None] * k[t][:, None, :]
            o[t] = (S * q[t][:, None, :]).sum(-1)
        state[slot, :, :, :dk] = S
    out.copy_(rmsnorm32(o.reshape(T, H * dv), gain.float(), eps) * torch.sigmoid(gate.float()))
    return out


def clamped_glu(g, u, limit: float):
    g, u = g.float().clamp(max=limit), u.float().clamp(-limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1.0)


def expert_outputs(x, idx, w, gate_up, down, act: str, limit: float = 0.0):
    E, F2, _ = gate_up.shape
    out = torch.zeros(x.shape[0], down.shape[1])
    for e in range(E):
        t, j = torch.nonzero(idx == e, as_tuple=True)
        if t.numel():
            y = linear(x[t], gate_up[e])
            h = (clamped_glu(y[:, :F2 // 2], y[:, F2 // 2:], limit) if act == "clamped" else {"geglu": geglu, "swiglu": swiglu}[act](y[:, :F2 // 2], y[:, F2 // 2:]))
            out.index_add_(0, t, linear(h.to(x.dtype), down[e]).float() * w[t, j][:, None])
    return out + (w * (idx >= E)).sum(-1, keepdim=True) * x.float()


def stream_step(h, a, m, routed, vec, keep, gains, eps, copy):
    s = torch.zeros_like(h) if a is None else a.float()
    s = m * (s if routed is None else s + routed)
    if keep:
        s = s + h
    if vec is not None:
        s = s + vec.float()
    h.copy_(s)
    if copy is not None:
        copy.copy_(h)
    return [rmsnorm32(h, g, eps) for g in gains]
