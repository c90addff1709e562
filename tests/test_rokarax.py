"""The Rokarax decoder and the mechanisms it is made of against the plain float64 oracle, on the host path and on the CUDA path (32-bit and
bf16): each mechanism alone, whole prompts, token-by-token decoding, portions, mixed batches, reuse of pages and state slots."""
import random
from types import SimpleNamespace

import pytest
import torch

from mary_b200 import ops
from mary_b200.models.mixers import LatentAttentionMixer, distance_buckets, yarn_frequencies
from mary_b200.models.registry import FAMILIES, make_engine
from mary_b200.oracle import rokarax as oracle
from mary_b200.runtime.batch import BatchMeta
from mary_b200.runtime.kv_cache import PagedKVCache

from paged_cases import Paged, bf16, error, prompt, schedule
from rokarax_cases import CONFIGS, attention, build, config, latent, mamba, random_weights

FAMILY = next(f for f in FAMILIES if f.name == "rokarax")
TARGETS = [pytest.param(("cpu", torch.float32), id="cpu"), pytest.param(("cuda", torch.float32), id="cuda-f32", marks=pytest.mark.gpu),
           pytest.param(("cuda", torch.bfloat16), id="cuda-bf16", marks=pytest.mark.gpu)]


@pytest.fixture(params=TARGETS)
def target(request):
    return request.param


def tol(target, f32=2e-5, b16=1.5e-2):
    return f32 if target[1] == torch.float32 else b16


def rand(g, *shape):
    return bf16(torch.randn(*shape, generator=g))


# --------------------------------------------------------------------------- mechanisms alone
@pytest.mark.parametrize("width", [8, 72, 50, 1024, 333, 2056])
def test_dynamic_tanh_around_the_stream(target, width):
    dev, dt = target
    g = torch.Generator().manual_seed(width)
    w = {n + s: v for n in "abc" for s, v in (("", rand(g, width)), (".b", rand(g, width)), (".alpha", bf16(torch.tensor(0.3) + ord(n) % 5)))}
    norm = {n: SimpleNamespace(w=w[n].to(dev, dt), b=w[n + ".b"].to(dev, dt), alpha=w[n + ".alpha"].reshape(1).to(dev)) for n in "abc"}
    wd = {k: v.double() for k, v in w.items()}
    table, ids = rand(g, 33, width), torch.tensor([0, 32, 7, 7, 1])
    h, x = ops.embed_dyt(ids.to(dev), table.to(dev, dt), 2.7, norm["a"])
    stream = table[ids].double() * 2.7
    assert h.dtype == torch.float32 and x.dtype == dt
    assert error(h, stream) < 1e-6 and error(x, oracle.dynamic_tanh(stream, wd, "a")) < tol(target, 1e-6, 4e-3)
    a = torch.randn(5, width + 8, generator=g)[:, :width] * 2
    x = ops.dyt_add(a.to(dev), norm["b"], h, norm["c"])
    stream = stream + oracle.dynamic_tanh(a.double(), wd, "b")
    assert error(h, stream) < 1e-6 and x.dtype == dt and error(x, oracle.dynamic_tanh(stream, wd, "c")) < tol(target, 1e-6, 4e-3)


@pytest.mark.parametrize("table", [(2, 3.0), (8, 60.0), (12, 7.0), (32, 128.0), (32, 500.0), (6, 1e5), (33, 90.0)], ids=str)
def test_distance_buckets(table):
    rows, far = table
    window = 700
    assert distance_buckets(window, rows, far).tolist() == [oracle.distance_bucket(n, rows, far) for n in range(window)]
    with pytest.raises(ValueError):
        distance_buckets(100, rows, rows // 2)


@pytest.mark.parametrize("rot", [(64, 10000.0, 4.0, 4096.0, 32.0, 1.0), (16, 1e6, 2.5, 512.0, 16.0, 2.0), (2, 100.0, 8.0, 64.0, 1.0, 1.0),
                                 (24, 50.0, 1.5, 1e6, 4.0, 0.01), (12, 300.0, None, 0, 0, 0)], ids=str)
def test_rotation_frequencies(rot):
    dims, base, *scaling = rot
    keys = dict(zip(("factor", "original", "fast", "slow"), scaling))
    want, gain = oracle.yarn_frequencies(dims, base, None if keys["factor"] is None else keys)
    got, g2 = yarn_frequencies(dims, base, **keys)
    assert torch.allclose(got, want, rtol=1e-12) and g2 == pytest.approx(gain, abs=1e-12)


ATTENTION = [(6, 2, 64, 64), (4, 4, 32, 48), (8, 1, 128, 128), (12, 2, 96, 40), (2, 2, 256, 256), (20, 1, 16, 24), (3, 1, 17, 33), (4, 2, 64, 128),
             (16, 2, 128, 128), (10, 1, 64, 64), (2, 1, 600, 24)]


@pytest.mark.parametrize("heads", ATTENTION, ids=str)
@pytest.mark.parametrize("page, window", [(16, 40), (64, 1), (64, 64), (64, 97), (16, 500)])
def test_attention_with_bias_window_and_gate(target, heads, page, window):
    dev, dt = target
    H, G, D, E = heads
    g = torch.Generator().manual_seed(H * D + E + window)
    lengths = {0: 150, 1: 1, 2: 77}
    q, k, v, gate = ({s: rand(g, n, hh * d) for s, n in lengths.items()} for hh, d in ((H, D), (G, D), (G, E), (H, E)))
    gq, gk = bf16(1 + 0.2 * torch.randn(H * D, generator=g)), bf16(1 + 0.2 * torch.randn(G * D, generator=g))
    rel = rand(g, 14, H) * 1.5
    at = distance_buckets(window, 14, 60.0)
    bias = rel[at].T.contiguous()
    eps, scale = 1e-3, 1.7 * D ** -0.5
    want = {}
    for s, n in lengths.items():
        qn, kn = oracle.rms(q[s].double(), gq.double(), eps).view(n, H, D), oracle.rms(k[s].double(), gk.double(), eps).view(n, G, D)
        o = oracle.window_attention(qn, kn, v[s].double().view(n, G, E), scale, window, lambda d, h: float(rel[oracle.distance_bucket(d, 14, 60.0), h]))
        want[s] = o.reshape(n, H * E) * oracle.sigmoid(gate[s].double())
    pool = Paged(page, device=dev)
    kc, vc = torch.zeros(96, page, G, D, dtype=dt, device=dev), torch.zeros(96, page, G, E, dtype=dt, device=dev)
    kw = dict(window=window, bias=bias.to(dev))
    at = [0, H * D, (H + G) * D, (H + G) * D + G * E, (H + G) * D + (G + H) * E]
    for step in schedule(lengths, random.Random(1)):
        meta = pool.step({s: n for s, (_, n) in step.items()})
        rows = torch.cat([torch.cat([x[s][a:a + n] for s, (a, n) in step.items()]) for x in (q, k, v, gate)], 1)
        rows = torch.cat([rows, torch.zeros(rows.shape[0], -rows.shape[1] % 8)], 1).to(dev, dt)
        pq, pk, pv, pg = (rows[:, at[i]:at[i + 1]] for i in range(4))
        qq = ops.row_norm_append(pq, pk, pv, H, G, D, E, gq.to(dev, dt), gk.to(dev, dt), meta, kc, vc, eps)
        out = ops.rows_buffer(rows.shape[0], H * E + 24, rows)
        out.fill_(7.0)
        ops.attention_exact(qq, kc, vc, meta, scale, out=out[:, :H * E], gate=pg, **kw)
        ref = torch.cat([want[s][a:a + n] for s, (a, n) in step.items()])
        assert error(out[:, :H * E], ref) < tol(target, 2e-5, 2e-2)
        assert bool((out[:, H * E:] == 7.0).all())
        # a layer that reads these keys: queries alone
        q2 = ops.row_norm_append(pq, None, None, H, G, D, E, gq.to(dev, dt), None, meta, kc, vc, eps)
        assert torch.equal(q2, qq)


@pytest.mark.parametrize("heads", [(4, 2, 64, 64), (2, 1, 128, 128), (4, 1, 40, 24), (2, 2, 256, 256)], ids=str)
@pytest.mark.parametrize("decoded", [False, True])
def test_attention_finds_one_key_at_the_window_edge(target, heads, decoded):
    """One key stands out for the last query: inside the window its value comes back whole, one position outside it must not be seen, nor
    one position after the query; at page borders and within a page, in a prompt and in decoding."""
    dev, dt = target
    H, G, D, E = heads
    page, T = 64, 330
    g = torch.Generator().manual_seed(5)
    v = rand(g, T + 1, G, E)
    for window in (1, 2, 63, 64, 65, 128, 129, 300, 330, 400):
        for back in {window - 1, window, 0, -1, min(window - 1, 64)}:
            j = T - 1 - back
            if not 0 <= j <= T:
                continue
            k, q = bf16(0.05 * torch.randn(T + 1, G, D, generator=g)), bf16(0.05 * torch.randn(T + 1, H, D, generator=g))
            k[j] = rand(g, G, D)
            q[T - 1] = 8.0 * k[j].repeat_interleave(H // G, 0)
            lo = max(0, T - window)
            want = oracle.window_attention(q[T - 1:T].double(), k[T - 1:T].double(), v[T - 1:T].double(), 1.0, 1)[0] if window == 1 else None
            s = torch.einsum("hd,khd->hk", q[T - 1].double(), k[lo:T].double().repeat_interleave(H // G, 1))
            want = torch.einsum("hk,khd->hd", torch.softmax(s, -1), v[lo:T].double().repeat_interleave(H // G, 1)) if want is None else want
            if 0 <= back < window:
                assert (want - v[j].double().repeat_interleave(H // G, 0)).abs().max() < 0.1       # the case shows what it should
            pool = Paged(page, 16, device=dev, seed=j)
            meta = pool.step({0: T - 1 if decoded else T})
            kc, vc = (torch.full((16, page, G, d), 0.25, dtype=dt, device=dev) for d in (D, E))
            put = lambda m, a, b: ops.ref.kv_append(k[a:b].to(dev, dt), v[a:b].to(dev, dt), kc, vc, m.slot_mapping)  # noqa: E731
            put(meta, 0, T - 1 if decoded else T)
            if decoded:
                meta = pool.step({0: 1})
                put(meta, T - 1, T)
            qq = q[T - 1:T] if decoded else q[:T]
            put(pool.step({0: 1}), T, T + 1)                         # the key after the query, already in the pages
            out = ops.attention_exact(qq.contiguous().to(dev, dt), kc, vc, meta, 1.0, window=window).view(-1, H, E)[-1]
            assert error(out, want) < tol(target, 2e-5, 2e-2), (window, back)


@pytest.mark.parametrize("decoded", [False, True])
@pytest.mark.parametrize("D", [64, 40])
def test_bias_of_one_distance_stands_out(target, decoded, D):
    """All keys alike and one distance with a large bias: the value that many positions back comes out, for every row of a prompt that has
    one, and in decoding."""
    dev, dt = target
    H, T, window, page = 2, 200, 150, 64
    g = torch.Generator().manual_seed(1)
    v = rand(g, T, 1, D)
    k = torch.zeros(T, 1, D)
    for dist in (0, 1, 15, 63, 64, 65, 127, 128, 149):
        bias = torch.zeros(H, window)
        bias[1, dist] = 30.0
        pool = Paged(page, 16, device=dev, seed=dist)
        kc, vc = (torch.zeros(16, page, 1, D, dtype=dt, device=dev) for _ in range(2))
        steps, outs = [T] if not decoded else [T - 40] + [1] * 40, []
        at = 0
        for n in steps:
            meta = pool.step({0: n})
            ops.ref.kv_append(k[at:at + n].to(dev, dt), v[at:at + n].to(dev, dt), kc, vc, meta.slot_mapping)
            outs.append(ops.attention_exact(torch.ones(n, H, D, dtype=dt, device=dev), kc, vc, meta, 1.0, window=window, bias=bias.to(dev)).view(n, H, D))
            at += n
        out = torch.cat(outs)
        assert error(out[dist:, 1], v[:T - dist, 0].double()) < tol(target, 1e-5, 6e-3), dist
        mean = torch.stack([v[max(0, i - window + 1):i + 1, 0].double().mean(0) for i in range(T)])
        assert error(out[:, 0], mean) < tol(target, 1e-5, 2e-2)


def latent_mixer(shape, window, scaling, target, g):
    H, D, R, E, Q, K = shape
    f, gain = oracle.yarn_frequencies(R, 500.0, scaling)
    m = LatentAttentionMixer(32, H, D, R, E, Q, K, 1.4 * (D + R) ** -0.5, window, f, gain, 1e-3, target[1], target[0])
    w = {"q_gain": bf16(1 + 0.2 * torch.randn(Q, generator=g)), "kv_gain": bf16(1 + 0.2 * torch.randn(K, generator=g)),
         "w_q": rand(g, H * (D + R), Q) * Q ** -0.5, "w_k": rand(g, H * D, K) * K ** -0.5, "w_v": rand(g, H * E, K) * K ** -0.5}
    w = {n: bf16(v) for n, v in w.items()}
    for n, v in w.items():
        getattr(m, n).data.copy_(v)
    m.finish()
    return m, w, (f, gain)


LATENT = [(4, 128, 64, 128, 40, 512), (16, 128, 64, 128, 64, 512), (3, 20, 12, 28, 24, 36), (5, 17, 6, 19, 23, 21), (20, 32, 16, 24, 48, 64), (2, 64, 64, 64, 32, 512),
          (2, 128, 64, 128, 16, 256)]


@pytest.mark.parametrize("shape", LATENT, ids=str)
@pytest.mark.parametrize("window", [1, 64, 90, 1000])
def test_latent_attention(target, shape, window):
    dev, dt = target
    H, D, R, E, Q, K = shape
    g = torch.Generator().manual_seed(sum(shape) + window)
    scaling = dict(factor=3.0, original=64.0, fast=8.0, slow=1.0) if window != 64 else None
    m, w, (f, gain) = latent_mixer(shape, window, scaling, target, g)
    lengths = {0: 150, 1: 1, 2: 77}
    y = {s: rand(g, n, Q + K + R) for s, n in lengths.items()}
    want = {}
    for s, n in lengths.items():
        d, wd = y[s].double(), {k: v.double() for k, v in w.items()}
        q = (oracle.rms(d[:, :Q], wd["q_gain"], m.eps) @ wd["w_q"].T).view(n, H, D + R)
        lat = oracle.rms(d[:, Q:Q + K], wd["kv_gain"], m.eps)
        kr = oracle.rotate_pairs(d[:, Q + K:], f, gain)
        k = torch.cat([(lat @ wd["w_k"].T).view(n, H, D), kr[:, None].expand(n, H, R)], -1)
        q = torch.cat([q[..., :D], oracle.rotate_pairs(q[..., D:], f, gain)], -1)
        want[s] = oracle.window_attention(q, k, (lat @ wd["w_v"].T).view(n, H, E), m.scale, window).reshape(n, H * E)
    pool = Paged(64, device=dev)
    cache = torch.zeros(96, 64, 1, K + R, dtype=dt, device=dev)
    pad = -(Q + K + R) % 8
    for step in schedule(lengths, random.Random(4)):
        meta = pool.step({s: n for s, (_, n) in step.items()})
        rows = torch.cat([y[s][a:a + n] for s, (a, n) in step.items()])
        rows = torch.cat([rows, torch.zeros(rows.shape[0], pad)], 1).to(dev, dt)
        c = ops.latent_prep(rows[:, :Q], rows[:, Q:Q + K + R], m.q_gain, m.kv_gain, m.freq, m.rot_gain, meta, cache, m.eps)
        out = ops.latent_attention(ops.linear(c, m.w_q), cache, meta, m)
        assert error(out, torch.cat([want[s][a:a + n] for s, (a, n) in step.items()])) < tol(target, 5e-5, 2.5e-2)


@pytest.mark.parametrize("shape", [(4, 128, 64, 128, 8, 512), (3, 20, 12, 28, 8, 36)], ids=str)
@pytest.mark.parametrize("decoded", [False, True])
def test_latent_attention_finds_one_key_at_the_window_edge(target, shape, decoded):
    dev, dt = target
    H, D, R, E, Q, K = shape
    page, T = 64, 300
    g = torch.Generator().manual_seed(9)
    for window in (1, 31, 32, 33, 64, 65, 127, 200, 300):
        m, w, _ = latent_mixer(shape, window, None, target, g)
        m.scale = 1.0
        for back in {0, window - 1, window, min(window - 1, 64)}:
            j = T - 1 - back
            if j < 0:
                continue
            rows, q = bf16(0.05 * torch.randn(T, K + R, generator=g)), bf16(0.02 * torch.randn(T, H, D + R, generator=g))
            rows[j, :K] = 3.0 * rand(g, K)
            key = (w["w_k"].double() @ rows[j, :K].double()).view(H, D)
            q[T - 1, :, :D] = (25.0 * key / key.pow(2).sum(-1, keepdim=True)).to(torch.bfloat16).float()
            q[T - 1, :, D:] = 0.0
            lo = max(0, T - window)
            k, v = (rows[lo:T, :K].double() @ w[n].double().T for n in ("w_k", "w_v"))
            s = torch.einsum("hd,khd->hk", q[T - 1, :, :D].double(), k.view(-1, H, D))
            want = torch.einsum("hk,khd->hd", torch.softmax(s, -1), v.view(-1, H, E))
            cache = torch.full((16, page, 1, K + R), 0.25, dtype=dt, device=dev)
            pool = Paged(page, 16, device=dev, seed=j)
            meta = pool.step({0: T - 1 if decoded else T})
            put = lambda mt, a, b: cache.view(-1, K + R).__setitem__(mt.slot_mapping.long(), rows[a:b].to(dev, dt))  # noqa: E731
            put(meta, 0, T - 1 if decoded else T)
            if decoded:
                meta = pool.step({0: 1})
                put(meta, T - 1, T)
            qq = q[T - 1:T] if decoded else q
            out = ops.latent_attention(qq.reshape(-1, H * (D + R)).to(dev, dt), cache, meta, m).view(-1, H, E)[-1]
            assert error(out, want) < tol(target, 5e-5, 4e-2), (window, back)


STATE_SPACE = [(4, 2, 64, 48, 4, 1), (6, 3, 24, 40, 3, 2), (3, 1, 19, 17, 1, 17), (8, 1, 128, 64, 4, 8), (2, 2, 200, 16, 2, 1), (5, 5, 32, 70, 9, 7),
               (4, 4, 8, 6, 2, 3), (4, 1, 64, 128, 4, 2), (2, 1, 256, 32, 4, 1), (6, 2, 16, 96, 4, 3)]


@pytest.mark.parametrize("shape", STATE_SPACE, ids=str)
@pytest.mark.parametrize("sizes", [(1, 1, 2, 3, 5, 17, 40, 70), (150,), (1,), (2, 64, 130)], ids=str)
def test_state_space(target, shape, sizes):
    dev, dt = target
    H, G, N, P, taps, parts = shape
    eps, inner = 1e-4, H * P
    g = torch.Generator().manual_seed(N * P)
    lengths = {0: 150, 1: 33, 2: 1, 3: 9, 4: 64}
    C = inner + 2 * G * N
    pad = lambda n: (n + 7) // 8 * 8  # noqa: E731
    at = [0, pad(inner), pad(inner) + pad(C)]
    x = {s: rand(g, n, at[2] + pad(H)) for s, n in lengths.items()}
    w, wb, gain = bf16(torch.randn(C, taps, generator=g) * taps ** -0.5), rand(g, C) * 0.5, bf16(1 + 0.2 * torch.randn(inner, generator=g))
    a_log, dt_bias, skip = torch.randn(H, generator=g), torch.randn(H, generator=g) - 1.0, 0.5 + torch.randn(H, generator=g).abs()
    a_log[0] = 6.0                                               # a head that forgets at once
    a_log[1] = -9.0                                              # and one that keeps (almost) everything
    want = {}
    for s, n in lengths.items():
        xs = x[s].double()
        y = oracle.silu(oracle.causal_conv(xs[:, at[1]:at[1] + C], w.double(), wb.double()))
        y = oracle.state_space(y[:, :inner].view(n, H, P), y[:, inner:inner + G * N].view(n, G, N), y[:, inner + G * N:].view(n, G, N),
                               oracle.softplus(xs[:, at[2]:at[2] + H] + dt_bias.double()), a_log.double(), skip.double())
        want[s] = oracle.rms_parts(y.reshape(n, inner) * oracle.silu(xs[:, :inner]), gain.double(), parts, eps)
    pool = Paged(device=dev)
    state = torch.full((6, H, P, (N + 3) // 4 * 4), 3.0, dtype=torch.float32, device=dev)      # what an earlier user of the slot left
    ring = torch.full((6, taps, C), 2.0, dtype=dt, device=dev)
    for step in schedule(lengths, random.Random(3), sizes):
        meta = pool.step({s: n for s, (_, n) in step.items()})
        rows = torch.cat([x[s][a:a + n] for s, (a, n) in step.items()]).to(dev, dt)
        out = ops.rows_buffer(rows.shape[0], inner, rows)
        ops.state_space(rows[:, at[1]:at[1] + C], w.to(dev, dt), wb.to(dev, dt), rows[:, at[2]:at[2] + H], dt_bias.to(dev), a_log.to(dev), skip.to(dev),
                        rows[:, :inner], gain.to(dev, dt), parts, ring, state, meta, G, H, N, P, eps, out)
        assert error(out, torch.cat([want[s][a:a + n] for s, (a, n) in step.items()])) < tol(target, 5e-5, 2e-2)


@pytest.mark.parametrize("N, P", [(32, 24), (64, 64)])
def test_state_space_keeps_one_write_over_a_long_distance(target, N, P):
    """(Almost) no decay, one token with a large step, then hundreds of tokens with (almost) none: its value is still read back."""
    dev, dt = target
    T, taps, H = 300, 2, 1
    C = P + 2 * N
    g = torch.Generator().manual_seed(0)
    x = bf16(torch.rand(T, 8 + C + (-C % 8) + P, generator=g) + 0.1)
    z0 = 8 + C + (-C % 8)
    x[:, 0] = -30.0                                              # step size ~ 0
    x[2, 0] = 3.0                                                # the write
    w = torch.zeros(C, taps)
    w[:, -1] = 1.0
    y = oracle.silu(x[:, 8:8 + C].double())
    dt2 = oracle.softplus(torch.tensor(3.0, dtype=torch.float64))
    read = dt2 * (y[2, P:P + N] @ y[T - 1, P + N:]) * y[2, :P] * oracle.silu(x[T - 1, z0:].double())
    want = oracle.rms(read[None], 1.0, 1e-6)
    pool = Paged(device=dev)
    state, ring = torch.zeros(6, H, P, N, device=dev), torch.zeros(6, taps, C, dtype=dt, device=dev)
    one = torch.ones(1, device=dev)
    for a, n in ((0, 3), (3, 150), (153, 146), (299, 1)):
        meta = pool.step({0: n})
        rows = x[a:a + n].to(dev, dt)
        out = ops.rows_buffer(n, P, rows)
        ops.state_space(rows[:, 8:8 + C], w.to(dev, dt), torch.zeros(C, dtype=dt, device=dev), rows[:, :1], 0 * one, -25.0 * one, 0 * one, rows[:, z0:],
                        torch.ones(P, device=dev, dtype=dt), 1, ring, state, meta, 1, H, N, P, 1e-6, out)
    assert error(out[-1:], want) < tol(target, 2e-3, 2e-2)


# --------------------------------------------------------------------------- the model through the engine
def engine(name, target, tokens=1024, seqs=4, seed=0, **kw):
    cfg = CONFIGS[name] if isinstance(name, str) else name
    w = random_weights(cfg, seed)
    m = build(cfg, w, *target)
    return cfg, w, make_engine(m, FAMILY, tokens, seqs, target[0], **kw)


LOGIT_TOL = dict(f32=1e-4, b16=8e-2)


@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_and_layers(target, name):
    cfg, w, eng = engine(name, target)
    ids = prompt(cfg, 140)
    logits, streams = oracle.run(cfg, w, ids)
    s = eng.open_sequence()
    got = eng.feed([(s, ids, range(len(ids)))])
    assert error(got, logits) < tol(target, **LOGIT_TOL)
    eng.close_sequence(s)
    s = eng.open_sequence()
    eng.cache.alloc.extend(s, len(ids))
    table, lens = eng.cache.alloc.page_table([s])
    meta = BatchMeta.build([len(ids)], lens, table, eng.cache.page_size, target[0], eng.cache.alloc.slots([s]))
    with torch.no_grad():
        states = eng.model.layer_states(torch.tensor(ids, dtype=torch.int32, device=target[0]), meta, eng.cache)
    for i in range(len(cfg["layers"])):
        assert error(states[i], streams[i]) < tol(target, 2e-5, 4e-2), i


@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("cut", ["ones", "twos", "changing"])
def test_portions_and_decoding(target, name, cut):
    cfg, w, eng = engine(name, target)
    ids = prompt(cfg, 140, 3)
    logits, _ = oracle.run(cfg, w, ids)
    sizes = {"ones": [1] * 140, "twos": [2] * 70, "changing": [63, 1, 1, 2, 30, 3, 17, 9, 8, 1, 1, 1, 3]}[cut]
    s, at, got = eng.open_sequence(), 0, []
    for n in sizes:
        got.append(eng.feed([(s, ids[at:at + n], range(n))]))
        at += n
    assert at == 140 and error(torch.cat(got), logits) < tol(target, **LOGIT_TOL)


@pytest.mark.parametrize("name", ["mixed", "odd", "tensor", "wide", "pages"])
def test_mixed_batches_pages_and_slots_reused(target, name):
    """More requests than slots and more tokens than the pool over time: portions of some beside single tokens of others; every logit
    equals the request's own, whatever ran beside it and whoever used its pages and slot before."""
    cfg, w, eng = engine(name, target, tokens=512, seqs=3)
    rng = random.Random(7)
    todo = [prompt(cfg, n, n) for n in (150, 3, 64, 65, 100, 128, 1, 70, 90)]
    want = [oracle.run(cfg, w, p)[0] for p in todo]
    queue, live, got = list(range(len(todo))), {}, {i: [] for i in range(len(todo))}
    while queue or live:
        while queue and len(live) < 3 and sum(-(-len(todo[i]) // 64) for i in [*live, queue[0]]) <= 8:
            live[queue.pop(0)] = [eng.open_sequence(), 0]
        step = [i for i in live if rng.random() < 0.75] or list(live)[:1]
        entries = []
        for i in step:
            n = min(rng.choice((1, 1, 1, 2, 9, 33, 64)), len(todo[i]) - live[i][1])
            entries.append((live[i][0], todo[i][live[i][1]:live[i][1] + n], range(n)))
        out = eng.feed(entries)
        k = 0
        for i, (_, t, _) in zip(step, entries):
            got[i].append(out[k:k + len(t)])
            k += len(t)
            live[i][1] += len(t)
        for i in step:
            if live[i][1] == len(todo[i]):
                eng.close_sequence(live.pop(i)[0])
    for i in range(len(todo)):
        assert error(torch.cat(got[i]), want[i]) < tol(target, **LOGIT_TOL), i
    assert eng.cache.alloc.free_pages == 8


@pytest.mark.gpu
@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16], ids=str)
def test_long_prompts(dt):
    """Prompts of more than a thousand tokens, whole and in long portions, time after time over the same pages and slots."""
    target = ("cuda", dt)
    layers = [attention(8, 2, 64, 64, 700, 400.0, 0.1, ff=192), mamba(4, 64, 128, 1, 4, 2, 192), latent(4, 128, 64, 128, 96, 512, 800, 0.06, ff=192),
              mamba(4, 64, 64, 2, 4, 1, None)]
    cfg, w, eng = engine(config(layers, vocab=64, width=128), target, tokens=6400)
    ids = prompt(cfg, 1100, 2)
    logits, _ = oracle.run(cfg, w, ids)
    for sizes in ([1100], [800, 300], [1100], [833, 1, 266]):
        s, at, got = eng.open_sequence(), 0, []
        for n in sizes:
            got.append(eng.feed([(s, ids[at:at + n], range(n))]))
            at += n
        assert error(torch.cat(got), logits) < tol(target, **LOGIT_TOL)
        eng.close_sequence(s)


def test_long_decoding(target):
    cfg = config([mamba(4, 16, 32, 2, 4, 4, 64), attention(4, 2, 64, 64, 50, 40.0, 0.2, ff=64), latent(4, 32, 16, 32, 24, 48, 100, 0.2)], vocab=97, width=64)
    cfg, w, eng = engine(cfg, target)
    n = 400 if target[0] == "cuda" else 150
    ids = prompt(cfg, n, 1)
    logits, _ = oracle.run(cfg, w, ids)
    s = eng.open_sequence()
    got = [eng.feed([(s, ids[:5], [4])])] + [eng.feed([(s, [t], [0])]) for t in ids[5:]]
    assert error(torch.cat(got), logits[4:]) < tol(target, **LOGIT_TOL)


@pytest.mark.parametrize("name", ["mixed", "tensor", "pages"])
def test_greedy_generation_through_the_scheduler(target, name):
    """Prompts of unequal lengths, more of them than are served together, chunked prefill: every generated token is the oracle's arg-max of
    the text before it (within rounding where two logits are as good as equal)."""
    cfg, w, eng = engine(name, target, tokens=768, seqs=3, prefill_chunk=50)
    prompts = [prompt(cfg, n, n) for n in (5, 120, 1, 64, 33)]
    outs = eng.generate(prompts, 12)
    slack = 1e-3 if target[1] == torch.float32 else 0.2
    for p, o in zip(prompts, outs):
        assert len(o) == 12
        logits, _ = oracle.run(cfg, w, p + o)
        at = logits[len(p) - 1:len(p) + 11]
        assert float((at.max(-1).values - at[torch.arange(12), torch.tensor(o)]).max()) <= slack
    assert eng.cache.alloc.free_pages == 12


@pytest.mark.parametrize("graph", [False, True])
@pytest.mark.parametrize("name", ["mixed", "tensor"])
def test_fixed_batch_decoder(target, graph, name):
    from mary_b200.runtime.spec_decode import SpecDecoder
    cfg, w, eng = engine(name, target)
    m = eng.model
    cache = PagedKVCache.for_model(m, num_pages=9, page_size=64, device=target[0], num_slots=3)
    dec = SpecDecoder(m, cache, 3, max_len=192, device=target[0], use_graph=graph)
    prompts = [prompt(cfg, 70, i) for i in range(3)]
    toks = [[int(t)] for t in dec.prefill(prompts, chunk=48)]
    dec.capture()
    for _ in range(10):
        dec.step()
        for b, t in enumerate(dec.emitted[:, 0].tolist()):
            toks[b].append(t)
    slack = 1e-3 if target[1] == torch.float32 else 0.2
    for p, o in zip(prompts, toks):
        at = oracle.run(cfg, w, p + o)[0][69:80]
        assert float((at.max(-1).values - at[torch.arange(11), torch.tensor(o)]).max()) <= slack


@pytest.mark.gpu
@pytest.mark.parametrize("sampled", [False, True])
def test_sampled_generation_on_the_gpu(sampled):
    from mary_b200.ops.sampling import sample
    cfg, w, eng = engine("tensor", ("cuda", torch.bfloat16), sampler=(lambda lg: sample(lg, 0.8, 5, 0.9, 3, 0)) if sampled else None)
    p = prompt(cfg, 40)
    out = eng.generate([p], 16)[0]
    logits = oracle.run(cfg, w, p + out)[0][39:55]
    rank = (logits > logits[torch.arange(16), torch.tensor(out)][:, None] + 0.2).sum(-1)
    assert int(rank.max()) < (5 if sampled else 1)
