"""The Tatizen decoder and the mechanisms it is made of against the plain float64 oracle, on the host path and on the CUDA path (32-bit and
bf16): each mechanism alone, whole prompts, token-by-token decoding, portions, mixed batches, reuse of pages and state slots."""
import random

import pytest
import torch

from mary_b200 import ops
from mary_b200.models.registry import FAMILIES, make_engine
from mary_b200.oracle import tatizen as oracle
from mary_b200.runtime.batch import BatchMeta
from mary_b200.runtime.kv_cache import PagedKVCache

from paged_cases import Paged, bf16, error, prompt, schedule
from tatizen_cases import CONFIGS, build, config, delta, parallel, random_weights

FAMILY = next(f for f in FAMILIES if f.name == "tatizen")
TARGETS = [pytest.param(("cpu", torch.float32), id="cpu"), pytest.param(("cuda", torch.float32), id="cuda-f32", marks=pytest.mark.gpu),
           pytest.param(("cuda", torch.bfloat16), id="cuda-bf16", marks=pytest.mark.gpu)]


@pytest.fixture(params=TARGETS)
def target(request):
    return request.param


def tol(target, f32=2e-5, b16=1.5e-2):
    return f32 if target[1] == torch.float32 else b16


# --------------------------------------------------------------------------- mechanisms alone
ATTENTION = [(6, 2, 64, 64), (4, 4, 32, 48), (8, 1, 128, 128), (12, 2, 96, 40), (2, 2, 256, 256), (20, 1, 16, 24), (3, 1, 17, 33), (4, 2, 64, 128),
             (16, 2, 128, 128), (10, 1, 64, 64)]


@pytest.mark.parametrize("heads", ATTENTION, ids=str)
@pytest.mark.parametrize("page", [16, 64])
def test_attention(target, heads, page):
    dev, dt = target
    H, G, D, E = heads
    g = torch.Generator().manual_seed(H * D + E)
    lengths = {0: 150, 1: 1, 2: 77}
    q, k, v = ({s: bf16(torch.randn(n, hh, d, generator=g)) for s, n in lengths.items()} for hh, d in ((H, D), (G, D), (G, E)))
    gq, gk = bf16(1 + 0.2 * torch.randn(D, generator=g)), bf16(1 + 0.2 * torch.randn(D, generator=g))
    eps, scale = 1e-3, 1.7 * D ** -0.5
    want = {s: oracle.causal_attention(oracle.rms(q[s].double(), gq.double(), eps), oracle.rms(k[s].double(), gk.double(), eps), v[s].double(), scale)
            for s in lengths}
    pool = Paged(page, device=dev)
    kc = torch.zeros(96, page, G, D, dtype=dt, device=dev)
    vc = torch.zeros(96, page, G, E, dtype=dt, device=dev)
    for step in schedule(lengths, random.Random(1)):
        meta = pool.step({s: n for s, (_, n) in step.items()})
        cut = lambda x: torch.cat([x[s][a:a + n].flatten(1) for s, (a, n) in step.items()]).to(dev, dt)  # noqa: E731
        rows = torch.cat([cut(q), cut(k), cut(v)], 1)
        pad = torch.zeros(rows.shape[0], -rows.shape[1] % 8, dtype=dt, device=dev)
        rows = torch.cat([rows, pad], 1)
        qq = ops.qk_norm_append(rows[:, :H * D], rows[:, H * D:(H + G) * D], rows[:, (H + G) * D:(H + G) * D + G * E], H, G, D, E, gq.to(dev, dt),
                                gk.to(dev, dt), meta, kc, vc, eps)
        out = ops.rows_buffer(rows.shape[0], H * E + 24, rows)
        out.fill_(7.0)
        ops.attention_exact(qq, kc, vc, meta, scale, out=out[:, :H * E])
        ref = torch.cat([want[s][a:a + n].flatten(1) for s, (a, n) in step.items()])
        assert error(out[:, :H * E], ref) < tol(target, 2e-5, 2e-2)
        assert bool((out[:, H * E:] == 7.0).all())              # the neighbouring columns are another branch's


@pytest.mark.parametrize("heads", [(4, 2, 64, 64), (2, 1, 128, 128), (4, 1, 40, 24)], ids=str)
@pytest.mark.parametrize("decoded", [False, True])
def test_attention_finds_one_far_key(target, heads, decoded):
    """One key stands out for the last query: its value must come back whole, wherever the key lies (first token, page borders, the token
    itself), in a prompt and in decoding; a key one position later than the query must not be seen."""
    dev, dt = target
    H, G, D, E = heads
    page, T = 64, 400
    g = torch.Generator().manual_seed(5)
    v = bf16(torch.randn(T + 1, G, E, generator=g))
    for j in (0, 1, 15, 16, 63, 64, 65, 127, 128, 200, 255, 256, 383, 384, T - 2, T - 1, T):
        k = bf16(0.05 * torch.randn(T + 1, G, D, generator=g))
        q = bf16(0.05 * torch.randn(T + 1, H, D, generator=g))
        k[j] = bf16(torch.randn(G, D, generator=g))
        q[T - 1] = 8.0 * k[j].repeat_interleave(H // G, 0)
        want = oracle.causal_attention(q[:T].double(), k[:T].double(), v[:T].double(), 1.0)[T - 1]
        if j < T:
            assert (want - v[j].double().repeat_interleave(H // G, 0)).abs().max() < 0.05       # the case shows what it should
        pool = Paged(page, 16, device=dev, seed=j)
        meta = pool.step({0: T - 1 if decoded else T})
        kc, vc = (torch.full((16, page, G, d), 0.25, dtype=dt, device=dev) for d in (D, E))
        slots = lambda m: m.slot_mapping  # noqa: E731
        if decoded:
            ops.ref.kv_append(k[:T - 1].to(dev, dt), v[:T - 1].to(dev, dt), kc, vc, slots(meta))
            meta = pool.step({0: 1})
            ops.ref.kv_append(k[T - 1:T].to(dev, dt), v[T - 1:T].to(dev, dt), kc, vc, slots(meta))
            qq = q[T - 1:T]
        else:
            ops.ref.kv_append(k[:T].to(dev, dt), v[:T].to(dev, dt), kc, vc, slots(meta))
            qq = q[:T]
        nxt = pool.step({0: 1})                                  # the key after the query, already in the pages
        ops.ref.kv_append(k[T:].to(dev, dt), v[T:].to(dev, dt), kc, vc, slots(nxt))
        out = ops.attention_exact(qq.contiguous().to(dev, dt), kc, vc, meta, 1.0).view(-1, H, E)[-1]
        assert error(out, want) < tol(target, 2e-5, 2e-2), j


LINEAR = [(2, 32, 64), (3, 48, 40), (1, 128, 64), (2, 200, 24), (2, 20, 17), (2, 256, 8), (1, 9, 130)]


@pytest.mark.parametrize("shape", LINEAR, ids=str)
@pytest.mark.parametrize("tau", [1.0, 12.0])
def test_decayed_linear_attention(target, shape, tau):
    dev, dt = target
    H, D, E = shape
    rank, eps = 11, 1e-4
    g = torch.Generator().manual_seed(D + E)
    lengths = {0: 90, 1: 33, 2: 1, 3: 9}
    sizes = [H * D, H * D, H * E, H * E, rank]
    width = sum(sizes)
    x = {s: bf16(torch.randn(n, width, generator=g)) for s, n in lengths.items()}
    a2, b2, gain = bf16(torch.randn(H * D, rank, generator=g)), bf16(2 * torch.randn(H * D, generator=g)), bf16(1 + 0.2 * torch.randn(E, generator=g))
    b2[0] = -60.0                                                # a channel that forgets at once
    want = {}
    for s, n in lengths.items():
        q, k, v, gate, low = x[s].double().split(sizes, 1)
        alpha = oracle.channel_decay(low, torch.eye(rank, dtype=torch.float64), a2.double(), b2.double(), tau).view(n, H, D)
        o = oracle.decayed_linear_attention(q.view(n, H, D) * D ** -0.5, k.view(n, H, D), v.view(n, H, E), alpha)
        want[s] = oracle.rms(o, gain.double(), eps).reshape(n, H * E) * oracle.silu(gate) * 0.37
    pool = Paged(device=dev)
    state = torch.full((6, H, E, (D + 3) // 4 * 4), 3.0, dtype=torch.float32, device=dev)      # what an earlier user of the slot left
    for step in schedule(lengths, random.Random(2)):
        meta = pool.step({s: n for s, (_, n) in step.items()})
        rows = torch.cat([x[s][a:a + n] for s, (a, n) in step.items()])
        rows = torch.cat([rows, torch.zeros(rows.shape[0], -width % 8)], 1).to(dev, dt)
        q, k, v, gate, low = rows[:, :width].split(sizes, 1)
        out = ops.rows_buffer(rows.shape[0], H * E, rows)
        ops.decayed_linear_attention(q, k, v, gate, low, a2.to(dev, dt), b2.to(dev, dt), 1.0 / tau, gain.to(dev, dt), state, meta, H, D, E, eps, 0.37, out)
        assert error(out, torch.cat([want[s][a:a + n] for s, (a, n) in step.items()])) < tol(target, 5e-5, 1e-2)


DELTA = [(4, 2, 64, 48, 4), (3, 3, 48, 40, 1), (6, 2, 128, 128, 3), (2, 1, 20, 17, 5), (2, 2, 200, 16, 2), (5, 1, 32, 70, 9)]


@pytest.mark.parametrize("shape", DELTA, ids=str)
def test_gated_delta_attention(target, shape):
    dev, dt = target
    H, K, D, E, taps = shape
    eps = 1e-4
    g = torch.Generator().manual_seed(D * E)
    lengths = {0: 90, 1: 33, 2: 1, 3: 9}
    C = 2 * K * D + H * E
    pad = lambda n: (n + 7) // 8 * 8  # noqa: E731
    at = [0, pad(C), pad(C) + pad(H * E), pad(C) + pad(H * E) + pad(H)]
    width = at[3] + pad(H)
    x = {s: bf16(torch.randn(n, width, generator=g)) for s, n in lengths.items()}
    w, gain = bf16(torch.randn(C, taps, generator=g) * taps ** -0.5), bf16(1 + 0.2 * torch.randn(E, generator=g))
    a_log, dt_bias = torch.randn(H, generator=g), torch.randn(H, generator=g)
    a_log[0] = 5.0                                               # a head that forgets at once
    want = {}
    for s, n in lengths.items():
        xs = x[s].double()
        y = oracle.silu(oracle.causal_conv(xs[:, :C], w.double()))
        q, k, v = y[:, :K * D].view(n, K, D), y[:, K * D:2 * K * D].view(n, K, D), y[:, 2 * K * D:].view(n, H, E)
        decay = torch.exp(-torch.exp(a_log.double()) * oracle.softplus(xs[:, at[3]:at[3] + H] + dt_bias.double()))
        o = oracle.gated_delta_rule(oracle.unit(q) * D ** -0.5, oracle.unit(k), v, decay, oracle.sigmoid(xs[:, at[2]:at[2] + H]))
        want[s] = (oracle.rms(o, gain.double(), eps) * oracle.silu(xs[:, at[1]:at[1] + H * E]).view(n, H, E)).reshape(n, H * E) * 1.9
    pool = Paged(device=dev)
    state = torch.full((6, H, E, (D + 3) // 4 * 4), 3.0, dtype=torch.float32, device=dev)
    ring = torch.full((6, taps, C), 2.0, dtype=dt, device=dev)
    for step in schedule(lengths, random.Random(3)):
        meta = pool.step({s: n for s, (_, n) in step.items()})
        rows = torch.cat([x[s][a:a + n] for s, (a, n) in step.items()]).to(dev, dt)
        out = ops.rows_buffer(rows.shape[0], H * E, rows)
        ops.gated_delta_attention(rows[:, :C], w.to(dev, dt), rows[:, at[2]:at[2] + H], rows[:, at[3]:at[3] + H], a_log.to(dev), dt_bias.to(dev),
                                  rows[:, at[1]:at[1] + H * E], gain.to(dev, dt), ring, state, meta, K, H, D, E, eps, 1.9, out)
        assert error(out, torch.cat([want[s][a:a + n] for s, (a, n) in step.items()])) < tol(target, 5e-5, 1e-2)


def test_delta_keeps_one_write_over_a_long_distance(target):
    """No decay, one token with write strength 1, then hundreds of tokens with (almost) none: the value must still be read back by its key."""
    dev, dt = target
    H = K = 1
    D, E, T, taps = 32, 24, 300, 2
    C = 2 * D + E
    g = torch.Generator().manual_seed(0)
    width = C + 8 + 8 + E
    x = bf16(torch.rand(T, width, generator=g) + 0.1)
    x[:, C] = -30.0                                              # beta ~ 0
    x[2, C] = 30.0                                               # the write
    x[:, C + 8] = -40.0                                          # softplus ~ 0: no decay
    x[T - 1, :D] = x[2, D:2 * D]                                 # the last query is the written key
    w = torch.zeros(C, taps)
    w[:, -1] = 1.0
    xs = x.double()
    y = oracle.silu(oracle.causal_conv(xs[:, :C], w.double()))
    v2 = y[2, 2 * D:]
    pool = Paged(device=dev)
    state, ring = torch.zeros(6, H, E, D, device=dev), torch.zeros(6, taps, C, dtype=dt, device=dev)
    for a, n in ((0, 3), (3, 150), (153, 146), (299, 1)):
        meta = pool.step({0: n})
        rows = x[a:a + n].to(dev, dt)
        out = ops.rows_buffer(n, E, rows)
        ops.gated_delta_attention(rows[:, :C], w.to(dev, dt), rows[:, C:C + 1], rows[:, C + 8:C + 9], torch.zeros(1, device=dev),
                                  torch.zeros(1, device=dev), rows[:, C + 16:], torch.ones(E, device=dev, dtype=dt), ring, state, meta, K, H, D, E, 1e-6,
                                  1.0, out)
    want = (oracle.rms(v2, torch.ones(E, dtype=torch.float64), 1e-6) * oracle.silu(xs[T - 1, C + 16:]))[None]
    assert error(out[-1:], want) < tol(target, 2e-3, 2e-2)


@pytest.mark.parametrize("width", [8, 72, 50, 1024, 333])
def test_residual_ops(target, width):
    dev, dt = target
    g = torch.Generator().manual_seed(width)
    a, h = torch.randn(19, width, generator=g), torch.randn(19, width, generator=g)
    w1, w2 = bf16(torch.randn(width, generator=g)), bf16(torch.randn(width, generator=g))
    eps = 0.05
    stream = h.double() + oracle.rms(a.double(), w1.double(), eps)
    for nxt in (None, w2):
        hd = h.clone().to(dev)
        x = ops.post_norm_add(a.to(dev), w1.to(dev, dt), hd, None if nxt is None else nxt.to(dev, dt), eps)
        assert error(hd, stream) < 1e-6
        assert x.dtype == dt and error(x, stream if nxt is None else oracle.rms(stream, w2.double(), eps)) < tol(target, 1e-6, 4e-3)
    assert error(ops.rmsnorm32(h.to(dev), w2.to(dev, dt), eps), oracle.rms(h.double(), w2.double(), eps)) < tol(target, 1e-6, 4e-3)
    table = bf16(torch.randn(33, width, generator=g))
    ids = torch.tensor([0, 32, 7, 7])
    hd, x = ops.embed32(ids.to(dev), table.to(dev, dt))
    assert torch.equal(hd.cpu(), table[ids]) and torch.equal(x.float().cpu(), table[ids])


@pytest.mark.parametrize("mkn", [(1, 72, 50), (1, 256, 512), (7, 50, 33), (130, 64, 200), (70, 333, 65), (300, 128, 96)], ids=str)
def test_linear_any_shape(target, mkn):
    dev, dt = target
    M, K, N = mkn
    g = torch.Generator().manual_seed(M)
    x, w = bf16(torch.randn(M, K, generator=g)), bf16(torch.randn(N, K, generator=g))
    want = x.double() @ w.double().T
    buf = ops.rows_buffer(M, K, torch.empty(0, dtype=dt, device=dev))
    buf.copy_(x)
    assert error(ops.linear_f32(buf, w.to(dev, dt), alpha=-0.3), -0.3 * want) < 2e-6
    assert error(ops.linear(buf, w.to(dev, dt)), want) < tol(target, 2e-6, 4e-3)
    if N % 2 == 0:
        gu = want[:, :N // 2], want[:, N // 2:]
        assert error(ops.linear_glu(buf, w.to(dev, dt), "geglu"), oracle.gelu(gu[0]) * gu[1]) < tol(target, 5e-6, 2e-2)


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


@pytest.mark.parametrize("name", ["mixed", "odd", "tensor", "group"])
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
    assert eng.cache.alloc.free_pages == 8 and eng.cache.alloc.free_slots == 3


@pytest.mark.gpu
@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16], ids=str)
def test_long_prompts(dt):
    """Prompts of more than a thousand tokens, whole and in long portions, time after time over the same pages and slots."""
    target = ("cuda", dt)
    cfg, w, eng = engine(config([parallel((8, 2, 64, 64), (2, 64, 64), ff=192)] * 2, vocab=64, width=128), target, tokens=6400)
    ids = prompt(cfg, 1500, 2)
    logits, _ = oracle.run(cfg, w, ids)
    for sizes in ([1500], [1100, 400], [1500], [1024, 1, 475]):
        s, at, got = eng.open_sequence(), 0, []
        for n in sizes:
            got.append(eng.feed([(s, ids[at:at + n], range(n))]))
            at += n
        assert error(torch.cat(got), logits) < tol(target, **LOGIT_TOL)
        eng.close_sequence(s)


def test_long_decoding(target):
    cfg = config([delta(4, 2, 32, 16, 4, 64), parallel((4, 2, 64, 64), (2, 16, 16), ff=64, tau=20.0)], vocab=97, width=64)
    cfg, w, eng = engine(cfg, target)
    n = 400 if target[0] == "cuda" else 150
    ids = prompt(cfg, n, 1)
    logits, _ = oracle.run(cfg, w, ids)
    s = eng.open_sequence()
    got = [eng.feed([(s, ids[:5], [4])])] + [eng.feed([(s, [t], [0])]) for t in ids[5:]]
    assert error(torch.cat(got), logits[4:]) < tol(target, **LOGIT_TOL)


@pytest.mark.parametrize("name", ["mixed", "tensor"])
def test_greedy_generation_through_the_scheduler(target, name):
    """Prompts of unequal lengths, more of them than state slots, chunked prefill: every generated token is the oracle's arg-max of the
    text before it (within rounding where two logits are as good as equal)."""
    cfg, w, eng = engine(name, target, tokens=768, seqs=3, prefill_chunk=50)
    prompts = [prompt(cfg, n, n) for n in (5, 120, 1, 64, 33)]
    outs = eng.generate(prompts, 12)
    slack = 1e-3 if target[1] == torch.float32 else 0.2
    for p, o in zip(prompts, outs):
        assert len(o) == 12
        logits, _ = oracle.run(cfg, w, p + o)
        at = logits[len(p) - 1:len(p) + 11]
        assert float((at.max(-1).values - at[torch.arange(12), torch.tensor(o)]).max()) <= slack
    assert eng.cache.alloc.free_slots == 3


@pytest.mark.parametrize("graph", [False, True])
def test_fixed_batch_decoder(target, graph):
    from mary_b200.runtime.spec_decode import SpecDecoder
    cfg, w, eng = engine("mixed", target)
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
    with pytest.raises(ValueError, match="recurrent"):
        SpecDecoder(m, PagedKVCache.for_model(m, num_pages=9, page_size=64, device=target[0], num_slots=3), 3, spec_k=1, max_len=192, device=target[0])


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
