"""Configuration, registry, weight loading (folder and pile), state slots, command line and trace replay of the Tatizen decoder, on the host."""
import io
import json
import os
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

from mary_b200.models.registry import family_of, make_engine, open_text_model
from mary_b200.models.tatizen.config import TatizenConfig
from mary_b200.oracle import tatizen as oracle
from mary_b200.runtime.engine import Engine
from mary_b200.runtime.kv_cache import OutOfPages, PageAllocator, PagedKVCache
from paged_cases import TRACE, error, prompt, trace_case, write_folder
from tatizen_cases import CONFIGS, build, config, delta, parallel, random_weights

ROOT = Path(__file__).resolve().parents[1]
DEVICES = [pytest.param("cpu", id="cpu"), pytest.param("cuda", id="cuda", marks=pytest.mark.gpu)]


# --------------------------------------------------------------------------- configuration and registry
@pytest.mark.parametrize("name", list(CONFIGS))
def test_config_round_trip(name):
    c = TatizenConfig.from_json(CONFIGS[name])
    assert c.to_json() == CONFIGS[name]
    assert TatizenConfig.from_json(json.loads(json.dumps(c.to_json()))) == c


@pytest.mark.parametrize("break_it, message", [
    (lambda c: c["layers"][0].update(type="other"), "unknown mixer"),
    (lambda c: c["layers"][0]["mlp"].update(kind="sparse"), "unknown feed-forward"),
    (lambda c: c["layers"][0]["mixer"]["left"].pop("scale"), "missing"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3), "divide"),
])
def test_config_refuses_what_it_does_not_know(break_it, message):
    c = json.loads(json.dumps(CONFIGS["mixed"]))
    break_it(c)
    with pytest.raises(ValueError, match=message):
        TatizenConfig.from_json(c)


def test_head_widths_beyond_the_kernels_are_refused():
    for layer in (delta(2, 2, 257, 16, 2, 32), parallel((2, 1, 64, 513)), parallel((2, 1, 513, 64)), parallel(right=(1, 260, 8))):
        cfg = config([layer], width=16)
        with pytest.raises(ValueError, match="exceed"):
            build(cfg, random_weights(cfg))


def test_registry_chooses_by_configuration():
    assert family_of({"architecture": "Tatizen"}).name == "tatizen"
    assert family_of({"model_type": "qwen3"}).name == "mistral"
    assert family_of({"model_type": "gemma4_text"}).name == "gemma4"
    with pytest.raises(LookupError):
        family_of({"architecture": "Nothing"})


@pytest.mark.parametrize("name", ["mixed", "odd", "recurrent"])
def test_folder_and_pile_give_the_same_model(tmp_path, name, tmp_pile):
    from mary_b200.format.persist import import_model_to_collection
    cfg = CONFIGS[name]
    w = random_weights(cfg, 4)
    write_folder(tmp_path, cfg, w)
    a, fam, tok = open_text_model(tmp_path)
    assert fam.name == "tatizen" and tok is None
    pile, key = tmp_pile
    import_model_to_collection(pile, key, str(tmp_path), name="t", source="test", dtype="bf16")
    b, _, _ = open_text_model(pile.path)
    want = build(cfg, w)
    for m in (a, b):
        for (n, p), (_, q) in zip(want.named_parameters(), m.named_parameters()):
            assert torch.equal(p, q), n


def test_every_tensor_is_used():
    """Changing any tensor of the checkpoint changes the logits."""
    cfg = config([parallel(), delta()], vocab=40, width=40)
    w = random_weights(cfg, 1)
    ids = prompt(cfg, 12)
    fam = family_of(cfg)

    def logits(weights):
        eng = make_engine(build(cfg, weights), fam, 64, 1)
        return eng.feed([(eng.open_sequence(), ids, range(12))])
    base = logits(w)
    for n in w:
        v = dict(w)
        v[n] = w[n] + 0.25 * torch.randn(w[n].shape, generator=torch.Generator().manual_seed(0))
        assert float((logits(v) - base).abs().max()) > 1e-3, n


@pytest.mark.parametrize("mutate", ["scale", "tau", "left_scale", "right_scale", "eps"])
def test_every_constant_is_read_from_the_configuration(mutate):
    cfg = config([parallel(), delta()], vocab=40, width=40)
    w, ids = random_weights(cfg, 1), prompt(cfg, 30)
    c2 = json.loads(json.dumps(cfg))
    m = c2["layers"][0]["mixer"]
    if mutate == "eps":
        c2["norm"]["eps"] = 0.3
    elif mutate == "scale":
        m["left"]["scale"] *= 3
    elif mutate == "tau":
        m["right"]["tau"] *= 3
    else:
        m[mutate] *= -2
    want, base = oracle.run(c2, w, ids)[0], oracle.run(cfg, w, ids)[0]
    assert error(base, want) > 1e-2
    eng = make_engine(build(c2, w), family_of(c2), 64, 1)
    assert error(eng.feed([(eng.open_sequence(), ids, range(30))]), want) < 1e-4


# --------------------------------------------------------------------------- state slots
def test_allocator_hands_out_each_slot_once_and_takes_it_back():
    a = PageAllocator(8, 16, num_slots=2)
    a.extend(1, 20), a.extend(2, 5)
    s = a.slots([1, 2])
    assert sorted(s.tolist()) == [0, 1] and a.free_slots == 0
    with pytest.raises(OutOfPages):
        a.extend(3, 1)
    assert a.free_pages == 5 and a.seq_len(3) == -1                  # nothing was reserved
    a.extend(1, 100 - 20 - 16)                                       # growing needs no further slot
    a.release(1)
    a.extend(3, 1)
    assert a.slots([3])[0] == s[0] and a.free_slots == 0
    with pytest.raises(KeyError):
        a.slots([1])
    with pytest.raises(OutOfPages):
        a.extend(2, 1000)
    assert a.seq_len(2) == 5
    assert PageAllocator(4).slots([0]) is None


def test_scheduler_admits_no_more_requests_than_slots():
    cfg = CONFIGS["recurrent"]
    model = build(cfg, random_weights(cfg))
    cache = PagedKVCache.for_model(model, num_pages=64, page_size=16, num_slots=2)
    eng = Engine(model, cache, max_seqs=16, prefill_chunk=4)
    for n in (9, 3, 5, 7):
        eng.add_request(prompt(cfg, n, n), 3)
    most = 0
    while eng.pending():
        eng.step()
        most = max(most, 2 - cache.alloc.free_slots)
        assert eng.lib.sched_num_running(eng.h) <= 2
    assert most == 2 and cache.alloc.free_slots == 2 and all(len(o) == 3 for o in eng.outputs.values())
    one = np.zeros(1, dtype=np.int32)
    eng.add_request([1, 2], 4)
    eng.step()
    assert eng.lib.sched_set_drafts(eng.h, 5, one.ctypes.data, 1) != 0           # no speculation over a recurrent state


def test_feed_refuses_a_batch_that_does_not_fit_and_keeps_the_state():
    cfg = CONFIGS["mixed"]
    w = random_weights(cfg)
    eng = make_engine(build(cfg, w), family_of(cfg), 128, 2)
    ids = prompt(cfg, 60)
    s, t = eng.open_sequence(), eng.open_sequence()
    eng.feed([(s, ids[:30], [])])
    with pytest.raises(OutOfPages):
        eng.feed([(s, ids[30:40], []), (t, ids * 2, [])])
    assert eng.cache.alloc.seq_len(s) == 30 and eng.cache.alloc.seq_len(t) == -1 and eng.cache.alloc.free_slots == 1
    got = eng.feed([(s, ids[30:], range(30))])
    assert error(got, oracle.run(cfg, w, ids)[0][30:]) < 1e-4
    for bad in ([(s, [], [])], [(s, [1], [1])], [(s, [1], []), (s, [2], [])]):
        with pytest.raises(ValueError):
            eng.feed(bad)


def test_state_is_sized_by_slots_and_never_quantised():
    model = build(CONFIGS["mixed"], random_weights(CONFIGS["mixed"]))
    c = PagedKVCache.for_model(model, num_pages=4, page_size=64, num_slots=3)
    assert [sorted(layer) for layer in c.state] == [["S"], ["S", "conv"], ["S", "conv"], ["S"]] and len(c.k) == 2
    assert all(layer["S"].dtype == torch.float32 and layer["S"].shape[0] == 3 for layer in c.state)
    assert c.k[0].shape[-1] == 32 and c.v[0].shape[-1] == 48 and c.bytes() > c.state_bytes() > 0
    with pytest.raises(ValueError):
        PagedKVCache.for_model(model, num_pages=4, page_size=64, num_slots=0)


# --------------------------------------------------------------------------- command line
@pytest.mark.parametrize("device", DEVICES)
def test_text_gen(tmp_path, capsys, device):
    from mary_b200.cli.text_gen import main
    cfg = CONFIGS["mixed"]
    w = random_weights(cfg, 2)
    write_folder(tmp_path, cfg, w)
    prompts = [prompt(cfg, n, n) for n in (4, 11, 7)]
    args = ["--model", str(tmp_path), "--ids", ";".join(",".join(map(str, p)) for p in prompts), "--max-new", "5", "--device", device, "--dtype", "float32",
            "--max-seqs", "2", "--prefill-chunk", "3"]
    assert main(args) == 0
    outs = [[int(x) for x in line.split(",")] for line in capsys.readouterr().out.splitlines()]
    for p, o in zip(prompts, outs):
        at = oracle.run(cfg, w, p + o)[0][len(p) - 1:len(p) + 4]
        assert float((at.max(-1).values - at[torch.arange(5), torch.tensor(o)]).max()) < 1e-3
    assert main(args + ["--temperature", "0.7", "--top-k", "4", "--seed", "5"]) == 0
    first = capsys.readouterr().out
    assert main(args + ["--temperature", "0.7", "--top-k", "4", "--seed", "5"]) == 0
    assert capsys.readouterr().out == first and len(first.splitlines()) == 3


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_run(tmp_path, monkeypatch, capsys, device, dtype):
    from mary_b200.cli.trace_run import main
    cfg = CONFIGS["mixed"]
    w = random_weights(cfg, 2)
    write_folder(tmp_path, cfg, w)
    lines, want = trace_case(cfg, w, oracle.run)
    out = tmp_path / "out"
    out.mkdir()
    monkeypatch.setattr(sys, "stdin", io.StringIO("\n".join(lines) + "\n"))
    assert main(["--model", str(tmp_path), "--dtype", dtype, "--out", str(out), "--max-tokens", "384", "--device", device]) == 0
    assert capsys.readouterr().out.split("\n")[:-1] == [f"done {s['step']}" for s in TRACE]
    assert sorted(os.listdir(out)) == sorted(f"{s}.f32" for s in want)
    for s, ref in want.items():
        got = np.fromfile(out / f"{s}.f32", dtype="<f4").reshape(-1, cfg["vocab"])
        assert error(got, ref) < (1e-4 if dtype == "float32" else 8e-2)


def test_trace_run_is_a_program(tmp_path):
    cfg = CONFIGS["recurrent"]
    w = random_weights(cfg, 2)
    write_folder(tmp_path, cfg, w)
    p = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "64",
                        "--device", "cpu"], input=json.dumps({"step": 4, "entries": [{"id": "x", "tokens": [1, 2], "want": [1]}], "end": ["x"]}) + "\n",
                       capture_output=True, text=True, timeout=120)
    assert p.returncode == 0 and p.stdout.strip() == "done 4"
    assert error(np.fromfile(tmp_path / "4.f32", dtype="<f4"), oracle.run(cfg, w, [1, 2])[0][1]) < 1e-4


def test_trace_run_refuses_32_bits_where_a_family_has_none(tmp_path):
    from mary_b200.cli.trace_run import main
    (tmp_path / "config.json").write_text(json.dumps({"model_type": "mistral"}))
    assert main(["--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "64"]) == 3


# --------------------------------------------------------------------------- partial kernel library
def test_partial_library_names_existing_sources():
    from mary_b200 import _build
    for fam in ("tatizen",):
        need = next(f for f in __import__("mary_b200.models.registry", fromlist=["FAMILIES"]).FAMILIES if f.name == fam).kernels
        assert {s.stem for s, _, _ in _build._kernel_sources(need)} == set(need)
    with pytest.raises(ValueError):
        _build._kernel_sources(("no_such_file",))
