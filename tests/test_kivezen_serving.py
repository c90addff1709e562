"""Configuration, registry, weight loading (folder and pile), cache pages and states per pass, state slots, command line and trace replay of the Kivezen
decoder."""
import io
import json
import os
import sys

import numpy as np
import pytest
import torch

from mary_b200.models.kivezen.config import KivezenConfig
from mary_b200.models.registry import family_of, make_engine, open_text_model
from mary_b200.oracle import kivezen as oracle
from mary_b200.runtime.kv_cache import OutOfPages, PagedKVCache
from kivezen_cases import CONFIGS, attention, build, config, dense, lightning, moe, random_weights
from paged_cases import TRACE, error, prompt, trace_case, write_folder

DEVICES = [pytest.param("cpu", id="cpu"), pytest.param("cuda", id="cuda", marks=pytest.mark.gpu)]


def copy(cfg):
    return json.loads(json.dumps(cfg))


# --------------------------------------------------------------------------- configuration and registry
@pytest.mark.parametrize("name", list(CONFIGS))
def test_config_round_trip(name):
    c = KivezenConfig.from_json(CONFIGS[name])
    assert c.to_json() == CONFIGS[name]
    assert KivezenConfig.from_json(copy(c.to_json())) == c


@pytest.mark.parametrize("break_it, message", [
    (lambda c: c["layers"][0].update(type="other"), "unknown mixer"),
    (lambda c: c["layers"][0]["mlp"].update(kind="other"), "unknown feed-forward"),
    (lambda c: c["layers"][0]["mlp"].pop("ff"), "missing"),
    (lambda c: c["layers"][0]["mixer"].pop("decay"), "missing"),
    (lambda c: c["layers"][0]["mixer"].update(decay=[0.5, 0.5]), "decays"),
    (lambda c: c["layers"][0]["mixer"].update(decay=[0.5, 0.5, 1.5]), "decays"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "missing"),
    (lambda c: c["layers"][1]["mixer"].update(dim=24.5), "whole"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "divide"),
    (lambda c: c["layers"][1]["mixer"].pop("rot"), "missing"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=26), "rotated"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), "rotated"),
    (lambda c: c["layers"][1]["mixer"].update(vdim=7), "rotated"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("slow"), "missing"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=6), "experts"),
    (lambda c: c.pop("norm"), "missing"),
    (lambda c: c.update(streams=17), "streams"),
    (lambda c: c.update(streams=0), "streams"),
    (lambda c: c["loop"].update(stop=6), "layers"),
    (lambda c: c["loop"].update(start=4), "layers"),
    (lambda c: c["loop"].update(times=0), "times"),
])
def test_config_refuses_what_it_does_not_know(break_it, message):
    c = copy(CONFIGS["mixed"])
    break_it(c)
    with pytest.raises(ValueError, match=message):
        KivezenConfig.from_json(c)


def test_absent_and_null_entries_mean_the_same():
    c = copy(CONFIGS["wide"])
    c["loop"] = c["streams"] = None
    c["layers"][3]["mixer"]["rot"]["scaling"] = None
    d = copy(CONFIGS["wide"])
    del d["layers"][0]["mlp"], d["streams"]
    d["layers"][3]["mixer"]["rot"].pop("scaling", None)
    assert KivezenConfig.from_json(c) == KivezenConfig.from_json(d)


def test_order_of_runs():
    assert KivezenConfig.from_json(CONFIGS["mixed"]).runs() == [0, 1, 2, 3, 1, 2, 3, 1, 2, 3, 4]
    for cfg in CONFIGS.values():
        assert KivezenConfig.from_json(cfg).runs() == oracle.layer_runs(cfg)


def test_sizes_beyond_the_kernels_are_refused():
    for layer, message in ((attention(2, 1, 641, 16, mlp=None), "640"), (attention(2, 1, 16, 514, mlp=None), "512"), (lightning((0.5,), 257), "256"),
                           (attention(mlp=moe(513, 2)), "router"), (attention(mlp=moe(40, 33)), "router")):
        cfg = config([layer], width=8)
        with pytest.raises(ValueError, match=message):
            build(cfg, random_weights(cfg))


def test_registry_chooses_by_configuration():
    assert family_of({"architecture": "Kivezen"}).name == "kivezen"
    assert family_of({"architecture": "Nipurax"}).name == "nipurax"


@pytest.mark.parametrize("name", ["mixed", "odd", "plain"])
def test_folder_and_pile_give_the_same_model(tmp_path, name, tmp_pile):
    from mary_b200.format.persist import import_model_to_collection
    cfg = CONFIGS[name]
    w = random_weights(cfg, 4)
    write_folder(tmp_path, cfg, w)
    a, fam, tok = open_text_model(tmp_path)
    assert fam.name == "kivezen" and tok is None
    pile, key = tmp_pile
    import_model_to_collection(pile, key, str(tmp_path), name="t", source="test", dtype="bf16")
    b, _, _ = open_text_model(pile.path)
    want = build(cfg, w)
    for m in (a, b):
        for (n, p), (_, q) in zip([*want.named_parameters(), *want.named_buffers()], [*m.named_parameters(), *m.named_buffers()]):
            assert torch.equal(p, q), n


SMALL = [attention(mlp=moe(4, 3)), lightning(), attention(mlp=None)]
SMALL_KW = dict(vocab=40, width=40, loop=(1, 2, 2))


def logits(cfg, w, ids):
    eng = make_engine(build(cfg, w), family_of(cfg), 128, 1)
    return eng.feed([(eng.open_sequence(), ids, range(len(ids)))])


def test_every_tensor_is_used():
    """Changing any tensor of the checkpoint changes the logits; the first sublayer's read weights only scale what its norm divides out, unless their sum
    changes its sign."""
    cfg = config(SMALL, **SMALL_KW)
    w = random_weights(cfg, 1)
    ids = prompt(cfg, 60)
    base = logits(cfg, w, ids)
    for n in w:
        v = dict(w)
        v[n] = -w[n] if n == "l0.hc1.in" else w[n] + 0.25 * torch.randn(w[n].shape, generator=torch.Generator().manual_seed(0))
        assert float((logits(cfg, v, ids) - base).abs().max()) > 1e-3, n


@pytest.mark.parametrize("path, value", [
    (("norm", "eps"), 0.3), (("logit_softcap",), 2.0), (("logit_softcap",), None), (("streams",), None), (("loop", "start"), 0), (("loop", "stop"), 3), (("loop", "times"), 3),
    (("loop",), None), ((0, "scale"), 0.9), ((0, "softcap"), 1.0), ((0, "rot", "base"), 20.0), ((0, "rot", "dims"), 6), ((0, "rot", "scaling", "factor"), 9.0),
    ((0, "rot", "scaling", "original"), 400.0), ((0, "rot", "scaling", "fast"), 2.0), ((0, "rot", "scaling", "slow"), 2.5), ((0, "rot", "scaling"), None),
    ((1, "decay"), [0.9, 0.4, 0.7]), ((0, "mlp", "router", "top"), 2), ((0, "mlp", "expert", "limit"), 0.3), ((0, "mlp", "shared", "limit"), 0.3),
    ((0, "mlp", "shared"), None), ((0, "mlp"), None)], ids=str)
def test_every_constant_is_read_from_the_configuration(path, value):
    cfg = config(SMALL, **SMALL_KW)
    w, ids = random_weights(cfg, 1), prompt(cfg, 60)
    c2 = copy(cfg)
    at = c2
    if not isinstance(path[0], str):
        at = c2["layers"][path[0]]
        at, path = (at, path[1:]) if path[1] == "mlp" else (at["mixer"], path[1:])
    for k in path[:-1]:
        at = at[k]
    at[path[-1]] = value
    want, base = oracle.run(c2, w, ids)[0], oracle.run(cfg, w, ids)[0]
    assert error(base, want) > 1e-3
    assert error(logits(c2, w, ids), want) < 2e-4


# --------------------------------------------------------------------------- cache pages and state slots
def test_every_pass_has_pages_or_a_state_of_its_own():
    m = build(CONFIGS["mixed"], random_weights(CONFIGS["mixed"]))
    c = PagedKVCache.for_model(m, num_pages=4, page_size=64, num_slots=2)
    assert [(tuple(k.shape[2:]), tuple(v.shape[2:])) for k, v in zip(c.k, c.v)] == [((2, 24), (2, 40))] * 7
    assert [[(n, tuple(t.shape), t.dtype) for n, t in layer.items()] for layer in c.state] == [[("S", (2, 3, 28, 20), torch.float32)]] * 4
    assert len(m.layers) == 5 and m.places == [0, 0, 1, 1, 2, 3, 2, 4, 5, 3, 6]


@pytest.mark.parametrize("layers", [[attention(mlp=dense(8))], [lightning()]], ids=["pages only", "states only"])
def test_one_kind_of_layer_alone(layers):
    cfg = config(layers, vocab=30, width=24)
    w, ids = random_weights(cfg), prompt(cfg, 70)
    assert error(logits(cfg, w, ids), oracle.run(cfg, w, ids)[0]) < 2e-4


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
    assert error(eng.feed([(s, ids[30:], range(30))]), oracle.run(cfg, w, ids)[0][30:]) < 2e-4


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
        assert float((at.max(-1).values - at[torch.arange(5), torch.tensor(o)]).max()) < 2e-3
    assert main(args + ["--temperature", "0.7", "--top-k", "4", "--seed", "5"]) == 0
    first = capsys.readouterr().out
    assert main(args + ["--temperature", "0.7", "--top-k", "4", "--seed", "5"]) == 0
    assert capsys.readouterr().out == first and len(first.splitlines()) == 3


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_trace_run(tmp_path, monkeypatch, capsys, device, dtype, name):
    from mary_b200.cli.trace_run import main
    cfg = CONFIGS[name]
    w = random_weights(cfg, 2)
    write_folder(tmp_path, cfg, w)
    lines, want = trace_case(cfg, w, oracle.run)
    out = tmp_path / "out"
    out.mkdir()
    monkeypatch.setattr(sys, "stdin", io.StringIO("\n".join(lines) + "\n"))
    assert main(["--model", str(tmp_path), "--dtype", dtype, "--out", str(out), "--max-tokens", "384", "--device", device]) == 0
    assert capsys.readouterr().out.split("\n")[:-1] == [f"done {s['step']}" for s in TRACE]
    assert sorted(os.listdir(out)) == sorted(f"{s}.f32" for s in want)
    got = torch.cat([torch.from_numpy(np.fromfile(out / f"{s}.f32", dtype="<f4").reshape(-1, cfg["vocab"])) for s in want])
    ref = torch.cat(list(want.values()))
    off = (got.double() - ref).pow(2).mean(-1).sqrt() / ref.pow(2).mean().sqrt()
    assert float(off.max()) < 2e-4 if dtype == "float32" else float((off > 8e-2).double().mean()) <= 0.25      # 16 bits: close calls of a router


def test_partial_library_names_existing_sources():
    from mary_b200 import _build
    need = family_of({"architecture": "Kivezen"}).kernels
    assert {s.stem for s, _, _ in _build._kernel_sources(need)} == set(need)
