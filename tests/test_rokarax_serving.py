"""Configuration, registry, weight loading (folder and pile), cache rows and state slots, command line and trace replay of the Rokarax decoder."""
import io
import json
import os
import sys

import numpy as np
import pytest
import torch

from mary_b200.models.registry import family_of, make_engine, open_text_model
from mary_b200.models.rokarax.config import RokaraxConfig
from mary_b200.oracle import rokarax as oracle
from mary_b200.runtime.kv_cache import OutOfPages, PagedKVCache
from paged_cases import TRACE, error, prompt, trace_case, write_folder
from rokarax_cases import CONFIGS, attention, build, config, latent, mamba, random_weights

DEVICES = [pytest.param("cpu", id="cpu"), pytest.param("cuda", id="cuda", marks=pytest.mark.gpu)]


def copy(cfg):
    return json.loads(json.dumps(cfg))


# --------------------------------------------------------------------------- configuration and registry
@pytest.mark.parametrize("name", list(CONFIGS))
def test_config_round_trip(name):
    c = RokaraxConfig.from_json(CONFIGS[name])
    assert c.to_json() == CONFIGS[name]
    assert RokaraxConfig.from_json(copy(c.to_json())) == c


@pytest.mark.parametrize("break_it, message", [
    (lambda c: c["layers"][0].update(type="other"), "unknown mixer"),
    (lambda c: c["layers"][0]["mlp"].update(kind="sparse"), "unknown feed-forward"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "missing"),
    (lambda c: c["layers"][0]["mixer"].pop("mask"), "missing"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "window"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "divide"),
    (lambda c: c["layers"][1]["mixer"].update(groups=4), "divide"),
    (lambda c: c["layers"][1]["mixer"].update(norm_groups=7), "divide"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=4), "rotated"),
    (lambda c: c["layers"][2]["mixer"]["rot"]["scaling"].pop("slow"), "missing"),
    (lambda c: c["layers"][4]["mixer"].update(kv_from=1), "no keys"),
    (lambda c: c["layers"][4]["mixer"].update(kv_from=4), "no keys"),
    (lambda c: c["layers"][4]["mixer"].update(kv_from=-1), "no keys"),
    (lambda c: c["layers"][4]["mixer"].update(dim=48), "differ"),
])
def test_config_refuses_what_it_does_not_know(break_it, message):
    c = copy(CONFIGS["mixed"])
    break_it(c)
    with pytest.raises(ValueError, match=message):
        RokaraxConfig.from_json(c)


def test_absent_and_null_entries_mean_the_same():
    c = copy(CONFIGS["mixed"])
    c["layers"][0]["mixer"]["kv_from"] = None
    c["layers"][5]["mixer"]["rot"]["scaling"] = None
    del c["layers"][3]["mlp"]
    assert RokaraxConfig.from_json(c) == RokaraxConfig.from_json(CONFIGS["mixed"])


def test_widths_beyond_the_kernels_are_refused():
    for layer in (mamba(2, 16, 257, 1, 2, 1), attention(2, 1, 641, 16), attention(2, 1, 16, 513), latent(kv_rank=513), latent(kv_rank=512, rot=130)):
        cfg = config([layer], width=16)
        with pytest.raises(ValueError, match="exceed"):
            build(cfg, random_weights(cfg))


def test_registry_chooses_by_configuration():
    assert family_of({"architecture": "Rokarax"}).name == "rokarax"
    assert family_of({"architecture": "Tatizen"}).name == "tatizen"


@pytest.mark.parametrize("name", ["mixed", "odd", "pages"])
def test_folder_and_pile_give_the_same_model(tmp_path, name, tmp_pile):
    from mary_b200.format.persist import import_model_to_collection
    cfg = CONFIGS[name]
    w = random_weights(cfg, 4)
    write_folder(tmp_path, cfg, w)
    a, fam, tok = open_text_model(tmp_path)
    assert fam.name == "rokarax" and tok is None
    pile, key = tmp_pile
    import_model_to_collection(pile, key, str(tmp_path), name="t", source="test", dtype="bf16")
    b, _, _ = open_text_model(pile.path)
    want = build(cfg, w)
    for m in (a, b):
        for (n, p), (_, q) in zip([*want.named_parameters(), *want.named_buffers()], [*m.named_parameters(), *m.named_buffers()]):
            assert torch.equal(p, q), n


SMALL = [attention(), mamba(), latent(), attention(kv_from=0, window=20, far=30.0)]


def logits(cfg, w, ids):
    eng = make_engine(build(cfg, w), family_of(cfg), 128, 1)
    return eng.feed([(eng.open_sequence(), ids, range(len(ids)))])


def test_every_tensor_is_used():
    """Changing any tensor of the checkpoint changes the logits."""
    cfg = config(SMALL, vocab=40, width=40)
    w = random_weights(cfg, 1)
    ids = prompt(cfg, 60)
    base = logits(cfg, w, ids)
    for n in w:
        v = dict(w)
        v[n] = w[n] + 0.25 * torch.randn(w[n].shape, generator=torch.Generator().manual_seed(0))
        assert float((logits(cfg, v, ids) - base).abs().max()) > 1e-3, n


@pytest.mark.parametrize("path, value", [
    (("norm", "eps"), 0.3), (("embedding", "scale"), 2.0), ((0, "scale"), 0.9), ((0, "bias_max"), 9.0), ((0, "mask", "size"), 7), ((3, "mask", "size"), 45),
    ((3, "scale"), 0.8), ((3, "bias_max"), 90.0), ((1, "norm_groups"), 3), ((1, "groups"), None), ((2, "scale"), 0.9), ((2, "mask", "size"), 4),
    ((2, "rot", "base"), 20.0), ((2, "rot", "scaling", "factor"), 9.0), ((2, "rot", "scaling", "original"), 500.0), ((2, "rot", "scaling", "fast"), 0.5),
    ((2, "rot", "scaling", "slow"), 0.1), ((2, "rot", "scaling"), None)], ids=str)
def test_every_constant_is_read_from_the_configuration(path, value):
    cfg = config(SMALL, vocab=40, width=40)
    w, ids = random_weights(cfg, 1), prompt(cfg, 60)
    c2 = copy(cfg)
    at = c2 if isinstance(path[0], str) else c2["layers"][path[0]]["mixer"]
    for k in path[:-1]:
        at = at[k] if isinstance(k, str) else at
    if path[-1] == "groups":                        # the same number of channels, grouped differently
        at.update(groups=6, state=at["state"] // 2)
    else:
        at[path[-1]] = value
    want, base = oracle.run(c2, w, ids)[0], oracle.run(cfg, w, ids)[0]
    assert error(base, want) > 1e-3
    assert error(logits(c2, w, ids), want) < 1e-4


# --------------------------------------------------------------------------- cache rows and state slots
def test_cache_holds_rows_of_own_keys_only():
    """Shared keys take no pages of their own, a latent layer stores one row per token and no values, slots exist for state layers alone."""
    m = build(CONFIGS["mixed"], random_weights(CONFIGS["mixed"]))
    c = PagedKVCache.for_model(m, num_pages=4, page_size=64, num_slots=3)
    assert [tuple(t.shape[2:]) for t in c.k] == [(2, 24), (1, 48), (1, 48)] and c.v[0].shape[-1] == 40 and c.v[1] is c.k[1]
    assert [layer.mixer.kv_index for layer in m.layers] == [0, -1, 1, -1, 0, 2]
    assert [sorted(layer) for layer in c.state] == [["S", "conv"]] * 2 and all(s["S"].dtype == torch.float32 for s in c.state)
    rows = 4 * 64 * 4 * (2 * (24 + 40) + 48 + 48)
    assert c.bytes() == rows + c.state_bytes()
    m = build(CONFIGS["pages"], random_weights(CONFIGS["pages"]))
    c = PagedKVCache.for_model(m, num_pages=4, page_size=64, num_slots=3)
    assert c.num_slots == 0 and not c.state and c.alloc.slots([0]) is None


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
    assert error(eng.feed([(s, ids[30:], range(30))]), oracle.run(cfg, w, ids)[0][30:]) < 1e-4


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
@pytest.mark.parametrize("name", ["mixed", "pages"])
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
    for s, ref in want.items():
        got = np.fromfile(out / f"{s}.f32", dtype="<f4").reshape(-1, cfg["vocab"])
        assert error(got, ref) < (1e-4 if dtype == "float32" else 8e-2)


def test_partial_library_names_existing_sources():
    from mary_b200 import _build
    need = family_of({"architecture": "Rokarax"}).kernels
    assert {s.stem for s, _, _ in _build._kernel_sources(need)} == set(need)
