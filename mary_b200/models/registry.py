"""Which text decoder a ``config.json`` describes, and how it is built, filled and served.

``open_text_model(path)`` takes a checkpoint folder (``config.json`` + safetensors) or a pile; the family is chosen by the configuration
alone.  ``make_engine`` puts a model behind the serving engine with the cache (pages, and state slots where it has recurrent layers) that
the model asks for."""
from __future__ import annotations

import json
from dataclasses import dataclass
from pathlib import Path
from typing import Callable

import torch

from ..nn.weight_loader import WeightLoader

_DENSE_KERNELS = ("runtime_support", "gemm_bf16", "gemm_simt", "attention_fa", "attention_decode", "attention_simt", "elementwise", "select", "layer_step")


@dataclass(frozen=True)
class Family:
    name: str
    matches: Callable[[dict], bool]
    load: Callable                      # (config dict, WeightLoader, device, dtype) -> model
    page_size: int = 16
    kernels: tuple | None = None        # kernel sources the decoder needs (None: the full library)
    f32_on_gpu: bool = False            # whether the CUDA path exists in 32 bits


def _load_tatizen(d, loader, device, dtype):
    from .tatizen.config import TatizenConfig
    from .tatizen.model import TatizenModel, decay_ranks, load_into
    cfg = TatizenConfig.from_json(d)
    model = TatizenModel(cfg, decay_ranks(cfg, loader.shape), dtype=dtype, device=device)
    load_into(model, loader)
    return model


def _load_rokarax(d, loader, device, dtype):
    from .rokarax.config import RokaraxConfig
    from .rokarax.model import RokaraxModel, bias_rows, load_into
    cfg = RokaraxConfig.from_json(d)
    model = RokaraxModel(cfg, bias_rows(cfg, loader.shape), dtype=dtype, device=device)
    load_into(model, loader)
    return model


def _load_nipurax(d, loader, device, dtype):
    from .nipurax.config import NipuraxConfig
    from .nipurax.model import NipuraxModel, load_into
    model = NipuraxModel(NipuraxConfig.from_json(d), loader.shape("bigram")[0], dtype=dtype, device=device)
    load_into(model, loader)
    return model


def _load_kivezen(d, loader, device, dtype):
    from .kivezen.config import KivezenConfig
    from .kivezen.model import KivezenModel, load_into
    model = KivezenModel(KivezenConfig.from_json(d), dtype=dtype, device=device)
    load_into(model, loader)
    return model


def _load_mistral(d, loader, device, dtype):
    from .mistral.model import MistralConfig, MistralModel, load_into
    model = MistralModel(MistralConfig.from_hf(d), dtype=dtype, device=device)
    load_into(model, loader)
    return model


def _load_gemma4(d, loader, device, dtype):
    from .gemma4 import Gemma4Model, Gemma4TextConfig
    from .gemma4.weights import load_into
    model = Gemma4Model(Gemma4TextConfig.from_json(d), dtype=dtype, device=device)
    load_into(model, loader)
    return model


FAMILIES = [
    Family("tatizen", lambda d: d.get("architecture") == "Tatizen", _load_tatizen, page_size=64, f32_on_gpu=True,
           kernels=_DENSE_KERNELS + ("attention_general", "residual32", "linear_attention", "recurrent_scan")),
    Family("rokarax", lambda d: d.get("architecture") == "Rokarax", _load_rokarax, page_size=64, f32_on_gpu=True,
           kernels=_DENSE_KERNELS + ("attention_general", "attention_mla", "residual32", "linear_attention", "recurrent_scan", "latent", "state_space", "ssd_chunk")),
    Family("nipurax", lambda d: d.get("architecture") == "Nipurax", _load_nipurax, page_size=64, f32_on_gpu=True,
           kernels=_DENSE_KERNELS + ("attention_general", "attention_gqa_tc", "residual32", "parallel_stream", "moe", "expert_step")),
    Family("kivezen", lambda d: d.get("architecture") == "Kivezen", _load_kivezen, page_size=64, f32_on_gpu=True,
           kernels=_DENSE_KERNELS + ("attention_general", "attention_gqa_tc", "residual32", "linear_attention", "recurrent_scan", "state_space", "ssd_chunk",
                                     "parallel_stream", "hyper_streams", "moe", "expert_step")),
    Family("gemma4", lambda d: str(d.get("model_type", "")).startswith("gemma4"), _load_gemma4),
    Family("mistral", lambda d: d.get("model_type") in ("mistral", "ministral", "qwen3", "mistral3"), _load_mistral),
]


def family_of(config: dict) -> Family:
    for f in FAMILIES:
        if f.matches(config):
            return f
    raise LookupError(f"no text decoder for architecture {config.get('architecture')!r}, model_type {config.get('model_type')!r}; known: "
                      f"{[f.name for f in FAMILIES]}")


def _read_folder(path: Path):
    files = sorted(path.glob("*.safetensors"))
    if not files:
        raise FileNotFoundError(f"{path}: no *.safetensors beside config.json")
    config = json.loads((path / "config.json").read_text())
    tok = None
    if (path / "tokenizer.json").is_file():
        from tokenizers import Tokenizer
        tok = Tokenizer.from_file(str(path / "tokenizer.json"))
    return config, WeightLoader.from_files(files), tok


def _read_pile(path: Path):
    from ..format.persist import load_config, read_model_pile
    from ..format.selection import SelectedModelIndex
    from ..format.tokenizer import build_tokenizer
    from ..pile import Pile
    pile = Pile.open(str(path), create=False)
    facts = read_model_pile(pile)
    index = SelectedModelIndex.from_snapshot(pile, facts)
    try:
        tok = build_tokenizer(pile, facts)
    except LookupError:
        tok = None
    loader = WeightLoader.from_pile(index)
    loader.pile = pile                      # leaf views alias the mapping
    return load_config(pile, facts, index.roots[0]), loader, tok


def read_config(path) -> dict:
    path = Path(path)
    return json.loads((path / "config.json").read_text()) if path.is_dir() else _read_pile(path)[0]


def open_text_model(path, device="cpu", dtype=torch.float32, compile_missing: bool = False):
    """``(model, family, tokenizer or None)``.  ``compile_missing``: compile the family's kernels when the checkout has no kernel library."""
    path = Path(path)
    config, loader, tok = _read_folder(path) if path.is_dir() else _read_pile(path)
    fam = family_of(config)
    if torch.device(device).type == "cuda":
        if dtype == torch.float32 and not fam.f32_on_gpu:
            raise TypeError(f"{fam.name} has no 32-bit CUDA path")
        if compile_missing and fam.kernels is not None:
            from .. import _native
            _native.require_kernels(fam.kernels)
    model = fam.load(config, loader, device, dtype)
    return model, fam, tok


def make_engine(model, family: Family, pool_tokens: int, max_seqs: int, device="cpu", max_tokens: int = 8192, prefill_chunk: int = 2048, **kw):
    """The serving engine with a pool for ``pool_tokens`` tokens (each sequence's count rounded up to whole pages) and ``max_seqs`` live
    sequences."""
    from ..runtime.engine import Engine
    from ..runtime.kv_cache import PagedKVCache
    pages = (pool_tokens + family.page_size - 1) // family.page_size
    cache = PagedKVCache.for_model(model, num_pages=pages, page_size=family.page_size, device=device, num_slots=max_seqs)
    return Engine(model, cache, max_tokens=max(max_tokens, max_seqs), max_seqs=max_seqs, prefill_chunk=prefill_chunk, device=device, **kw)
