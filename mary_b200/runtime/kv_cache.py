"""Paged KV cache: native page allocator (``_core.so``) + the device tensors that hold the pages.

Pages are 16 tokens by default.  One cache instance serves all layers: ``k[layer]`` / ``v[layer]`` have shape
``[num_pages, page_size, kv_heads, head_dim]``; MLA models use a single latent tensor per layer
(``[num_pages, page_size, kv_lora + rope_dim]``).  A sequence's page list is shared by every layer."""
from __future__ import annotations

import ctypes

import numpy as np
import torch

from .. import _native


def _declare(lib):
    if getattr(lib, "_kv_declared", False):
        return
    c = ctypes
    lib.kv_create.restype = c.c_void_p
    lib.kv_create.argtypes = [c.c_int32, c.c_int32]
    lib.kv_destroy.argtypes = [c.c_void_p]
    lib.kv_free_pages.argtypes = [c.c_void_p]
    lib.kv_peak_used.restype = c.c_int64
    lib.kv_peak_used.argtypes = [c.c_void_p]
    lib.kv_seq_len.restype = c.c_int64
    lib.kv_seq_len.argtypes = [c.c_void_p, c.c_int64]
    lib.kv_extend.restype = c.c_int64
    lib.kv_extend.argtypes = [c.c_void_p, c.c_int64, c.c_int64]
    lib.kv_truncate.restype = c.c_int64
    lib.kv_truncate.argtypes = [c.c_void_p, c.c_int64, c.c_int64]
    lib.kv_release.argtypes = [c.c_void_p, c.c_int64]
    lib.kv_pages.argtypes = [c.c_void_p, c.c_int64, c.c_void_p, c.c_int32]
    lib.kv_set_slots.argtypes = [c.c_void_p, c.c_int32]
    lib.kv_free_slots.argtypes = [c.c_void_p]
    lib.kv_seq_slots.argtypes = [c.c_void_p, c.c_void_p, c.c_int32, c.c_void_p]
    lib.kv_page_table.argtypes = [c.c_void_p, c.c_void_p, c.c_int32, c.c_void_p, c.c_int32, c.c_void_p]
    lib.sched_create.restype = c.c_void_p
    lib.sched_create.argtypes = [c.c_void_p, c.c_int32, c.c_int32, c.c_int32]
    lib.sched_destroy.argtypes = [c.c_void_p]
    lib.sched_add.argtypes = [c.c_void_p, c.c_int64, c.c_void_p, c.c_int32, c.c_int32]
    lib.sched_add.restype = c.c_int32
    lib.sched_num_waiting.argtypes = [c.c_void_p]
    lib.sched_num_running.argtypes = [c.c_void_p]
    lib.sched_set_drafts.argtypes = [c.c_void_p, c.c_int64, c.c_void_p, c.c_int32]
    lib.sched_next.argtypes = [c.c_void_p] + [c.c_void_p] * 9
    lib.sched_commit.argtypes = [c.c_void_p, c.c_int64, c.c_int32, c.c_int32, c.c_int32, c.c_int32]
    lib.sched_is_finished.argtypes = [c.c_void_p, c.c_int64]
    lib.sched_remove.argtypes = [c.c_void_p, c.c_int64]
    lib._kv_declared = True


class OutOfPages(RuntimeError):
    pass


class PageAllocator:
    """Pages, and for models with recurrent layers one state slot per sequence (``num_slots`` of them): a sequence takes its slot
    when it is created and returns it with its pages."""

    def __init__(self, num_pages: int, page_size: int = 16, num_slots: int = 0):
        self.lib = _native.core()
        _declare(self.lib)
        self.num_pages, self.page_size, self.num_slots = num_pages, page_size, num_slots
        self.h = self.lib.kv_create(num_pages, page_size)
        if num_slots:
            self.lib.kv_set_slots(self.h, num_slots)

    def extend(self, seq: int, tokens: int) -> int:
        n = self.lib.kv_extend(self.h, seq, tokens)
        if n < 0:
            raise OutOfPages(f"sequence {seq}: no room for {tokens} more tokens ({self.free_pages} of {self.num_pages} pages free"
                             + (f", {self.free_slots} of {self.num_slots} state slots free)" if self.num_slots else ")"))
        return n

    def slots(self, seqs):
        """State slots of the sequences as an int32 NumPy array, or ``None`` for an allocator without slots."""
        if not self.num_slots:
            return None
        s = np.asarray(seqs, dtype=np.int64)
        out = np.empty(len(s), dtype=np.int32)
        if self.lib.kv_seq_slots(self.h, s.ctypes.data, len(s), out.ctypes.data):
            raise KeyError(f"unknown sequence among {s.tolist()}")
        return out

    @property
    def free_slots(self) -> int:
        return self.lib.kv_free_slots(self.h)

    def truncate(self, seq: int, new_len: int) -> None:
        if self.lib.kv_truncate(self.h, seq, new_len) < 0:
            raise ValueError(f"cannot truncate sequence {seq} to {new_len}")

    def release(self, seq: int) -> None:
        self.lib.kv_release(self.h, seq)

    def seq_len(self, seq: int) -> int:
        return self.lib.kv_seq_len(self.h, seq)

    @property
    def free_pages(self) -> int:
        return self.lib.kv_free_pages(self.h)

    @property
    def peak_used(self) -> int:
        return self.lib.kv_peak_used(self.h)

    def pages(self, seq: int) -> list[int]:
        buf = np.empty(self.num_pages, dtype=np.int32)
        n = self.lib.kv_pages(self.h, seq, buf.ctypes.data, buf.size)
        if n < 0:
            raise KeyError(seq)
        return buf[:n].tolist()

    def page_table(self, seqs, max_pages: int | None = None):
        """``(table int32[n, max_pages] padded with -1, kv_lens int32[n])`` as NumPy arrays."""
        s = np.asarray(seqs, dtype=np.int64)
        if max_pages is None:
            max_pages = max(1, max((self.seq_len(int(x)) + self.page_size - 1) // self.page_size for x in s))
        table = np.empty((len(s), max_pages), dtype=np.int32)
        lens = np.empty(len(s), dtype=np.int32)
        rc = self.lib.kv_page_table(self.h, s.ctypes.data, len(s), table.ctypes.data, max_pages, lens.ctypes.data)
        if rc != 0:
            raise ValueError("page table: unknown sequence or max_pages too small")
        return table, lens

    def __del__(self):
        try:
            self.lib.kv_destroy(self.h)
        except Exception:
            pass


class Q8Pages:
    """The pages of one layer's K (or V) as 8-bit codes: ``codes [pages, page, Hkv, D]`` unsigned bytes and ``sz [pages, page, Hkv, 2]``
    f32 ``(scale, zero)`` per (token, kv head); element = ``code * scale + zero``, ``scale = (max - min) / 255``, ``zero = min`` — the
    grouping and rounding of the reference's device cache quantiser (src/models/gemma/gpu_quant.rs:28-166), which packs four codes
    per 32-bit word where this keeps plain bytes.  Half the bytes of a bf16 cache plus 8 bytes per (token, head)."""

    def __init__(self, num_pages: int, page_size: int, kv_heads: int, head_dim: int, device="cpu"):
        self.codes = torch.zeros(num_pages, page_size, kv_heads, head_dim, dtype=torch.uint8, device=device)
        self.sz = torch.zeros(num_pages, page_size, kv_heads, 2, dtype=torch.float32, device=device)
        self.sz[..., 0] = 1.0

    shape = property(lambda self: self.codes.shape)
    device = property(lambda self: self.codes.device)
    is_cuda = property(lambda self: self.codes.is_cuda)

    def dim(self) -> int:
        return 4

    def nbytes(self) -> int:
        return self.codes.numel() + self.sz.numel() * 4

    @staticmethod
    def quantize(rows):
        """``rows [..., D]`` -> ``(codes uint8, sz [..., 2] f32)`` by the rule above (round half up, as the device kernel)."""
        x = rows.float()
        lo, hi = x.min(-1, keepdim=True).values, x.max(-1, keepdim=True).values
        rng = hi - lo
        sc = torch.where(rng > 0, rng / 255.0, torch.ones_like(rng))
        codes = torch.floor((x - lo) / sc + 0.5).clamp(0, 255).to(torch.uint8)
        return codes, torch.cat([sc, lo], -1)

    def append(self, rows, slots) -> None:
        """Quantise ``rows [T, Hkv, D]`` into the flat slots ``slots [T]`` (page * page_size + offset)."""
        codes, sz = self.quantize(rows)
        self.codes.view(-1, *self.codes.shape[2:])[slots.long()] = codes
        self.sz.view(-1, *self.sz.shape[2:])[slots.long()] = sz

    def dequantize(self, pages=None, dtype=torch.bfloat16):
        """bf16 pages ``[n, page, Hkv, D]`` of the listed pages (all when ``None``)."""
        c = self.codes if pages is None else self.codes[pages.long()]
        z = self.sz if pages is None else self.sz[pages.long()]
        return (c.float() * z[..., :1] + z[..., 1:]).to(dtype)


class PagedKVCache:
    """Device storage for the pages of every layer.  ``kv_dtype="int8"`` keeps K and V as :class:`Q8Pages`.  ``v_head_dim`` gives
    values a width of their own; a layer with width 0 stores none (its values are part of its key rows, ``v[layer] is k[layer]``).  ``state_spec`` (one ``{name: (shape, dtype)}`` per recurrent layer) adds ``state[layer][name]``
    tensors ``[num_slots, *shape]``: the per-sequence recurrent state, addressed by ``BatchMeta.state_slots``.  A slot is never
    cleared: the kernels take a sequence whose rows start at position 0 to have zero state."""

    def __init__(self, num_layers: int, num_pages: int, page_size: int, kv_heads: int | list[int], head_dim: int | list[int],
                 dtype=torch.bfloat16, device="cpu", latent_dim: int | None = None, alias_v_to_k: bool = False, kv_dtype: str | None = None,
                 v_head_dim: int | list[int] | None = None, state_spec: list[dict] | None = None, num_slots: int = 0):
        if state_spec and num_slots < 1:
            raise ValueError("recurrent layers need at least one state slot")
        self.alloc = PageAllocator(num_pages, page_size, num_slots if state_spec else 0)
        self.num_slots = num_slots if state_spec else 0
        self.state = [{n: torch.zeros(num_slots, *shape, dtype=dt, device=device) for n, (shape, dt) in spec.items()}
                      for spec in (state_spec or [])]
        self.page_size, self.num_pages, self.num_layers = page_size, num_pages, num_layers
        self.latent = latent_dim is not None
        heads = kv_heads if isinstance(kv_heads, list) else [kv_heads] * num_layers
        dims = head_dim if isinstance(head_dim, list) else [head_dim] * num_layers
        vdims = dims if v_head_dim is None else v_head_dim if isinstance(v_head_dim, list) else [v_head_dim] * num_layers
        self.kv_dtype = kv_dtype
        if kv_dtype not in (None, "int8"):
            raise ValueError(f"kv_dtype {kv_dtype!r}: only None (the activation dtype) and 'int8' are implemented")
        if kv_dtype == "int8":
            if self.latent or alias_v_to_k or vdims != dims:
                raise ValueError("the 8-bit cache holds separate K and V pages of attention heads, not a latent or aliased cache")
            self.k = [Q8Pages(num_pages, page_size, heads[i], dims[i], device) for i in range(num_layers)]
            self.v = [Q8Pages(num_pages, page_size, heads[i], dims[i], device) for i in range(num_layers)]
        elif self.latent:
            self.k = [torch.zeros(num_pages, page_size, latent_dim, dtype=dtype, device=device) for _ in range(num_layers)]
            self.v = self.k
        else:
            self.k = [torch.zeros(num_pages, page_size, heads[i], dims[i], dtype=dtype, device=device) for i in range(num_layers)]
            self.v = self.k if alias_v_to_k else [torch.zeros(num_pages, page_size, heads[i], vdims[i], dtype=dtype, device=device) if vdims[i]
                                                  else self.k[i] for i in range(num_layers)]

    @staticmethod
    def for_model(model, num_pages: int, page_size: int, device="cpu", num_slots: int = 0, **kw) -> "PagedKVCache":
        """The cache a model asks for through ``kv_spec()`` (attention layers) and, where it has one, ``state_spec()``."""
        spec = dict(model.kv_spec())
        if hasattr(model, "state_spec"):
            spec.update(state_spec=model.state_spec(), num_slots=num_slots)
        return PagedKVCache(num_pages=num_pages, page_size=page_size, dtype=model.dtype, device=device, **spec, **kw)

    def state_bytes(self) -> int:
        return sum(t.numel() * t.element_size() for layer in self.state for t in layer.values())

    def save_state(self):
        """Copy of every recurrent state (a step that is run twice, such as a warm-up before a capture, has to start from it again)."""
        return [{n: t.clone() for n, t in layer.items()} for layer in self.state]

    def restore_state(self, saved) -> None:
        for layer, old in zip(self.state, saved):
            for n, t in layer.items():
                t.copy_(old[n])

    def bytes(self) -> int:
        if self.kv_dtype == "int8":
            return sum(t.nbytes() for t in self.k) + sum(t.nbytes() for t in self.v)
        n = sum(t.numel() * t.element_size() for t in self.k)
        if not (self.latent or self.v is self.k):
            n += sum(t.numel() * t.element_size() for i, t in enumerate(self.v) if t is not self.k[i])
        return n + self.state_bytes()
