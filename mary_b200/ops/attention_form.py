"""What a call of ``attention_exact`` may ask for beyond causal attention with a window."""
from __future__ import annotations

from dataclasses import dataclass

import torch


@dataclass(frozen=True)
class AttentionForm:
    """``chunk``: a query sees the keys of its own chunk of that many positions, counted from the start of the sequence (0: all).  ``cap``:
    ``score <- cap * tanh(score / cap)`` after the scale (0: none).  ``sink [Hq]`` f32: a score per head that enters the sum of weights only.
    ``temperature = (coef, every)``: the query at position ``p`` times ``1 + coef * ln(floor((p + 1) / every) + 1)``.  ``difference = (mix, post,
    eps)``: query and key rows hold two maps side by side that read the same values; the result is ``rms(a0 - mix * a1) * post`` over the value
    width of every head.  ``turn [T, value width / 2, 2]`` f32 (one map): cosine and sine by which the pairs ``2 m, 2 m + 1`` of every head's result are turned
    back."""

    chunk: int = 0
    cap: float = 0.0
    sink: torch.Tensor | None = None
    temperature: tuple[float, int] | None = None
    difference: tuple[float, float, float] | None = None
    turn: torch.Tensor | None = None

    @property
    def maps(self) -> int:
        return 1 if self.difference is None else 2
