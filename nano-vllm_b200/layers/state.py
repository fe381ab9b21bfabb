"""Per-sequence state of fixed size: what a layer run keeps besides (or instead of) the paged cache."""
from __future__ import annotations

import torch


class SlotState:
    """`state` [slots, *shape], allocated and bound by the runner; dtype None = the model's.  A sequence holds one slot while it
    lives; a sequence at position 0 starts from zero whatever its slot holds."""

    def __init__(self, shape: tuple[int, ...], dtype: torch.dtype | None = None):
        self.shape, self.dtype = tuple(shape), dtype
        self.state: torch.Tensor | None = None
