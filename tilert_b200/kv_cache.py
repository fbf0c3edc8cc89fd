"""Key/value cache of one attention layer for one sequence: a ring of rows per key/value head.

A layer that sees only the last ``window`` positions needs no more rows than its window plus the positions that are
written in one go (a query of a portion must still find the window of the portion's first token after its last token
has been written).  A layer without a window, or with one that covers the whole sequence, keeps ``max_len`` rows.
Position p is row ``p % ring``; rows of an earlier sequence need no clearing, because a query only reads positions up
to its own and every one of them has been written since the sequence began."""

from __future__ import annotations

import torch


class RingKVCache:
    def __init__(self, kv_heads: int, dim: int, vdim: int, window: int | None, max_len: int, portion: int, device, dtype):
        pad16 = lambda n: (n + 15) // 16 * 16  # noqa: E731
        self.window = window if window is not None and window < max_len else 0  # 0: nothing is ever outside
        self.ring = max_len if self.window == 0 else self.window - 1 + portion
        self.k = torch.zeros(kv_heads, self.ring, pad16(dim), dtype=dtype, device=device)
        self.v = torch.zeros(kv_heads, self.ring, pad16(vdim), dtype=dtype, device=device)

    def visible(self, length: int) -> int:
        """Keys the last of ``length`` positions sees."""
        return length if self.window == 0 else min(length, self.window)

    def bytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in (self.k, self.v))
