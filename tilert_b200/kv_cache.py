"""Caches of one attention layer for one sequence: rings of rows, one row per position.

A layer that sees only the last ``window`` positions needs no more rows than its window plus the positions that are
written in one go (a query of a portion must still find the window of the portion's first token after its last token
has been written).  A layer without a window, or with one that covers the whole sequence, keeps ``max_len`` rows.
Position p is row ``p % ring``; rows of an earlier sequence need no clearing, because a query only reads positions up
to its own and every one of them has been written since the sequence began."""

from __future__ import annotations

import torch


def _pad(n: int, m: int) -> int:
    return (n + m - 1) // m * m


class Ring:
    def __init__(self, window: int | None, max_len: int, portion: int):
        self.window = window if window is not None and window < max_len else 0  # 0: nothing is ever outside
        self.ring = max_len if self.window == 0 else self.window - 1 + portion

    def visible(self, length: int, tokens: int = 1) -> int:
        """Keys the last ``tokens`` of ``length`` positions see together."""
        return length if self.window == 0 else min(length, self.window + tokens - 1)

    def _tensors(self) -> tuple[torch.Tensor, ...]:
        raise NotImplementedError

    def bytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in self._tensors())


class RingKVCache(Ring):
    """Keys and values per key/value head."""

    def __init__(self, kv_heads: int, dim: int, vdim: int, window: int | None, max_len: int, portion: int, device, dtype):
        super().__init__(window, max_len, portion)
        self.k = torch.zeros(kv_heads, self.ring, _pad(dim, 16), dtype=dtype, device=device)
        self.v = torch.zeros(kv_heads, self.ring, _pad(vdim, 16), dtype=dtype, device=device)

    def _tensors(self):
        return self.k, self.v


class LatentCache(Ring):
    """One row per position for all heads: the latent that keys and values are expanded from, zeros up to a multiple of
    16, the rotated key part, zeros up to a multiple of 32."""

    def __init__(self, rank: int, rot: int, window: int | None, max_len: int, portion: int, device, dtype):
        super().__init__(window, max_len, portion)
        self.rank, self.rot = rank, rot
        self.rows = torch.zeros(self.ring, _pad(_pad(rank, 16) + rot, 32), dtype=dtype, device=device)

    def _tensors(self):
        return (self.rows,)
