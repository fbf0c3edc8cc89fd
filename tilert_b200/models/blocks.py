"""What the models with bf16 weight rows share: weights as the kernels want them, work buffers, and the residual stream
of a one-token step and of a portion of tokens."""

from __future__ import annotations

import math
from dataclasses import dataclass

import torch

from tilert_b200 import gqa_ops as ops
from tilert_b200.gqa_ops import BF16, F32, pad


def padded_rows(w: torch.Tensor, device) -> torch.Tensor:
    """bf16 [.., n, pad8(k)] on the device, zeros beyond k."""
    w = w.to(device, BF16)
    k = w.shape[-1]
    return w.contiguous() if k % 8 == 0 else torch.nn.functional.pad(w, (0, pad(k) - k)).contiguous()


def one_plus(w: torch.Tensor, device) -> torch.Tensor:
    """f32 gain of a norm whose weight is an offset from one, zeros beyond its length."""
    g = 1.0 + w.to(device, F32)
    return torch.nn.functional.pad(g, (0, pad(g.numel()) - g.numel())).contiguous()


def padded_vec(w: torch.Tensor, device, scale: float = 1.0) -> torch.Tensor:
    """f32 vector times ``scale``, zeros beyond its length."""
    v = w.to(device, F32) * scale
    return torch.nn.functional.pad(v, (0, pad(v.numel()) - v.numel())).contiguous()


def layer_norm(sd, name: str, device, scale: float = 1.0) -> ops.Norm:
    """The layer norm of a checkpoint's ``name`` and ``name.b``, its result times ``scale``."""
    return ops.Norm(padded_vec(sd[name], device, scale), padded_vec(sd[f"{name}.b"], device, scale), centered=True)


class Scratch:
    """Named work buffers shared by the layers (they run one after the other).  A buffer is identified by its name
    and shape, and starts as zeros: what lies beyond a logical length is then zero for good."""

    def __init__(self, device):
        self.device = torch.device(device)
        self._bufs: dict = {}

    def get(self, name: str, *shape: int, dtype=F32) -> torch.Tensor:
        key = (name, shape, dtype)
        if key not in self._bufs:
            self._bufs[key] = torch.zeros(*shape, dtype=dtype, device=self.device)
        return self._bufs[key]

    def flat(self, name: str, *shape: int, dtype=F32) -> torch.Tensor:
        """A contiguous buffer of this shape in memory that grows as needed (never inside a graph: it may move); the
        contents are whatever was left there, but finite."""
        n, key = math.prod(shape), (name, dtype)
        if key not in self._bufs or self._bufs[key].numel() < n:
            self._bufs[key] = torch.zeros(n, dtype=dtype, device=self.device)
        return self._bufs[key][:n].view(*shape)


@dataclass
class Pending:
    """A sublayer output whose norm and residual step the next launch will do."""

    y: torch.Tensor
    norm: torch.Tensor | ops.Norm  # (a bare tensor: the gain of an RMS norm)


class Stream:
    """The residual vector of a one-token step: two buffers, because a launch that advances it reads the old one."""

    def __init__(self, scratch: Scratch, dim: int):
        self.bufs = [scratch.get("x0", pad(dim)), scratch.get("x1", pad(dim))]
        self.at = 0
        self.pending: Pending | None = None
        self.add: torch.Tensor | None = None  # a constant vector, added behind the pending output

    @property
    def x(self) -> torch.Tensor:
        return self.bufs[self.at]

    def _advance(self) -> tuple[torch.Tensor, dict]:
        """The residual to read, and what the launch that reads it has to do with it first."""
        if self.pending is None and self.add is None:
            return self.x, {}
        old, kw = self.x, {"add": self.add, "x_out": self.bufs[self.at ^ 1]}
        if self.pending is not None:
            kw |= {"y": self.pending.y, "gain": self.pending.norm}
        self.at ^= 1
        self.pending = self.add = None
        return old, kw

    def dense(self, w, out, n: int, k: int, eps: float, **kw) -> None:
        """A product of the up-to-date vector (or of its norm ``gain2``); advances the residual."""
        x, todo = self._advance()
        ops.vec_dense(x, w, out, n, k, eps=eps, **todo, **kw)

    def gated(self, w, out, n: int, k: int, limit: float, alpha: float, eps: float, **kw) -> None:
        """The same into the gated unit of a dense feed-forward."""
        x, todo = self._advance()
        ops.vec_gated(x, w, out, n, k, limit, alpha, eps=eps, **todo, **kw)


class RowStream:
    """The residual rows of a portion, f32 ``x`` and ``xh``, what the next sublayer reads.  As in a one-token step a
    sublayer's output waits: the launch that adds it also norms the next sublayer's input."""

    def __init__(self, x: torch.Tensor, xh: torch.Tensor, rows: int, dim: int, eps: float):
        self.x, self.xh, self.rows, self.dim, self.eps = x, xh, rows, dim, eps
        self.pending: Pending | None = None
        self.add: torch.Tensor | None = None  # a constant vector, added behind the pending output

    def _advance(self, xh, norm2) -> None:
        p = self.pending
        ops.residual_norm(self.x, xh, None if p is None else p.norm, self.eps, self.dim, self.rows, y=None if p is None else p.y,
                          add=self.add, norm2=norm2)
        self.pending = self.add = None

    def normed(self, norm) -> torch.Tensor:
        """The norm of the up-to-date rows as activations."""
        self._advance(self.xh, norm)
        return self.xh

    def settle(self) -> torch.Tensor:
        """The up-to-date rows."""
        if self.pending is not None or self.add is not None:
            self._advance(None, None)
        return self.x
