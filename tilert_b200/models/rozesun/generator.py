"""Generation with a Rozesun model through the shared generator."""

from __future__ import annotations

from ..generator import PortionGenerator


class RozesunGenerator(PortionGenerator):
    pass
