"""Generation with a Ralasun model through the shared generator."""

from __future__ import annotations

from ..generator import PortionGenerator


class RalasunGenerator(PortionGenerator):
    pass
