"""Matulorn: a layer-list decoder (hybrid.py) — minGRU, latent-attention and gated-delta mixers in any order, grouped RMS norms
before and after every sublayer, clamped gated feed-forwards."""
from __future__ import annotations

from .hybrid_driver import HybridDriver


class Matulorn(HybridDriver):
    architecture = "Matulorn"
