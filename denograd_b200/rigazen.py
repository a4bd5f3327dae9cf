"""Rigazen: a layer-list decoder (hybrid.py) — mLSTM mixers, and mixers with window attention and lightning attention side by
side, in any order; sublayers read the stream itself and only their outputs are normed (weights stored around zero); squared-
ReLU feed-forwards; a per-layer input from a second token table; logits from the embedding table."""
from __future__ import annotations

from .hybrid_driver import HybridDriver


class Rigazen(HybridDriver):
    architecture = "Rigazen"
