"""Gagotar model family: attention whose heads exchange scores before the softmax, in chunks of positions, side by side with gated linear
attention; both normed before they are averaged; per-column layer scales; experts with limited activations."""
from .config import GagotarConfig
from .model import Gagotar

__all__ = ["Gagotar", "GagotarConfig"]
