"""Nilatar model family: latent attention with a query latent and slowed-down long waves, linear attention with a constant decay per head,
windowed sink attention whose keys and values several layers can share; per-column layer scales; dense feed-forwards."""
from .config import NilatarConfig
from .model import Nilatar

__all__ = ["Nilatar", "NilatarConfig"]
