"""Cached decode of twin-norm decoders (``models/nugosun.py``): one row per sequence, one CUDA graph per step."""
from __future__ import annotations

from .layered_decode import LayeredDecode


class TwinNormDecode(LayeredDecode):
    pass
