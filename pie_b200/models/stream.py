"""The 32-bit residual stream of designs that norm a sublayer's output: x += y / rms(y) * gain is pending until the next
norm reads the stream, and both run in one pass."""
from __future__ import annotations

from ..ops import latent as lops
from .config import ModelConfig


class ResidualStream:
    """x [N, padded width] fp32, and a sublayer output y not yet normed and added to it."""

    def __init__(self, x):
        self.x, self.y, self.y_norm = x, None, None
        self.values = None          # values of the first layer that mixes them (32-bit, one row per token)

    def finish(self, cfg: ModelConfig):
        """The stream with everything pending added."""
        if self.y is not None:
            self.x, _, _ = lops.stream_norm(self.x, cfg.hidden_size, cfg.rms_norm_eps, self.y, self.y_norm, dtype=self.y.dtype)
            self.y = self.y_norm = None
        return self.x

    def normed(self, cfg: ModelConfig, gain, dtype):
        """Add what is pending, then RMSNorm(x) * gain in `dtype`."""
        self.x, h, _ = lops.stream_norm(self.x, cfg.hidden_size, cfg.rms_norm_eps, self.y, self.y_norm, gain, dtype=dtype)
        self.y = self.y_norm = None
        return h

    def plain(self, cfg: ModelConfig, dtype):
        """Add what is pending; the stream itself in `dtype`."""
        self.x, h, _ = lops.stream_norm(self.x, cfg.hidden_size, cfg.rms_norm_eps, self.y, self.y_norm, dtype=dtype, copy=True)
        self.y = self.y_norm = None
        return h
