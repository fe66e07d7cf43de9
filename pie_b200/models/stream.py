"""The 32-bit residual stream of designs that norm a sublayer's output: x += y / rms(y) * gain is pending until the next
norm reads the stream, and both run in one pass."""
from __future__ import annotations

import torch

from ..ops import latent as lops, stream_conv as conv
from .config import ModelConfig


class ResidualStream:
    """x [N, padded width] fp32, and a sublayer output y not yet normed and added to it."""

    def __init__(self, x):
        self.x, self.y, self.y_norm = x, None, None
        self.pair = ()              # (sublayer output, gain) pairs, each to be normed and added
        self.values = None          # values of the first layer that mixes them (32-bit, one row per token)

    def finish(self, cfg: ModelConfig):
        """The stream with everything pending added."""
        if self.pair:
            self.x, _ = conv.conv_norm(self.x, cfg.hidden_size, cfg.rms_norm_eps, self.pair)
            self.pair = ()
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

    def convolved(self, cfg: ModelConfig, lw: dict, half: str, li: int, rs, dtype):
        """Add what is pending, then the layer norm and the convolution ahead of a sublayer, in `dtype`."""
        history = rs.history_of(li, half) if cfg.conv_taps > 1 else None
        self.x, h = conv.conv_norm(self.x, cfg.hidden_size, cfg.rms_norm_eps, self.pair, lw["gain" + half], lw["offset" + half],
                                   lw.get("taps" + half), history, rs, dtype)
        self.pair = ()
        return h

    def add_product(self, a, w):
        """x += a @ w.T, accumulated in 32-bit (bf16 on the device: in the product's epilogue)."""
        if a.is_cuda and a.dtype == torch.bfloat16:
            lops.gemm_stream(a, w, None, self.x)
        else:
            self.x = self.x + torch.matmul(a, w.t()).float()
