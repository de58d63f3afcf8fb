"""The residual stream of models that keep it in 32-bit and normalise every sublayer's output.

A sublayer's output does not join the stream by itself: it is left pending, with its post-norm, and the
kernel that produces the next sublayer's input performs the add on its way (``ops.mixers.stream_norm``), so a
stretch "post-norm, residual add, pre-norm (, token shift)" is one pass over the rows.
"""
from __future__ import annotations

from typing import Optional

import torch

from ..ops import mixers as mx


class ResidualStream:
    def __init__(self, x: torch.Tensor, fmt: str):
        self.x, self.fmt = x, fmt                  # fp32 [T, W]
        self.y: Optional[torch.Tensor] = None      # pending sublayer output and its post-norm
        self.post = None

    @property
    def shape(self):
        return self.x.shape

    def add(self, y: torch.Tensor, post) -> "ResidualStream":
        assert self.y is None
        self.y, self.post = y, post
        return self

    def _step(self, **kw):
        x, h, mixes, h32 = mx.stream_norm(self.x, self.fmt, y=self.y, post=self.post, **kw)
        self.x, self.y, self.post = x, None, None
        return h, mixes, h32

    def norm(self, pre) -> torch.Tensor:
        """The next sublayer's input, pre(x)."""
        return self._step(pre=pre)[0]

    def shift(self, pre, mu, state, batch, write_state: bool, want_h32: bool):
        """pre(x), its five token-shift mixes and (on request) its fp32 rows."""
        return self._step(pre=pre, mu=mu, state=state, batch=batch, write_state=write_state, want_h32=want_h32)

    def raw(self) -> torch.Tensor:
        """x itself in the activation type."""
        return self._step(raw=True)[0]

    @property
    def value(self) -> torch.Tensor:
        return self.resolve()

    def resolve(self) -> torch.Tensor:
        """x in fp32, nothing pending."""
        if self.y is not None:
            self._step()
        return self.x
