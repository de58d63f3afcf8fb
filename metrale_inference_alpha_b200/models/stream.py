"""The residual stream of models that keep it in 32-bit.

A sublayer's output does not join the stream by itself: it is left pending (with its post-norm, where the model
has one, and with a mixture of experts' unsummed rows), and the kernel that produces the next sublayer's input
performs the add on its way (``ops.mixers.stream_norm``, ``stream_rms``), so a stretch "post-norm or expert sum,
residual add, pre-norm (, token shift)" is one pass over the rows.
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import ops
from ..ops import mixers as mx


class ResidualStream:
    def __init__(self, x: torch.Tensor, fmt: str, pair: Optional[torch.Tensor] = None):
        self.x, self.fmt = x, fmt                  # fp32 [T, W]
        self.pair = pair                           # looped models: [T, 2 W], the right half holds the embedding output
        self.y: Optional[torch.Tensor] = None      # pending sublayer output and its post-norm
        self.post = None
        self.routed: Optional[mx.Routed] = None    # pending expert rows

    @property
    def shape(self):
        return self.x.shape

    def add(self, y: torch.Tensor, post=None, routed: Optional[mx.Routed] = None) -> "ResidualStream":
        assert self.y is None
        self.y, self.post, self.routed = y, post, routed
        return self

    def _step(self, pre=None, raw: bool = False, out=None, **kw):
        if self.post is None and (self.y is not None or out is not None or isinstance(pre, mx.RmsNorm)):
            x, h = mx.stream_rms(self.x, self.fmt, y=self.y, routed=self.routed, pre=pre, raw=raw, out=out)
            mixes = h32 = None
        else:
            x, h, mixes, h32 = mx.stream_norm(self.x, self.fmt, y=self.y, post=self.post, pre=pre, raw=raw, **kw)
        self.x, self.y, self.post, self.routed = x, None, None, None
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

    def enter_pass(self, w_in, step: torch.Tensor) -> None:
        """In front of a pass of looped layers: x <- w_in [x; embedding output] + step."""
        self._step(raw=True, out=self.pair[:, :self.x.shape[1]])
        self.x = ops.linear(mx.act_of(self.pair, self.fmt), w_in, out_f32=True, bias=step)

    @property
    def value(self) -> torch.Tensor:
        return self.resolve()

    def resolve(self) -> torch.Tensor:
        """x in fp32, nothing pending."""
        if self.y is not None:
            self._step()
        return self.x
