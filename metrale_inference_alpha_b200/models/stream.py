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
from ..ops import canon, mixers as mx


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

    def take(self, rows: torch.Tensor) -> torch.Tensor:
        """Chosen rows of x in fp32."""
        return self.resolve().index_select(0, rows)

    @property
    def value(self) -> torch.Tensor:
        return self.resolve()

    def resolve(self) -> torch.Tensor:
        """x in fp32, nothing pending."""
        if self.y is not None:
            self._step()
        return self.x


class HyperStream:
    """The residual of models with static hyper-connections: S fp32 streams per token, read and written by every sublayer
    with its own weights (``ops.mixers.HyperW``). One kernel joins the pending sublayer output and makes the next input."""

    def __init__(self, x: torch.Tensor, streams: int, fmt: str):
        self.x, self.S, self.fmt = x, streams, fmt      # [T, W] until the first sublayer has joined, then [T, S, W]
        self.pending: Optional[mx.SublayerOut] = None
        self.hc: Optional[mx.HyperW] = None
        self.ones = None

    @property
    def shape(self):
        return torch.Size((self.x.shape[0], self.x.shape[-1]))

    def norm(self, pre: mx.DytNorm, hc: mx.HyperW) -> torch.Tensor:
        """The next sublayer's input, pre(sum_s w_in[s] x_s)."""
        return self._step(w_in=hc.w_in, pre=pre)

    def add(self, out: mx.SublayerOut, hc: mx.HyperW) -> "HyperStream":
        assert self.pending is None
        self.pending, self.hc = out, hc
        return self

    def _step(self, **kw):
        self.x, h = mx.stream_hyper(self.x, self.S, self.fmt, pending=self.pending, hc=self.hc, **kw)
        if kw.get("rows") is None:
            self.pending = self.hc = None
        return h

    def _sum(self, rows=None) -> torch.Tensor:
        if self.ones is None:
            self.ones = torch.ones(self.S, dtype=torch.float32, device=self.x.device)
        return self._step(w_in=self.ones, out_f32=True, rows=rows)

    def take(self, rows: torch.Tensor) -> torch.Tensor:
        """The sum of the streams at chosen tokens, fp32; the streams themselves are left as they are."""
        return self._sum(rows)

    def resolve(self) -> torch.Tensor:
        """The sum of the streams in fp32, nothing pending."""
        return self._sum()

    @property
    def value(self) -> torch.Tensor:
        return self.resolve()


class CanonStream:
    """The residual of models whose sublayers read x + conv(x), a short causal convolution, and join through an RMS norm of
    their output: one fp32 stream. One kernel joins the pending output and makes the next input."""

    def __init__(self, x: torch.Tensor, fmt: str):
        self.x, self.fmt = x, fmt                       # fp32 [T, W]
        self.pending: Optional[mx.SublayerOut] = None
        self.post: Optional[mx.RmsNorm] = None

    @property
    def shape(self):
        return self.x.shape

    def read(self, filt: torch.Tensor, window: "canon.Window", batch, stash=None) -> torch.Tensor:
        """The next sublayer's input; the window moves on, or waits for the accepted rows of a verify step."""
        h = self._step(filt=filt, window=window, batch=batch, write_state=stash is None)
        if stash is not None and filt.shape[0] > 1:
            x, taps = self.x, filt.shape[0]
            stash.later[window.rows.data_ptr(), window.at] = lambda cb: canon.canon_commit(x, taps, window, cb)
        return h

    def add(self, out: mx.SublayerOut, post: mx.RmsNorm) -> "CanonStream":
        assert self.pending is None
        self.pending, self.post = out, post
        return self

    def _step(self, **kw):
        self.x, h = canon.stream_canon(self.x, self.fmt, pending=self.pending, norm=self.post, **kw)
        self.pending = self.post = None
        return h

    def take(self, rows: torch.Tensor) -> torch.Tensor:
        """Chosen rows of x in fp32."""
        return self.resolve().index_select(0, rows)

    def resolve(self) -> torch.Tensor:
        """x in fp32, nothing pending."""
        self._step()
        return self.x

    @property
    def value(self) -> torch.Tensor:
        return self.resolve()
