"""Short causal convolutions over time with a carried window: around the residual stream (a sublayer's output joins it
through an RMS norm, the next sublayer's input is convolved) and on columns of a projection. CUDA tensors run the kernels
in ``csrc/canon.cu``, CPU tensors the restatements below.

A window is the last taps - 1 inputs of a sequence, oldest first, in fp32. Windows live in a state pool's flat rows:
``Window(rows, at, width)`` is columns at, at + 1, ... of ``rows`` [slots, N].
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import Optional

import torch

from . import _count, _native, _ptr, _stream, runtime
from .mixers import DTYPE, RmsNorm, SublayerOut, _f32


@dataclass
class Window:
    rows: torch.Tensor         # fp32 [slots, N]
    at: int
    width: int                 # channels

    def view(self, taps: int) -> torch.Tensor:
        """[slots, taps - 1, width]"""
        return self.rows[:, self.at:self.at + (taps - 1) * self.width].view(self.rows.shape[0], taps - 1, self.width)

    def args(self, batch, write: bool):
        a = _WindowArgs(self.rows.data_ptr() + 4 * self.at if self.rows.numel() else None, self.rows.stride(0))
        a.q_start, a.q_len, a.positions, a.slots = (_ptr(batch.q_start), _ptr(batch.q_len), _ptr(batch.positions), _ptr(batch.state_slots))
        a.num_seqs, a.num_slots, a.max_q_len, a.write = batch.q_len.numel(), self.rows.shape[0], int(batch.max_q_len), int(write)
        a.status = _ptr(runtime(self.rows.device).status)
        return a


class _WindowArgs(C.Structure):
    _fields_ = [("base", C.c_void_p), ("ld", C.c_longlong), ("q_start", C.c_void_p), ("q_len", C.c_void_p), ("positions", C.c_void_p),
                ("slots", C.c_void_p), ("num_seqs", C.c_int), ("num_slots", C.c_int), ("max_q_len", C.c_int), ("write", C.c_int),
                ("status", C.c_void_p)]


class _StreamCanonArgs(C.Structure):
    _fields_ = [("T", C.c_int), ("W", C.c_int), ("taps", C.c_int), ("f32", C.c_int), ("K", C.c_int), ("plus_one", C.c_int),
                ("x", C.c_void_p), ("y", C.c_void_p), ("ye", C.c_void_p), ("ye_ld", C.c_longlong), ("pair_row", C.c_void_p),
                ("pair_w", C.c_void_p), ("norm_w", C.c_void_p), ("eps", C.c_float), ("x_out", C.c_void_p), ("filt", C.c_void_p),
                ("out", C.c_void_p), ("win", _WindowArgs)]


class _ShortConvArgs(C.Structure):
    _fields_ = [("C", C.c_int), ("taps", C.c_int), ("f32", C.c_int), ("write_out", C.c_int), ("x", C.c_void_p),
                ("x_ld", C.c_longlong), ("filt", C.c_void_p), ("out", C.c_void_p), ("win", _WindowArgs)]


_native.register_optional("mb_stream_canon", [C.POINTER(_StreamCanonArgs), C.c_void_p])
_native.register_optional("mb_canon_commit", [C.c_void_p, C.c_int, C.c_int, C.POINTER(_WindowArgs), C.c_void_p])
_native.register_optional("mb_short_conv", [C.POINTER(_ShortConvArgs), C.c_void_p])


_LONG_PORTION = 96               # portions this long take the join and the convolution as two launches


def _sequences(batch):
    """(first row, rows, state slot, starts at position 0) of every sequence with rows."""
    for r, n, slot in zip(batch.q_start.tolist(), batch.q_len.tolist(), batch.state_slots.tolist()):
        if n > 0:
            yield r, n, slot, int(batch.positions[r]) == 0


def _convolve_ref(x: torch.Tensor, filt: torch.Tensor, window: torch.Tensor, batch, write: bool) -> torch.Tensor:
    """x [T, C] fp32, filt [taps, C], window [slots, taps - 1, C]."""
    taps = filt.shape[0]
    out = torch.zeros_like(x)
    for r, n, slot, fresh in _sequences(batch):
        old = torch.zeros_like(window[slot]) if fresh else window[slot]
        z = torch.cat([old, x[r:r + n]])
        out[r:r + n] = sum(filt[j].float() * z[j:j + n] for j in range(taps))
        if write and taps > 1:
            window[slot] = z[n:]
    return out


def stream_canon(x: torch.Tensor, fmt: str, *, pending: Optional[SublayerOut] = None, norm: Optional[RmsNorm] = None,
                 filt: Optional[torch.Tensor] = None, window: Optional[Window] = None, batch=None, write_state: bool = True):
    """x [T, W] fp32. With ``pending`` (y, routed rows, or both): x' = x + norm(pending), else x' = x. With ``filt``
    [taps, W]: h = x' + the causal convolution of x' along each sequence, the window advanced. Returns (x', h or None);
    x' is x itself when nothing is pending."""
    T, W = x.shape
    if not x.is_cuda:
        x1 = x
        if pending is not None:
            y = torch.zeros(T, W) if pending.y is None else pending.y.float()
            x1 = x + norm.ref(y if pending.routed is None else y + pending.routed.y)
        if filt is None:
            return x1, None
        return x1, (x1 + _convolve_ref(x1, filt, window.view(filt.shape[0]), batch, write_state)).to(DTYPE[fmt])
    a = _StreamCanonArgs(T=T, W=W, f32=_f32(fmt), x=_ptr(x))
    x1 = h = None
    if pending is not None:
        assert pending.gate is None
        x1 = torch.empty_like(x)
        y, r = pending.y, pending.routed
        if y is not None:
            assert y.dtype == DTYPE[fmt] and y.is_contiguous() and y.shape == (T, W)
            a.y = _ptr(y)
        if r is not None:
            a.ye, a.ye_ld, a.pair_row, a.pair_w, a.K = _ptr(r.y), r.y.stride(0), _ptr(r.pair_row), _ptr(r.w), r.w.shape[1]
        a.norm_w, a.eps, a.plus_one, a.x_out = _ptr(norm.w), norm.eps, int(norm.plus_one), _ptr(x1)
        assert norm.scale == 1.0
    if filt is not None:
        h = torch.empty(T, W, dtype=DTYPE[fmt], device=x.device)
        a.taps, a.filt, a.out, a.win = filt.shape[0], _ptr(filt), _ptr(h), window.args(batch, write_state)
    if x1 is None and h is None:
        return x, None
    _native.check(_native.lib().mb_stream_canon(C.byref(a), _stream()), f"stream_canon[T={T} W={W}]")
    _count(2 if filt is not None and int(batch.max_q_len) >= _LONG_PORTION else 1)
    return (x if x1 is None else x1), h


def canon_commit(x: torch.Tensor, taps: int, window: Window, batch) -> None:
    """Advance the window by each sequence's rows of x in ``batch`` (sequences of zero rows keep theirs)."""
    if taps < 2:
        return
    if not x.is_cuda:
        _convolve_ref(x, torch.zeros(taps, x.shape[1]), window.view(taps), batch, True)
        return
    a = window.args(batch, True)
    _native.check(_native.lib().mb_canon_commit(_ptr(x), x.shape[1], taps, C.byref(a), _stream()), "canon_commit")
    _count()


def short_conv(x: torch.Tensor, filt: torch.Tensor, window: Window, batch, fmt: str, *, write_state: bool = True,
               write_out: bool = True) -> Optional[torch.Tensor]:
    """Causal convolution of x's columns [T, C] (a column range, activation type) with ``filt`` [taps, C] fp32, through
    SiLU; the window advanced. ``write_out`` off: only that."""
    T, Cn = x.shape
    taps = filt.shape[0]
    if not x.is_cuda:
        y = _convolve_ref(x.float(), filt, window.view(taps), batch, write_state)
        return torch.nn.functional.silu(y).to(DTYPE[fmt]) if write_out else None
    assert x.stride(1) == 1 and x.dtype == DTYPE[fmt] and filt.dtype == torch.float32 and window.width == Cn
    out = torch.empty(T, Cn, dtype=x.dtype, device=x.device) if write_out else None
    a = _ShortConvArgs(Cn, taps, _f32(fmt), int(write_out), _ptr(x), x.stride(0), _ptr(filt), _ptr(out), window.args(batch, write_state))
    _native.check(_native.lib().mb_short_conv(C.byref(a), _stream()), f"short_conv[T={T} C={Cn}]")
    _count()
    return out
