"""Ops of models with a 32-bit residual stream: Dynamic-Tanh and RMS norms fused around the stream, static
hyper-connections, token-shift mixes, attention with separate query/key and value head sizes (sinks, windows with kept
first tokens, output gates), decaying linear attention (per-head or per-channel decay), gated group norms and the
token side input.

CUDA tensors run the kernels in ``csrc/{stream_norm,stream_hyper,attention,attention_tc,attention_simt,linear_attn,
linear_chunked,gemm_simt}.cu``; CPU tensors run the restatements below, which compute the same quantities
in fp32 and round where the kernels round. The activation type is bf16, or fp32 for models served in
32-bit (``Act.fmt`` "bf16" / "fp32").
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import Optional, Tuple

import torch

from . import Act, _count, _native, _ptr, _stream, runtime
from . import reference as ref

ADD = {None: 0, "dyt": 1, "rms": 2}
DTYPE = {"bf16": torch.bfloat16, "fp32": torch.float32}


@dataclass
class DytNorm:
    """tanh(alpha x) w + b."""
    alpha: float
    w: torch.Tensor        # bf16 [W]
    b: torch.Tensor        # bf16 [W]


@dataclass
class RmsNorm:
    """x / sqrt(mean(x^2) + eps) * w * scale, or 1 + w for weights that are stored around zero."""
    w: torch.Tensor        # bf16 [W]
    eps: float
    plus_one: bool = False
    scale: float = 1.0

    def ref(self, x: torch.Tensor) -> torch.Tensor:
        w = self.w.float() + 1.0 if self.plus_one else self.w.float()
        return x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + self.eps) * w * self.scale


@dataclass
class Routed:
    """A mixture of experts' output that has not been summed: row pair_row[t K + j] of y, times w[t, j]. With
    ``pair_row`` None (CPU) y is the sum itself, [T, W]."""
    y: torch.Tensor                        # fp32 [pairs, >= W]
    pair_row: Optional[torch.Tensor]       # int32 [T K], -1 = no row
    w: Optional[torch.Tensor]              # fp32 [T, K]


def act_of(t: torch.Tensor, fmt: str) -> Act:
    """`t` (already of the activation type) as a GEMM operand; on CPU operands are kept in fp32."""
    d = t if t.is_cuda else t.float()
    return Act(fmt, t.shape[0], t.shape[1], d, bf16=t if fmt == "bf16" else None)


def _f32(fmt: str) -> int:
    return int(fmt == "fp32")


# ----------------------------------------------------------------------------- stream norm
class _StreamNormArgs(C.Structure):
    _fields_ = [("T", C.c_int), ("W", C.c_int), ("f32", C.c_int), ("add_mode", C.c_int), ("out_mode", C.c_int),
                ("x", C.c_void_p), ("y", C.c_void_p), ("post_alpha", C.c_float), ("post_w", C.c_void_p), ("post_b", C.c_void_p),
                ("pre_alpha", C.c_float), ("pre_w", C.c_void_p), ("pre_b", C.c_void_p), ("eps", C.c_float),
                ("x_out", C.c_void_p), ("out", C.c_void_p), ("h32", C.c_void_p), ("mu", C.c_void_p), ("mixes", C.c_void_p),
                ("state", C.c_void_p), ("q_start", C.c_void_p), ("q_len", C.c_void_p), ("positions", C.c_void_p),
                ("slots", C.c_void_p), ("num_seqs", C.c_int), ("num_slots", C.c_int), ("write_state", C.c_int),
                ("status", C.c_void_p)]


class _StreamRmsArgs(C.Structure):
    _fields_ = [("T", C.c_int), ("W", C.c_int), ("f32", C.c_int), ("out_mode", C.c_int), ("x", C.c_void_p), ("y", C.c_void_p),
                ("ye", C.c_void_p), ("ye_ld", C.c_longlong), ("pair_row", C.c_void_p), ("pair_w", C.c_void_p), ("K", C.c_int),
                ("w", C.c_void_p), ("eps", C.c_float), ("x_out", C.c_void_p), ("out", C.c_void_p), ("out_ld", C.c_longlong),
                ("plus_one", C.c_int), ("scale", C.c_float)]


_native.register_optional("mb_stream_norm", [C.POINTER(_StreamNormArgs), C.c_void_p])
_native.register_optional("mb_stream_rms", [C.POINTER(_StreamRmsArgs), C.c_void_p])
_native.register_optional("mb_shift_commit", [C.c_void_p, C.c_int] + [C.c_void_p] * 4 + [C.c_int, C.c_int, C.c_void_p, C.c_void_p])


def dyt_ref(x: torch.Tensor, n: DytNorm) -> torch.Tensor:
    return torch.tanh(n.alpha * x.float()) * n.w.float() + n.b.float()


def stream_rms(x: torch.Tensor, fmt: str, *, y: Optional[torch.Tensor] = None, routed: Optional[Routed] = None,
               pre: Optional[RmsNorm] = None, raw: bool = False, out: Optional[torch.Tensor] = None):
    """x' = x (+ y) (+ the routed experts' weighted sum), x [T, W] fp32, y of the activation type. Output pre(x'), or x'
    itself with ``raw``, or none; ``out`` may be a column range of a wider matrix. Returns (x', output); x' is x itself
    when nothing is added."""
    T, W = x.shape
    wanted = pre is not None or raw
    if wanted and out is None:
        out = torch.empty(T, W, dtype=DTYPE[fmt], device=x.device)
    if not x.is_cuda:
        x1 = x if y is None else x + y.float()
        x1 = x1 if routed is None else x1 + routed.y
        if wanted:
            out.copy_(x1 if raw else pre.ref(x1))
        return x1, out
    a = _StreamRmsArgs()
    a.T, a.W, a.f32, a.x = T, W, _f32(fmt), _ptr(x)
    x1 = x
    if y is not None or routed is not None:
        x1 = torch.empty_like(x)
        a.x_out = _ptr(x1)
    if y is not None:
        assert y.dtype == DTYPE[fmt] and y.is_contiguous()
        a.y = _ptr(y)
    if routed is not None:
        a.ye, a.ye_ld, a.pair_row, a.pair_w, a.K = _ptr(routed.y), routed.y.stride(0), _ptr(routed.pair_row), _ptr(routed.w), routed.w.shape[1]
    if wanted:
        assert out.stride(1) == 1 and out.dtype == DTYPE[fmt]
        a.out_mode, a.out, a.out_ld = (2 if raw else 1), _ptr(out), out.stride(0)
        if pre is not None:
            a.w, a.eps, a.plus_one, a.scale = _ptr(pre.w), pre.eps, int(pre.plus_one), pre.scale
    _native.check(_native.lib().mb_stream_rms(C.byref(a), _stream()), f"stream_rms[T={T} W={W}]")
    _count()
    return x1, out


def stream_norm(x: torch.Tensor, fmt: str, *, y: Optional[torch.Tensor] = None, post=None, pre: Optional[DytNorm] = None,
                raw: bool = False, want_x: bool = True, mu: Optional[torch.Tensor] = None, state: Optional[torch.Tensor] = None,
                batch=None, write_state: bool = True, want_h32: bool = False):
    """x [T, W] fp32. With ``y`` (activation type) and ``post`` (DytNorm | RmsNorm): x' = x + post(y), else
    x' = x. Output h = pre(x'), or x' itself with ``raw``, or none. With ``mu`` [5, W] (and ``state``
    [slots, W] fp32, ``batch``): the five token-shift mixes of h, and the state advanced to each sequence's
    last row. Returns (x', h, mixes [5, T, W] or None, h in fp32 or None); x' is x itself when nothing is added."""
    T, W = x.shape
    out_dt = DTYPE[fmt]
    if not x.is_cuda:
        x1 = x
        if y is not None:
            add = dyt_ref(y, post) if isinstance(post, DytNorm) else \
                y.float() * torch.rsqrt(y.float().pow(2).mean(-1, keepdim=True) + post.eps) * post.w.float()
            x1 = x + add
        if pre is None and not raw:
            return x1, None, None, None
        h = x1 if raw else dyt_ref(x1, pre)
        mixes = None
        if mu is not None:
            prev = torch.zeros_like(h)
            qs, ql, sl = batch.q_start.tolist(), batch.q_len.tolist(), batch.state_slots.tolist()
            for s, n in enumerate(ql):
                if n <= 0:
                    continue
                r = qs[s]
                if int(batch.positions[r]) != 0:
                    prev[r] = state[sl[s]]
                prev[r + 1:r + n] = h[r:r + n - 1]
            mixes = (h[None] + (prev - h)[None] * mu.float()[:, None, :]).to(out_dt)
            if write_state:
                for s, n in enumerate(ql):
                    if n > 0:
                        state[sl[s]] = h[qs[s] + n - 1]
        return x1, h.to(out_dt), mixes, (h if want_h32 else None)
    dev = x.device
    a = _StreamNormArgs()
    a.T, a.W, a.f32 = T, W, _f32(fmt)
    a.x = _ptr(x)
    x1 = x
    if y is not None:
        assert y.dtype == out_dt and y.is_contiguous()
        a.y, a.post_w = _ptr(y), _ptr(post.w)
        if isinstance(post, DytNorm):
            a.add_mode, a.post_alpha, a.post_b = 1, post.alpha, _ptr(post.b)
        else:
            a.add_mode, a.eps = 2, post.eps
        if want_x:
            x1 = torch.empty_like(x)
            a.x_out = _ptr(x1)
    h = mixes = h32 = None
    if pre is not None or raw:
        h = torch.empty(T, W, dtype=out_dt, device=dev)
        a.out, a.out_mode = _ptr(h), 2 if raw else 1
        if pre is not None:
            a.pre_alpha, a.pre_w, a.pre_b = pre.alpha, _ptr(pre.w), _ptr(pre.b)
        if want_h32:
            h32 = torch.empty(T, W, dtype=torch.float32, device=dev)
            a.h32 = _ptr(h32)
    if mu is not None:
        mixes = torch.empty(5, T, W, dtype=out_dt, device=dev)
        a.mu, a.mixes, a.state = _ptr(mu), _ptr(mixes), _ptr(state)
        a.q_start, a.q_len, a.positions, a.slots = (_ptr(batch.q_start), _ptr(batch.q_len), _ptr(batch.positions),
                                                    _ptr(batch.state_slots))
        a.num_seqs, a.num_slots, a.write_state = batch.q_len.numel(), state.shape[0], int(write_state)
    a.status = _ptr(runtime(dev).status)
    _native.check(_native.lib().mb_stream_norm(C.byref(a), _stream()), f"stream_norm[T={T} W={W}]")
    _count()
    return x1, h, mixes, h32


# ----------------------------------------------------------------------------- several residual streams
@dataclass
class HyperW:
    """Static hyper-connection of one sublayer over S residual streams: it reads sum_s w_in[s] x_s, and every stream becomes
    sum_s w_mix[s, t] x_s + w_out[t] y."""
    w_in: torch.Tensor     # fp32 [S]
    w_out: torch.Tensor    # fp32 [S]
    w_mix: torch.Tensor    # fp32 [S (from), S (to)]


@dataclass
class SublayerOut:
    """What a sublayer leaves for the streams: y (activation type), times the sigmoid of ``gate`` [T] (fp32 logits, may be
    a column), plus the routed experts' sum; any of them may be missing."""
    y: Optional[torch.Tensor] = None
    gate: Optional[torch.Tensor] = None
    routed: Optional[Routed] = None


class _StreamHyperArgs(C.Structure):
    _fields_ = [("T", C.c_int), ("W", C.c_int), ("S", C.c_int), ("f32", C.c_int), ("x_one", C.c_int), ("out_mode", C.c_int), ("K", C.c_int),
                ("x", C.c_void_p), ("y", C.c_void_p), ("y_gate", C.c_void_p), ("y_gate_ld", C.c_longlong), ("ye", C.c_void_p),
                ("ye_ld", C.c_longlong), ("pair_row", C.c_void_p), ("pair_w", C.c_void_p), ("w_mix", C.c_void_p), ("w_out", C.c_void_p),
                ("x_out", C.c_void_p), ("w_in", C.c_void_p), ("alpha", C.c_float), ("norm_w", C.c_void_p), ("norm_b", C.c_void_p),
                ("out", C.c_void_p), ("rows", C.c_void_p), ("num_rows", C.c_longlong), ("status", C.c_void_p)]


_native.register_optional("mb_stream_hyper", [C.POINTER(_StreamHyperArgs), C.c_void_p])
_HYPER_IN_PLACE = 4              # the kernel holds this many streams in registers


def stream_hyper(x: torch.Tensor, S: int, fmt: str, *, pending: Optional[SublayerOut] = None, hc: Optional[HyperW] = None,
                 w_in: Optional[torch.Tensor] = None, pre: Optional[DytNorm] = None, out_f32: bool = False,
                 rows: Optional[torch.Tensor] = None):
    """x [T, S, W] fp32, or [T, W] while all S streams are one row. ``pending`` joins the streams through ``hc``; the
    output is pre(u), or u itself in fp32 (``out_f32``) or the activation type, u = sum_s w_in[s] x_s of the new streams.
    ``rows`` (int64): only those tokens, the streams stay. Returns (streams, output); streams that are given whole may be
    updated in place."""
    one = x.dim() == 2
    T, W = x.shape[0], x.shape[-1]
    n = T if rows is None else rows.numel()
    out = torch.empty(n, W, dtype=torch.float32 if out_f32 else DTYPE[fmt], device=x.device)
    if not x.is_cuda:
        xs = x[:, None, :].expand(T, S, W) if one else x
        if pending is not None:
            y = torch.zeros(T, W)
            if pending.y is not None:
                y = pending.y.float() * (torch.sigmoid(pending.gate.float())[:, None] if pending.gate is not None else 1.0)
            if pending.routed is not None:
                y = y + pending.routed.y
            xs = torch.einsum("tsw,so->tow", xs, hc.w_mix) + hc.w_out[None, :, None] * y[:, None, :]
        u = torch.einsum("tsw,s->tw", xs, w_in)
        u = u if rows is None else u[rows.long()]
        out.copy_(u if pre is None else dyt_ref(u, pre))
        return (xs if pending is not None and rows is None else x), out
    a = _StreamHyperArgs()
    a.T, a.W, a.S, a.f32, a.x_one = n, W, S, _f32(fmt), int(one)
    a.x, a.out, a.w_in, a.status = _ptr(x), _ptr(out), _ptr(w_in), _ptr(runtime(x.device).status)
    a.out_mode = 3 if out_f32 else 1 if pre is not None else 2
    if pre is not None:
        assert not out_f32
        a.alpha, a.norm_w, a.norm_b = pre.alpha, _ptr(pre.w), _ptr(pre.b)
    x1 = x
    if rows is not None:
        assert rows.dtype == torch.int64
        a.rows, a.num_rows = _ptr(rows), T
    if pending is not None:
        a.w_mix, a.w_out = _ptr(hc.w_mix), _ptr(hc.w_out)
        y, g, r = pending.y, pending.gate, pending.routed
        if y is not None:
            assert y.dtype == DTYPE[fmt] and y.is_contiguous() and y.shape == (T, W)
            a.y = _ptr(y)
            if g is not None:
                assert g.dtype == torch.float32 and g.dim() == 1
                a.y_gate, a.y_gate_ld = _ptr(g), g.stride(0)
        if r is not None:
            a.ye, a.ye_ld, a.pair_row, a.pair_w, a.K = _ptr(r.y), r.y.stride(0), _ptr(r.pair_row), _ptr(r.w), r.w.shape[1]
        if rows is None:
            x1 = torch.empty(T, S, W, dtype=torch.float32, device=x.device) if one or S > _HYPER_IN_PLACE else x
            a.x_out = _ptr(x1)
    _native.check(_native.lib().mb_stream_hyper(C.byref(a), _stream()), f"stream_hyper[T={n} S={S} W={W}]")
    _count()
    return x1, out


def shift_commit(h32: torch.Tensor, state: torch.Tensor, batch) -> None:
    """state[slot] := h of each sequence's last row in ``batch`` (sequences of zero rows keep theirs)."""
    if not h32.is_cuda:
        for s, n in enumerate(batch.q_len.tolist()):
            if n > 0:
                state[int(batch.state_slots[s])] = h32[int(batch.q_start[s]) + n - 1]
        return
    rc = _native.lib().mb_shift_commit(_ptr(h32), h32.shape[1], _ptr(state), _ptr(batch.q_start), _ptr(batch.q_len),
                                       _ptr(batch.state_slots), batch.q_len.numel(), state.shape[0],
                                       _ptr(runtime(h32.device).status), _stream())
    _native.check(rc, "shift_commit")
    _count()


# ----------------------------------------------------------------------------- projections of the token-shift mixes
def grouped_ok(width: int, rows: int, fmt: str) -> bool:
    """Whether the r, k, v, g projections can be one grouped tcgen05 GEMM: whole 128-row weight tiles each."""
    return fmt == "bf16" and rows % 128 == 0 and width % 8 == 0


_GROUP_LISTS: dict = {}          # never evicted: captured graphs hold the lists' addresses (a few KB per row count)
_GROUPED_MAX_ROWS = 256          # above this, one full-width GEMM per projection fills the GPU by itself


def _group_list(T: int, groups: int, device):
    """Work list of a grouped GEMM whose group s owns rows [s T, (s + 1) T): (expert, first row, rows) per tile."""
    tn = 16
    while tn < T and tn < 64:
        tn <<= 1
    key = (T, groups, str(device))
    if key not in _GROUP_LISTS:
        tiles = [(s, s * T + r, min(tn, T - r)) for s in range(groups) for r in range(0, T, tn)]
        cols = [torch.tensor(c, dtype=torch.int32).to(device) for c in zip(*tiles)]
        _GROUP_LISTS[key] = (*cols, len(tiles))
    e, r0, nr, n = _GROUP_LISTS[key]
    return e, r0, nr, n, tn


def mix_projections(mixes: torch.Tensor, w, fmt: str):
    """r, k, v, g [T, H D] from the first four token-shift mixes, each through its own matrix."""
    from . import linear
    _, T, W = mixes.shape
    if w.rkvg_stack is None or not mixes.is_cuda:
        return tuple(linear(act_of(mixes[s], fmt), w.rkvg[s]) for s in range(4))
    n = w.rkvg_stack.N // 4
    if T > _GROUPED_MAX_ROWS:
        from . import QuantWeight
        if not w.rkvg:
            w.rkvg = [QuantWeight(fmt, n, W, w.rkvg_stack.data[s * n:(s + 1) * n]) for s in range(4)]
        return tuple(linear(act_of(mixes[s], fmt), w.rkvg[s]) for s in range(4))
    e, r0, nr, tiles, tn = _group_list(T, 4, mixes.device)
    y = linear(act_of(mixes[:4].reshape(4 * T, W), fmt), w.rkvg_stack, grouped=(e, r0, nr, n, tiles, tn))
    return tuple(y[s * T:(s + 1) * T] for s in range(4))


# ----------------------------------------------------------------------------- gated norm
class _GatedNormArgs(C.Structure):
    _fields_ = [("T", C.c_int), ("K", C.c_int), ("group", C.c_int), ("f32", C.c_int), ("x", C.c_void_p), ("w", C.c_void_p),
                ("gate", C.c_void_p), ("gate_ld", C.c_longlong), ("sigmoid_gate", C.c_int), ("eps", C.c_float),
                ("scale", C.c_float), ("out", C.c_void_p), ("out_ld", C.c_longlong)]


_native.register_optional("mb_gated_norm", [C.POINTER(_GatedNormArgs), C.c_void_p])


def gated_norm(x: torch.Tensor, w: torch.Tensor, gate: torch.Tensor, fmt: str, *, group: int, gate_act: str, eps: float,
               scale: float = 1.0, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """scale * act(gate) * w * x / rms(x over groups of `group` channels). x [T, K] fp32; ``gate`` [T, K] may
    be a column range; ``gate_act`` "silu" | "sigmoid"; ``out`` may be a column range of a wider matrix."""
    T, K = x.shape
    if out is None:
        out = torch.empty(T, K, dtype=DTYPE[fmt], device=x.device)
    if not x.is_cuda:
        g = x.view(T, K // group, group)
        n = (g * torch.rsqrt(g.pow(2).mean(-1, keepdim=True) + eps)).reshape(T, K)
        z = gate.float()
        act = torch.sigmoid(z) if gate_act == "sigmoid" else torch.nn.functional.silu(z)
        out.copy_(n * w.float() * act * scale)
        return out
    assert x.is_contiguous() and gate.stride(1) == 1 and out.stride(1) == 1 and gate.dtype == out.dtype == DTYPE[fmt]
    a = _GatedNormArgs(T, K, group, _f32(fmt), _ptr(x), _ptr(w), _ptr(gate), gate.stride(0), int(gate_act == "sigmoid"),
                       float(eps), float(scale), _ptr(out), out.stride(0))
    _native.check(_native.lib().mb_gated_norm(C.byref(a), _stream()), f"gated_norm[T={T} K={K}]")
    _count()
    return out


# ----------------------------------------------------------------------------- embedding, token side input
class _EmbedArgs(C.Structure):
    _fields_ = [("M", C.c_int), ("W", C.c_int), ("vocab", C.c_int), ("copy_f32", C.c_int), ("tokens", C.c_void_p), ("table", C.c_void_p),
                ("out", C.c_void_p), ("scale", C.c_float), ("copy", C.c_void_p), ("copy_ld", C.c_longlong), ("positions", C.c_void_p),
                ("pos", C.c_void_p), ("max_pos", C.c_int), ("norm_alpha", C.c_float), ("norm_w", C.c_void_p), ("norm_b", C.c_void_p),
                ("status", C.c_void_p)]


_native.register_optional("mb_embed_scaled", [C.POINTER(_EmbedArgs), C.c_void_p])
_native.register_optional("mb_side_gate", [C.c_void_p, C.c_void_p, C.c_void_p, C.c_longlong] + [C.c_int] * 4 +
                          [C.c_void_p, C.c_int, C.c_void_p, C.c_void_p])


def embed_scaled(ids: torch.Tensor, table: torch.Tensor, scale: float, copy: Optional[torch.Tensor] = None, *,
                 pos: Optional[torch.Tensor] = None, positions: Optional[torch.Tensor] = None, norm: Optional[DytNorm] = None) -> torch.Tensor:
    """fp32 [T, W] = norm(table[ids] * scale + pos[positions]), `pos` and `norm` optional; ``copy`` (may be a column
    range) takes the same in the activation type."""
    if not table.is_cuda:
        x = table[ids.long()].float() * scale
        if pos is not None:
            x = x + pos[positions.long()].float()
        if norm is not None:
            x = dyt_ref(x, norm)
        if copy is not None:
            copy.copy_(x)
        return x
    M, W = ids.numel(), table.shape[1]
    out = torch.empty(M, W, dtype=torch.float32, device=table.device)
    a = _EmbedArgs(M=M, W=W, vocab=table.shape[0], copy_f32=int(copy is not None and copy.dtype == torch.float32), tokens=_ptr(ids),
                   table=_ptr(table), out=_ptr(out), scale=float(scale), status=_ptr(runtime(table.device).status))
    if copy is not None:
        a.copy, a.copy_ld = _ptr(copy), copy.stride(0)
    if pos is not None:
        a.positions, a.pos, a.max_pos = _ptr(positions), _ptr(pos), pos.shape[0]
    if norm is not None:
        a.norm_alpha, a.norm_w, a.norm_b = norm.alpha, _ptr(norm.w), _ptr(norm.b)
    _native.check(_native.lib().mb_embed_scaled(C.byref(a), _stream()), "embed_scaled")
    _count()
    return out


def side_gate(z: torch.Tensor, ids: torch.Tensor, table: torch.Tensor, off: int, fmt: str) -> torch.Tensor:
    """gelu_tanh(z) * table[ids, off : off + dim]; z [T, dim] fp32."""
    T, dim = z.shape
    if not z.is_cuda:
        e = table[ids.long(), off:off + dim].float()
        return (torch.nn.functional.gelu(z, approximate="tanh") * e).to(DTYPE[fmt])
    out = torch.empty(T, dim, dtype=DTYPE[fmt], device=z.device)
    rc = _native.lib().mb_side_gate(_ptr(z), _ptr(ids), _ptr(table), table.stride(0), off, dim, T, table.shape[0], _ptr(out),
                                    _f32(fmt), _ptr(runtime(z.device).status), _stream())
    _native.check(rc, "side_gate")
    _count()
    return out


# ----------------------------------------------------------------------------- attention with its own head sizes
class _RopeDimsArgs(C.Structure):
    _fields_ = [("M", C.c_int), ("Hq", C.c_int), ("Hkv", C.c_int), ("dk", C.c_int), ("dv", C.c_int), ("rot", C.c_int),
                ("dkp", C.c_int), ("dvp", C.c_int), ("f32", C.c_int), ("qkv", C.c_void_p), ("qkv_ld", C.c_longlong),
                ("positions", C.c_void_p), ("slots", C.c_void_p), ("cos_tab", C.c_void_p), ("sin_tab", C.c_void_p),
                ("max_pos", C.c_int), ("q_out", C.c_void_p), ("k_cache", C.c_void_p), ("v_cache", C.c_void_p),
                ("num_slots", C.c_longlong), ("status", C.c_void_p), ("q_norm", C.c_void_p), ("k_norm", C.c_void_p), ("eps", C.c_float)]


class _SimtAttnArgs(C.Structure):
    _fields_ = [("q", C.c_void_p), ("k_cache", C.c_void_p), ("v_cache", C.c_void_p), ("block_table", C.c_void_p),
                ("max_blocks", C.c_int), ("q_start", C.c_void_p), ("q_len", C.c_void_p), ("ctx_len", C.c_void_p),
                ("total_rows", C.c_int), ("num_seqs", C.c_int), ("Hq", C.c_int), ("Hkv", C.c_int), ("dk", C.c_int),
                ("dv", C.c_int), ("dkp", C.c_int), ("dvp", C.c_int), ("block_size", C.c_int), ("num_blocks", C.c_longlong),
                ("scale", C.c_float), ("out_scale", C.c_float), ("sink", C.c_int), ("f32", C.c_int), ("out", C.c_void_p),
                ("out_ld", C.c_longlong), ("status", C.c_void_p), ("sink_w", C.c_void_p), ("window", C.c_int), ("keep", C.c_int),
                ("gate", C.c_void_p), ("gate_ld", C.c_longlong), ("gate_mode", C.c_int), ("softcap", C.c_float)]


_native.register_optional("mb_rope_dims", [C.POINTER(_RopeDimsArgs), C.c_void_p])
_native.register_optional("mb_attn_simt", [C.POINTER(_SimtAttnArgs), C.c_void_p])


def padded_head_dims(dk: int, dv: int, fmt: str) -> Tuple[int, int]:
    """Row lengths of the K and V pools: the tensor-core kernels' tiles (64 or 128 each, or 256 both) for bf16
    caches, the head sizes themselves where only the fp32 kernel serves the shape."""
    if fmt != "bf16" or max(dk, dv) > 256:
        return dk, dv
    if max(dk, dv) > 128:
        return 256, 256
    tile = lambda d: 64 if d <= 64 else 128
    return tile(dk), tile(dv)


def rope_dims(qkv: torch.Tensor, *, Hq: int, Hkv: int, dk: int, dv: int, positions, slots, k_cache, v_cache, cos, sin,
              fmt: str, q_norm: Optional[RmsNorm] = None, k_norm: Optional[RmsNorm] = None) -> torch.Tensor:
    """qkv [T, Hq dk | Hkv dk | Hkv dv | ...]: norm every q and k head (``q_norm`` / ``k_norm`` over dk), rotate the first 2 * cos.shape[1] dimensions of every q and k head
    (rotate-half pairing) and scatter k, v into caches [blocks, block, Hkv, padded]. Returns q [T, Hq, padded dk]."""
    M = qkv.shape[0]
    dkp, dvp = k_cache.shape[3], v_cache.shape[3]
    rot = 2 * cos.shape[1] if cos is not None else 0
    if not qkv.is_cuda:
        x = qkv.float()
        q = x[:, :Hq * dk].view(M, Hq, dk)
        k = x[:, Hq * dk:(Hq + Hkv) * dk].view(M, Hkv, dk)
        v = x[:, (Hq + Hkv) * dk:(Hq + Hkv) * dk + Hkv * dv].reshape(M, Hkv, dv)
        rms = lambda t, n: t if n is None else t * torch.rsqrt(t.pow(2).mean(-1, keepdim=True) + n.eps) * n.w.float()
        q, k = rms(q, q_norm), rms(k, k_norm)
        if rot:
            q, k = ref.apply_rope_neox(q, positions, cos, sin), ref.apply_rope_neox(k, positions, cos, sin)
        pad = torch.nn.functional.pad
        ok = slots >= 0
        idx = slots[ok].long()
        k_cache.view(-1, Hkv, dkp)[idx] = pad(k, (0, dkp - dk))[ok].to(k_cache.dtype)
        v_cache.view(-1, Hkv, dvp)[idx] = pad(v, (0, dvp - dv))[ok].to(v_cache.dtype)
        return pad(q, (0, dkp - dk)).to(DTYPE[fmt])
    assert qkv.dtype == k_cache.dtype == v_cache.dtype == DTYPE[fmt]
    q_out = torch.empty(M, Hq, dkp, dtype=DTYPE[fmt], device=qkv.device)
    a = _RopeDimsArgs(M, Hq, Hkv, dk, dv, rot, dkp, dvp, _f32(fmt), _ptr(qkv), qkv.stride(0), _ptr(positions), _ptr(slots),
                      _ptr(cos) if rot else None, _ptr(sin) if rot else None, cos.shape[0] if rot else 0, _ptr(q_out),
                      _ptr(k_cache), _ptr(v_cache), k_cache.shape[0] * k_cache.shape[1], _ptr(runtime(qkv.device).status))
    if q_norm is not None or k_norm is not None:
        a.q_norm, a.k_norm = _ptr(q_norm.w if q_norm else None), _ptr(k_norm.w if k_norm else None)
        a.eps = (q_norm or k_norm).eps
        assert q_norm is None or k_norm is None or q_norm.eps == k_norm.eps
    _native.check(_native.lib().mb_rope_dims(C.byref(a), _stream()), f"rope_dims[T={M}]")
    _count()
    return q_out


class _AttnRowsArgs(C.Structure):
    _fields_ = [("M", C.c_int), ("Hq", C.c_int), ("Hkv", C.c_int), ("dk", C.c_int), ("dv", C.c_int), ("rot", C.c_int), ("dkp", C.c_int),
                ("dvp", C.c_int), ("f32", C.c_int), ("y", C.c_void_p), ("ld", C.c_longlong), ("q_at", C.c_int), ("k_at", C.c_int),
                ("v_at", C.c_int), ("positions", C.c_void_p), ("slots", C.c_void_p), ("cos_tab", C.c_void_p), ("sin_tab", C.c_void_p),
                ("v_cos", C.c_void_p), ("v_sin", C.c_void_p), ("max_pos", C.c_int), ("q_norm", C.c_void_p), ("k_norm", C.c_void_p),
                ("eps", C.c_float), ("q_out", C.c_void_p), ("k_cache", C.c_void_p), ("v_cache", C.c_void_p), ("num_slots", C.c_longlong),
                ("status", C.c_void_p)]


_native.register_optional("mb_attention_rows", [C.POINTER(_AttnRowsArgs), C.c_void_p])
_native.register_optional("mb_turn_rows", [C.c_void_p, C.c_longlong] + [C.c_int] * 4 + [C.c_void_p] * 3 + [C.c_int, C.c_void_p, C.c_void_p])


def attention_rows(y: torch.Tensor, *, cols: Tuple[int, int, int], Hq: int, Hkv: int, dk: int, dv: int, positions, slots, k_cache, v_cache, rot,
                   fmt: str, q_norm: Optional[RmsNorm] = None, k_norm: Optional[RmsNorm] = None, v_rot=None) -> torch.Tensor:
    """Queries, keys and values at columns ``cols`` of y [T, *] (values may be the keys' own columns): norms over all
    heads of the projection (weights [Hq dk] and [Hkv dk]), rotation of q and k by ``rot`` = (cos, sin) tables over their leading
    dimensions and of v by ``v_rot`` over all of dv, k and v into caches [blocks, block, Hkv, padded]. Returns q
    [T, Hq, padded dk]."""
    M = y.shape[0]
    dkp, dvp = k_cache.shape[3], v_cache.shape[3]
    cos, sin = rot if rot is not None else (None, None)
    if not y.is_cuda:
        q, k, v = (y[:, at:at + n].float() for at, n in zip(cols, (Hq * dk, Hkv * dk, Hkv * dv)))
        q = (q if q_norm is None else q_norm.ref(q)).view(M, Hq, dk)
        k = (k if k_norm is None else k_norm.ref(k)).view(M, Hkv, dk)
        v = v.reshape(M, Hkv, dv)
        if cos is not None:
            q, k = ref.apply_rope_neox(q, positions, cos, sin), ref.apply_rope_neox(k, positions, cos, sin)
        if v_rot is not None:
            v = ref.apply_rope_neox(v, positions, *v_rot)
        pad = torch.nn.functional.pad
        ok = slots >= 0
        idx = slots[ok].long()
        k_cache.view(-1, Hkv, dkp)[idx] = pad(k, (0, dkp - dk))[ok].to(k_cache.dtype)
        v_cache.view(-1, Hkv, dvp)[idx] = pad(v, (0, dvp - dv))[ok].to(v_cache.dtype)
        return pad(q, (0, dkp - dk)).to(DTYPE[fmt])
    assert y.dtype == k_cache.dtype == v_cache.dtype == DTYPE[fmt] and y.stride(1) == 1
    for n in (q_norm, k_norm):
        assert n is None or not n.plus_one and n.scale == 1.0
    assert q_norm is None or k_norm is None or q_norm.eps == k_norm.eps
    q_out = torch.empty(M, Hq, dkp, dtype=DTYPE[fmt], device=y.device)
    a = _AttnRowsArgs(M, Hq, Hkv, dk, dv, 2 * cos.shape[1] if cos is not None else 0, dkp, dvp, _f32(fmt), _ptr(y), y.stride(0), *cols,
                      _ptr(positions), _ptr(slots), _ptr(cos), _ptr(sin))
    a.max_pos = (1 << 30) if cos is None and v_rot is None else min(t.shape[0] for t in (cos, v_rot and v_rot[0]) if t is not None)
    if v_rot is not None:
        a.v_cos, a.v_sin = _ptr(v_rot[0]), _ptr(v_rot[1])
    a.q_norm, a.k_norm = _ptr(q_norm.w if q_norm else None), _ptr(k_norm.w if k_norm else None)
    a.eps = (q_norm or k_norm).eps if q_norm or k_norm else 0.0
    a.q_out, a.k_cache, a.v_cache, a.num_slots = _ptr(q_out), _ptr(k_cache), _ptr(v_cache), k_cache.shape[0] * k_cache.shape[1]
    a.status = _ptr(runtime(y.device).status)
    _native.check(_native.lib().mb_attention_rows(C.byref(a), _stream()), f"attention_rows[T={M}]")
    _count()
    return q_out


def turn_rows(x: torch.Tensor, H: int, dv: int, positions, rot, fmt: str) -> torch.Tensor:
    """Every head's row of x [T, H dv] (may be a column range) turned by minus its position, in place."""
    cos, sin = rot
    if not x.is_cuda:
        x.copy_(ref.apply_rope_neox(x.reshape(-1, H, dv), positions, cos, -sin).reshape(-1, H * dv))
        return x
    assert x.stride(1) == 1 and x.dtype == DTYPE[fmt]
    rc = _native.lib().mb_turn_rows(_ptr(x), x.stride(0), x.shape[0], H, dv, _f32(fmt), _ptr(positions), _ptr(cos), _ptr(sin), cos.shape[0],
                                    _ptr(runtime(x.device).status), _stream())
    _native.check(rc, f"turn_rows[T={x.shape[0]}]")
    _count()
    return x


@dataclass
class OutputGate:
    """Sigmoid gates on an attention output: logits [T, heads] (one per head) or [T, heads * dv], may be a column range."""
    logits: torch.Tensor
    per_head: bool

    def values(self, Hq: int, dv: int) -> torch.Tensor:
        g = torch.sigmoid(self.logits.float())
        return g[:, :, None] if self.per_head else g.view(-1, Hq, dv)

    def into(self, a) -> None:
        assert self.logits.stride(1) == 1
        a.gate, a.gate_ld, a.gate_mode = _ptr(self.logits), self.logits.stride(0), 1 if self.per_head else 2


def attention_dims(q: torch.Tensor, k_cache, v_cache, batch, *, dk: int, dv: int, scale: float, sink, fmt: str,
                   out: torch.Tensor, out_scale: float = 1.0, kernel: str = "auto", window: int = 0, keep: int = 0,
                   gate: Optional[OutputGate] = None, softcap: float = 0.0, turn_back=None) -> torch.Tensor:
    """Causal paged attention of q [T, Hq, padded dk] into ``out`` [T, Hq * dv] (may be a column range), times
    ``out_scale`` and the ``gate``. ``sink``: True adds one to the softmax denominator, a tensor [Hq] (fp32) exp(sink) per
    head. ``softcap`` > 0: scores become softcap tanh(score / softcap). ``turn_back`` = (cos, sin) tables over dv / 2: every
    output row is turned by minus its position, in the kernel's own store where that has both halves. ``window`` > 0: a position sees itself, the window - 1 before it and the first ``keep``. The softmax weights keep
    32-bit precision: they enter the product with V as two bf16 terms. ``kernel``: auto | simt | mma | tc (tests)."""
    if turn_back is not None and not (q.is_cuda and gate is None and _turns(q, k_cache, v_cache, batch, dv, fmt, kernel, out)):
        kw = dict(dk=dk, dv=dv, scale=scale, sink=sink, fmt=fmt, out=out, out_scale=out_scale, window=window, keep=keep, softcap=softcap)
        assert gate is None
        return turn_rows(attention_dims(q, k_cache, v_cache, batch, kernel=kernel, **kw), q.shape[1], dv, batch.positions, turn_back, fmt)
    sink_w = sink if isinstance(sink, torch.Tensor) else None
    sink = sink_w is not None or bool(sink)
    keep = keep if window > 0 else 0
    T, Hq, dkp = q.shape
    nb, bs, Hkv, _ = k_cache.shape
    dvp = v_cache.shape[3]
    if not q.is_cuda:
        qs, ql, cl = batch.q_start.tolist(), batch.q_len.tolist(), batch.ctx_len.tolist()
        G = Hq // Hkv
        for s, n in enumerate(ql):
            if n <= 0:
                continue
            ctx = cl[s]
            blocks = batch.block_table[s, :(ctx + bs - 1) // bs].long()
            k = k_cache[blocks].reshape(-1, Hkv, dkp)[:ctx, :, :dk].float().repeat_interleave(G, 1)
            v = v_cache[blocks].reshape(-1, Hkv, dvp)[:ctx, :, :dv].float().repeat_interleave(G, 1)
            sc = torch.einsum("ihd,jhd->hij", q[qs[s]:qs[s] + n, :, :dk].double(), k.double()) * scale
            if softcap > 0:
                sc = softcap * torch.tanh(sc / softcap)
            i = torch.arange(ctx - n, ctx)[:, None]
            j = torch.arange(ctx)[None, :]
            hide = j > i
            if window > 0:
                hide = hide | ((i - j >= window) & (j >= keep))
            sc.masked_fill_(hide, float("-inf"))
            m = sc.amax(-1, keepdim=True)
            sk = sink_w.double()[:, None, None] if sink_w is not None else torch.zeros(1, 1, 1, dtype=torch.double)
            if sink:
                m = torch.maximum(m, sk)
            e = torch.exp(sc - m)
            den = e.sum(-1, keepdim=True) + (torch.exp(sk - m) if sink else 0.0)
            o = torch.einsum("hij,jhd->ihd", e / den, v.double()) * out_scale
            if gate is not None:
                o = o * gate.values(Hq, dv)[qs[s]:qs[s] + n].double()
            out[qs[s]:qs[s] + n] = o.reshape(n, Hq * dv).to(out.dtype)
        return out
    L, rt = _native.lib(), runtime(q.device)
    S, mq = batch.q_len.numel(), int(batch.max_q_len)
    assert out.stride(1) == 1 and out.dtype == DTYPE[fmt]
    G = Hq // Hkv
    if kernel == "auto":
        kernel = _attention_kernel(dkp, dvp, dv, G, mq, fmt, out, gate)
    if kernel == "simt":
        a = _SimtAttnArgs(_ptr(q), _ptr(k_cache), _ptr(v_cache), _ptr(batch.block_table), batch.block_table.stride(0),
                          _ptr(batch.q_start), _ptr(batch.q_len), _ptr(batch.ctx_len), T, S, Hq, Hkv, dk, dv, dkp, dvp, bs, nb,
                          float(scale), float(out_scale), int(sink), _f32(fmt), _ptr(out), out.stride(0), _ptr(rt.status), _ptr(sink_w),
                          window, keep)
        a.softcap = float(softcap)
        if gate is not None:
            gate.into(a)
        _native.check(L.mb_attn_simt(C.byref(a), _stream()), f"attn_simt[T={T}]")
        _count()
        return out
    if kernel == "tc":
        t = _native.AttnTcArgs()
        t.q, t.k_cache, t.v_cache, t.block_table = _ptr(q), _ptr(k_cache), _ptr(v_cache), _ptr(batch.block_table)
        t.q_start, t.q_len, t.ctx_len = _ptr(batch.q_start), _ptr(batch.q_len), _ptr(batch.ctx_len)
        t.out, t.status, t.num_blocks, t.max_blocks, t.num_seqs, t.max_q_len = _ptr(out), _ptr(rt.status), nb, \
            batch.block_table.stride(0), S, mq
        t.Hq, t.Hkv, t.D, t.block_size, t.scale, t.v_mn = Hq, Hkv, dkp, bs, float(scale), 1
        t.out_ld, t.out_scale, t.sink, t.split_p = out.stride(0), float(out_scale), int(sink), 1
        if turn_back is not None:
            t.turn_cos, t.turn_sin, t.turn_max = _ptr(turn_back[0]), _ptr(turn_back[1]), turn_back[0].shape[0]
        t.sink_w, t.window, t.keep, t.softcap = _ptr(sink_w), window, keep, float(softcap)
        if gate is not None:
            gate.into(t)
        _native.check(L.mb_attn_prefill_tc(C.byref(t), _stream()), "attn_prefill_tc")
        _count()
        return out
    from . import _ATTN_PART_TOKENS
    a = _native.AttnArgs()
    a.q, a.k_cache, a.v_cache = _ptr(q), _ptr(k_cache), _ptr(v_cache)
    a.block_table, a.max_blocks = _ptr(batch.block_table), batch.block_table.stride(0)
    a.q_start, a.q_len, a.ctx_len = _ptr(batch.q_start), _ptr(batch.q_len), _ptr(batch.ctx_len)
    a.num_seqs, a.max_q_len, a.max_ctx = S, mq, int(batch.max_ctx)
    a.Hq, a.Hkv, a.D, a.block_size, a.num_blocks, a.scale = Hq, Hkv, dkp, bs, nb, float(scale)
    a.out, a.total_rows, a.part_tokens, a.status = _ptr(out), T, _ATTN_PART_TOKENS, _ptr(rt.status)
    a.DV, a.dv, a.out_ld, a.out_scale, a.sink, a.split_p = dvp, dv, out.stride(0), float(out_scale), int(sink), 1
    if turn_back is not None:
        a.turn_cos, a.turn_sin, a.turn_max = _ptr(turn_back[0]), _ptr(turn_back[1]), turn_back[0].shape[0]
    a.sink_w, a.window, a.keep, a.softcap = _ptr(sink_w), window, keep, float(softcap)
    if gate is not None:
        gate.into(a)
    if G * mq <= 32:
        seen = L.mb_attn_visible(int(batch.max_ctx), mq, window, keep)
        rt.ensure_attn_ws(L.mb_attn_ws_bytes(T, Hq, dvp, seen, _ATTN_PART_TOKENS))
    a.ws, a.ws_bytes = _ptr(rt.attn_ws), rt.attn_ws.numel()
    _native.check(L.mb_paged_attention(C.byref(a), _stream()), f"attention_dims[T={T}]")
    _count()
    return out


def _attention_kernel(dkp: int, dvp: int, dv: int, G: int, mq: int, fmt: str, out: torch.Tensor, gate) -> str:
    """Which kernel serves a step: simt (fp32, or sizes without tiles), tc (long portions on tcgen05) or mma."""
    if not (fmt == "bf16" and dkp in (64, 128, 256) and dvp in (64, 128, 256) and (dkp == dvp or max(dkp, dvp) <= 128)
            and (dv != dvp or (out.stride(0) % 2 == 0 and out.data_ptr() % 4 == 0))):
        return "simt"
    if tc_serves(dkp, dvp, dv, out, gate) and mq >= 128:
        return "tc"
    return "simt" if dkp == 256 and 16 < G * mq <= 32 else "mma"    # between the two row-tile limits of the 256-wide tiles


def _turns(q, k_cache, v_cache, batch, dv: int, fmt: str, kernel: str, out: torch.Tensor) -> bool:
    """Whether the kernel that serves a step turns its output rows back itself."""
    G, mq, dvp = q.shape[1] // k_cache.shape[2], int(batch.max_q_len), v_cache.shape[3]
    if kernel == "auto":
        kernel = _attention_kernel(q.shape[2], dvp, dv, G, mq, fmt, out, None)
    return kernel == "tc" or (kernel == "mma" and dv % 8 == 0 and (G * mq <= 32 or dv == dvp))


def tc_serves(dkp: int, dvp: int, dv: int, out: torch.Tensor, gate: Optional[OutputGate] = None) -> bool:
    """Shapes of the tcgen05 prefill kernel: equal 128- or 256-wide tiles stored (and gated) whole in 16-byte vectors."""
    from . import _ATTN_TC
    if gate is not None and not gate.per_head and (gate.logits.stride(0) % 8 or gate.logits.data_ptr() % 16):
        return False
    return _ATTN_TC and dkp == dvp == dv and dkp in (128, 256) and out.stride(0) % 8 == 0 and out.data_ptr() % 16 == 0


# ----------------------------------------------------------------------------- decaying linear attention
class _LinearAttnArgs(C.Structure):
    _fields_ = [("q", C.c_void_p), ("k", C.c_void_p), ("v", C.c_void_p), ("q_ld", C.c_longlong), ("k_ld", C.c_longlong),
                ("v_ld", C.c_longlong), ("H", C.c_int), ("DK", C.c_int), ("DV", C.c_int), ("f32", C.c_int), ("log_w", C.c_void_p),
                ("decay", C.c_void_p), ("u", C.c_void_p), ("state", C.c_void_p), ("out", C.c_void_p), ("q_start", C.c_void_p),
                ("q_len", C.c_void_p), ("positions", C.c_void_p), ("slots", C.c_void_p), ("num_seqs", C.c_int),
                ("num_slots", C.c_int), ("write_state", C.c_int), ("write_out", C.c_int), ("status", C.c_void_p),
                ("decode", C.c_int), ("norm_w", C.c_void_p), ("gate", C.c_void_p), ("gate_ld", C.c_longlong),
                ("sigmoid_gate", C.c_int), ("eps", C.c_float), ("scale", C.c_float), ("norm_out", C.c_void_p),
                ("norm_out_ld", C.c_longlong), ("lr_a1", C.c_void_p), ("lr_a1_ld", C.c_longlong), ("lr_a2", C.c_void_p),
                ("lr_bias", C.c_void_p), ("lr_rank", C.c_int), ("lr_c", C.c_float)]


class _LinearChunkedArgs(C.Structure):
    _fields_ = [("q", C.c_void_p), ("k", C.c_void_p), ("v", C.c_void_p), ("q_ld", C.c_longlong), ("k_ld", C.c_longlong),
                ("v_ld", C.c_longlong), ("H", C.c_int), ("DK", C.c_int), ("DV", C.c_int), ("total_rows", C.c_int), ("log_w", C.c_void_p),
                ("decay", C.c_void_p), ("u", C.c_void_p), ("state", C.c_void_p), ("out", C.c_void_p), ("ws", C.c_void_p),
                ("ws_bytes", C.c_size_t), ("q_start", C.c_void_p), ("q_len", C.c_void_p), ("positions", C.c_void_p),
                ("slots", C.c_void_p), ("num_seqs", C.c_int), ("num_slots", C.c_int), ("max_q_len", C.c_int),
                ("write_state", C.c_int), ("status", C.c_void_p)]


_native.register_optional("mb_linear_attn", [C.POINTER(_LinearAttnArgs), C.c_void_p])
_native.register_optional("mb_linear_chunked", [C.POINTER(_LinearChunkedArgs), C.c_void_p])
_CHUNK_MIN_TOKENS = 48           # portions at least this long take the chunked kernels
_CHUNK_WS_MAX = 4 << 30
_chunk_ws: dict = {}


def _linear_chunked(q, k, v, state, batch, H, dk, dv, log_w, decay, u, write_state):
    """Chunked kernels (csrc/linear_chunked.cu); None for shapes, layouts or sizes they do not take."""
    if dk not in (64, 128) or dv not in (64, 128) or q.dtype != torch.bfloat16 or (u is not None and log_w is None):
        return None
    if any(t.data_ptr() % 16 or t.stride(0) % 8 for t in (q, k, v)):
        return None
    L, dev, T, S = _native.lib(), q.device, q.shape[0], batch.q_len.numel()
    L.mb_linear_chunked_ws_bytes.restype, L.mb_linear_chunked_ws_bytes.argtypes = C.c_size_t, [C.c_int] * 5
    need = int(L.mb_linear_chunked_ws_bytes(T, S, H, dk, dv))
    if need > _CHUNK_WS_MAX:
        return None
    ws = _chunk_ws.get(dev)
    if ws is None or ws.numel() < need:
        if torch.cuda.is_current_stream_capturing():
            return None
        ws = _chunk_ws[dev] = torch.empty(int(need * 1.25), dtype=torch.uint8, device=dev)
    out = torch.empty(T, H * dv, dtype=torch.float32, device=dev)
    a = _LinearChunkedArgs(_ptr(q), _ptr(k), _ptr(v), q.stride(0), k.stride(0), v.stride(0), H, dk, dv, T, _ptr(log_w), _ptr(decay),
                           _ptr(u), _ptr(state), _ptr(out), _ptr(ws), ws.numel(), _ptr(batch.q_start), _ptr(batch.q_len),
                           _ptr(batch.positions), _ptr(batch.state_slots), S, state.shape[0], int(batch.max_q_len), int(write_state),
                           _ptr(runtime(dev).status))
    _native.check(L.mb_linear_chunked(C.byref(a), _stream()), f"linear_chunked[T={T} H={H}]")
    _count(3)
    return out


@dataclass
class LowRankDecay:
    """Decays sigmoid(a2 a1 + bias)^c per token and key channel, a1 [T, rank] being their projection's first half."""
    a1: torch.Tensor                       # activation type, may be a column range
    a2: torch.Tensor                       # bf16 [H dk, rank]
    bias: torch.Tensor                     # fp32 [H dk]
    c: float
    a2_lin: object = None                  # bf16 QuantWeight of a2: prefill-sized steps run on the tensor cores

    def log(self) -> torch.Tensor:
        """c log(sigmoid(a2 a1 + bias)), fp32 [T, H dk]."""
        if not self.a1.is_cuda:
            z = (self.a1.double() @ self.a2.double().t()).float() + self.bias
            return self.c * ref.log_sigmoid(z)
        if self.a2_lin is not None and self.a1.shape[0] >= _DECAY_TC_MIN_ROWS:
            from . import linear
            a1 = self.a1 if self.a1.stride(0) % 8 == 0 and self.a1.data_ptr() % 16 == 0 else self.a1.contiguous()
            return linear(act_of(a1, "bf16"), self.a2_lin, out_f32=True, log_sigmoid=(self.bias, self.c))
        out = torch.empty(self.a1.shape[0], self.a2.shape[0], dtype=torch.float32, device=self.a1.device)
        return gemm_simt(self.a1, self.a2, out, epilogue=7, bias=self.bias, epi_a=self.c)


def _decode_ok(batch, dk: int, dv: int, kernel: str) -> bool:
    """The streaming decode kernel: one row per sequence, whole 16-byte vectors, heads up to 256 x 256."""
    return kernel in ("auto", "decode") and int(batch.max_q_len) == 1 and dv % 4 == 0 and max(dk, dv) <= 256


def linear_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, state: torch.Tensor, batch, *, heads: int, dk: int, dv: int,
                     fmt: str, log_w: Optional[torch.Tensor] = None, decay: Optional[torch.Tensor] = None,
                     u: Optional[torch.Tensor] = None, write_state: bool = True, write_out: bool = True,
                     kernel: str = "auto", norm: Optional[dict] = None, low_rank: Optional[LowRankDecay] = None) -> Optional[torch.Tensor]:
    """Per head S_t = diag(w_t) S_(t-1) + k_t v_t^T over a ragged batch; w_t = ``decay`` [H], or exp(``log_w``
    [T, H dk]), or ``low_rank`` (computed inside the decode kernel where that serves the step). Output q_t^T S_t, or with ``u`` [H, dk] q_t^T (S_(t-1) + diag(u) k_t v_t^T). q, k, v [T, *]
    may be column ranges; state [slots, H, dk, dv] fp32. Returns fp32 [T, H dv]. ``kernel``: auto | seq |
    chunked | decode (tests). ``norm`` (keyword arguments of ``gated_norm`` with group = dv, and ``w``, ``gate``,
    ``out``): the gated per-head norm of the output goes to norm["out"], inside the decode kernel where that
    serves the step; nothing is returned then."""
    T, H = q.shape[0], heads
    if low_rank is not None and not (q.is_cuda and _decode_ok(batch, dk, dv, kernel)):
        log_w, low_rank = low_rank.log(), None
    if norm is not None:
        kw = dict(heads=H, dk=dk, dv=dv, fmt=fmt, log_w=log_w, decay=decay, u=u, write_state=write_state, kernel=kernel)
        if not (q.is_cuda and _decode_ok(batch, dk, dv, kernel)):
            core = linear_attention(q, k, v, state, batch, **kw)
            gated_norm(core, norm["w"], norm["gate"], fmt, group=dv, gate_act=norm["gate_act"], eps=norm["eps"], scale=norm["scale"],
                       out=norm["out"])
            return None
    if not q.is_cuda:
        out = torch.zeros(T, H * dv, dtype=torch.float32)
        qs, ql, sl = batch.q_start.tolist(), batch.q_len.tolist(), batch.state_slots.tolist()
        qf, kf, vf = q.float().view(T, H, dk), k.float().view(T, H, dk), v.float().view(T, H, dv)
        w = torch.exp(log_w).view(T, H, dk) if log_w is not None else decay.float()[None, :, None].expand(T, H, dk)
        for s, n in enumerate(ql):
            if n <= 0:
                continue
            S = torch.zeros(H, dk, dv) if int(batch.positions[qs[s]]) == 0 else state[sl[s]].clone()
            for t in range(qs[s], qs[s] + n):
                kv = kf[t][:, :, None] * vf[t][:, None, :]
                if u is not None:
                    out[t] = ((S + u[:, :, None] * kv) * qf[t][:, :, None]).sum(1).reshape(-1)
                S = w[t][:, :, None] * S + kv
                if u is None:
                    out[t] = (S * qf[t][:, :, None]).sum(1).reshape(-1)
            if write_state:
                state[sl[s]] = S
        return out if write_out else None
    assert q.dtype == k.dtype == v.dtype == DTYPE[fmt] and q.stride(1) == k.stride(1) == v.stride(1) == 1
    dev = q.device
    if kernel == "chunked" or (kernel == "auto" and write_out and int(batch.max_q_len) >= _CHUNK_MIN_TOKENS):
        out = _linear_chunked(q, k, v, state, batch, H, dk, dv, log_w, decay, u, write_state)
        if out is not None:
            return out
        assert kernel == "auto", "the chunked kernels do not take this shape"
    out = torch.empty(T, H * dv, dtype=torch.float32, device=dev) if write_out and norm is None else None
    a = _LinearAttnArgs(_ptr(q), _ptr(k), _ptr(v), q.stride(0), k.stride(0), v.stride(0), H, dk, dv, _f32(fmt), _ptr(log_w),
                        _ptr(decay), _ptr(u), _ptr(state), _ptr(out), _ptr(batch.q_start), _ptr(batch.q_len),
                        _ptr(batch.positions), _ptr(batch.state_slots), batch.q_len.numel(), state.shape[0], int(write_state),
                        int(write_out), _ptr(runtime(dev).status))
    a.decode = int(_decode_ok(batch, dk, dv, kernel))
    if low_rank is not None:
        lr = low_rank
        assert lr.a1.stride(1) == 1 and lr.a1.dtype == DTYPE[fmt] and lr.a2.is_contiguous()
        a.lr_a1, a.lr_a1_ld, a.lr_a2, a.lr_bias, a.lr_rank, a.lr_c = (_ptr(lr.a1), lr.a1.stride(0), _ptr(lr.a2), _ptr(lr.bias),
                                                                     lr.a2.shape[1], float(lr.c))
    if norm is not None:
        g, o = norm["gate"], norm["out"]
        assert g.stride(1) == 1 and o.stride(1) == 1 and g.dtype == o.dtype == DTYPE[fmt]
        a.norm_w, a.gate, a.gate_ld, a.sigmoid_gate = _ptr(norm["w"]), _ptr(g), g.stride(0), int(norm["gate_act"] == "sigmoid")
        a.eps, a.scale, a.norm_out, a.norm_out_ld = float(norm["eps"]), float(norm["scale"]), _ptr(o), o.stride(0)
    _native.check(_native.lib().mb_linear_attn(C.byref(a), _stream()), f"linear_attn[T={T} H={H}]")
    _count()
    return out


# ----------------------------------------------------------------------------- CUDA-core GEMM
class _SimtGemmArgs(C.Structure):
    _fields_ = [("M", C.c_int), ("N", C.c_int), ("K", C.c_int), ("x_bf16", C.c_int), ("w_bf16", C.c_int), ("out_bf16", C.c_int),
                ("X", C.c_void_p), ("ldx", C.c_longlong), ("W", C.c_void_p), ("ldw", C.c_longlong), ("out", C.c_void_p),
                ("ldo", C.c_longlong), ("a_op", C.c_int), ("epilogue", C.c_int), ("bias", C.c_void_p), ("epi_a", C.c_float),
                ("epi_b", C.c_float), ("epi_n", C.c_int), ("tile_expert", C.c_void_p), ("tile_row0", C.c_void_p), ("tile_nrows", C.c_void_p),
                ("max_tiles", C.c_int), ("tile_rows", C.c_int), ("row_index", C.c_void_p), ("row_div", C.c_int)]


_native.register_optional("mb_gemm_simt", [C.POINTER(_SimtGemmArgs), C.c_void_p])


def gemm_simt(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor, *, tanh_in: bool = False, epilogue: int = 0, bias=None,
              epi_a: float = 0.0, epi_b: float = 0.0, epi_n: int = 0, grouped=None, row_index=None, row_div: int = 1) -> torch.Tensor:
    """out = epilogue(x w^T). ``grouped`` = (tile_expert, tile_row0, tile_nrows, rows of w per expert, max_tiles,
    tile_rows): x's rows are sorted by expert, or read as x[row_index // row_div]."""
    M, K = x.shape
    N = w.shape[0]
    if row_index is not None:
        M = row_index.numel()
    assert x.stride(1) == 1 and w.stride(1) == 1 and out.stride(1) == 1
    bf = torch.bfloat16
    a = _SimtGemmArgs(M, N, K, int(x.dtype == bf), int(w.dtype == bf), int(out.dtype == bf), _ptr(x), x.stride(0), _ptr(w),
                      w.stride(0), _ptr(out), out.stride(0), int(tanh_in), epilogue, _ptr(bias), float(epi_a), float(epi_b), epi_n)
    if grouped is not None:
        a.tile_expert, a.tile_row0, a.tile_nrows = _ptr(grouped[0]), _ptr(grouped[1]), _ptr(grouped[2])
        a.N, a.max_tiles, a.tile_rows = grouped[3], grouped[4], grouped[5]
    if row_index is not None:
        a.row_index, a.row_div = _ptr(row_index), row_div
    _native.check(_native.lib().mb_gemm_simt(C.byref(a), _stream()), f"gemm_simt[M={M} N={N} K={K}]")
    _count()
    return out


_native.register_optional("mb_tanh_split", [C.c_void_p, C.c_void_p, C.c_int, C.c_int, C.c_void_p])
_DECAY_TC_MIN_ROWS = 256         # from here on the tensor cores, below the CUDA-core GEMM


def log_decay(z: torch.Tensor, w2: torch.Tensor, w0: torch.Tensor, w2_twice=None) -> torch.Tensor:
    """-exp(tanh(z) w2^T + w0) in fp32: the logarithm of the decay exp(-exp(.)). z [T, rank] fp32. ``w2_twice``
    (bf16 QuantWeight [w2 | w2]): prefill-sized steps run it on the tensor cores, tanh(z) entering as two bf16 terms."""
    if z.is_cuda and w2_twice is not None and z.shape[0] >= _DECAY_TC_MIN_ROWS:
        from . import linear
        T, R = z.shape
        zs = torch.empty(T, 2 * R, dtype=torch.bfloat16, device=z.device)
        _native.check(_native.lib().mb_tanh_split(_ptr(z), _ptr(zs), T, R, _stream()), "tanh_split")
        _count()
        return linear(act_of(zs, "bf16"), w2_twice, out_f32=True, neg_exp_bias=w0)
    if not z.is_cuda:
        return -torch.exp((torch.tanh(z).double() @ w2.double().t()).float() + w0)
    out = torch.empty(z.shape[0], w2.shape[0], dtype=torch.float32, device=z.device)
    return gemm_simt(z, w2, out, tanh_in=True, epilogue=4, bias=w0)
