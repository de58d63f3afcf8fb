"""Delta-rule linear attention over a ragged batch: the gated rule (one decay and step size per head) and the general one
(a decay and a removal rate per key channel, the key itself written). CUDA tensors run ``csrc/delta_attn.cu`` and
``csrc/delta_chunked.cu``, CPU tensors the restatement below.
"""
from __future__ import annotations

import ctypes as C
import math
from dataclasses import dataclass
from typing import Optional, Union

import torch

from . import _count, _native, _ptr, _stream, runtime
from .canon import _sequences
from .mixers import _DECAY_TC_MIN_ROWS, DTYPE, _f32, act_of, gated_norm, gemm_simt

UNIT_EPS = 1e-6


@dataclass
class GatedRule:
    """S <- g S; S <- S + k (beta (v - S^T k))^T, g = exp(-exp(A_log) softplus(decay + dt_bias)), beta = sigmoid(step)."""
    decay: torch.Tensor            # logits [T, H], may be a column range
    step: torch.Tensor             # logits [T, H], rows as far apart as decay's
    A_log: torch.Tensor            # fp32 [H]
    dt_bias: torch.Tensor          # fp32 [H]


@dataclass
class BoundedDecay:
    """Log decays c sigmoid(tanh(z) w2^T + bias) of every key channel, c < 0: z [T, rank] is their projection's first half."""
    z: torch.Tensor                # activation type, may be a column range
    w2: torch.Tensor               # bf16 [H dk, rank]
    bias: torch.Tensor             # fp32 [H dk]
    c: float
    w2_twice: object = None        # bf16 QuantWeight [w2 | w2]: prefill-sized steps run on the tensor cores, tanh as two terms

    def log(self) -> torch.Tensor:
        """fp32 [T, H dk]."""
        T, R = self.z.shape
        if not self.z.is_cuda:
            return self.c * torch.sigmoid((torch.tanh(self.z.double()) @ self.w2.double().t()).float() + self.bias)
        if self.w2_twice is not None and T >= _DECAY_TC_MIN_ROWS:
            from . import linear
            zs = torch.empty(T, 2 * R, dtype=torch.bfloat16, device=self.z.device)
            rc = _native.lib().mb_tanh_split_cols(_ptr(self.z), self.z.stride(0), int(self.z.dtype == torch.bfloat16), _ptr(zs), T, R, _stream())
            _native.check(rc, "tanh_split_cols")
            _count()
            return linear(act_of(zs, "bf16"), self.w2_twice, out_f32=True, sigmoid=(self.bias, self.c))
        out = torch.empty(T, self.w2.shape[0], dtype=torch.float32, device=self.z.device)
        return gemm_simt(self.z, self.w2, out, tanh_in=True, epilogue=9, bias=self.bias, epi_a=self.c)


@dataclass
class GeneralRule:
    """S <- diag(w) S - (a u) (u^T S)^T + k v^T, u = k / |k|, a = sigmoid(removal), w from ``decay``."""
    removal: torch.Tensor          # logits [T, H dk], may be a column range
    decay: Union[BoundedDecay, torch.Tensor]     # or the log decays, fp32 [T, H dk]
    bound: float = -math.inf       # no log decay is below this (BoundedDecay: its own constant)

    def logs(self) -> "GeneralRule":
        """The same with the decays as a tensor."""
        return GeneralRule(self.removal, self.decay.log(), self.decay.c) if isinstance(self.decay, BoundedDecay) else self


class _DeltaInputs(C.Structure):
    _fields_ = [("q", C.c_void_p), ("k", C.c_void_p), ("v", C.c_void_p), ("q_ld", C.c_longlong), ("k_ld", C.c_longlong),
                ("v_ld", C.c_longlong), ("H", C.c_int), ("HK", C.c_int), ("DK", C.c_int), ("DV", C.c_int), ("f32", C.c_int),
                ("general", C.c_int), ("decay", C.c_void_p), ("step", C.c_void_p), ("gate_ld", C.c_longlong), ("A_log", C.c_void_p),
                ("dt_bias", C.c_void_p), ("removal", C.c_void_p), ("removal_ld", C.c_longlong), ("log_w", C.c_void_p)]


class _DeltaAttnArgs(C.Structure):
    _fields_ = [("inp", _DeltaInputs), ("lr_z", C.c_void_p), ("lr_ld", C.c_longlong), ("lr_w2", C.c_void_p), ("lr_bias", C.c_void_p),
                ("lr_rank", C.c_int), ("lr_c", C.c_float), ("state", C.c_void_p), ("out", C.c_void_p), ("q_start", C.c_void_p),
                ("q_len", C.c_void_p), ("positions", C.c_void_p), ("slots", C.c_void_p), ("num_seqs", C.c_int), ("num_slots", C.c_int),
                ("write_state", C.c_int), ("write_out", C.c_int), ("status", C.c_void_p), ("decode", C.c_int), ("norm_w", C.c_void_p),
                ("gate", C.c_void_p), ("gate_ld", C.c_longlong), ("sigmoid_gate", C.c_int), ("eps", C.c_float), ("scale", C.c_float),
                ("norm_out", C.c_void_p), ("norm_out_ld", C.c_longlong)]


class _DeltaChunkedArgs(C.Structure):
    _fields_ = [("inp", _DeltaInputs), ("state", C.c_void_p), ("out", C.c_void_p), ("ws", C.c_void_p), ("ws_bytes", C.c_size_t),
                ("q_start", C.c_void_p), ("q_len", C.c_void_p), ("positions", C.c_void_p), ("slots", C.c_void_p), ("total_rows", C.c_int),
                ("num_seqs", C.c_int), ("num_slots", C.c_int), ("max_q_len", C.c_int), ("write_state", C.c_int), ("status", C.c_void_p),
                ("norm_w", C.c_void_p), ("gate", C.c_void_p), ("gate_ld", C.c_longlong), ("sigmoid_gate", C.c_int), ("eps", C.c_float),
                ("scale", C.c_float), ("norm_out", C.c_void_p), ("norm_out_ld", C.c_longlong)]


_native.register_optional("mb_delta_chunked", [C.POINTER(_DeltaChunkedArgs), C.c_void_p])
_native.register_optional("mb_delta_attn", [C.POINTER(_DeltaAttnArgs), C.c_void_p])
_native.register_optional("mb_tanh_split_cols", [C.c_void_p, C.c_longlong, C.c_int, C.c_void_p, C.c_int, C.c_int, C.c_void_p])
_LOW_RANK_MAX = 64               # ranks up to here are computed inside the decode kernel
_CHUNK = 64
_CHUNK_MIN_TOKENS = 48           # portions at least this long take the chunked kernels
_CHUNK_WS_MAX = 4 << 30
_chunk_ws: dict = {}


def _unit(x: torch.Tensor) -> torch.Tensor:
    return x * torch.rsqrt(x.pow(2).sum(-1, keepdim=True) + UNIT_EPS)


def _delta_ref(q, k, v, rule, state, batch, H, HK, dk, dv, write_state):
    T = q.shape[0]
    rep = lambda x: x.float().view(T, HK, dk).repeat_interleave(H // HK, 1)
    qf, kf, vf = rep(q), rep(k), v.float().reshape(T, H, dv)
    u = _unit(kf)
    if isinstance(rule, GatedRule):
        g = torch.exp(-torch.exp(rule.A_log) * torch.nn.functional.softplus(rule.decay.float() + rule.dt_bias, threshold=40.0))
        beta, qf = torch.sigmoid(rule.step.float()), _unit(qf) * dk ** -0.5
    else:
        w, a = torch.exp(rule.decay).view(T, H, dk), torch.sigmoid(rule.removal.float()).view(T, H, dk)
    out = torch.zeros(T, H * dv)
    for r, n, slot, fresh in _sequences(batch):
        S = torch.zeros(H, dk, dv) if fresh else state[slot].clone()
        for t in range(r, r + n):
            d = (S * u[t][:, :, None]).sum(1)                            # S^T u, [H, dv]
            if isinstance(rule, GatedRule):
                S = g[t][:, None, None] * S + u[t][:, :, None] * (beta[t][:, None] * (vf[t] - g[t][:, None] * d))[:, None, :]
            else:
                S = w[t][:, :, None] * S - (a[t] * u[t])[:, :, None] * d[:, None, :] + kf[t][:, :, None] * vf[t][:, None, :]
            out[t] = (S * qf[t][:, :, None]).sum(1).reshape(-1)
        if write_state:
            state[slot] = S
    return out


def _chunked_serves(q, k, v, rule, dk: int, dv: int) -> bool:
    """Head sizes of the chunked kernels, whole 16-byte vectors, and decays whose factors stay in range over a chunk."""
    if q.dtype != torch.bfloat16 or dk not in (64, 128) or dv not in (64, 128):
        return False
    rows = [q, k, v]
    if isinstance(rule, GeneralRule):
        rows.append(rule.removal)
        bound = rule.decay.c if isinstance(rule.decay, BoundedDecay) else rule.bound
        if bound * _CHUNK * math.log2(math.e) < -100:
            return False
    return not any(t.data_ptr() % 16 or t.stride(0) % 8 for t in rows)


def _norm_args(a, norm, fmt: str) -> None:
    g, o = norm["gate"], norm["out"]
    assert g.stride(1) == 1 and o.stride(1) == 1 and g.dtype == o.dtype == DTYPE[fmt]
    a.norm_w, a.gate, a.gate_ld, a.sigmoid_gate = _ptr(norm["w"]), _ptr(g), g.stride(0), int(norm["gate_act"] == "sigmoid")
    a.eps, a.scale, a.norm_out, a.norm_out_ld = float(norm["eps"]), float(norm["scale"]), _ptr(o), o.stride(0)


def _delta_chunked(i, state, batch, T: int, write_state: bool, norm):
    """Chunked kernels (csrc/delta_chunked.cu); False when their workspace would be unreasonably large. Returns the rows,
    or None where they went to norm["out"]."""
    L, dev, S = _native.lib(), state.device, batch.q_len.numel()
    L.mb_delta_chunked_ws_bytes.restype, L.mb_delta_chunked_ws_bytes.argtypes = C.c_size_t, [C.c_int] * 5
    need = int(L.mb_delta_chunked_ws_bytes(T, S, i.H, i.DK, i.DV))
    if need > _CHUNK_WS_MAX:
        return False
    ws = _chunk_ws.get(dev)
    if ws is None or ws.numel() < need:
        if torch.cuda.is_current_stream_capturing():
            return False
        ws = _chunk_ws[dev] = torch.empty(int(need * 1.25), dtype=torch.uint8, device=dev)
    if norm is not None and any(t.stride(0) % 2 or t.data_ptr() % 4 for t in (norm["gate"], norm["out"])):
        return False
    out = None if norm is not None else torch.empty(T, i.H * i.DV, dtype=torch.float32, device=dev)
    a = _DeltaChunkedArgs(i, _ptr(state), _ptr(out), _ptr(ws), ws.numel(), _ptr(batch.q_start), _ptr(batch.q_len), _ptr(batch.positions),
                          _ptr(batch.state_slots), T, S, state.shape[0], int(batch.max_q_len), int(write_state), _ptr(runtime(dev).status))
    if norm is not None:
        _norm_args(a, norm, "bf16")
    _native.check(L.mb_delta_chunked(C.byref(a), _stream()), f"delta_chunked[T={T} H={i.H}]")
    _count(3)
    return out


def delta_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, rule, state: torch.Tensor, batch, *, heads: int, dk: int, dv: int,
                    fmt: str, key_heads: Optional[int] = None, write_state: bool = True, write_out: bool = True, kernel: str = "auto",
                    norm: Optional[dict] = None) -> Optional[torch.Tensor]:
    """q, k [T, key_heads dk], v [T, heads dv] (may be column ranges), state [slots, heads, dk, dv] fp32, ``rule`` a GatedRule
    or a GeneralRule. Returns S^T q after every update, fp32 [T, heads dv]. ``norm`` (keyword arguments of ``gated_norm``
    with group = dv, and ``w``, ``gate``, ``out``): the gated per-head norm of the output goes to norm["out"], inside the
    decode kernel where that serves the step; nothing is returned then. ``kernel``: auto | seq | decode | chunked (tests)."""
    T, H, HK = q.shape[0], heads, key_heads or heads
    general = isinstance(rule, GeneralRule)
    decode = q.is_cuda and kernel in ("auto", "decode") and int(batch.max_q_len) == 1 and dv % 4 == 0 and dv <= 256
    low_rank = rule.decay if general and isinstance(rule.decay, BoundedDecay) else None
    if low_rank is not None and not (decode and low_rank.w2.shape[1] <= _LOW_RANK_MAX):
        rule, low_rank = rule.logs(), None
    chunked = q.is_cuda and write_out and _chunked_serves(q, k, v, rule, dk, dv) and \
        (kernel == "chunked" or (kernel == "auto" and int(batch.max_q_len) >= _CHUNK_MIN_TOKENS))
    if norm is not None and not decode and not chunked:
        core = delta_attention(q, k, v, rule, state, batch, heads=H, dk=dk, dv=dv, fmt=fmt, key_heads=HK, write_state=write_state, kernel=kernel)
        gated_norm(core, norm["w"], norm["gate"], fmt, group=dv, gate_act=norm["gate_act"], eps=norm["eps"], scale=norm["scale"], out=norm["out"])
        return None
    if not q.is_cuda:
        out = _delta_ref(q, k, v, rule, state, batch, H, HK, dk, dv, write_state)
        return out if write_out else None
    assert q.dtype == k.dtype == v.dtype == DTYPE[fmt] and q.stride(1) == k.stride(1) == v.stride(1) == 1
    dev = q.device
    i = _DeltaInputs(_ptr(q), _ptr(k), _ptr(v), q.stride(0), k.stride(0), v.stride(0), H, HK, dk, dv, _f32(fmt), int(general))
    if general:
        assert rule.removal.dtype == DTYPE[fmt] and rule.removal.stride(1) == 1
        i.removal, i.removal_ld = _ptr(rule.removal), rule.removal.stride(0)
        if low_rank is None:
            assert rule.decay.is_contiguous() and rule.decay.dtype == torch.float32
            i.log_w = _ptr(rule.decay)
    else:
        assert rule.decay.dtype == rule.step.dtype == DTYPE[fmt] and rule.decay.stride() == rule.step.stride() and rule.decay.stride(1) == 1
        i.decay, i.step, i.gate_ld, i.A_log, i.dt_bias = (_ptr(rule.decay), _ptr(rule.step), rule.decay.stride(0), _ptr(rule.A_log),
                                                          _ptr(rule.dt_bias))
    if chunked:
        out = _delta_chunked(i, state, batch, T, write_state, norm)
        if out is not False:
            return out
        return delta_attention(q, k, v, rule, state, batch, heads=H, dk=dk, dv=dv, fmt=fmt, key_heads=HK, write_state=write_state, kernel="seq",
                               norm=norm)
    assert kernel != "chunked", "the chunked kernels do not take this shape"
    out = torch.empty(T, H * dv, dtype=torch.float32, device=dev) if write_out and norm is None else None
    a = _DeltaAttnArgs(inp=i, state=_ptr(state), out=_ptr(out), q_start=_ptr(batch.q_start), q_len=_ptr(batch.q_len),
                       positions=_ptr(batch.positions), slots=_ptr(batch.state_slots), num_seqs=batch.q_len.numel(), num_slots=state.shape[0],
                       write_state=int(write_state), write_out=int(write_out), status=_ptr(runtime(dev).status), decode=int(decode))
    if low_rank is not None:
        lr = low_rank
        assert lr.z.stride(1) == 1 and lr.z.dtype == DTYPE[fmt] and lr.w2.is_contiguous()
        a.lr_z, a.lr_ld, a.lr_w2, a.lr_bias, a.lr_rank, a.lr_c = (_ptr(lr.z), lr.z.stride(0), _ptr(lr.w2), _ptr(lr.bias), lr.w2.shape[1],
                                                                 float(lr.c))
    if norm is not None:
        _norm_args(a, norm, fmt)
    _native.check(_native.lib().mb_delta_attn(C.byref(a), _stream()), f"delta_attn[T={T} H={H}]")
    _count()
    return out
