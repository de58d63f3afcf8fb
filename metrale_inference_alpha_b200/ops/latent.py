"""Ops of latent attention with per-layer sizes (queries through a normed latent, keys and values linear in a cached
latent, one rotated key part for all heads), in absorbed form: multi-query attention over the cached rows, whose
first part serves as the values too.

One cache row per token: [latent | zeros | rotated key | zeros], laid out for the attention kernel that serves the
sizes (``latent_row``). CUDA tensors run ``csrc/latent.cu`` for the norms, rotations and cache rows and one of the
attention kernels (``csrc/{mla,attention,attention_simt}.cu``); CPU tensors run the restatements below.
"""
from __future__ import annotations

import ctypes as C
from typing import NamedTuple

import torch

from . import _count, _native, _ptr, _stream, mla_cuda, runtime
from . import reference as ref
from .mixers import DTYPE, _f32, attention_dims


class LatentRow(NamedTuple):
    row: int           # elements of a cached row
    rope_at: int       # first element of the rotated key part
    kernel: str        # tile: the paged attention kernels with equal K and V tiles | mla: the 576-wide kernels | simt


def latent_row(rank: int, rot: int, fmt: str) -> LatentRow:
    d = rank + rot
    if fmt == "bf16" and d <= 256:
        return LatentRow(64 if d <= 64 else 128 if d <= 128 else 256, rank, "tile")
    if fmt == "bf16" and rank <= mla_cuda.LATENT and rot <= mla_cuda.ROW - mla_cuda.LATENT:
        return LatentRow(mla_cuda.ROW, mla_cuda.LATENT, "mla")
    return LatentRow(d, rank, "simt")


class _LatentNormArgs(C.Structure):
    _fields_ = [("T", C.c_int), ("in_f32", C.c_int), ("f32", C.c_int), ("q_rank", C.c_int), ("L", C.c_int), ("R", C.c_int), ("row", C.c_int),
                ("rope_at", C.c_int), ("x", C.c_void_p), ("x_ld", C.c_longlong), ("q_w", C.c_void_p), ("kv_w", C.c_void_p),
                ("eps", C.c_float), ("cos_tab", C.c_void_p), ("sin_tab", C.c_void_p), ("max_pos", C.c_int), ("positions", C.c_void_p),
                ("slots", C.c_void_p), ("num_slots", C.c_longlong), ("cache", C.c_void_p), ("cq", C.c_void_p), ("status", C.c_void_p)]


class _LatentQueryArgs(C.Structure):
    _fields_ = [("T", C.c_int), ("H", C.c_int), ("f32", C.c_int), ("dim", C.c_int), ("R", C.c_int), ("L", C.c_int), ("row", C.c_int),
                ("rope_at", C.c_int), ("q", C.c_void_p), ("cos_tab", C.c_void_p), ("sin_tab", C.c_void_p), ("max_pos", C.c_int),
                ("positions", C.c_void_p), ("qq", C.c_void_p), ("status", C.c_void_p)]


_native.register_optional("mb_latent_norm", [C.POINTER(_LatentNormArgs), C.c_void_p])
_native.register_optional("mb_latent_query", [C.POINTER(_LatentQueryArgs), C.c_void_p])


def norm_and_cache(x: torch.Tensor, fmt: str, *, q_rank: int, L: int, R: int, q_w, kv_w, eps: float, cos, sin, positions, slots,
                   cache: torch.Tensor, lay: LatentRow) -> torch.Tensor:
    """x [T, >= q_rank + L + R] (fp32 or the activation type): the query latent's RMS norm [T, q_rank], and one cache row
    per token [norm(latent) | rotated key part] at its slot (rows without a slot write nothing)."""
    T = x.shape[0]
    if not x.is_cuda:
        xf = x.float()
        cq = ref.rms_norm(xf[:, :q_rank], q_w, eps).to(DTYPE[fmt])
        row = torch.zeros(T, lay.row)
        row[:, :L] = ref.rms_norm(xf[:, q_rank:q_rank + L], kv_w, eps)
        kr = xf[:, None, q_rank + L:q_rank + L + R]
        row[:, lay.rope_at:lay.rope_at + R] = ref.apply_rope_neox(kr, positions, cos, sin)[:, 0] if R else kr[:, 0]
        ok = slots >= 0
        cache.view(-1, lay.row)[slots[ok].long()] = row[ok].to(cache.dtype)
        return cq
    assert x.stride(1) == 1 and cache.dtype == DTYPE[fmt] and cache.shape[-1] == lay.row
    cq = torch.empty(T, q_rank, dtype=DTYPE[fmt], device=x.device)
    a = _LatentNormArgs(T, int(x.dtype == torch.float32), _f32(fmt), q_rank, L, R, lay.row, lay.rope_at, _ptr(x), x.stride(0), _ptr(q_w),
                        _ptr(kv_w), float(eps), _ptr(cos), _ptr(sin), cos.shape[0] if R else 0, _ptr(positions), _ptr(slots),
                        cache.shape[0] * cache.shape[1], _ptr(cache), _ptr(cq), _ptr(runtime(x.device).status))
    _native.check(_native.lib().mb_latent_norm(C.byref(a), _stream()), f"latent_norm[T={T}]")
    _count()
    return cq


def absorbed_query(q: torch.Tensor, w_uk: torch.Tensor, fmt: str, *, H: int, dim: int, R: int, cos, sin, positions,
                   lay: LatentRow) -> torch.Tensor:
    """q [T, H (dim + R)] -> [T, H, row]: the unrotated part times the head's key matrix [H, dim, L] in the latent
    columns, the rotated part in its place, zeros elsewhere."""
    T, L = q.shape[0], w_uk.shape[2]
    q = q.view(T, H, dim + R)
    if not q.is_cuda:
        qf = q.float()
        out = torch.zeros(T, H, lay.row)
        out[..., :L] = torch.einsum("thd,hdl->thl", qf[..., :dim].double(), w_uk.double()).float()
        if R:
            out[..., lay.rope_at:lay.rope_at + R] = ref.apply_rope_neox(qf[..., dim:], positions, cos, sin)
        return out.to(DTYPE[fmt])
    qq = torch.empty(T, H, lay.row, dtype=DTYPE[fmt], device=q.device)
    torch.bmm(q[..., :dim].transpose(0, 1), w_uk, out=qq[..., :L].transpose(0, 1))
    if lay.row > L:
        a = _LatentQueryArgs(T, H, _f32(fmt), dim, R, L, lay.row, lay.rope_at, _ptr(q), _ptr(cos), _ptr(sin), cos.shape[0] if R else 0,
                             _ptr(positions), _ptr(qq), _ptr(runtime(q.device).status))
        _native.check(_native.lib().mb_latent_query(C.byref(a), _stream()), f"latent_query[T={T}]")
        _count()
    return qq


def attention(qq: torch.Tensor, cache: torch.Tensor, batch, w_uv: torch.Tensor, scale: float, fmt: str, lay: LatentRow,
              out: torch.Tensor, kernel: str = "auto") -> torch.Tensor:
    """Causal attention of qq [T, H, row] over the cached rows, mapped to head values by w_uv [H, vdim, L], into
    ``out`` [T, H vdim] (may be a column range). The softmax weights keep 32-bit precision."""
    T, H, _ = qq.shape
    dv, L = w_uv.shape[1], w_uv.shape[2]
    if qq.is_cuda and lay.kernel == "mla" and kernel in ("auto", "mma", "tc"):
        o = mla_cuda.mla_attention(qq, cache, batch.block_table, batch.q_start, batch.q_len, batch.ctx_len, max_q_len=int(batch.max_q_len),
                                   max_ctx=max(int(batch.max_ctx), 1), scale=scale, impl={"auto": 0, "mma": 1, "tc": 2}[kernel], split_p=True,
                                   out_bf16=True)
    else:
        o = torch.empty(T, H, L, dtype=qq.dtype, device=qq.device)
        if lay.kernel == "simt":
            kernel = "simt"
        attention_dims(qq, cache, cache, batch, dk=lay.row, dv=L, scale=scale, sink=False, fmt=fmt, out=o.view(T, H * L), kernel=kernel)
    if not qq.is_cuda:
        out.copy_(torch.einsum("thl,hvl->thv", o[..., :L].double(), w_uv.double()).reshape(T, H * dv))
        return out
    torch.bmm(o[..., :L].transpose(0, 1), w_uv.transpose(1, 2), out=out.view(T, H, dv).transpose(0, 1))
    return out

