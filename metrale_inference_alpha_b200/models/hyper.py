"""Layers over several residual streams (static hyper-connections): x_t <- sum_s mix[s, t] x_s + out[t] sublayer(norm(u)),
u = sum_s in[s] x_s, for a mixer and then a feed-forward.

The mixer is softmax attention with its own head sizes and any of: rotary positions on the leading dimensions, per-head
norms on queries and keys, a window with kept first tokens, a sink per head, output gates per head or per element. The
feed-forward is a clamped GLU or a mixture of such experts with a gated shared one. Each sublayer's output stays pending on
the streams, and the kernel that makes the next input joins it (``models/stream.py::HyperStream``).
"""
from __future__ import annotations

import torch

from .. import ops
from ..ops import mixers as mx


def gated_attention(dec, a, w, batch, kc, vc, fmt: str):
    """One projection for queries, keys, values and gate logits; norms, rotation and cache rows; attention with the gate
    in its epilogue; output projection."""
    qkvg = ops.linear(a, w.qkvg)
    cos, sin = dec.rotary(w.rot_dims, w.rot_base, w.rot_scaling)
    q = mx.rope_dims(qkvg, Hq=w.heads, Hkv=w.kv_heads, dk=w.dim, dv=w.vdim, positions=batch.positions, slots=batch.slot_mapping,
                     k_cache=kc, v_cache=vc, cos=cos, sin=sin, fmt=fmt, q_norm=w.q_norm, k_norm=w.k_norm)
    n, at = w.heads * w.vdim, w.heads * w.dim + w.kv_heads * (w.dim + w.vdim)
    gate = None
    if w.gate is not None:
        gate = mx.OutputGate(qkvg[:, at:at + (w.heads if w.gate == "head" else n)], w.gate == "head")
    out = torch.empty(a.M, n, dtype=qkvg.dtype, device=qkvg.device)
    mx.attention_dims(q, kc, vc, batch, dk=w.dim, dv=w.vdim, scale=w.scale, sink=w.sink if w.sink is not None else False, fmt=fmt, out=out,
                      window=w.window, keep=w.keep, gate=gate)
    return ops.linear(mx.act_of(out, fmt), w.o)


def gated_moe(dec, a, w) -> mx.SublayerOut:
    """Routed experts, unsummed, beside the shared expert and its gate's logits: router and gate are one projection."""
    from .moe import routed_rows
    E = w.spec.num_experts
    logits = ops.linear(a, w.router, out_f32=True)
    out = mx.SublayerOut(routed=routed_rows(dec, a, logits[:, :E], w))
    if w.shared is not None:
        out.y, out.gate = dec.dense_ffn(a, w.shared, None), logits[:, E]
    return out


def hyper_layer(dec, x, lw, batch, caches, run: int):
    fmt, j = x.fmt, caches.kv_index[run]
    a = mx.act_of(x.norm(lw.ln1, lw.hc_attn), fmt)
    x.add(mx.SublayerOut(gated_attention(dec, a, lw.mixer, batch, caches.kv.k[j], caches.kv.v[j], fmt)), lw.hc_attn)
    if lw.ffn_kind == "none":
        return x
    a = mx.act_of(x.norm(lw.ln2, lw.hc_ffn), fmt)
    return x.add(gated_moe(dec, a, lw.ffn) if lw.ffn_kind == "moe" else mx.SublayerOut(dec.dense_ffn(a, lw.ffn, None)), lw.hc_ffn)
