"""Mixers of the 32-bit-stream decoders: sink attention beside RWKV-style time mixing ("parallel"), lightning
attention, and the per-layer token side input. Each takes the residual stream, produces its input with the
stream's own kernel and leaves its output pending on the stream (``models/stream.py``).

The time mixing keeps the previous token's input in the state pool's window tensor [slots, W] and the
per-head matrices in its state tensor; lightning attention keeps the matrices only.
"""
from __future__ import annotations

import torch

from .. import ops
from ..ops import mixers as mx


def parallel_block(dec, x, lw, batch, kv, j: int, pool, sidx: int):
    """left_scale * sink attention + right_scale * time mixing on one normalised input. Both scales are
    applied in fp32 where each half's output is produced, so that one GEMM over [left | right] projects both."""
    c, w = dec.cfg, lw.mixer
    L, R = w.left, w.right
    fmt = x.fmt
    stash = getattr(batch, "spec_stash", None)
    ws = stash is None                                               # verify steps commit the state afterwards
    h, mixes, h32 = x.shift(lw.ln1, R.mu, pool.conv[sidx], batch, ws, not ws)
    T = h.shape[0]
    nl, nr = L.heads * L.vdim, R.heads * R.dim
    cat = torch.empty(T, nl + nr, dtype=h.dtype, device=h.device)
    # ---- left: sink attention
    qkv = ops.linear(mx.act_of(h, fmt), L.qkv)
    cos, sin = dec.rotary(L.rot_dims, L.rot_base)
    q = mx.rope_dims(qkv, Hq=L.heads, Hkv=L.kv_heads, dk=L.dim, dv=L.vdim, positions=batch.positions, slots=batch.slot_mapping,
                     k_cache=kv.k[j], v_cache=kv.v[j], cos=cos, sin=sin, fmt=fmt)
    mx.attention_dims(q, kv.k[j], kv.v[j], batch, dk=L.dim, dv=L.vdim, scale=L.scale, sink=True, fmt=fmt, out=cat[:, :nl],
                      out_scale=w.left_scale)
    # ---- right: time mixing
    r, k, v, g = mx.mix_projections(mixes, R, fmt)
    log_w = mx.log_decay(ops.linear(mx.act_of(mixes[4], fmt), R.w1, out_f32=True), R.w2, R.w0, R.w2_twice)
    mx.linear_attention(r, k, v, pool.ssm[sidx], batch, heads=R.heads, dk=R.dim, dv=R.dim, fmt=fmt, log_w=log_w, u=R.u, write_state=ws,
                        norm=dict(w=R.norm, gate=g, gate_act="silu", eps=c.rms_eps, scale=w.right_scale, out=cat[:, nl:]))
    if stash is not None:
        stash.layers[sidx] = ("parallel", lw, h32, (r, k, v), log_w)
    return x.add(ops.linear(mx.act_of(cat, fmt), w.o), lw.post_attn)


def lightning_block(dec, x, lw, batch, pool, sidx: int):
    """silu(q), silu(k), silu(v), decaying linear attention read after the update, RMS norm over all heads,
    sigmoid gate, projection."""
    c, w, fmt = dec.cfg, lw.mixer, x.fmt
    H, dk, dv = w.heads, w.dim, w.vdim
    stash = getattr(batch, "spec_stash", None)
    n = 2 * H * dk + H * dv
    qkvg = ops.linear(mx.act_of(x.norm(lw.ln1), fmt), w.qkvg, silu_cols=n)
    q, k, v, g = qkvg[:, :H * dk], qkvg[:, H * dk:2 * H * dk], qkvg[:, 2 * H * dk:n], qkvg[:, n:]
    core = mx.linear_attention(q, k, v, pool.ssm[sidx], batch, heads=H, dk=dk, dv=dv, fmt=fmt, decay=w.decay,
                               write_state=stash is None)
    if stash is not None:
        stash.layers[sidx] = ("lightning", lw, None, (q, k, v), None)
    y = mx.gated_norm(core, w.norm, g, fmt, group=H * dv, gate_act="sigmoid", eps=c.rms_eps)
    return x.add(ops.linear(mx.act_of(y, fmt), w.o), lw.post_attn)


def token_side(dec, x, w, batch):
    """x + rms(proj(gelu(gate x) * e)) with e this layer's slice of the token's side embedding."""
    fmt = x.fmt
    z = ops.linear(mx.act_of(x.raw(), fmt), w.gate, out_f32=True)
    g = mx.side_gate(z, batch.token_ids, dec.w.side_embed, w.offset, fmt)
    return x.add(ops.linear(mx.act_of(g, fmt), w.proj), w.norm)


def commit(kind: str, lw, x_in, qkv, log_w, pool, sidx: int, cb) -> None:
    """State-only pass over the accepted rows of a verify step (``models.recurrent.commit_recurrent``)."""
    w = lw.mixer.right if kind == "parallel" else lw.mixer
    dv = w.dim if kind == "parallel" else w.vdim
    fmt = "fp32" if qkv[0].dtype == torch.float32 else "bf16"
    kw = dict(log_w=log_w, u=w.u) if kind == "parallel" else dict(log_w=log_w) if kind == "gla" else dict(decay=w.decay)
    mx.linear_attention(*qkv, pool.ssm[sidx], cb, heads=w.heads, dk=w.dim, dv=dv, fmt=fmt, write_out=False, **kw)
    if kind == "parallel":
        mx.shift_commit(x_in, pool.conv[sidx], cb)
