"""Layers that read the residual stream through a short convolution and norm what they write back:
x <- x + norm(sublayer(x + conv(x))), for a mixer and then a feed-forward.

Mixers: the gated delta rule ("delta"), and attention beside a recurrence on one input ("twin"), either attention with
rotated values and capped scores beside lightning attention, or windowed attention whose values are its keys beside the
general delta rule. The feed-forward is a mixture of squared-ReLU experts with a shared one. A sublayer's output stays
pending on the stream, and the kernel that makes the next input joins it (``models/stream.py::CanonStream``).

Every layer keeps, per sequence, the last inputs of both convolutions (and of the delta rule's own) in one flat row of the
state pool's window tensor, and its matrices in the state tensor.
"""
from __future__ import annotations

import torch

from .. import ops
from ..ops import mixers as mx
from ..ops.canon import Window, short_conv
from ..ops.delta import BoundedDecay, GatedRule, GeneralRule, delta_attention


def windows(cfg, lw, rows: torch.Tensor):
    """The layer's windows inside its rows of the pool: (mixer input, feed-forward input, projection or None)."""
    W, n = cfg.hidden_size, (cfg.canon_taps - 1) * cfg.hidden_size
    second = n if lw.ffn_kind != "none" else 0
    conv = Window(rows, n + second, lw.mixer.conv.shape[1]) if lw.kind == "delta" else None
    return Window(rows, 0, W), Window(rows, n, W), conv


def window_floats(cfg, lw) -> int:
    """Length of the layer's row."""
    n = (cfg.canon_taps - 1) * cfg.hidden_size * (1 if lw.ffn_kind == "none" else 2)
    return n + ((lw.mixer.conv.shape[0] - 1) * lw.mixer.conv.shape[1] if lw.kind == "delta" else 0)


def _cols(y: torch.Tensor, span) -> torch.Tensor:
    return y[:, span[0]:span[0] + span[1]]


def delta_mixer(dec, a, lw, batch, window: Window, state, fmt: str, stash):
    """One projection for queries, keys, values, gates and both logits; short convolution; gated delta rule with the head
    norm in it; output projection."""
    w = lw.mixer
    y = ops.linear(a, w.in_proj)
    at, ws = w.at, stash is None                                     # verify steps commit the state afterwards
    qkv = short_conv(_cols(y, at["qkv"]), w.conv, window, batch, fmt, write_state=ws)
    nk = w.kv_heads * w.dim
    q, k, v = qkv[:, :nk], qkv[:, nk:2 * nk], qkv[:, 2 * nk:]
    rule = GatedRule(_cols(y, at["a"]), _cols(y, at["b"]), w.A_log, w.dt_bias)
    out = torch.empty(a.M, w.heads * w.vdim, dtype=y.dtype, device=y.device)
    kw = dict(heads=w.heads, key_heads=w.kv_heads, dk=w.dim, dv=w.vdim, fmt=fmt)
    delta_attention(q, k, v, rule, state, batch, write_state=ws, **kw,
                    norm=dict(w=w.norm, gate=_cols(y, at["g"]), gate_act="silu", eps=dec.cfg.rms_eps, scale=1.0, out=out))
    if stash is not None:
        x = _cols(y, at["qkv"])
        stash.later[window.rows.data_ptr(), window.at] = lambda cb: short_conv(x, w.conv, window, cb, fmt, write_out=False)
        stash.later[state.data_ptr()] = lambda cb: delta_attention(q, k, v, rule, state, cb, write_out=False, kernel="seq", **kw)
    return ops.linear(mx.act_of(out, fmt), w.o)


def twin_attention(dec, y, w, batch, kc, vc, fmt: str, out, out_scale: float) -> None:
    """The attention half, times its factor, into ``out``: norms over the whole projection, rotation, cache, attention."""
    rot = dec.rotary(w.rot_dims, w.rot_base, w.rot_scaling)
    turn = dec.rotary(w.vdim, w.rot_base) if w.turn_values else None
    q = mx.attention_rows(y, cols=w.cols, Hq=w.heads, Hkv=w.kv_heads, dk=w.dim, dv=w.vdim, positions=batch.positions, slots=batch.slot_mapping,
                          k_cache=kc, v_cache=vc, rot=rot if rot[0] is not None else None, fmt=fmt, q_norm=w.q_norm, k_norm=w.k_norm, v_rot=turn)
    mx.attention_dims(q, kc, vc, batch, dk=w.dim, dv=w.vdim, scale=w.scale, sink=False, fmt=fmt, out=out, out_scale=out_scale,
                      window=w.window, softcap=w.softcap, turn_back=turn)


def twin_mixer(dec, a, lw, batch, kc, vc, state, fmt: str, stash):
    """left_scale * attention + right_scale * recurrence on one input: one projection for everything both read, both halves
    side by side with their factors, one output projection over [left | right]."""
    w = lw.mixer
    L, R = w.left, w.right
    general = R.rule == "general"
    y = ops.linear(a, w.in_proj, bias=w.bias) if w.bias is not None else ops.linear(a, w.in_proj, silu_cols=w.silu_cols)
    nl, nr, ws = L.heads * L.vdim, R.heads * R.vdim, stash is None
    cat = torch.empty(a.M, nl + nr, dtype=y.dtype, device=y.device)
    twin_attention(dec, y, L, batch, kc, vc, fmt, cat[:, :nl], w.left_scale)
    q, k, v, g = (_cols(y, R.at[n]) for n in ("q", "k", "v", "g"))
    norm = dict(w=R.norm, gate=g, gate_act="sigmoid", eps=dec.cfg.rms_eps, scale=w.right_scale, out=cat[:, nl:])
    if general:
        decay = BoundedDecay(_cols(y, R.at["w1"]), R.w2, R.w0, R.decay_scale, R.w2_twice)
        rule = GeneralRule(_cols(y, R.at["a"]), decay)
        rule = rule if ws else rule.logs()
        delta_attention(q, k, v, rule, state, batch, heads=R.heads, dk=R.dim, dv=R.vdim, fmt=fmt, write_state=ws, norm=norm)
        if stash is not None:
            stash.later[state.data_ptr()] = lambda cb: delta_attention(q, k, v, rule, state, cb, heads=R.heads, dk=R.dim, dv=R.vdim, fmt=fmt,
                                                                       write_out=False, kernel="seq")
    else:
        kw = dict(heads=R.heads, dk=R.dim, dv=R.vdim, fmt=fmt, decay=R.decay)
        core = mx.linear_attention(q, k, v, state, batch, write_state=ws, **kw)
        mx.gated_norm(core, norm.pop("w"), norm.pop("gate"), fmt, group=nr, **norm)
        if stash is not None:
            stash.later[state.data_ptr()] = lambda cb: mx.linear_attention(q, k, v, state, cb, write_out=False, **kw)
    return ops.linear(mx.act_of(cat, fmt), w.o)


def relu2_moe(dec, a, w) -> mx.SublayerOut:
    """Routed experts, unsummed, beside the shared expert."""
    from .moe import routed_rows
    logits = ops.linear(a, w.router, out_f32=True)
    out = mx.SublayerOut(routed=routed_rows(dec, a, logits[:, :w.spec.num_experts], w))
    if w.shared is not None:
        out.y = ops.linear(mx.act_of(ops.linear(a, w.shared.gate_up, relu2=True), a.fmt), w.shared.down)
    return out


def canon_layer(dec, x, lw, batch, caches, run: int):
    fmt, j = x.fmt, caches.state_index[run]
    stash = getattr(batch, "spec_stash", None)
    win1, win2, conv = windows(dec.cfg, lw, caches.state.conv[j])
    state = caches.state.ssm[j]
    a = mx.act_of(x.read(lw.canon[0], win1, batch, stash), fmt)
    if lw.kind == "delta":
        y = delta_mixer(dec, a, lw, batch, conv, state, fmt, stash)
    else:
        c = caches.kv_index[run]
        y = twin_mixer(dec, a, lw, batch, caches.kv.k[c], caches.kv.v[c], state, fmt, stash)
    x.add(mx.SublayerOut(y), lw.post_attn)
    if lw.ffn_kind == "none":
        return x
    a = mx.act_of(x.read(lw.canon[1], win2, batch, stash), fmt)
    return x.add(relu2_moe(dec, a, lw.ffn), lw.post_ffn)
