"""Layers whose mixer and feed-forward read one norm of a 32-bit stream and join it together:
x <- x + mixer(norm(x)) + ff(norm(x)).

Mixer output and feed-forward activation (the dense one, or a mixture's shared expert) are written side by side,
one GEMM over both projects them back, and the routed experts' rows stay where the grouped GEMM left them until
the next norm's kernel adds everything to the stream.
"""
from __future__ import annotations

import torch

from .. import ops
from ..ops import mixers as mx


def joint_layer(dec, x, lw, batch, caches, run: int):
    fmt = x.fmt
    h = x.norm(lw.ln1)
    a = mx.act_of(h, fmt)
    cat = torch.empty(h.shape[0], lw.out.K, dtype=h.dtype, device=h.device)
    nm = lw.mixer.out_width
    logits = None
    if lw.kind == "latent":
        from .mla import latent_mixer
        logits = latent_mixer(dec, a, lw.mixer, batch, caches.kv.k[caches.kv_index[run]], fmt, cat[:, :nm])
    else:
        from .recurrent import gla_mixer
        gla_mixer(dec, a, lw, batch, caches.state, caches.state_index[run], fmt, cat[:, :nm])
    ff = lw.ffn.shared if lw.ffn_kind == "moe" else lw.ffn
    if ff is not None:
        glu = dict(swiglu=True) if lw.ffn_kind == "moe" else dict(geglu=True)
        ops.linear(a, ff.gate_up, out=cat[:, nm:], **glu)
    routed = None
    if lw.ffn_kind == "moe":
        from .moe import routed_rows
        if lw.ffn.router is not None:
            logits = ops.linear(a, lw.ffn.router, out_f32=True)
        routed = routed_rows(dec, a, logits[:, :lw.ffn.spec.num_experts], lw.ffn)
    return x.add(ops.linear(mx.act_of(cat, fmt), lw.out), None, routed)
