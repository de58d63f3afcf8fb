"""Finelix checkpoints: tensor names and shapes of a configuration, and their typed serving weights.

Names: ``embed``, ``head``, ``final.norm``, ``loop.in`` / ``loop.step`` and per layer ``l<i>.norm1``, ``l<i>.mix.*``,
``l<i>.mlp.*`` (a mixture of experts: ``mlp.router``, ``mlp.router.b``, ``mlp.e<j>.*``, ``mlp.shared.*``). Matrices
are stored [out, in] under the bare name. Both sublayers of a layer read one norm and are added together, which is
what the fusions at load build on:
  * a linear-attention layer's q | k | v | g and the first half of its decay projection are one matrix; so are a
    latent layer's query latent | key-value latent and its router, whose outputs stay 32-bit;
  * the mixer's output projection and the down projection of the dense (or shared) feed-forward are stacked along
    their inputs: one GEMM over [mixer | feed-forward] projects both;
  * gate and up rows are interleaved, experts are stacked, each padded with zero rows to whole 128-row weight tiles.
"""
from __future__ import annotations

from typing import Dict, Tuple

import torch

from .. import ops
from ..config.model_config import ModelConfig
from ..ops import QuantWeight
from ..ops.mixers import DTYPE, RmsNorm
from ..ops.moe import GroupedExperts, RouterSpec
from .loader import FfnW, GlaW, LatentW, LayerW, ModelW, MoeW


def tensor_shapes(c: ModelConfig) -> Dict[str, Tuple[tuple, str]]:
    """name -> (shape, kind of synthetic values) of every tensor. The rank of the decay projection is not part of
    the configuration: synthetic checkpoints use 16."""
    W, out, rank = c.hidden_size, {}, 16

    def lin(name, n, k):
        out[name] = ((n, k), "linear")

    def ffn(name, ff):
        lin(f"{name}.gate", ff, W)
        lin(f"{name}.up", ff, W)
        lin(f"{name}.down", W, ff)

    out["embed"] = ((c.vocab_size, W), "small")
    if c.loop:
        lin("loop.in", W, 2 * W)
        out["loop.step"] = ((c.loop["times"], W), "small")
    for i, (t, sp) in enumerate(zip(c.layer_types, c.layer_specs)):
        p, q, m, mlp = f"l{i}", f"l{i}.mix", sp["mixer"], sp["mlp"]
        out[f"{p}.norm1"] = ((W,), "ones")
        H = m["heads"]
        if t == "latent":
            L, R = m["kv_rank"], m["rot_dim"]
            lin(f"{q}.dq", m["q_rank"], W)
            out[f"{q}.dq.norm"] = ((m["q_rank"],), "ones")
            lin(f"{q}.uq", H * (m["dim"] + R), m["q_rank"])
            lin(f"{q}.dkv", L + R, W)
            out[f"{q}.dkv.norm"] = ((L,), "ones")
            lin(f"{q}.uk", H * m["dim"], L)
            lin(f"{q}.uv", H * m["vdim"], L)
            lin(f"{q}.o", W, H * m["vdim"])
        else:
            dk, dv = H * m["dim"], H * m["vdim"]
            for n, rows in (("q", dk), ("k", dk), ("v", dv), ("g", dv)):
                lin(f"{q}.{n}", rows, W)
            lin(f"{q}.o", W, dv)
            out[f"{q}.norm"] = ((m["vdim"],), "ones")
            lin(f"{q}.a1", rank, W)
            lin(f"{q}.a2", dk, rank)
            out[f"{q}.a2.b"] = ((dk,), "mix")
        if mlp is None:
            continue
        if mlp["kind"] == "dense":
            ffn(f"{p}.mlp", mlp["ff"])
            continue
        E = mlp["router"]["experts"]
        for e in range(E):
            ffn(f"{p}.mlp.e{e}", mlp["expert"]["ff"])
        lin(f"{p}.mlp.router", E, W)
        out[f"{p}.mlp.router.b"] = ((E,), "bias")
        if mlp.get("shared"):
            ffn(f"{p}.mlp.shared", mlp["shared"]["ff"])
    out["final.norm"] = ((W,), "ones")
    lin("head", c.vocab_size, W)
    return out


def load_finelix(ld) -> ModelW:
    c: ModelConfig = ld.cfg
    if ld.tp_size > 1 or ld.ep_size > 1:
        raise NotImplementedError("Finelix models are served on one rank")
    if c.weight_format not in ("bf16", "fp32"):
        raise NotImplementedError(f"Finelix weights are served in bf16 or fp32, not {c.weight_format}")
    fmt, W = c.weight_format, c.hidden_size

    def raw(*names):
        return torch.cat([ld.src.get(n).to(ld.dev) for n in names], 0).to(DTYPE[fmt]).contiguous()

    def weight(w) -> QuantWeight:
        return QuantWeight(fmt, w.shape[0], w.shape[1], w.contiguous())

    def norm(name) -> RmsNorm:
        return RmsNorm(ld.vec(name), c.rms_eps)

    def pad_rows(w, multiple):
        n = -w.shape[0] % multiple
        return torch.cat([w, w.new_zeros(n, w.shape[1])], 0) if n else w

    def gate_up(name):
        return ops.interleave_gate_up(raw(f"{name}.gate"), raw(f"{name}.up"))

    def gla(q, m) -> GlaW:
        H, dk, dv = m["heads"], m["dim"], m["vdim"]
        # rows padded to a whole 16-byte vector, so that every row of the output starts on one
        w = GlaW(in_proj=weight(pad_rows(raw(*(f"{q}.{n}" for n in ("q", "k", "v", "g", "a1"))), 8)), a2=ld.vec(f"{q}.a2"),
                 a2_bias=ld.vec(f"{q}.a2.b", torch.float32), norm=ld.vec(f"{q}.norm").repeat(H).contiguous(), heads=H, dim=dk, vdim=dv,
                 tau=float(m["tau"]))
        if fmt == "bf16" and w.a2.shape[1] % 8 == 0:
            w.a2_lin = weight(w.a2)
        return w

    def latent(q, m, router) -> LatentW:
        H, dim, R, L, dv = m["heads"], m["dim"], m["rot_dim"], m["kv_rank"], m["vdim"]
        parts = [f"{q}.dq", f"{q}.dkv"] + ([router] if router else [])
        q_norm = ld.vec(f"{q}.dq.norm")
        return LatentW(in_proj=weight(pad_rows(raw(*parts), 4)), q_norm=q_norm, kv_norm=ld.vec(f"{q}.dkv.norm"),
                       uq=weight(raw(f"{q}.uq")), w_uk=raw(f"{q}.uk").view(H, dim, L), w_uv=raw(f"{q}.uv").view(H, dv, L), heads=H, dim=dim,
                       rot_dim=R, vdim=dv, kv_rank=L, q_rank=q_norm.numel(), scale=float(m["scale"]), rot_base=float(m["rot"]["base"]))

    def experts(p, mlp) -> GroupedExperts:
        gu = [pad_rows(gate_up(f"{p}.e{e}"), 128) for e in range(mlp["router"]["experts"])]
        ff = gu[0].shape[0] // 2                     # the padding's gates and ups are zero, so are its activations
        down = []
        for e in range(len(gu)):
            d = raw(f"{p}.e{e}.down")
            down.append(pad_rows(torch.cat([d, d.new_zeros(W, ff - d.shape[1])], 1) if ff > d.shape[1] else d, 128))
        return GroupedExperts(weight(torch.cat(gu, 0)), weight(torch.cat(down, 0)), len(gu), 2 * ff, down[0].shape[0], interleaved=True)

    m = ModelW()
    m.embed = ld.vec("embed")
    m.lm_head = weight(raw("head"))
    m.vocab_lo, m.vocab_hi = 0, c.vocab_size
    m.final_norm = norm("final.norm")
    if c.loop:
        m.loop_in, m.loop_step = weight(raw("loop.in")), ld.vec("loop.step", torch.float32)
    for i, (t, sp) in enumerate(zip(c.layer_types, c.layer_specs)):
        p, mlp = f"l{i}", sp["mlp"]
        L = LayerW(kind=t, ffn_kind=c.ffn_types[i], ln1=norm(f"{p}.norm1"))
        fold = t == "latent" and L.ffn_kind == "moe"                 # the router's rows ride in the mixer's input projection
        L.mixer = latent(f"{p}.mix", sp["mixer"], f"{p}.mlp.router" if fold else None) if t == "latent" else gla(f"{p}.mix", sp["mixer"])
        side = None                                                  # the feed-forward every token runs
        if L.ffn_kind == "dense":
            side = f"{p}.mlp"
            L.ffn = FfnW(weight(gate_up(side)), interleaved=True)
        elif L.ffn_kind == "moe":
            L.ffn = MoeW(bias=ld.vec(f"{p}.mlp.router.b", torch.float32), grouped=experts(f"{p}.mlp", mlp),
                         spec=RouterSpec(mlp["router"]["experts"], mlp["router"]["top"]))
            if not fold:
                L.ffn.router = weight(raw(f"{p}.mlp.router"))
            if mlp.get("shared"):
                side = f"{p}.mlp.shared"
                L.ffn.shared = FfnW(weight(gate_up(side)), interleaved=True)
        L.out = weight(torch.cat([raw(f"{p}.mix.o")] + ([raw(f"{side}.down")] if side else []), 1))
        m.layers.append(L)
    return m
