"""Fabulix checkpoints: tensor names and shapes of a configuration, and their typed serving weights.

Names: ``embed``, ``side.embed``, ``final.norm`` and per layer ``l<i>.norm1`` / ``norm1b`` / ``norm2`` /
``norm2b`` (each with ``.alpha`` and ``.b``), ``l<i>.mix.*``, ``l<i>.mlp.*``, ``l<i>.side.*``. Matrices are stored
[out, in] under the bare name. Fused at load: the attention's q | k | v; the two output projections of a
parallel mixer along their inputs (one GEMM over [left | right]); the time mixing's r | k | v | g (when their
height suits the grouped GEMM); a lightning mixer's q | k | v | g; gate and up rows interleaved.
"""
from __future__ import annotations

from typing import Dict, Tuple

import torch

from .. import ops
from ..config.model_config import ModelConfig
from ..ops import QuantWeight
from ..ops.mixers import DytNorm, RmsNorm
from .loader import FfnW, LayerW, LightningW, ModelW, ParallelW, SinkAttnW, TimeMixW, TokenSideW


def tensor_shapes(c: ModelConfig) -> Dict[str, Tuple[tuple, str]]:
    """name -> (shape, kind of synthetic values) of every tensor. The rank of the decay projection is not
    part of the configuration: synthetic checkpoints use a fortieth of the width, at least 16 and a multiple of 8."""
    W, out = c.hidden_size, {}
    rank = max(16, W // 40 // 8 * 8)

    def norm(name):
        out[name], out[name + ".b"], out[name + ".alpha"] = ((W,), "ones"), ((W,), "bias"), ((), "alpha")

    def lin(name, n, k):
        out[name] = ((n, k), "linear")

    out["embed"] = ((c.vocab_size, W), "small")
    if c.token_side_dim:
        out["side.embed"] = ((c.vocab_size, c.num_layers * c.token_side_dim), "mix")
    for i, (t, sp) in enumerate(zip(c.layer_types, c.layer_specs)):
        p, m, mlp = f"l{i}", sp["mixer"], sp["mlp"]
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if mlp else ()):
            norm(f"{p}.{n}")
        if t == "parallel":
            a, r, q = m["left"], m["right"], f"{p}.mix.left"
            for n, rows in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"])):
                lin(f"{q}.{n}", rows, W)
            lin(f"{q}.o", W, a["heads"] * a["vdim"])
            q, hd = f"{p}.mix.right", r["heads"] * r["dim"]
            for n in "rkvgw":
                out[f"{q}.mu.{n}"] = ((W,), "mix")
            for n in "rkvg":
                lin(f"{q}.{n}", hd, W)
            lin(f"{q}.w1", rank, W)
            lin(f"{q}.w2", hd, rank)
            out[f"{q}.w0"], out[f"{q}.u"], out[f"{q}.norm"] = ((hd,), "mix"), ((r["heads"], r["dim"]), "mix"), ((hd,), "ones")
            lin(f"{q}.o", W, hd)
        else:
            q, dk, dv = f"{p}.mix", m["heads"] * m["dim"], m["heads"] * m["vdim"]
            for n, rows in (("q", dk), ("k", dk), ("v", dv), ("g", dv)):
                lin(f"{q}.{n}", rows, W)
            lin(f"{q}.o", W, dv)
            out[f"{q}.norm"] = ((dv,), "ones")
        if mlp:
            lin(f"{p}.mlp.gate", mlp["ff"], W)
            lin(f"{p}.mlp.up", mlp["ff"], W)
            lin(f"{p}.mlp.down", W, mlp["ff"])
        if c.token_side_dim:
            lin(f"{p}.side.gate", c.token_side_dim, W)
            lin(f"{p}.side.proj", W, c.token_side_dim)
            out[f"{p}.side.norm"] = ((W,), "ones")
    norm("final.norm")
    return out


def load_fabulix(ld) -> ModelW:
    c: ModelConfig = ld.cfg
    if ld.tp_size > 1 or ld.ep_size > 1:
        raise NotImplementedError("Fabulix models are served on one rank")
    if c.weight_format not in ("bf16", "fp32"):
        raise NotImplementedError(f"Fabulix weights are served in bf16 or fp32, not {c.weight_format}")
    fmt = c.weight_format

    def lin(*names) -> QuantWeight:
        """One linear layer, or several that share their input stacked along the output."""
        w = torch.cat([ld.src.get(n).to(ld.dev) for n in names], 0)
        return QuantWeight(fmt, w.shape[0], w.shape[1], w.to(ops.mixers.DTYPE[fmt]).contiguous())

    def norm(name) -> DytNorm:
        return DytNorm(float(ld.src.get(name + ".alpha").float()), ld.vec(name), ld.vec(name + ".b"))

    def parallel(p, m) -> ParallelW:
        a, r = m["left"], m["right"]
        q = f"{p}.left"
        left = SinkAttnW(lin(f"{q}.q", f"{q}.k", f"{q}.v"), a["heads"], a["kv_heads"], a["dim"], a["vdim"], float(a["scale"]),
                         a["rot"]["dims"], float(a["rot"]["base"]))
        q = f"{p}.right"
        right = TimeMixW(mu=torch.stack([ld.vec(f"{q}.mu.{n}") for n in "rkvgw"]).contiguous(), w1=lin(f"{q}.w1"),
                         w2=ld.vec(f"{q}.w2"), w0=ld.vec(f"{q}.w0", torch.float32), u=ld.vec(f"{q}.u", torch.float32),
                         norm=ld.vec(f"{q}.norm"), heads=r["heads"], dim=r["dim"])
        if fmt == "bf16" and right.w2.shape[1] % 4 == 0:
            right.w2_twice = QuantWeight("bf16", right.w2.shape[0], 2 * right.w2.shape[1], torch.cat([right.w2, right.w2], 1).contiguous())
        if ops.mixers.grouped_ok(c.hidden_size, r["heads"] * r["dim"], fmt) and ld.dev.type == "cuda":
            right.rkvg_stack = lin(*(f"{q}.{n}" for n in "rkvg"))
        else:
            right.rkvg = [lin(f"{q}.{n}") for n in "rkvg"]
        o = torch.cat([ld.src.get(f"{p}.{s}.o").to(ld.dev) for s in ("left", "right")], 1).to(ops.mixers.DTYPE[fmt]).contiguous()
        return ParallelW(left, right, QuantWeight(fmt, o.shape[0], o.shape[1], o), float(m["left_scale"]), float(m["right_scale"]))

    m = ModelW()
    m.embed = ld.vec("embed")
    m.lm_head = QuantWeight(fmt, c.vocab_size, c.hidden_size, m.embed.to(ops.mixers.DTYPE[fmt]))
    m.vocab_lo, m.vocab_hi = 0, c.vocab_size
    m.final_norm = norm("final.norm")
    if c.token_side_dim:
        m.side_embed = ld.vec("side.embed")
    for i, (t, sp) in enumerate(zip(c.layer_types, c.layer_specs)):
        p, mx, mlp = f"l{i}", sp["mixer"], sp["mlp"]
        L = LayerW(kind=t, ffn_kind=c.ffn_types[i], ln1=norm(f"{p}.norm1"), post_attn=norm(f"{p}.norm1b"))
        if t == "parallel":
            L.mixer = parallel(f"{p}.mix", mx)
        else:
            q = f"{p}.mix"
            L.mixer = LightningW(lin(f"{q}.q", f"{q}.k", f"{q}.v", f"{q}.g"), lin(f"{q}.o"), ld.vec(f"{q}.norm"),
                                 torch.tensor(mx["decay"], dtype=torch.float32, device=ld.dev), mx["heads"], mx["dim"], mx["vdim"])
        if mlp:
            L.ln2, L.post_ffn = norm(f"{p}.norm2"), norm(f"{p}.norm2b")
            gu = lin(f"{p}.mlp.gate", f"{p}.mlp.up")
            I = gu.N // 2
            perm = torch.stack([torch.arange(I), torch.arange(I) + I], 1).reshape(-1).to(gu.data.device)
            L.ffn = FfnW(ops.permute_rows(gu, perm), lin(f"{p}.mlp.down"), interleaved=True,
                         clamp_glu=(c.glu_alpha, float(mlp["limit"])))
        if c.token_side_dim:
            L.side = TokenSideW(lin(f"{p}.side.gate"), lin(f"{p}.side.proj"), RmsNorm(ld.vec(f"{p}.side.norm"), c.rms_eps),
                                i * c.token_side_dim)
        m.layers.append(L)
    return m
