"""Ledinex checkpoints: tensor names and shapes of a configuration, and their typed serving weights.

Names: ``embed`` (also the output head), ``final.norm`` and per layer ``l<i>.norm1`` / ``norm2`` (around zero), ``l<i>.canon1`` /
``canon2`` [width, taps], ``l<i>.mix.*`` (a mixer of two halves: ``mix.left.*``, ``mix.right.*``), ``l<i>.mlp.router``,
``mlp.e<j>.*``, ``mlp.shared.*``. Matrices are stored [out, in] under the bare name.
Fused at load: everything a mixer projects, every part's rows starting at a multiple of eight (zero rows between), so that
its columns of the output are whole vectors; both output projections of a two-half mixer along their inputs; experts
stacked and padded with zero rows to whole 128-row weight tiles (a padded unit is relu(0)^2); filters transposed to
[taps, channels]; the logits' factor into the final norm.
"""
from __future__ import annotations

import math
from typing import Dict, Tuple

import torch

from .. import ops
from ..config.model_config import ModelConfig
from ..ops import QuantWeight
from ..ops.mixers import DTYPE, RmsNorm
from ..ops.moe import GroupedExperts, RouterSpec
from .loader import DeltaW, FfnW, LayerW, ModelW, MoeW, RecurrenceW, TwinAttnW, TwinW

LOG_DECAY_SCALE = -math.exp(-0.5)        # log decays of the general delta rule lie between this and zero


def tensor_shapes(c: ModelConfig) -> Dict[str, Tuple[tuple, str]]:
    """name -> (shape, kind of synthetic values) of every tensor. The rank of the decay projection is not part of the
    configuration: synthetic checkpoints use a fortieth of the width, at least 16 and a multiple of 8."""
    W, out = c.hidden_size, {}
    rank = max(16, W // 40 // 8 * 8)

    def lin(name, n, k):
        out[name] = ((n, k), "linear")

    out["embed"] = ((c.vocab_size, W), "small")
    for i, (t, sp) in enumerate(zip(c.spec_types, c.layer_specs)):
        p, q, m, mlp = f"l{i}", f"l{i}.mix", sp["mixer"], sp["mlp"]
        for n in ("1", "2") if mlp else ("1",):
            out[f"{p}.norm{n}"], out[f"{p}.canon{n}"] = ((W,), "bias"), ((W, c.canon_taps), "conv")
        if t == "delta":
            H, nk, nv = m["heads"], m["kv_heads"] * m["dim"], m["heads"] * m["vdim"]
            for n, rows in (("q", nk), ("k", nk), ("v", nv)):
                lin(f"{q}.{n}", rows, W)
                out[f"{q}.{n}.conv"] = ((rows, m["conv"]), "conv")
            for n, rows in (("a", H), ("b", H), ("g", nv)):
                lin(f"{q}.{n}", rows, W)
            out[f"{q}.A_log"], out[f"{q}.dt_bias"], out[f"{q}.norm"] = ((H,), "alog"), ((H,), "bias"), ((m["vdim"],), "ones")
            lin(f"{q}.o", W, nv)
        else:
            a, r = m["left"], m["right"]
            hq, hk = a["heads"] * a["dim"], a["kv_heads"] * a["dim"]
            lin(f"{q}.left.q", hq, W)
            lin(f"{q}.left.k", hk, W)
            out[f"{q}.left.q.norm"], out[f"{q}.left.k.norm"] = ((hq,), "ones"), ((hk,), "ones")
            dk = r["heads"] * r["dim"]
            if t == "parallel":
                lin(f"{q}.left.v", a["kv_heads"] * a["vdim"], W)
                lin(f"{q}.left.o", W, a["heads"] * a["vdim"])
                dv = r["heads"] * r["vdim"]
                rows = (("q", dk), ("k", dk), ("v", dv), ("g", dv))
            else:
                out[f"{q}.left.q.b"], out[f"{q}.left.k.b"] = ((hq,), "bias"), ((hk,), "bias")
                lin(f"{q}.left.o", W, hq)
                dv = dk
                rows = (("r", dk), ("k", dk), ("v", dk), ("g", dk), ("a", dk), ("w1", rank))
                lin(f"{q}.right.w2", dk, rank)
                out[f"{q}.right.w0"], out[f"{q}.right.a.b"] = ((dk,), "mix"), ((dk,), "bias")
            for n, k in rows:
                lin(f"{q}.right.{n}", k, W)
            out[f"{q}.right.norm"] = ((dv,), "ones")
            lin(f"{q}.right.o", W, dv)
        if mlp is None:
            continue
        names = [(f"e{e}", mlp["expert"]["ff"]) for e in range(mlp["router"]["experts"])]
        for n, ff in names + ([("shared", mlp["shared"]["ff"])] if mlp.get("shared") else []):
            lin(f"{p}.mlp.{n}.up", ff, W)
            lin(f"{p}.mlp.{n}.down", W, ff)
        lin(f"{p}.mlp.router", mlp["router"]["experts"], W)
    out["final.norm"] = ((W,), "bias")
    return out


def load_ledinex(ld) -> ModelW:
    c: ModelConfig = ld.cfg
    if ld.tp_size > 1 or ld.ep_size > 1:
        raise NotImplementedError("Ledinex models are served on one rank")
    if c.weight_format not in ("bf16", "fp32"):
        raise NotImplementedError(f"Ledinex weights are served in bf16 or fp32, not {c.weight_format}")
    fmt, W = c.weight_format, c.hidden_size

    def raw(name):
        return ld.src.get(name).to(ld.dev).to(DTYPE[fmt]).contiguous()

    def f32(name):
        return ld.vec(name, torch.float32)

    def weight(w) -> QuantWeight:
        return QuantWeight(fmt, w.shape[0], w.shape[1], w.contiguous())

    def pad_rows(w, multiple):
        n = -w.shape[0] % multiple
        return torch.cat([w, w.new_zeros(n, w.shape[1])], 0) if n else w

    def stack(*parts):
        """Rows of [(label, names)] under each other, every part from a multiple of eight rows on: (weight, label -> span)."""
        rows, at, n = [], {}, 0
        for label, names in parts:
            w = torch.cat([raw(x) for x in names], 0)
            at[label] = (n, w.shape[0])
            rows.append(pad_rows(w, 8))
            n += rows[-1].shape[0]
        return weight(torch.cat(rows, 0)), at

    def norm(name) -> RmsNorm:
        return RmsNorm(ld.vec(name), c.rms_eps, plus_one=True)

    def delta(q, m) -> DeltaW:
        w, at = stack(("qkv", [f"{q}.{n}" for n in "qkv"]), ("g", [f"{q}.g"]), ("a", [f"{q}.a"]), ("b", [f"{q}.b"]))
        conv = torch.cat([f32(f"{q}.{n}.conv") for n in "qkv"], 0)
        return DeltaW(in_proj=w, at=at, conv=conv.t().contiguous(), A_log=f32(f"{q}.A_log"), dt_bias=f32(f"{q}.dt_bias"),
                      norm=ld.vec(f"{q}.norm").repeat(m["heads"]).contiguous(), o=weight(raw(f"{q}.o")), heads=m["heads"],
                      kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"])

    def rotation(rot):
        s = rot.get("scaling")
        if s and "original" in s:
            s = {"rope_type": "yarn", "factor": float(s["factor"]), "original_max_position_embeddings": float(s["original"]),
                 "beta_fast": float(s["fast"]), "beta_slow": float(s["slow"]), "attention_factor": 0.1 * math.log(s["factor"]) + 1.0}
        elif s:
            s = {"rope_type": "linear", "factor": float(s["factor"])}
        return dict(rot_dims=rot["dims"], rot_base=float(rot["base"]), rot_scaling=s or None)

    def twin(q, t, m) -> TwinW:
        a, r = m["left"], m["right"]
        first = [("lq", [f"{q}.left.q"]), ("lk", [f"{q}.left.k"])]
        if t == "parallel":                              # what passes through SiLU comes first
            w, at = stack(*((n, [f"{q}.right.{n}"]) for n in "qkvg"), *first, ("lv", [f"{q}.left.v"]))
            tw = TwinW(in_proj=w, silu_cols=at["g"][0])
            R = RecurrenceW("lightning", decay=torch.tensor(r["decay"], dtype=torch.float32, device=ld.dev))
        else:
            w, at = stack(*first, ("q", [f"{q}.right.r"]), *((n, [f"{q}.right.{n}"]) for n in ("k", "v", "g", "a", "w1")))
            at["lv"] = at["lk"]
            bias = torch.zeros(w.N, dtype=torch.float32, device=ld.dev)
            for n, b in (("lq", "left.q.b"), ("lk", "left.k.b"), ("a", "right.a.b")):
                bias[at[n][0]:at[n][0] + at[n][1]] = f32(f"{q}.{b}")
            tw = TwinW(in_proj=w, bias=bias)
            R = RecurrenceW("general", w2=ld.vec(f"{q}.right.w2"), w0=f32(f"{q}.right.w0"), decay_scale=LOG_DECAY_SCALE)
            if fmt == "bf16" and R.w2.shape[1] % 4 == 0:
                R.w2_twice = weight(torch.cat([R.w2, R.w2], 1))
        R.at, R.norm, R.heads, R.dim, R.vdim = at, ld.vec(f"{q}.right.norm"), r["heads"], r["dim"], r.get("vdim", r["dim"])
        tw.right = R
        tw.left = TwinAttnW(cols=tuple(at[n][0] for n in ("lq", "lk", "lv")), heads=a["heads"], kv_heads=a["kv_heads"], dim=a["dim"],
                            vdim=a["vdim"] if t == "parallel" else a["dim"], scale=float(a["scale"]),
                            q_norm=RmsNorm(ld.vec(f"{q}.left.q.norm"), c.rms_eps), k_norm=RmsNorm(ld.vec(f"{q}.left.k.norm"), c.rms_eps),
                            turn_values=t == "parallel", window=int((a.get("mask") or {}).get("size", 0)),
                            softcap=float(a.get("softcap") or 0.0), **rotation(a["rot"]))
        tw.o = weight(torch.cat([raw(f"{q}.left.o"), raw(f"{q}.right.o")], 1))
        tw.left_scale, tw.right_scale = float(m["left_scale"]), float(m["right_scale"])
        return tw

    def moe(p, mlp) -> MoeW:
        E = mlp["router"]["experts"]
        up = [pad_rows(raw(f"{p}.e{e}.up"), 128) for e in range(E)]
        ff, down = up[0].shape[0], []
        for e in range(E):
            d = raw(f"{p}.e{e}.down")
            down.append(pad_rows(torch.cat([d, d.new_zeros(W, ff - d.shape[1])], 1) if ff > d.shape[1] else d, 128))
        ge = GroupedExperts(weight(torch.cat(up, 0)), weight(torch.cat(down, 0)), E, ff, down[0].shape[0], interleaved=False)
        w = MoeW(router=weight(pad_rows(raw(f"{p}.router"), 4)), grouped=ge,
                 spec=RouterSpec(E, mlp["router"]["top"], router="softmax", ffn_act="relu2"))
        if mlp.get("shared"):
            w.shared = FfnW(weight(pad_rows(raw(f"{p}.shared.up"), 8)), None)
            d = raw(f"{p}.shared.down")
            w.shared.down = weight(torch.cat([d, d.new_zeros(W, w.shared.gate_up.N - d.shape[1])], 1))
        return w

    m = ModelW()
    m.embed = ld.vec("embed")
    m.lm_head = QuantWeight(fmt, c.vocab_size, W, m.embed.to(DTYPE[fmt]))
    m.vocab_lo, m.vocab_hi = 0, c.vocab_size
    m.final_norm = RmsNorm(ld.vec("final.norm"), c.rms_eps, plus_one=True, scale=c.logit_scale)
    for i, (t, sp) in enumerate(zip(c.spec_types, c.layer_specs)):
        p, mlp = f"l{i}", sp["mlp"]
        filt = lambda n: ld.vec(f"{p}.canon{n}").t().contiguous()
        L = LayerW(kind=c.layer_types[i], ffn_kind=c.ffn_types[i], post_attn=norm(f"{p}.norm1"),
                   mixer=delta(f"{p}.mix", sp["mixer"]) if t == "delta" else twin(f"{p}.mix", t, sp["mixer"]))
        L.canon = (filt(1), filt(2) if mlp else None)
        if mlp:
            L.post_ffn, L.ffn = norm(f"{p}.norm2"), moe(f"{p}.mlp", mlp)
        m.layers.append(L)
    return m
