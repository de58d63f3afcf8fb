"""Pivipel checkpoints: tensor names and shapes of a configuration, and their typed serving weights.

Names: ``embed`` (also the output head), ``pos``, ``embed.norm``, ``final.norm`` and per layer ``l<i>.norm1`` / ``norm2``
(norms with ``.alpha`` and ``.b`` beside the weight), ``l<i>.hc1.*`` / ``hc2.*``, ``l<i>.mix.*``, ``l<i>.mlp.*`` (a mixture of
experts: ``mlp.router``, ``mlp.e<j>.*``, ``mlp.shared.*``, ``mlp.shared.sg``). Matrices are stored [out, in] under the bare
name. A layer that uses another one's tensors has none, and is served by the same weights object.
Fused at load: q | k | v | gate logits; the router's rows and the shared expert's gate row; gate and up rows interleaved;
experts stacked and padded with zero rows to whole 128-row weight tiles (a padded gate is zero, so is its activation).
"""
from __future__ import annotations

from typing import Dict, Tuple

import torch

from .. import ops
from ..config.model_config import ModelConfig
from ..ops import QuantWeight
from ..ops.mixers import DTYPE, DytNorm, HyperW, RmsNorm
from ..ops.moe import GroupedExperts, RouterSpec
from .loader import FfnW, GatedAttnW, LayerW, ModelW, MoeW

GATES = {"attention": "head", "attention_2": "element"}


def tensor_shapes(c: ModelConfig) -> Dict[str, Tuple[tuple, str]]:
    """name -> (shape, kind of synthetic values) of every tensor."""
    W, S, out = c.hidden_size, c.streams, {}

    def lin(name, n, k):
        out[name] = ((n, k), "linear")

    def norm(name):
        out[name], out[name + ".b"], out[name + ".alpha"] = ((W,), "ones"), ((W,), "bias"), ((), "alpha")

    def hyper(name):
        out[name + ".in"], out[name + ".out"], out[name + ".mix"] = ((S,), "hyper"), ((S,), "hyper"), ((S, S), "hyper")

    def ffn(name, ff):
        lin(f"{name}.gate", ff, W)
        lin(f"{name}.up", ff, W)
        lin(f"{name}.down", W, ff)

    out["embed"], out["pos"] = ((c.vocab_size, W), "small"), ((c.max_position, W), "small")
    norm("embed.norm")
    for i, (t, sp) in enumerate(zip(c.spec_types, c.layer_specs)):
        if c.layer_owner(i) != i:
            continue
        p, q, m, mlp = f"l{i}", f"l{i}.mix", sp["mixer"], sp["mlp"]
        norm(f"{p}.norm1")
        hyper(f"{p}.hc1")
        H = m["heads"]
        for n, rows in (("q", H * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * m["vdim"])):
            lin(f"{q}.{n}", rows, W)
        lin(f"{q}.g", H if GATES[t] == "head" else H * m["vdim"], W)
        lin(f"{q}.o", W, H * m["vdim"])
        if t == "attention":
            out[f"{q}.sink"] = ((H,), "mix")
        else:
            out[f"{q}.q.norm"] = out[f"{q}.k.norm"] = ((m["dim"],), "ones")
        if mlp is None:
            continue
        norm(f"{p}.norm2")
        hyper(f"{p}.hc2")
        if mlp["kind"] == "dense":
            ffn(f"{p}.mlp", mlp["ff"])
            continue
        E = mlp["router"]["experts"]
        for e in range(E):
            ffn(f"{p}.mlp.e{e}", mlp["expert"]["ff"])
        lin(f"{p}.mlp.router", E, W)
        if mlp.get("shared"):
            ffn(f"{p}.mlp.shared", mlp["shared"]["ff"])
            lin(f"{p}.mlp.shared.sg", 1, W)
    norm("final.norm")
    return out


def load_pivipel(ld) -> ModelW:
    c: ModelConfig = ld.cfg
    if ld.tp_size > 1 or ld.ep_size > 1:
        raise NotImplementedError("Pivipel models are served on one rank")
    if c.weight_format not in ("bf16", "fp32"):
        raise NotImplementedError(f"Pivipel weights are served in bf16 or fp32, not {c.weight_format}")
    fmt, W = c.weight_format, c.hidden_size

    def raw(*names):
        parts = [ld.src.get(n).to(ld.dev) for n in names]
        return torch.cat([p.reshape(-1, p.shape[-1]) for p in parts], 0).to(DTYPE[fmt]).contiguous()

    def weight(w) -> QuantWeight:
        return QuantWeight(fmt, w.shape[0], w.shape[1], w.contiguous())

    def pad_rows(w, multiple):
        n = -w.shape[0] % multiple
        return torch.cat([w, w.new_zeros(n, w.shape[1])], 0) if n else w

    def norm(name) -> DytNorm:
        return DytNorm(float(ld.src.get(name + ".alpha").float()), ld.vec(name), ld.vec(name + ".b"))

    def hyper(name) -> HyperW:
        return HyperW(*(ld.vec(f"{name}.{n}", torch.float32) for n in ("in", "out", "mix")))

    def attention(q, t, m) -> GatedAttnW:
        # rows padded to a whole 16-byte vector, so that every row of the output starts on one
        w = GatedAttnW(qkvg=weight(pad_rows(raw(*(f"{q}.{n}" for n in "qkvg")), 8)), o=weight(raw(f"{q}.o")), heads=m["heads"],
                       kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], scale=float(m["scale"]), gate=GATES[t])
        mask, rot = m.get("mask") or {}, m.get("rot")
        w.window, w.keep = int(mask.get("size", 0)), int(mask.get("keep_first", 0))
        if t == "attention":
            w.sink = ld.vec(f"{q}.sink", torch.float32)
        else:
            w.q_norm, w.k_norm = (RmsNorm(ld.vec(f"{q}.{n}.norm"), c.rms_eps) for n in "qk")
        if rot:
            w.rot_dims, w.rot_base, s = rot["dims"], float(rot["base"]), rot.get("scaling")
            if s:
                w.rot_scaling = {"rope_type": "llama3", "factor": float(s["factor"]), "low_freq_factor": float(s["low"]),
                                 "high_freq_factor": float(s["high"]), "original_max_position_embeddings": float(s["original"])}
        return w

    def ffn(name, limit) -> FfnW:
        return FfnW(weight(ops.interleave_gate_up(raw(f"{name}.gate"), raw(f"{name}.up"))), weight(raw(f"{name}.down")), interleaved=True,
                    clamp_glu=(c.glu_alpha, float(limit)))

    def moe(p, mlp) -> MoeW:
        r, x, sh = mlp["router"], mlp["expert"], mlp.get("shared")
        gu = [pad_rows(ops.interleave_gate_up(raw(f"{p}.e{e}.gate"), raw(f"{p}.e{e}.up")), 128) for e in range(r["experts"])]
        ff, down = gu[0].shape[0] // 2, []
        for e in range(len(gu)):
            d = raw(f"{p}.e{e}.down")
            down.append(pad_rows(torch.cat([d, d.new_zeros(W, ff - d.shape[1])], 1) if ff > d.shape[1] else d, 128))
        ge = GroupedExperts(weight(torch.cat(gu, 0)), weight(torch.cat(down, 0)), len(gu), 2 * ff, down[0].shape[0], interleaved=True,
                            clamp_glu=(c.glu_alpha, float(x["limit"])))
        g = r.get("groups") or {"count": 1, "keep": 1}
        spec = RouterSpec(r["experts"], r["top"], router="softmax_grouped", router_n_group=g["count"], router_topk_group=g["keep"],
                          router_renormalize=False, router_scaling=float(r.get("scale", 1.0)))
        w = MoeW(router=weight(pad_rows(raw(f"{p}.router", *([f"{p}.shared.sg"] if sh else [])), 4)), grouped=ge, spec=spec)
        if sh:
            w.shared = ffn(f"{p}.shared", sh["limit"])
        return w

    m = ModelW()
    m.embed, m.pos_embed, m.embed_norm = ld.vec("embed"), ld.vec("pos"), norm("embed.norm")
    m.lm_head = QuantWeight(fmt, c.vocab_size, W, m.embed.to(DTYPE[fmt]))
    m.vocab_lo, m.vocab_hi = 0, c.vocab_size
    m.final_norm = norm("final.norm")
    for i, (t, sp) in enumerate(zip(c.spec_types, c.layer_specs)):
        if c.layer_owner(i) != i:
            m.layers.append(None)
            continue
        p, mlp = f"l{i}", sp["mlp"]
        L = LayerW(kind=c.layer_types[i], ffn_kind=c.ffn_types[i], ln1=norm(f"{p}.norm1"), hc_attn=hyper(f"{p}.hc1"),
                   mixer=attention(f"{p}.mix", t, sp["mixer"]))
        if mlp is not None:
            L.ln2, L.hc_ffn = norm(f"{p}.norm2"), hyper(f"{p}.hc2")
            L.ffn = moe(f"{p}.mlp", mlp) if L.ffn_kind == "moe" else ffn(f"{p}.mlp", mlp["limit"])
        m.layers.append(L)
    m.layers = [m.layers[c.layer_owner(i)] for i in range(c.num_layers)]
    return m
