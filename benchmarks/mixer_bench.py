#!/usr/bin/env python
"""The kernels of the Fabulix, Finelix, Pivipel or Ledinex decoder next to the like kernels of the engine's attention / MLA /
Kimi-delta-attention / Mamba2 hybrids and of its gated-attention MoE models at equal size, each with its distance from the roofline (measured copy
bandwidth and measured bf16 GEMM rate), and the throughput of a whole model next to an equal-size hybrid. CUDA
events around one call, L2 flushed by a 512 MB write before every call, median of the timed calls. Reached as
`bench.py --mixers`, `--design` naming the decoder.
"""
from __future__ import annotations

import json
import os
import statistics
import sys

import torch

sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
from metrale_inference_alpha_b200 import ops  # noqa: E402
from metrale_inference_alpha_b200.engine.batch import ForwardBatch  # noqa: E402
from metrale_inference_alpha_b200.ops import QuantWeight, mixers as mx, recurrent as rops, reference as ref  # noqa: E402

DEV, BF = "cuda", torch.bfloat16


def peaks():
    p = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "MEASURED_PEAKS.json")
    d = json.load(open(p)) if os.path.exists(p) else {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}
    return d["hbm_gbs"] * 1e9, d["bf16_tflops"] * 1e12


class Timer:
    def __init__(self):
        self.flush = torch.empty(512 << 20, dtype=torch.uint8, device=DEV)

    def __call__(self, fn, iters=9, warm=3):
        ts = []
        for i in range(warm + iters):
            self.flush.fill_(i & 1)
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            fn()
            b.record()
            torch.cuda.synchronize()
            if i >= warm:
                ts.append(a.elapsed_time(b) * 1e-3)
        return statistics.median(ts)


def batch(lens, start=0):
    nb = (max(lens) + start) // 16 + 2
    seqs = [dict(tokens=[1] * n, start_pos=start, blocks=list(range(1 + i * nb, 1 + (i + 1) * nb)), state_slot=i + 1, logits="last")
            for i, n in enumerate(lens)]
    return ForwardBatch.build(seqs, 16, device=DEV), 2 + len(lens) * nb


def rnd(*s, dtype=BF, std=1.0):
    return (torch.randn(*s, device=DEV) * std).to(dtype)


def pairing(rows):
    """pair(shape, name, new, bytes, flops, like name, like, bytes, flops): times both and appends one row."""
    t, bw, fl = Timer(), *peaks()

    def pair(shape, name, new, nb, nf, like_name, like, lb, lf):
        a, b = t(new), t(like)
        ra, rb = max(nb / bw, nf / fl), max(lb / bw, lf / fl)
        rows.append({"shape": shape, "kernel": name, "us": round(a * 1e6, 1), "x_roofline": round(a / ra, 2), "like": like_name,
                     "like_us": round(b * 1e6, 1), "like_x_roofline": round(b / rb, 2), "ratio": round(a / ra / (b / rb), 2)})
        print(rows[-1], file=sys.stderr, flush=True)
    return pair


SHAPES = (("decode 128 seqs, ctx 1024", [1] * 128, 1023), ("prefill 1 x 4096", [4096], 0), ("prefill 8 x 1024", [1024] * 8, 0))


def kernels(W=2560, H=20, G=4, D=128, FF=6912, R=64, side=128):
    """Rows: (shape, mechanism, new us, new bytes, new flops, like name, like us, like bytes, like flops)."""
    rows = []
    HD, pair = H * D, pairing(rows)
    for shape, lens, start in SHAPES:
        b, nblk = batch(lens, start)
        T, S = sum(lens), len(lens)
        ctx = lens[0] + start
        # ---- norms
        x, y = rnd(T, W, dtype=torch.float32), rnd(T, W)
        n1 = mx.DytNorm(0.5, rnd(W), rnd(W))
        mu, st = rnd(5, W), torch.zeros(S + 2, W, device=DEV)
        xb, wv = rnd(T, W), rnd(W)
        rms = lambda: ops.row_op(xb, "bf16", ops.IN_RMSNORM, w=wv, residual=y, write_residual=True)
        pair(shape, "stream_norm (post + add + pre)", lambda: mx.stream_norm(x, "bf16", y=y, post=n1, pre=n1), T * W * 12, 0,
             "residual + RMSNorm", rms, T * W * 8, 0)
        pair(shape, "stream_norm + token-shift mixes", lambda: mx.stream_norm(x, "bf16", y=y, post=mx.RmsNorm(wv, 1e-5), pre=n1, mu=mu, state=st, batch=b),
             T * W * 22, 0, "residual + RMSNorm", rms, T * W * 8, 0)
        core, gate, gw = rnd(T, HD, dtype=torch.float32), rnd(T, HD), rnd(HD)
        for name, grp in (("gated_norm, per head", D), ("gated_norm, all heads", HD)):
            pair(shape, name, lambda: mx.gated_norm(core, gw, gate, "bf16", group=grp, gate_act="silu", eps=1e-5), T * HD * 8, 0,
                 "gated RMSNorm", lambda: ops.row_op(core, "bf16", ops.IN_GATED_RMSNORM, gate=gate, w=gw, group=grp), T * HD * 8, 0)
        # ---- attention
        cos, sin = ref.rope_tables(8192, D, 1e4, device=DEV)
        kc, vc = rnd(nblk, 16, G, D), rnd(nblk, 16, G, D)
        qkv = rnd(T, (H + 2 * G) * D)
        byt = 2 * qkv.numel() * 2
        pair(shape, "rope_dims", lambda: mx.rope_dims(qkv, Hq=H, Hkv=G, dk=D, dv=D, positions=b.positions, slots=b.slot_mapping, k_cache=kc,
                                                      v_cache=vc, cos=cos, sin=sin, fmt="bf16"), byt, 0,
             "rope + KV write", lambda: ops.qk_norm_rope_kvwrite(qkv, Hq=H, Hkv=G, D=D, positions=b.positions, slots=b.slot_mapping, k_cache=kc,
                                                                 v_cache=vc, cos=cos, sin=sin), byt, 0)
        q, out = rnd(T, H, D), torch.empty(T, HD, dtype=BF, device=DEV)
        byt = S * ctx * G * D * 4 + T * HD * 4
        flo = sum(4 * HD * (n * start + n * (n + 1) / 2) for n in lens)
        pair(shape, "attention with sink", lambda: mx.attention_dims(q, kc, vc, b, dk=D, dv=D, scale=0.09, sink=True, fmt="bf16", out=out), byt, flo,
             "attention", lambda: ops.paged_attention(q, kc, vc, b.block_table, b.q_start, b.q_len, b.ctx_len, max_q_len=b.max_q_len,
                                                      max_ctx=b.max_ctx, scale=0.09), byt, flo)
        # ---- recurrences
        r, k, v = rnd(T, HD), rnd(T, HD), rnd(T, HD)
        lw, u = -torch.exp(torch.randn(T, HD, device=DEV) - 3), torch.rand(H, D, device=DEV)
        ssm = torch.zeros(S + 2, H, D, D, device=DEV)
        dec = torch.linspace(0.6, 0.999, H, device=DEV)
        sb = 2 * S * H * D * D * 4
        conv, graw, braw = rnd(T, 3 * HD, dtype=torch.float32), rnd(T, HD, dtype=torch.float32), rnd(T, H, dtype=torch.float32)
        A, dtb = torch.zeros(H, device=DEV), torch.zeros(HD, device=DEV)
        kda = lambda: rops.kda_recurrence(conv, graw, braw, A, dtb, -5.0, ssm, b, heads=H, dim=D)
        pair(shape, "time-mix recurrence", lambda: mx.linear_attention(r, k, v, ssm, b, heads=H, dk=D, dv=D, fmt="bf16", log_w=lw, u=u),
             T * HD * 14 + sb, 0, "Kimi delta attention", kda, T * HD * 20 + sb, 0)
        P, N, Hm = 64, 128, 2 * H
        xbc, dtm, Dm = rnd(T, Hm * P + 2 * Hm * N, dtype=torch.float32), rnd(T, Hm), torch.zeros(Hm, device=DEV)
        ssm2 = torch.zeros(S + 2, Hm, P, N, device=DEV)
        pair(shape, "lightning recurrence", lambda: mx.linear_attention(r, k, v, ssm, b, heads=H, dk=D, dv=D, fmt="bf16", decay=dec),
             T * HD * 10 + sb, 0, "Mamba2 scan (64 x 128 states, as many bytes)",
             lambda: rops.mamba2_scan(xbc, dtm, Dm, Dm, Dm, ssm2, b, heads=Hm, groups=Hm, head_dim=P, state=N), xbc.numel() * 4 + T * Hm * P * 4 + sb, 0)
        del conv, graw, xbc
        # ---- matrix products with their epilogues
        act = mx.act_of(rnd(T, W), "bf16")
        gu = QuantWeight("bf16", 2 * FF, W, rnd(2 * FF, W, std=0.02))
        gb, gf = (2 * FF * W + T * W + T * FF) * 2, 2 * T * 2 * FF * W
        pair(shape, "GEMM + clamped GLU", lambda: ops.linear(act, gu, clamp_glu=(1.702, 3.0)), gb, gf, "GEMM + SwiGLU",
             lambda: ops.linear(act, gu, swiglu=True), gb, gf)
        w4 = QuantWeight("bf16", 4 * HD, W, rnd(4 * HD, W, std=0.02))
        gb, gf = (4 * HD * W + T * W + T * 4 * HD) * 2, 2 * T * 4 * HD * W
        pair(shape, "GEMM + SiLU columns", lambda: ops.linear(act, w4, silu_cols=3 * HD), gb, gf, "GEMM", lambda: ops.linear(act, w4), gb, gf)
        mixes = rnd(5, T, W)
        from metrale_inference_alpha_b200.weights.loader import TimeMixW
        tw = TimeMixW(rkvg_stack=w4)
        pair(shape, "r, k, v, g of their own mixes", lambda: mx.mix_projections(mixes, tw, "bf16"), gb + 3 * T * W * 2, gf, "GEMM",
             lambda: ops.linear(act, w4), gb, gf)
        z, w2, w0 = rnd(T, R, dtype=torch.float32), rnd(HD, R, std=0.1), torch.zeros(HD, device=DEV)
        zb, w2q = mx.act_of(rnd(T, R), "bf16"), QuantWeight("bf16", HD, R, w2)
        w2t = QuantWeight("bf16", HD, 2 * R, torch.cat([w2, w2], 1))
        pair(shape, "log decay (32-bit low-rank)", lambda: mx.log_decay(z, w2, w0, w2t), T * HD * 4 + T * R * 4 + HD * R * 2, 0, "low-rank decay GEMM, bf16",
             lambda: ops.linear(zb, w2q, out_f32=True), T * HD * 4 + T * R * 2 + HD * R * 2, 0)
        ids, tab, zz = torch.randint(0, 60000, (T,), dtype=torch.int32, device=DEV), rnd(60000, side * 4), rnd(T, side, dtype=torch.float32)
        et = rnd(60000, W)
        pair(shape, "token side gate", lambda: mx.side_gate(zz, ids, tab, side, "bf16"), T * side * 8, 0, "embedding gather", lambda: ops.embed(ids, et),
             T * W * 4, 0)
        pair(shape, "scaled embedding, fp32", lambda: mx.embed_scaled(ids, et, 2.0), T * W * 6, 0, "embedding gather", lambda: ops.embed(ids, et), T * W * 4, 0)
    return rows


def finelix_kernels(W=2560, H=20, D=128, FF=6912, rank=16, Hl=32, dim=128, R=64, dv=128, L=512, QR=1536, E=64, top=6, EF=1024):
    """The same rows for Finelix: the like kernels are those of MLA + Kimi-delta hybrids with experts."""
    from metrale_inference_alpha_b200.ops import latent as lt, mla_cuda, moe as moe_ops, moe_cuda
    from metrale_inference_alpha_b200.weights.loader import MoeW
    rows = []
    HD, pair, lay = H * D, pairing(rows), lt.latent_row(L, R, "bf16")
    f32 = torch.float32
    for shape, lens, start in SHAPES:
        b, nblk = batch(lens, start)
        T, S, ctx = sum(lens), len(lens), lens[0] + start
        # ---- the stream
        x, y, xb, wv = rnd(T, W, dtype=f32), rnd(T, W), rnd(T, W), rnd(W)
        n1 = mx.RmsNorm(wv, 1e-5)
        pair(shape, "stream_rms (add + norm)", lambda: mx.stream_rms(x, "bf16", y=y, pre=n1), T * W * 12, 0, "residual + RMSNorm",
             lambda: ops.row_op(xb, "bf16", ops.IN_RMSNORM, w=wv, residual=y, write_residual=True), T * W * 8, 0)
        # ---- experts
        gu, dn = QuantWeight("bf16", E * 2 * EF, W, rnd(E * 2 * EF, W, std=0.02)), QuantWeight("bf16", E * W, EF, rnd(E * W, EF, std=0.02))
        w = MoeW(grouped=moe_ops.GroupedExperts(gu, dn, E, 2 * EF, W, True), bias=rnd(E, dtype=f32), spec=moe_ops.RouterSpec(E, top))
        act, logits = mx.act_of(rnd(T, W), "bf16"), rnd(T, E, dtype=f32)
        soft = moe_ops.RouterSpec(E, top, "softmax")
        pair(shape, "route (biased, over the chosen)", lambda: moe_ops.route(logits, w.spec, w.bias), T * (E + 2 * top) * 4, 0, "route (softmax)",
             lambda: moe_ops.route(logits, soft), T * (E + 2 * top) * 4, 0)
        wt, idx = moe_ops.route(logits, w.spec, w.bias)
        hit = len(set(idx.flatten().tolist()))
        eb, ef = hit * 3 * EF * W * 2 + T * W * 2 + T * top * (W * 4 + 2 * EF * 2), T * top * 6 * EF * W
        pair(shape, "experts, unsummed", lambda: moe_cuda.grouped_pairs(w.spec, act, idx, w), eb, ef, "experts + combine + residual",
             lambda: moe_cuda.grouped_ffn(w.spec, act, wt, idx, w, finish=(y, None, xb)), eb + T * W * 6, ef)
        ye, sp = moe_cuda.grouped_pairs(w.spec, act, idx, w)
        routed = mx.Routed(ye, sp.pair_row, wt)

        def combine():
            out = torch.empty(T, W, dtype=BF, device=DEV)
            ops._native.lib().mb_moe_finish(ops._ptr(ye), ye.stride(0), ops._ptr(sp.pair_row), ops._ptr(wt), T, top, W, ops._ptr(y), W, None, 0,
                                            ops._ptr(xb), ops._ptr(out), ops._stream())
        pair(shape, "stream_rms with the experts' sum", lambda: mx.stream_rms(x, "bf16", y=y, routed=routed, pre=n1), T * W * (12 + 4 * top), 0,
             "expert combine", combine, T * W * (6 + 4 * top), 0)
        del gu, dn, w, ye, sp, routed
        # ---- latent attention
        cos, sin = ref.rope_tables(8192, R, 1e4, device=DEV)
        cache, p = rnd(nblk, 16, 1, lay.row), rnd(T, QR + L + R + E, dtype=f32)
        qn, kn = rnd(QR), rnd(L)
        kw = dict(q_rank=QR, L=L, R=R, q_w=qn, kv_w=kn, eps=1e-5, cos=cos, sin=sin, positions=b.positions, slots=b.slot_mapping, cache=cache, lay=lay)
        qa = rnd(T, QR)
        pair(shape, "latent_norm (+ cache row)", lambda: lt.norm_and_cache(p, "bf16", **kw), T * ((QR + L + R) * 4 + QR * 2 + lay.row * 2), 0,
             "RMSNorm of the query latent", lambda: ops.row_op(qa, "bf16", ops.IN_RMSNORM, w=qn), T * QR * 4, 0)
        q, uk, ckv = rnd(T, Hl * (dim + R)), rnd(Hl, dim, L, std=0.05), rnd(T, L + R)
        q3 = q.view(T, Hl, dim + R)

        def like_query():
            ql = torch.bmm(q3[..., :dim].transpose(0, 1), uk)
            return mla_cuda.prepare(q3, ql, ckv, kn, cos, sin, b.positions, b.slot_mapping, cache, dim, 1e-5)
        nb = T * Hl * (dim + R + lay.row) * 2 + uk.numel() * 2
        pair(shape, "absorbed queries", lambda: lt.absorbed_query(q, uk, "bf16", H=Hl, dim=dim, R=R, cos=cos, sin=sin, positions=b.positions, lay=lay),
             nb, 2 * T * Hl * dim * L, "absorbed queries + cache row", like_query, nb + T * (L + R) * 4, 2 * T * Hl * dim * L)
        qq, uv = rnd(T, Hl, lay.row, std=0.3), rnd(Hl, dv, L, std=0.05)
        out = torch.empty(T, Hl * dv, dtype=BF, device=DEV)
        akw = dict(max_q_len=b.max_q_len, max_ctx=b.max_ctx, scale=0.07)
        pairs_ = sum(n * start + n * (n + 1) / 2 for n in lens)
        nb, nf = S * ctx * lay.row * 2 + T * Hl * (lay.row * 2 + L * 2), 2 * Hl * (lay.row + L) * pairs_

        def like_att():
            o = mla_cuda.mla_attention(qq, cache, b.block_table, b.q_start, b.q_len, b.ctx_len, **akw)
            return torch.bmm(o.to(BF).transpose(0, 1), uv.transpose(1, 2)).transpose(0, 1).reshape(T, Hl * dv)
        nb, nf = nb + uv.numel() * 2 + T * Hl * (L + dv) * 2, nf + 2 * T * Hl * L * dv
        pair(shape, "latent attention + value product", lambda: lt.attention(qq, cache, b, uv, 0.07, "bf16", lay, out), nb, nf,
             "MLA attention + value product", like_att, nb, nf)
        del qq, q, cache
        # ---- gated linear attention
        z = rnd(T, 4 * HD + rank)
        q, k, v, g, a1 = z[:, :HD], z[:, HD:2 * HD], z[:, 2 * HD:3 * HD], z[:, 3 * HD:4 * HD], z[:, 4 * HD:]
        a2, bias, gw = rnd(HD, rank, std=0.1), rnd(HD, dtype=f32), rnd(HD)
        lr = mx.LowRankDecay(a1, a2, bias, 1 / 16, QuantWeight("bf16", HD, rank, a2))
        ssm, out = torch.zeros(S + 2, H, D, D, device=DEV), torch.empty(T, HD, dtype=BF, device=DEV)
        sb = 2 * S * H * D * D * 4
        conv, graw, braw = rnd(T, 3 * HD, dtype=f32), rnd(T, HD, dtype=f32), rnd(T, H, dtype=f32)
        A, dtb = torch.zeros(H, device=DEV), torch.zeros(HD, device=DEV)
        nw = rnd(D, dtype=f32)
        norm = dict(w=gw, gate=g, gate_act="silu", eps=1e-5, scale=1.0, out=out)
        pair(shape, "gated linear attention (decay, recurrence, norm)",
             lambda: mx.linear_attention(q, k, v, ssm, b, heads=H, dk=D, dv=D, fmt="bf16", low_rank=lr, norm=norm), T * HD * 10 + T * rank * 2 + sb, 0,
             "Kimi delta attention (recurrence, norm)",
             lambda: rops.kda_recurrence(conv, graw, braw, A, dtb, -5.0, ssm, b, heads=H, dim=D, norm=(nw, g, 1e-5)), T * HD * 20 + sb, 0)
        zb, a2q = mx.act_of(rnd(T, rank), "bf16"), QuantWeight("bf16", HD, rank, a2)
        pair(shape, "log decay (log sigmoid / tau)", lr.log, T * HD * 4 + T * rank * 2 + HD * rank * 2, 0, "low-rank decay GEMM, bf16",
             lambda: ops.linear(zb, a2q, out_f32=True), T * HD * 4 + T * rank * 2 + HD * rank * 2, 0)
        del conv, graw
        # ---- matrix products with their epilogues
        gu = QuantWeight("bf16", 2 * FF, W, rnd(2 * FF, W, std=0.02))
        cat = torch.empty(T, HD + FF, dtype=BF, device=DEV)
        gb, gf = (2 * FF * W + T * W + T * FF) * 2, 2 * T * 2 * FF * W
        pair(shape, "GEMM + tanh-GELU GLU", lambda: ops.linear(act, gu, geglu=True, out=cat[:, HD:]), gb, gf, "GEMM + SwiGLU",
             lambda: ops.linear(act, gu, swiglu=True), gb, gf)
        wo, wm, wd = (QuantWeight("bf16", W, n, rnd(W, n, std=0.02)) for n in (HD + FF, HD, FF))
        ca, cm, cd = (mx.act_of(rnd(T, n), "bf16") for n in (HD + FF, HD, FF))
        gb, gf = ((HD + FF) * (W + T) + T * W) * 2, 2 * T * (HD + FF) * W
        pair(shape, "joint output GEMM", lambda: ops.linear(ca, wo), gb, gf, "o_proj + down_proj, residual", lambda:
             ops.linear(cd, wd, residual=ops.linear(cm, wm, residual=xb)), gb + T * W * 6, gf)
        wi, pa, step = QuantWeight("bf16", W, 2 * W, rnd(W, 2 * W, std=0.02)), mx.act_of(rnd(T, 2 * W), "bf16"), rnd(W, dtype=f32)
        gb, gf = 2 * W * (W + T) * 2 + T * W * 4, 4 * T * W * W
        pair(shape, "pass entry GEMM (32-bit out + step)", lambda: ops.linear(pa, wi, out_f32=True, bias=step), gb, gf, "GEMM, 32-bit out",
             lambda: ops.linear(pa, wi, out_f32=True), gb, gf)
        ids, et = torch.randint(0, 60000, (T,), dtype=torch.int32, device=DEV), rnd(60000, W)
        pr = torch.empty(T, 2 * W, dtype=BF, device=DEV)
        pair(shape, "scaled embedding (+ copy)", lambda: mx.embed_scaled(ids, et, 2.0, pr[:, W:]), T * W * 8, 0, "embedding gather",
             lambda: ops.embed(ids, et), T * W * 4, 0)
    return rows


def pivipel_kernels(W=2560, H=32, G=8, D=128, FF=6912, E=64, top=6, EF=1024, S=2, window=512, keep=4, groups=8, keep_groups=4):
    """The same rows for Pivipel: the like kernels are those of windowed, gated attention models with experts."""
    from metrale_inference_alpha_b200.ops import moe as moe_ops, moe_cuda
    from metrale_inference_alpha_b200.weights.loader import MoeW
    rows = []
    HD, pair, f32 = H * D, pairing(rows), torch.float32
    for shape, lens, start in SHAPES:
        b, nblk = batch(lens, start)
        T, ctx = sum(lens), lens[0] + start
        # ---- the streams
        x, y, xb, wv = rnd(T, S, W, dtype=f32), rnd(T, W), rnd(T, W), rnd(W)
        hw = mx.HyperW(*(torch.full(s, 0.4, device=DEV) for s in ((S,), (S,), (S, S))))
        n1 = mx.DytNorm(0.5, rnd(W), rnd(W))
        one = mx.SublayerOut(y)
        pair(shape, f"stream_hyper ({S} streams, join + read + norm)", lambda: mx.stream_hyper(x, S, "bf16", pending=one, hc=hw, w_in=hw.w_in, pre=n1),
             T * W * (8 * S + 4), 0, "residual + RMSNorm", lambda: ops.row_op(xb, "bf16", ops.IN_RMSNORM, w=wv, residual=y, write_residual=True),
             T * W * 8, 0)
        ids, et, pt = torch.randint(0, 60000, (T,), dtype=torch.int32, device=DEV), rnd(60000, W), rnd(8192, W)
        pair(shape, "embedding + position + norm, fp32", lambda: mx.embed_scaled(ids, et, 1.0, pos=pt, positions=b.positions, norm=n1), T * W * 8, 0,
             "embedding gather", lambda: ops.embed(ids, et), T * W * 4, 0)
        # ---- experts
        gu, dn = QuantWeight("bf16", E * 2 * EF, W, rnd(E * 2 * EF, W, std=0.02)), QuantWeight("bf16", E * W, EF, rnd(E * W, EF, std=0.02))
        soft = moe_ops.RouterSpec(E, top, "softmax")
        spec = moe_ops.RouterSpec(E, top, "softmax_grouped", router_n_group=groups, router_topk_group=keep_groups, router_renormalize=False)
        w = MoeW(grouped=moe_ops.GroupedExperts(gu, dn, E, 2 * EF, W, True, clamp_glu=(1.702, 7.0)), spec=spec)
        lw = MoeW(grouped=moe_ops.GroupedExperts(gu, dn, E, 2 * EF, W, True), spec=soft)
        act, logits = mx.act_of(rnd(T, W), "bf16"), rnd(T, E, dtype=f32)
        pair(shape, "route (softmax, groups)", lambda: moe_ops.route(logits, spec), T * (E + 2 * top) * 4, 0, "route (softmax)",
             lambda: moe_ops.route(logits, soft), T * (E + 2 * top) * 4, 0)
        rw = QuantWeight("bf16", E + 4, W, rnd(E + 4, W, std=0.02))
        rl = QuantWeight("bf16", E, W, rw.data[:E])
        pair(shape, "router + shared gate GEMM", lambda: ops.linear(act, rw, out_f32=True), ((E + 4 + T) * W) * 2 + T * (E + 4) * 4, 2 * T * W * (E + 4),
             "router GEMM", lambda: ops.linear(act, rl, out_f32=True), ((E + T) * W) * 2 + T * E * 4, 2 * T * W * E)
        wt, idx = moe_ops.route(logits, soft)
        hit = len(set(idx.flatten().tolist()))
        eb, ef = hit * 3 * EF * W * 2 + T * W * 2 + T * top * (W * 4 + 2 * EF * 2), T * top * 6 * EF * W
        pair(shape, "experts (clamped GLU), unsummed", lambda: moe_cuda.grouped_pairs(spec, act, idx, w), eb, ef, "experts (SwiGLU)",
             lambda: moe_cuda.grouped_pairs(soft, act, idx, lw), eb, ef)
        ye, sp = moe_cuda.grouped_pairs(spec, act, idx, w)
        gate = rnd(T, dtype=f32)
        full = mx.SublayerOut(y, gate, mx.Routed(ye, sp.pair_row, wt))

        def combine():
            out = torch.empty(T, W, dtype=BF, device=DEV)
            ops._native.lib().mb_moe_finish(ops._ptr(ye), ye.stride(0), ops._ptr(sp.pair_row), ops._ptr(wt), T, top, W, ops._ptr(y), W, ops._ptr(gate), 1,
                                            ops._ptr(xb), ops._ptr(out), ops._stream())
        pair(shape, "stream_hyper with gated shared expert and experts' sum",
             lambda: mx.stream_hyper(x, S, "bf16", pending=full, hc=hw, w_in=hw.w_in, pre=n1), T * W * (8 * S + 4 + 4 * top), 0,
             "expert combine (gated shared)", combine, T * W * (6 + 4 * top), 0)
        del gu, dn, w, lw, ye, sp, full
        # ---- attention
        cos, sin = ref.rope_tables(8192, D, 1e4, device=DEV)
        kc, vc = rnd(nblk, 16, G, D), rnd(nblk, 16, G, D)
        qkvg, qn = rnd(T, (H + 2 * G) * D + HD), rnd(D)
        byt = 2 * T * (H + 2 * G) * D * 2
        nm = mx.RmsNorm(qn, 1e-5)
        pos = dict(Hq=H, Hkv=G, positions=b.positions, slots=b.slot_mapping, k_cache=kc, v_cache=vc)
        plain = qkvg[:, :(H + 2 * G) * D].contiguous()
        like = lambda c, s, n: (lambda: ops.qk_norm_rope_kvwrite(plain, D=D, cos=c, sin=s, q_norm_w=n, k_norm_w=n, **pos))
        pair(shape, "rope_dims (rotation)", lambda: mx.rope_dims(qkvg, dk=D, dv=D, cos=cos, sin=sin, fmt="bf16", **pos), byt, 0, "rope + KV write",
             like(cos, sin, None), byt, 0)
        pair(shape, "rope_dims (head norms)", lambda: mx.rope_dims(qkvg, dk=D, dv=D, cos=None, sin=None, fmt="bf16", q_norm=nm, k_norm=nm, **pos), byt, 0,
             "head norms + KV write", like(None, None, qn), byt, 0)
        q, out, sink = rnd(T, H, D), torch.empty(T, HD, dtype=BF, device=DEV), rnd(H, dtype=f32)
        seen = sum(min(window, p + 1) for n in lens for p in range(start, start + n))
        byt = sum(min(ctx, n + window) for n in lens) * G * D * 4 + T * HD * 4
        ge, gh = qkvg[:, (H + 2 * G) * D:], qkvg[:, (H + 2 * G) * D:(H + 2 * G) * D + H]
        kw = dict(dk=D, dv=D, scale=0.09, fmt="bf16", out=out, window=window)
        like = lambda: ops.paged_attention(q, kc, vc, b.block_table, b.q_start, b.q_len, b.ctx_len, max_q_len=b.max_q_len, max_ctx=b.max_ctx, scale=0.09,
                                           window=window)
        pair(shape, "windowed attention, sinks, head gates", lambda: mx.attention_dims(q, kc, vc, b, sink=sink, gate=mx.OutputGate(gh, True), **kw),
             byt + T * H * 2, 4 * HD * seen, "windowed attention", like, byt, 4 * HD * seen)
        gq = rnd(T, 2 * HD)
        pair(shape, "windowed attention, kept tokens, element gates",
             lambda: mx.attention_dims(q, kc, vc, b, sink=False, keep=keep, gate=mx.OutputGate(ge, False), **kw), byt + T * HD * 2, 4 * HD * (seen + T * keep),
             "windowed attention + gate", lambda: ops.row_op(like().view(T, HD), "bf16", ops.IN_SIGMOID_GATE, gate=gq, head_dim=D, gate_head_stride=2 * D,
                                                             gate_head_off=D), byt + T * HD * 6, 4 * HD * seen)
        del q, qkvg, gq, plain
        # ---- matrix products with their epilogues
        gu = QuantWeight("bf16", 2 * FF, W, rnd(2 * FF, W, std=0.02))
        gb, gf = (2 * FF * W + T * W + T * FF) * 2, 2 * T * 2 * FF * W
        pair(shape, "GEMM + clamped GLU", lambda: ops.linear(act, gu, clamp_glu=(1.702, 7.0)), gb, gf, "GEMM + SwiGLU",
             lambda: ops.linear(act, gu, swiglu=True), gb, gf)
    return rows


def ledinex_kernels(W=2560, H=32, G=8, D=128, FF=6912, E=64, top=6, EF=1024, SF=2048, HR=20, window=512, rank=64, taps=3, conv=4):
    """The same rows for Ledinex: the like kernels are those of attention / gated-delta-net / Kimi-delta models with experts."""
    from metrale_inference_alpha_b200.ops import canon, delta as dl, moe as moe_ops, moe_cuda
    from metrale_inference_alpha_b200.weights.loader import MoeW
    rows = []
    HD, RD, pair, f32 = H * D, HR * D, pairing(rows), torch.float32
    for shape, lens, start in SHAPES:
        b, nblk = batch(lens, start)
        T, S, ctx = sum(lens), len(lens), lens[0] + start
        # ---- the stream
        x, y, xb, wv = rnd(T, W, dtype=f32), rnd(T, W), rnd(T, W), rnd(W)
        nm, filt = mx.RmsNorm(wv, 1e-6, plus_one=True), rnd(taps, W)
        win = canon.Window(torch.zeros(S + 2, (taps - 1) * W, device=DEV), 0, W)
        kw = dict(norm=nm, filt=filt, window=win, batch=b)
        one, wb = mx.SublayerOut(y), 2 * S * (taps - 1) * W * 4
        pair(shape, "stream_canon (norm + add + convolution)", lambda: canon.stream_canon(x, "bf16", pending=one, **kw), T * W * 12 + wb, 0,
             "residual + RMSNorm", lambda: ops.row_op(xb, "bf16", ops.IN_RMSNORM, w=wv, residual=y, write_residual=True), T * W * 8, 0)
        # ---- experts
        up, gu = QuantWeight("bf16", E * EF, W, rnd(E * EF, W, std=0.02)), QuantWeight("bf16", E * 2 * EF, W, rnd(E * 2 * EF, W, std=0.02))
        dn = QuantWeight("bf16", E * W, EF, rnd(E * W, EF, std=0.02))
        soft, spec = moe_ops.RouterSpec(E, top, "softmax"), moe_ops.RouterSpec(E, top, "softmax", ffn_act="relu2")
        w = MoeW(grouped=moe_ops.GroupedExperts(up, dn, E, EF, W, False), spec=spec)
        lw = MoeW(grouped=moe_ops.GroupedExperts(gu, dn, E, 2 * EF, W, True), spec=soft)
        act, logits = mx.act_of(rnd(T, W), "bf16"), rnd(T, E, dtype=f32)
        wt, idx = moe_ops.route(logits, soft)
        hit = len(set(idx.flatten().tolist()))
        eb = lambda n: hit * n * EF * W * 2 + T * W * 2 + T * top * (W * 4 + 2 * EF * 2)
        pair(shape, "experts (squared ReLU), unsummed", lambda: moe_cuda.grouped_pairs(spec, act, idx, w), eb(2), T * top * 4 * EF * W, "experts (SwiGLU)",
             lambda: moe_cuda.grouped_pairs(soft, act, idx, lw), eb(3), T * top * 6 * EF * W)
        ye, sp = moe_cuda.grouped_pairs(spec, act, idx, w)
        full = mx.SublayerOut(y, None, mx.Routed(ye, sp.pair_row, wt))

        def combine():
            out = torch.empty(T, W, dtype=BF, device=DEV)
            ops._native.lib().mb_moe_finish(ops._ptr(ye), ye.stride(0), ops._ptr(sp.pair_row), ops._ptr(wt), T, top, W, ops._ptr(y), W, None, 0,
                                            ops._ptr(xb), ops._ptr(out), ops._stream())
        pair(shape, "stream_canon with shared expert and experts' sum", lambda: canon.stream_canon(x, "bf16", pending=full, **kw),
             T * W * (12 + 4 * top) + wb, 0, "expert combine (shared)", combine, T * W * (6 + 4 * top), 0)
        del gu, dn, w, lw, ye, sp, full, up
        su = QuantWeight("bf16", SF, W, rnd(SF, W, std=0.02))
        gb, gf = (SF * W + T * W + T * SF) * 2, 2 * T * SF * W
        pair(shape, "GEMM + squared ReLU", lambda: ops.linear(act, su, relu2=True), gb, gf, "GEMM", lambda: ops.linear(act, su), gb, gf)
        N = (H + G) * D + 5 * RD + rank
        wi, bias = QuantWeight("bf16", N, W, rnd(N, W, std=0.02)), rnd(N, dtype=f32)
        gb, gf = (N * W + T * W + T * N) * 2, 2 * T * N * W
        pair(shape, "twin projection GEMM + bias", lambda: ops.linear(act, wi, bias=bias), gb, gf, "GEMM", lambda: ops.linear(act, wi), gb, gf)
        # ---- attention
        cos, sin = ref.rope_tables(8192, D, 1e4, device=DEV)
        kc, vc = rnd(nblk, 16, G, D), rnd(nblk, 16, G, D)
        qkv, hn = rnd(T, (H + 2 * G) * D), rnd(D)
        pos = dict(Hq=H, Hkv=G, positions=b.positions, slots=b.slot_mapping, k_cache=kc, v_cache=vc)
        qn, kn = mx.RmsNorm(rnd(HD), 1e-6), mx.RmsNorm(rnd(G * D), 1e-6)
        like = lambda: ops.qk_norm_rope_kvwrite(qkv, D=D, cos=cos, sin=sin, q_norm_w=hn, k_norm_w=hn, **pos)
        byt, cols = 2 * qkv.numel() * 2, (0, HD, HD + G * D)
        pair(shape, "attention_rows (norms over all heads, rotated values)",
             lambda: mx.attention_rows(qkv, cols=cols, dk=D, dv=D, rot=(cos, sin), fmt="bf16", q_norm=qn, k_norm=kn, v_rot=(cos, sin), **pos), byt, 0,
             "head norms + rope + KV write", like, byt, 0)
        pair(shape, "attention_rows (values are the keys)",
             lambda: mx.attention_rows(qkv, cols=(0, HD, HD), dk=D, dv=D, rot=(cos, sin), fmt="bf16", q_norm=qn, k_norm=kn, **pos), byt - T * G * D * 2, 0,
             "head norms + rope + KV write", like, byt, 0)
        q, cat = rnd(T, H, D), torch.empty(T, HD + RD, dtype=BF, device=DEV)
        o2, turn = cat[:, :HD], (cos, sin)
        flo = sum(4 * HD * (n * start + n * (n + 1) / 2) for n in lens)
        byt = S * ctx * G * D * 4 + T * HD * 4
        att = lambda win_: (lambda: ops.paged_attention(q, kc, vc, b.block_table, b.q_start, b.q_len, b.ctx_len, max_q_len=b.max_q_len, max_ctx=b.max_ctx,
                                                        scale=0.09, window=win_))
        new = lambda win_, cap, turn_: (lambda: mx.attention_dims(q, kc, vc, b, dk=D, dv=D, scale=0.09, sink=False, fmt="bf16", out=o2, out_scale=0.7,
                                                                  window=win_, softcap=cap, turn_back=turn_))
        pair(shape, "capped attention, output turned back", new(0, 30.0, turn), byt, flo, "attention", att(0), byt, flo)
        seen = sum(min(window, p + 1) for n in lens for p in range(start, start + n))
        byt = sum(min(ctx, n + window) for n in lens) * G * D * 4 + T * HD * 4
        pair(shape, "windowed attention", new(window, 0.0, None), byt, 4 * HD * seen, "windowed attention (other models)", att(window), byt, 4 * HD * seen)
        del q, qkv
        # ---- recurrences
        C3, sb = 3 * RD, 2 * S * HR * D * D * 4
        px, fl = rnd(T, C3 + RD + 64), rnd(conv, C3, dtype=f32)
        wn = canon.Window(torch.zeros(S + 2, (conv - 1) * C3, device=DEV), 0, C3)
        cst, cwt = torch.zeros(S + 2, C3, conv - 1, device=DEV), fl.t().contiguous()
        pair(shape, "short_conv", lambda: canon.short_conv(px[:, :C3], fl, wn, b, "bf16"), T * C3 * 4 + 2 * S * C3 * (conv - 1) * 4, 0, "causal_conv1d",
             lambda: rops.causal_conv1d(px, C3, cwt, None, cst, b), T * C3 * 6 + 2 * S * C3 * (conv - 1) * 4, 0)
        ssm = torch.zeros(S + 2, HR, D, D, device=DEV)
        cv, cf = rnd(T, C3), rnd(T, C3, dtype=f32)
        q, k, v = cv[:, :RD], cv[:, RD:2 * RD], cv[:, 2 * RD:]
        A, dtb, ba = torch.zeros(HR, device=DEV), torch.zeros(HR, device=DEV), rnd(T, 2 * HR, dtype=f32)
        gate, nw, ab = px[:, C3:C3 + RD], rnd(RD), px[:, C3 + RD:]
        rule = dl.GatedRule(ab[:, :HR], ab[:, 32:32 + HR], A, dtb)
        nrm = dict(w=nw, gate=gate, gate_act="silu", eps=1e-6, scale=1.0, out=torch.empty(T, RD, dtype=BF, device=DEV))
        gdn = lambda: ops.row_op(rops.gdn_recurrence(cf, ba, A, dtb, ssm, b, k_heads=HR, v_heads=HR, k_dim=D, v_dim=D), "bf16", ops.IN_GATED_RMSNORM,
                                 gate=gate, w=nw, group=D)
        hk = dict(heads=HR, dk=D, dv=D, fmt="bf16")
        pair(shape, "gated delta rule (recurrence, norm)", lambda: dl.delta_attention(q, k, v, rule, ssm, b, norm=nrm, **hk), T * RD * 10 + sb, 0,
             "gated delta net (recurrence, norm)", gdn, T * RD * 16 + sb, 0)
        rw2 = rnd(RD, rank, std=0.1)
        z, tw = rnd(T, rank), QuantWeight("bf16", RD, 2 * rank, torch.cat([rw2, rw2], 1).contiguous())
        bd = dl.BoundedDecay(z, rw2, rnd(RD, dtype=f32), -0.6065, tw)
        lin, za = QuantWeight("bf16", RD, rank, rw2), mx.act_of(z, "bf16")
        pair(shape, "log decay (bounded, 32-bit low-rank)", bd.log, T * (rank * 2 + RD * 4), 2 * T * rank * RD, "low-rank decay GEMM, bf16",
             lambda: ops.linear(za, lin, out_f32=True), T * (rank * 2 + RD * 4), 2 * T * rank * RD)
        aa = rnd(T, RD)
        gen = dl.GeneralRule(aa, bd)
        nrm2 = dict(nrm, gate_act="sigmoid")
        graw, braw, ng, dt2 = rnd(T, RD, dtype=f32), rnd(T, HR, dtype=f32), torch.ones(D, device=DEV), torch.zeros(RD, device=DEV)
        kda = lambda: rops.kda_recurrence(cf, graw, braw, A, dt2, -5.0, ssm, b, heads=HR, dim=D, norm=(ng, gate, 1e-6))
        pair(shape, "general delta rule (decay, recurrence, norm)", lambda: dl.delta_attention(q, k, v, gen, ssm, b, norm=nrm2, **hk), T * RD * 12 + sb, 0,
             "Kimi delta attention (recurrence, norm)", kda, T * RD * 20 + sb, 0)
        dec = torch.linspace(0.6, 0.999, HR, device=DEV)

        def light():
            core = mx.linear_attention(q, k, v, ssm, b, decay=dec, **hk)
            mx.gated_norm(core, nw, gate, "bf16", group=RD, gate_act="sigmoid", eps=1e-6, out=nrm["out"])
        pair(shape, "lightning attention (recurrence, norm)", light, T * RD * 10 + sb, 0, "gated delta net (recurrence, norm)", gdn, T * RD * 16 + sb, 0)
        del cv, cf, px, graw, q, k, v
    return rows


def ledinex_models():
    """(label, name -> configuration): Ledinex and a hybrid of equal size: attention where Ledinex runs two mixers side by
    side, gated delta net where it runs the gated delta rule, SwiGLU experts with as many rows; bf16."""
    from metrale_inference_alpha_b200.config.model_config import ModelConfig, preset
    for label, kw in (("1B-like layers", dict(width=2048, heads=16, kv_heads=4, right_heads=16, delta_heads=16, delta_kv_heads=16, experts=32, top=4,
                                              expert_ff=768, shared_ff=1536, vocab=32768)),
                      ("3B-like layers", {})):
        p = preset("ledinex-3b", num_layers=6, window=512, **kw)
        m, d, mlp = p.layer_specs[1]["mixer"]["left"], p.layer_specs[0]["mixer"], p.layer_specs[1]["mlp"]
        h = ModelConfig(name="gdn-attention-moe", arch="qwen_hybrid", vocab_size=p.vocab_size, hidden_size=p.hidden_size, num_layers=6,
                        num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"], rotary_dim=m["dim"], qk_norm=True, attn_output_gate=True,
                        norm_plus_one=True, layer_types=["gdn" if t == "delta" else "attention" for t in p.layer_types], ffn_types=list(p.ffn_types),
                        gdn_k_heads=d["kv_heads"], gdn_v_heads=d["heads"], gdn_k_dim=d["dim"], gdn_v_dim=d["vdim"], conv_kernel=d["conv"],
                        num_experts=mlp["router"]["experts"], experts_per_token=mlp["router"]["top"], moe_intermediate_size=mlp["expert"]["ff"],
                        intermediate_size=mlp["expert"]["ff"], num_shared_experts=mlp["shared"]["ff"] // mlp["expert"]["ff"], shared_expert_gate=True,
                        router="softmax", tie_embeddings=True, weight_format="bf16", kv_dtype="bf16", max_position=16384)
        yield label, {"ledinex": p, "gated-delta-net / attention MoE": h}


def pivipel_models():
    """(label, name -> configuration): Pivipel and a model of equal size with the same experts, windows, head norms and
    output gates on one bf16 residual; bf16."""
    from metrale_inference_alpha_b200.config.model_config import ModelConfig, preset
    for label, kw in (("1B-like layers", dict(width=2048, heads=16, kv_heads=4, ff=5632, experts=32, top=4, expert_ff=768, shared_ff=1536, vocab=32768)),
                      ("3B-like layers", {})):
        p = preset("pivipel-3b", num_layers=6, window=512, **kw)
        m, mlp = p.layer_specs[1]["mixer"], p.layer_specs[1]["mlp"]
        h = ModelConfig(name="gated-attention-moe", arch="qwen_hybrid", vocab_size=p.vocab_size, hidden_size=p.hidden_size, num_layers=6,
                        num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"], rotary_dim=m["dim"], qk_norm=True, attn_output_gate=True,
                        norm_plus_one=True, layer_types=["attention"] * 6, ffn_types=list(p.ffn_types), sliding_window=m["mask"]["size"],
                        intermediate_size=p.intermediate_size, num_experts=mlp["router"]["experts"], experts_per_token=mlp["router"]["top"],
                        moe_intermediate_size=mlp["expert"]["ff"], num_shared_experts=mlp["shared"]["ff"] // mlp["expert"]["ff"], shared_expert_gate=True,
                        router="softmax", tie_embeddings=True, weight_format="bf16", kv_dtype="bf16", max_position=16384)
        yield label, {"pivipel": p, "gated-attention MoE": h}


def finelix_models():
    """(label, name -> configuration): Finelix, the same with two layers looped three times, and a hybrid of
    equal size: MLA and experts where Finelix has latent attention, Kimi delta attention and SwiGLU elsewhere; bf16."""
    from metrale_inference_alpha_b200.config.model_config import ModelConfig, preset
    for label, kw in (("1B-like layers", dict(width=2048, heads=16, lin_heads=16, ff=5632, experts=32, top=4, expert_ff=768, shared_ff=1536, vocab=32768)),
                      ("3B-like layers", {})):
        looped = preset("finelix-3b", num_layers=6, **kw)
        f = looped.scaled(loop=None)
        m, mlp = f.layer_specs[1]["mixer"], f.layer_specs[1]["mlp"]
        g = f.layer_specs[0]["mixer"]
        h = ModelConfig(name="mla-kda-hybrid", arch="deepseek_mla", vocab_size=f.vocab_size, hidden_size=f.hidden_size, num_layers=6,
                        num_heads=m["heads"], num_kv_heads=m["heads"], head_dim=m["dim"] + m["rot_dim"], rope_theta=10000.0,
                        layer_types=["mla" if t == "latent" else "kda" for t in f.layer_types], ffn_types=list(f.ffn_types),
                        dense_intermediate_size=f.intermediate_size, intermediate_size=f.intermediate_size, q_lora_rank=m["q_rank"],
                        kv_lora_rank=m["kv_rank"], qk_nope_dim=m["dim"], qk_rope_dim=m["rot_dim"], v_head_dim=m["vdim"],
                        num_experts=mlp["router"]["experts"], experts_per_token=mlp["router"]["top"], moe_intermediate_size=mlp["expert"]["ff"],
                        num_shared_experts=mlp["shared"]["ff"] // mlp["expert"]["ff"], router="sigmoid", kda_heads=g["heads"], kda_head_dim=g["dim"],
                        kda_gate_rank=64, weight_format="bf16", kv_dtype="bf16", max_position=16384)
        yield label, {"finelix": f, "MLA / Kimi-delta hybrid": h, "finelix, two layers looped three times": looped}


def models():
    """(label, Fabulix configuration, hybrid of equal size: attention where Fabulix runs two mixers in parallel,
    Kimi delta attention where it runs lightning attention; SwiGLU; bf16)."""
    from metrale_inference_alpha_b200.config.model_config import ModelConfig, preset
    for label, kw in (("1B-like layers", dict(num_layers=6, width=2048, heads=16, kv_heads=4, right_heads=16, lin_heads=16, ff=5632, dim=128, vdim=128,
                                              rot_dims=128, right_dim=128, lin_dim=128, lin_vdim=128, vocab=32768)),
                      ("3B-like layers", dict(num_layers=6))):
        f = preset("fabulix-3b", **kw)
        a = f.layer_specs[0]["mixer"]["left"]
        h = ModelConfig(name="kda-hybrid", arch="qwen_hybrid", vocab_size=f.vocab_size, hidden_size=f.hidden_size, num_layers=f.num_layers,
                        num_heads=a["heads"], num_kv_heads=a["kv_heads"], head_dim=a["dim"], rotary_dim=a["dim"], qk_norm=True,
                        layer_types=["kda" if t == "lightning" else "attention" for t in f.layer_types], ffn_types=["dense"] * f.num_layers,
                        intermediate_size=f.intermediate_size, kda_heads=a["heads"], kda_head_dim=128, kda_gate_rank=64, tie_embeddings=True,
                        norm_plus_one=True, weight_format="bf16", kv_dtype="bf16", max_position=16384)
        yield label, {"fabulix": f, "attention / Kimi-delta hybrid": h}


def throughput(cfg, decode_batches=(1, 32, 128), prefills=((1, 4096), (8, 1024)), ctx=1024):
    """Device-timed: prefill tokens/s of whole prompts (one forward each) and decode tokens/s of graph replays."""
    from metrale_inference_alpha_b200.engine.llm_engine import EngineArgs, LLMEngine
    from metrale_inference_alpha_b200.scheduler.types import Request, SeqStep, Sequence, StepPlan
    from metrale_inference_alpha_b200.sampling.params import SamplingParams
    t, out = Timer(), {"params": cfg.param_count()}
    eng = LLMEngine(EngineArgs(model=cfg, device=DEV, max_num_seqs=128, max_model_len=8192, max_prefill_tokens=8192, num_kv_blocks=128 * (ctx // 16 + 2) + 64,
                               enable_prefix_caching=False))
    r = eng.runner

    def seqs(n, length):
        res, nb = [], length // 16 + 2
        for i in range(n):
            s = Sequence(Request(f"b{i}", [3 + (7 * i + j) % 1000 for j in range(length)], SamplingParams(max_tokens=4)), i + 1)
            s.blocks, s.state_slot = list(range(1 + i * nb, 1 + (i + 1) * nb)), (i + 1 if r.pool is not None else 0)
            res.append(s)
        return res

    for n, length in prefills:
        ss = seqs(n, length)
        b = r._stage(StepPlan("prefill", [SeqStep(s, s.tokens, 0) for s in ss]))
        dt = t(lambda: r.decoder.forward(b, r.caches), iters=5)
        out[f"prefill {n}x{length}"] = {"ms": round(dt * 1e3, 3), "tok_s": round(n * length / dt)}
    for n in decode_batches:
        plan = StepPlan("decode", [SeqStep(s, [5], ctx - 1) for s in seqs(n, ctx)])
        r._decode_graph(plan, True, False)
        torch.cuda.synchronize()
        g = r.graphs[(r._rung(n), True, False)][0]
        dt = t(g.replay)
        out[f"decode {n}"] = {"ms": round(dt * 1e3, 4), "tok_s": round(n / dt)}
    ops.check_status(DEV)
    eng.close()
    return out


def run(what="all", design="fabulix"):
    res = {"design": design}
    if what in ("all", "kernels"):
        res["kernels"] = {"fabulix": kernels, "finelix": finelix_kernels, "pivipel": pivipel_kernels, "ledinex": ledinex_kernels}[design]()
    if what in ("all", "models"):
        res["models"] = {}
        for label, cfgs in {"fabulix": models, "finelix": finelix_models, "pivipel": pivipel_models, "ledinex": ledinex_models}[design]():
            res["models"][label] = {}
            for name, cfg in cfgs.items():
                res["models"][label][name] = throughput(cfg)
                print(label, name, res["models"][label][name], file=sys.stderr, flush=True)
                torch.cuda.empty_cache()
    ops.check_status(DEV)
    return res


if __name__ == "__main__":
    print(json.dumps(run(*sys.argv[1:3])))
