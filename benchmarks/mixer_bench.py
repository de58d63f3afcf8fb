#!/usr/bin/env python
"""The kernels of the Fabulix decoder next to the like kernels of the engine's attention / Kimi-delta-attention /
Mamba2 hybrids at equal size, each with its distance from the roofline (measured copy bandwidth and measured
bf16 GEMM rate), and the throughput of a whole model next to an equal-size hybrid. CUDA events around one call,
L2 flushed by a 512 MB write before every call, median of the timed calls. Reached as `bench.py --mixers`.
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


def kernels(W=2560, H=20, G=4, D=128, FF=6912, R=64, side=128):
    """Rows: (shape, mechanism, new us, new bytes, new flops, like name, like us, like bytes, like flops)."""
    t, rows, bw, fl = Timer(), [], *peaks()
    HD = H * D

    def pair(shape, name, new, nb, nf, like_name, like, lb, lf):
        a, b = t(new), t(like)
        ra, rb = max(nb / bw, nf / fl), max(lb / bw, lf / fl)
        rows.append({"shape": shape, "kernel": name, "us": round(a * 1e6, 1), "x_roofline": round(a / ra, 2), "like": like_name,
                     "like_us": round(b * 1e6, 1), "like_x_roofline": round(b / rb, 2), "ratio": round(a / ra / (b / rb), 2)})
        print(rows[-1], file=sys.stderr, flush=True)

    for shape, lens, start in (("decode 128 seqs, ctx 1024", [1] * 128, 1023), ("prefill 1 x 4096", [4096], 0), ("prefill 8 x 1024", [1024] * 8, 0)):
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
        yield label, f, h


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


def run(what="all"):
    res = {}
    if what in ("all", "kernels"):
        res["kernels"] = kernels()
    if what in ("all", "models"):
        res["models"] = {}
        for label, f, h in models():
            res["models"][label] = {}
            for name, cfg in (("fabulix", f), ("attention / Kimi-delta hybrid", h)):
                res["models"][label][name] = throughput(cfg)
                print(label, name, res["models"][label][name], file=sys.stderr, flush=True)
                torch.cuda.empty_cache()
    ops.check_status(DEV)
    return res


if __name__ == "__main__":
    print(json.dumps(run(sys.argv[1] if len(sys.argv) > 1 else "all")))
