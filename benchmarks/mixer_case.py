"""One launch sequence on a small case, for a profiler: decode | chunk (recurrence, time-mix mode), gla (the same
recurrence read after its update, with low-rank decays and the head norm), latent-decode | latent (latent attention),
hyper (residual streams: join, read, norm), window-decode | window (windowed attention with kept tokens and gates),
gated-delta | general-delta (delta rules with their head norm; -decode: one token each), canon (join and convolution), capped-decode | capped
(attention with capped scores whose outputs are turned back)."""
import os
import sys

import torch

sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
from benchmarks.mixer_bench import batch, rnd  # noqa: E402
from metrale_inference_alpha_b200.ops import check_status, mixers as mx  # noqa: E402

case = sys.argv[1]
H, D = 20, 128
if case.startswith("latent"):
    from metrale_inference_alpha_b200.ops import latent as lt
    lens, start = ([1] * 64, 1023) if case == "latent-decode" else ([1024], 0)
    b, blocks = batch(lens, start)
    T, heads, lay = sum(lens), 32, lt.latent_row(512, 64, "bf16")
    cache, q, uv = rnd(blocks, 16, 1, lay.row), rnd(T, heads, lay.row, std=0.3), rnd(heads, 128, 512, std=0.05)
    out = torch.empty(T, heads * 128, dtype=q.dtype, device="cuda")
    run = lambda: lt.attention(q, cache, b, uv, 0.07, "bf16", lay, out)
elif case == "hyper":
    T, W, S = 8192, 2560, 2
    x, pre = rnd(T, S, W, dtype=torch.float32), mx.DytNorm(0.5, rnd(W), rnd(W))
    hc, out = mx.HyperW(*(torch.full(s, 0.4, device="cuda") for s in ((S,), (S,), (S, S)))), mx.SublayerOut(rnd(T, W))
    run = lambda: mx.stream_hyper(x, S, "bf16", pending=out, hc=hc, w_in=hc.w_in, pre=pre)
elif "delta" in case:
    from metrale_inference_alpha_b200.ops import delta as dl
    lens, start = ([1] * 128, 63) if case.endswith("-decode") else ([4096], 0)
    b, _ = batch(lens, start)
    T = sum(lens)
    q, k, v, g, a = (rnd(T, H * D) for _ in range(5))
    ssm, A = torch.zeros(len(lens) + 2, H, D, D, device="cuda"), torch.zeros(H, device="cuda")
    low = dl.BoundedDecay(rnd(T, 64), rnd(H * D, 64, std=0.1), rnd(H * D, dtype=torch.float32), -0.6065)
    rule = dl.GatedRule(a[:, :H], a[:, 64:64 + H], A, A) if case.startswith("gated") else dl.GeneralRule(a, low)
    norm = dict(w=rnd(H * D), gate=g, gate_act="silu", eps=1e-6, scale=1.0, out=torch.empty_like(g))
    run = lambda: dl.delta_attention(q, k, v, rule, ssm, b, heads=H, dk=D, dv=D, fmt="bf16", norm=norm)
elif case == "canon":
    from metrale_inference_alpha_b200.ops import canon
    T, W = 8192, 2560
    b, _ = batch([T], 0)
    x, y, win = rnd(T, W, dtype=torch.float32), mx.SublayerOut(rnd(T, W)), canon.Window(torch.zeros(4, 2 * W, device="cuda"), 0, W)
    nm, filt = mx.RmsNorm(rnd(W), 1e-6, plus_one=True), rnd(3, W)
    run = lambda: canon.stream_canon(x, "bf16", pending=y, norm=nm, filt=filt, window=win, batch=b)
elif case.startswith("capped"):
    from metrale_inference_alpha_b200.ops import reference as ref
    lens, start = ([1] * 128, 1023) if case == "capped-decode" else ([4096], 0)
    b, blocks = batch(lens, start)
    T, H, G = sum(lens), 32, 8
    kc, vc, q = rnd(blocks, 16, G, D), rnd(blocks, 16, G, D), rnd(T, H, D)
    out, turn = torch.empty(T, H * D, dtype=q.dtype, device="cuda"), ref.rope_tables(8192, D, 1e4, device="cuda")
    run = lambda: mx.attention_dims(q, kc, vc, b, dk=D, dv=D, scale=0.09, sink=False, fmt="bf16", out=out, softcap=30.0, turn_back=turn)
elif case.startswith("window"):
    lens, start = ([1] * 128, 1023) if case == "window-decode" else ([4096], 0)
    b, blocks = batch(lens, start)
    T, H, G = sum(lens), 32, 8
    kc, vc, q, z = rnd(blocks, 16, G, D), rnd(blocks, 16, G, D), rnd(T, H, D), rnd(T, H * D)
    out = torch.empty_like(z)
    run = lambda: mx.attention_dims(q, kc, vc, b, dk=D, dv=D, scale=0.09, sink=False, fmt="bf16", out=out, window=512, keep=4,
                                    gate=mx.OutputGate(z, False))
else:
    lens, start = ([1] * 128, 63) if case == "decode" else ([4096], 0)
    b, _ = batch(lens, start)
    T = sum(lens)
    q, k, v, g = (rnd(T, H * D) for _ in range(4))
    ssm = torch.zeros(len(lens) + 2, H, D, D, device="cuda")
    kw = dict(heads=H, dk=D, dv=D, fmt="bf16")
    if case == "gla":
        lr = mx.LowRankDecay(rnd(T, 16), rnd(H * D, 16, std=0.1), rnd(H * D, dtype=torch.float32), 1 / 16)
        kw.update(low_rank=lr, norm=dict(w=rnd(H * D), gate=g, gate_act="silu", eps=1e-5, scale=1.0, out=torch.empty_like(g)))
    else:
        kw.update(log_w=-torch.exp(torch.randn(T, H * D, device="cuda") - 3), u=torch.rand(H, D, device="cuda"))
    run = lambda: mx.linear_attention(q, k, v, ssm, b, **kw)
for _ in range(3):
    run()
torch.cuda.synchronize()
check_status("cuda")
