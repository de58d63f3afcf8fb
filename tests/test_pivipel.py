"""The Pivipel decoder against a plain restatement (pivipel_oracle.py): every mechanism alone, then whole models through
the engine's own entry points. The CPU runs cover the engine's host logic and its op restatements, the GPU runs the
kernels."""
import json
import math

import pytest
import torch

import pivipel_cases as pc
import pivipel_oracle as po
from metrale_inference_alpha_b200 import ops
from metrale_inference_alpha_b200.config.model_config import from_hf_config, from_pivipel_config, preset
from metrale_inference_alpha_b200.engine.llm_engine import EngineArgs, LLMEngine
from metrale_inference_alpha_b200.engine.replay import TraceReplay
from metrale_inference_alpha_b200.ops import mixers as mx, moe as moe_ops, reference as ref
from metrale_inference_alpha_b200.sampling.params import SamplingParams

DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]
DTYPES = ["fp32", "bf16"]
TOL = 3e-5                                  # 32-bit models: of the logits' rms
dt = lambda fmt: mx.DTYPE[fmt]


def gen(*shape, seed=0, std=1.0, mean=0.0):
    g = torch.Generator().manual_seed(seed)
    return torch.randn(*shape, generator=g) * std + mean


def b16(t):
    return t.to(torch.bfloat16)


def close(got, want, rel):
    got, want = got.double().cpu(), want.double()
    err = float((got - want).abs().max())
    assert err <= rel * float(want.abs().max()) + 1e-12, (err, float(want.abs().max()))


def near(got, want, dtype):
    """32-bit models: every row. bf16 models: single rows may round badly (a sharp softmax), most do not."""
    d = got.double() - want
    d = (d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    if dtype == "fp32":
        return float(d.max()) < TOL
    return float(d.max()) < 0.2 and float(d.quantile(0.9)) < 0.05 * (1 if len(d) > 9 else 2)


# ------------------------------------------------------------------ the streams
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", DTYPES)
@pytest.mark.parametrize("S,W", [(1, 37), (2, 96), (3, 100), (4, 2560), (5, 52), (9, 37)])
def test_streams_join_and_read(device, fmt, S, W):
    T, K = 11, 3
    hc, nx = (mx.HyperW(gen(S, seed=s), gen(S, seed=s + 1), gen(S, S, seed=s + 2)) for s in (1, 4))
    on = lambda h: mx.HyperW(h.w_in.to(device), h.w_out.to(device), h.w_mix.to(device))
    pre = mx.DytNorm(0.7, b16(gen(W, seed=7)), b16(gen(W, seed=8)))
    pre_d = mx.DytNorm(0.7, pre.w.to(device), pre.b.to(device))
    y, logit = gen(T, W, seed=9).to(dt(fmt)), gen(T, 5, seed=10, std=2.0)
    ye, pw = gen(T * K, W + 4, seed=11), gen(T, K, seed=12).abs()
    place = torch.randperm(T * K, generator=torch.Generator().manual_seed(1)).int()
    place[4] = place[20] = -1                                        # pairs that no row stands for
    esum = torch.zeros(T, W, dtype=torch.float64)
    for t in range(T):
        for j in range(K):
            if place[t * K + j] >= 0:
                esum[t] += pw[t, j].double() * ye[int(place[t * K + j]), :W].double()
    routed = mx.Routed(esum.float(), None, None) if device == "cpu" else mx.Routed(ye.to(device), place.to(device), pw.to(device))
    sg = logit.to(device)[:, 3]                                      # a column
    gated = y.double() * po.sigmoid(logit[:, 3].double())[:, None]
    tol = 1e-5 if fmt == "fp32" else 6e-3
    rows = torch.tensor([10, 0, 3, 3], dtype=torch.int64)
    for one in (True, False):
        x = gen(T, W, seed=2, std=3.0) if one else gen(T, S, W, seed=3, std=3.0)
        xs = (x[:, None].expand(T, S, W) if one else x).double().transpose(0, 1)
        for out, Y in ((mx.SublayerOut(y.to(device)), y.double()), (mx.SublayerOut(y.to(device), sg), gated),
                       (mx.SublayerOut(y.to(device), sg, routed), gated + esum), (mx.SublayerOut(routed=routed), esum), (None, None)):
            new = xs if out is None else po.write_streams(xs, Y, hc.w_mix.double(), hc.w_out.double())
            u = po.read_streams(new, nx.w_in.double())
            kw = dict(pending=out, hc=on(hc) if out else None, w_in=on(nx).w_in)
            xd = x.to(device)
            close(mx.stream_hyper(xd, S, fmt, rows=rows.to(device), out_f32=True, **kw)[1], u[rows], 1e-5)
            assert torch.equal(xd.cpu(), x)                          # chosen rows leave the streams as they are
            x1, h = mx.stream_hyper(xd.clone(), S, fmt, pre=pre_d, **kw)
            close(h, po.dynamic_tanh(u, pre.alpha, pre.w.double(), pre.b.double()), tol)
            if out is not None:
                close(x1, new.transpose(0, 1), 2e-6)                 # the streams are 32-bit in both formats
            close(mx.stream_hyper(xd.clone(), S, fmt, **kw)[1], u, tol)
            x2, s = mx.stream_hyper(xd.clone(), S, fmt, out_f32=True, **kw)
            close(s, u, 1e-5)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("W", [37, 128])
def test_embedding_with_positions_and_norm(device, W):
    table, pos = b16(gen(30, W, seed=1)), b16(gen(50, W, seed=2))
    n = mx.DytNorm(0.8, b16(gen(W, seed=3)), b16(gen(W, seed=4)))
    ids, at = torch.tensor([3, 29, 0, 7, 7], dtype=torch.int32), torch.tensor([0, 49, 1, 17, 16], dtype=torch.int32)
    d = lambda t: t.to(device)
    got = mx.embed_scaled(d(ids), d(table), 1.0, pos=d(pos), positions=d(at), norm=mx.DytNorm(0.8, d(n.w), d(n.b)))
    x = table[ids.long()].double() + pos[at.long()].double()
    close(got, po.dynamic_tanh(x, 0.8, n.w.double(), n.b.double()), 2e-6)
    close(mx.embed_scaled(d(ids), d(table), 2.0, pos=d(pos), positions=d(at)), x + table[ids.long()].double(), 1e-6)


# ------------------------------------------------------------------ head norms, rotation, cache rows
def test_scaled_frequencies():
    """Every band: frequencies that stay, that are divided, and between."""
    for rot in ({"base": 3000.0, "dims": 32, "scaling": {"factor": 6.0, "low": 1.0, "high": 3.0, "original": 96}},
                {"base": 1e4, "dims": 10, "scaling": {"factor": 3.0, "low": 0.5, "high": 3.0, "original": 30}}, {"base": 500.0, "dims": 6}):
        s = rot.get("scaling")
        hf = s and {"rope_type": "llama3", "factor": s["factor"], "low_freq_factor": s["low"], "high_freq_factor": s["high"],
                    "original_max_position_embeddings": s["original"]}
        want = torch.tensor(po.frequencies(rot), dtype=torch.float64)
        assert float((ref.rope_inv_freq(rot["dims"], rot["base"], hf)[0] / want - 1).abs().max()) < 1e-12
        if s:
            wave = [2 * math.pi * rot["base"] ** (2 * i / rot["dims"]) for i in range(rot["dims"] // 2)]
            bands = [0 if w < s["original"] / s["high"] else 2 if w > s["original"] / s["low"] else 1 for w in wave]
            assert set(bands) == {0, 1, 2}


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", DTYPES)
@pytest.mark.parametrize("H,G,dk,dv,rot", [(4, 2, 64, 64, 0), (3, 1, 22, 30, 10), (6, 2, 128, 40, 128), (2, 1, 264, 12, 8), (9, 3, 20, 20, 0)])
@pytest.mark.parametrize("which", ["qk", "q", "k", ""])
def test_head_norms_and_rotation(device, fmt, H, G, dk, dv, rot, which):
    T, eps, block = 7, 1e-2, 16
    n = (H + G) * dk + G * dv
    x = gen(T, n + 8, seed=1).to(dt(fmt)).to(device)                      # gate logits behind the values
    pos = torch.tensor([0, 1, 15, 16, 17, 900, 3], dtype=torch.int32)
    slots = torch.tensor([40, 3, 17, 16, -1, 79, 47], dtype=torch.int64)
    w = {k: b16(gen(dk, seed=s, std=0.3, mean=1.0)) for k, s in (("q", 2), ("k", 3))}
    nm = {k: mx.RmsNorm(w[k].to(device), eps) if k in which else None for k in "qk"}
    dkp, dvp = mx.padded_head_dims(dk, dv, fmt)
    kc = torch.full((5, block, G, dkp), 9.0, dtype=dt(fmt), device=device)
    vc = torch.full((5, block, G, dvp), 9.0, dtype=dt(fmt), device=device)
    cos, sin = ref.rope_tables(1000, rot, 700.0, device=device) if rot else (None, None)
    q = mx.rope_dims(x, Hq=H, Hkv=G, dk=dk, dv=dv, positions=pos.to(device), slots=slots.to(device), k_cache=kc, v_cache=vc, cos=cos, sin=sin,
                     fmt=fmt, q_norm=nm["q"], k_norm=nm["k"])
    xc, tol = x.double().cpu(), 1e-5 if fmt == "fp32" else 6e-3
    qw, kw = xc[:, :H * dk].view(T, H, dk), xc[:, H * dk:(H + G) * dk].view(T, G, dk)
    if nm["q"]:
        qw = po.rms_norm(qw, w["q"].double(), eps)
    if nm["k"]:
        kw = po.rms_norm(kw, w["k"].double(), eps)
    if rot:
        r = {"base": 700.0, "dims": rot}
        qw, kw = (torch.stack([po.rotate(t[i], int(pos[i]), r) for i in range(T)]) for t in (qw, kw))
    close(q[..., :dk], qw, tol)
    assert bool((q[..., dk:] == 0).all())
    kc, vc = kc.cpu().view(-1, G, dkp), vc.cpu().view(-1, G, dvp)
    live = slots >= 0
    close(kc[slots[live], :, :dk], kw[live], tol)
    close(vc[slots[live], :, :dv], xc[live, (H + G) * dk:n].view(-1, G, dv), 1e-9)
    assert bool((kc[slots[live], :, dk:] == 0).all()) and bool((vc[slots[live], :, dv:] == 0).all())
    untouched = [s for s in range(80) if s not in slots.tolist()]
    assert bool((kc[untouched] == 9).all()) and bool((vc[untouched] == 9).all())


# ------------------------------------------------------------------ attention
# H, G, dk, dv: the 64-, 128- and 256-wide tiles (equal and not), past them, away from whole vectors
ATT = {"t64": (4, 2, 64, 64), "t64/128": (4, 4, 40, 128), "t128": (6, 2, 128, 128), "t128/64": (3, 1, 100, 48), "t256": (2, 1, 200, 72),
       "t256 full": (4, 2, 256, 256), "past": (2, 1, 264, 20), "odd": (3, 1, 22, 30)}
# window, kept, sink, gate
MASKS = {"window": (19, 0, True, "head"), "one": (1, 0, True, None), "kept": (17, 3, False, "element"), "kept all": (5, 90, False, "element"),
         "two tiles kept": (33, 70, True, "head"), "wide": (64, 16, True, "element"), "past it": (500, 5, False, "head"), "none": (0, 0, True, "element")}


def qkv_of(dims, n, fmt, seed=0, far=()):
    """Random rows, with keys that stand out: query i finds key j far above all others."""
    H, G, dk, dv = dims
    q, k, v = gen(n, H, dk, seed=seed), gen(n, G, dk, seed=seed + 1), gen(n, G, dv, seed=seed + 2)
    for i, j in far:
        k[j] *= 3.0 / k[j].abs().max()
        q[i] = k[j].repeat_interleave(H // G, 0) * 2
    return tuple(t.to(dt(fmt)) for t in (q, k, v))


def run_attention(device, fmt, qkv, dims, cuts, scale, window, keep, sink=None, gate=None, kernel="auto", block=16):
    """One sequence fed in portions through the paged cache beside a short second sequence. gate: [n, H] or [n, H, dv]
    logits. Returns [n, H, dv]."""
    H, G, dk, dv = dims
    q, k, v = qkv
    n = q.shape[0]
    dkp, dvp = mx.padded_head_dims(dk, dv, fmt)
    nb = (n + block - 1) // block
    full = lambda d: torch.full((2 * nb + 8, block, G, d), float("nan"), dtype=dt(fmt), device=device)   # unwritten slots must not matter
    kc, vc = full(dkp), full(dvp)
    pages = list(range(nb + 4, 4, -1))                                # descending: pages are not in order
    z = None if gate is None else gate.reshape(n, -1)
    rows = torch.cat([q.reshape(n, -1), k.reshape(n, -1), v.reshape(n, -1)] + ([z.to(dt(fmt))] if z is not None else []), 1)
    at_g = (H + G) * dk + G * dv
    rows = torch.cat([rows, rows.new_zeros(n, -rows.shape[1] % 8)], 1)
    outs, at, i = [], 0, 0
    while at < n:
        m = min(cuts[min(i, len(cuts) - 1)], n - at)
        o1 = min(at, 15)                                              # the neighbour's position this step
        b = pc.batch([m, 1], [at + m, o1 + 1], device=device, block=block, pages=[pages[:(at + m + block - 1) // block], [1]])
        x = torch.cat([rows[at:at + m], rows[o1:o1 + 1]]).to(device)
        qq = mx.rope_dims(x, Hq=H, Hkv=G, dk=dk, dv=dv, positions=b.positions, slots=b.slot_mapping, k_cache=kc, v_cache=vc, cos=None, sin=None, fmt=fmt)
        wide = torch.full((m + 1, H * dv + 8), 5.0, dtype=dt(fmt), device=device)
        g = None if z is None else mx.OutputGate(x[:, at_g:at_g + z.shape[1]], gate.dim() == 2)
        mx.attention_dims(qq, kc, vc, b, dk=dk, dv=dv, scale=scale, sink=False if sink is None else sink.to(device), fmt=fmt, out=wide[:, 8:],
                          window=window, keep=keep, gate=g, kernel=kernel)
        assert bool((wide[:, :8] == 5.0).all())
        outs.append(wide[:m, 8:])
        at, i = at + m, i + 1
    return torch.cat(outs).view(n, H, dv).double().cpu()


def plain(qkv, scale, window, keep, sink=None, gate=None, fmt="fp32"):
    mask = {"size": window, "keep_first": keep} if window else {}
    o = po.attend(*(t.double() for t in qkv), mask, scale, None if sink is None else sink.double())
    if gate is not None:
        g = po.sigmoid(gate.to(dt(fmt)).double())
        o = o * (g[:, :, None] if g.dim() == 2 else g)
    return o


FAR = ((0, 0), (15, 0), (16, 15), (17, 16), (32, 31), (33, 32), (47, 1), (48, 0), (63, 48), (69, 0), (69, 16), (50, 33), (51, 32), (40, 2), (41, 3))


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", DTYPES)
@pytest.mark.parametrize("name,mask", [(a, "kept") for a in ATT] + [(a, "window") for a in ("t64", "t128", "odd")] + [("t64", m) for m in MASKS] +
                         [("t128/64", "two tiles kept"), ("past", "kept all"), ("t256", "none")])
@pytest.mark.parametrize("cuts", [[70], [2], [33, 1], [1]])
def test_windowed_attention(device, fmt, name, mask, cuts):
    dims, (window, keep, sink, gate) = ATT[name], MASKS[mask]
    H, G, dk, dv = dims
    qkv = qkv_of(dims, 70, fmt, far=FAR)
    sink = gen(H, seed=5, mean=1.0) if sink else None
    gate = None if gate is None else gen(70, H, seed=6) if gate == "head" else gen(70, H, dv, seed=6)
    want = plain(qkv, 0.13, window, keep, sink, gate, fmt)
    close(run_attention(device, fmt, qkv, dims, cuts, 0.13, window, keep, sink, gate), want, 2e-5 if fmt == "fp32" else 8e-3)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", DTYPES)
@pytest.mark.parametrize("window,keep", [(1, 1), (16, 0), (17, 3), (20, 16), (64, 2), (31, 17)])
def test_single_keys_at_the_edges(device, fmt, window, keep):
    """One key outshines all others: queries that see it return its value, the first one past the window does not, and kept
    tokens stay visible for good."""
    dims, n, scale = (2, 1, 16, 24), 90, 4.0
    q, k, v = gen(n, 2, 16, seed=1, std=0.05), gen(n, 1, 16, seed=2, std=0.05), gen(n, 1, 24, seed=3)
    q[..., 0] = 4.0
    for j in (0, keep - 1, keep, 15, 16, 33):
        if j < 0:
            continue
        kj = k.clone()
        kj[j, 0, 0] = 4.0
        qkv = tuple(t.to(dt(fmt)) for t in (q, kj, v))
        for cuts in ([n], [17, 16, 2, 1]):
            got = run_attention(device, fmt, qkv, dims, cuts, scale, window, keep)
            for i in range(j, n):
                hit = float((got[i] - qkv[2][j].double()).abs().max()) < 2e-2
                assert hit == (i - j < window or j < keep), (i, j)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", DTYPES)
def test_sinks_far_above_and_below(device, fmt):
    """A sink above every score takes nearly all, one far below nothing; heads differ."""
    dims = (4, 2, 64, 64)
    qkv = qkv_of(dims, 40, fmt, seed=4)
    sink = torch.tensor([-60.0, 0.0, 9.0, 80.0])
    for cuts in ([40], [1]):
        got = run_attention(device, fmt, qkv, dims, cuts, 0.2, 11, 0, sink)
        want = plain(qkv, 0.2, 11, 0, sink)
        for h in range(3):
            close(got[:, h], want[:, h], 2e-5 if fmt == "fp32" else 8e-3)
        assert float(got[:, 3].abs().max()) < 1e-20


@pytest.mark.gpu
@pytest.mark.parametrize("kernel,name", [("mma", "t64"), ("mma", "t128"), ("tc", "t128"), ("auto", "t128"), ("auto", "t256"), ("tc", "t256 full"), ("mma", "t128/64"),
                                         ("simt", "t64"), ("mma", "t64/128")])
@pytest.mark.parametrize("window,keep", [(300, 5), (129, 64), (1100, 130), (64, 65), (700, 0), (0, 0)])
def test_attention_kernels_long(kernel, name, window, keep):
    """Long contexts: many tiles in and past the window, several partitions of what is seen, kept tokens over several
    tiles, far keys on both sides of every edge. Rows are rounded to bf16 on both sides."""
    dims, n, scale = ATT[name], 1250, 0.09
    H, G, dk, dv = dims
    q, k, v = (b16(gen(n, h, d, seed=s)) for h, d, s in ((H, dk, 1), (G, dk, 2), (G, dv, 3)))
    w = window or n
    for i, j in [(i, j) for i in (700, 1199, 1210, 1249) for j in (i, i - w + 1, i - w, 0, keep - 1, keep, 64) if 0 <= j <= i]:
        k[j] = k[j] * 1.5
        q[i, ::2] = k[j].repeat_interleave(H // G, 0)[::2]
    sink, gate = gen(H, seed=5, mean=2.0), b16(gen(n, H, dv, seed=6))
    s = torch.einsum("ihd,jhd->hij", q.double(), k.double().repeat_interleave(H // G, 1)) * scale
    i, j = torch.arange(n)[:, None], torch.arange(n)[None]
    s.masked_fill_((j > i) | ((i - j >= w) & (j >= keep)), float("-inf"))
    p = torch.softmax(torch.cat([s, sink.double()[:, None, None].expand(H, n, 1)], -1), -1)[..., :-1]
    want = torch.einsum("hij,jhd->ihd", p, v.double().repeat_interleave(H // G, 1)) * po.sigmoid(gate.double())
    dkp, dvp = mx.padded_head_dims(dk, dv, "bf16")
    nb = n // 16 + 2
    pages = list(range(nb + 7, 7, -1))
    idx = torch.tensor([pages[t // 16] * 16 + t % 16 for t in range(n)])
    kc, vc = (torch.full((nb + 9, 16, G, d), float("nan"), dtype=torch.bfloat16) for d in (dkp, dvp))
    pad = torch.nn.functional.pad
    kc.view(-1, G, dkp)[idx], vc.view(-1, G, dvp)[idx] = pad(k, (0, dkp - dk)), pad(v, (0, dvp - dv))
    kc, vc, qd, gd = kc.cuda(), vc.cuda(), pad(q, (0, dkp - dk)).cuda(), gate.reshape(n, -1).cuda()
    cuts = [(t, t + 1) for t in range(1195, 1250, 3)] + [(0, 256), (512, 513), (256, 257), (0, 1190), (1000, 1007), (630, 800), (1210, 1211), (1249, 1250)]
    for lo, hi in cuts:
        b = pc.batch([hi - lo], [hi], pages=[pages[:(hi + 15) // 16]], device="cuda")
        out = torch.empty(hi - lo, H * dv, dtype=torch.bfloat16, device="cuda")
        mx.attention_dims(qd[lo:hi].contiguous(), kc, vc, b, dk=dk, dv=dv, scale=scale, sink=sink.cuda(), fmt="bf16", out=out, window=window, keep=keep,
                          gate=mx.OutputGate(gd[lo:hi], False), kernel=kernel if kernel != "mma" or dkp < 256 or hi - lo == 1 else "auto")
        close(out.view(-1, H, dv), want[lo:hi], 1e-2)
    ops.check_status("cuda")


# ------------------------------------------------------------------ feed-forwards
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("E,k,groups,keep", [(6, 2, 3, 2), (40, 8, 4, 2), (1, 1, 1, 1), (64, 6, 8, 4), (30, 3, 30, 5), (12, 5, 1, 1)])
def test_router(device, E, k, groups, keep):
    """Softmax over all experts, chosen inside the best groups: strong experts in groups that lose, ties, far-apart logits."""
    z = gen(30, E, seed=1, std=2.0)
    z[3] *= 40
    z[4] = 0.5                                                                           # all equal: the lowest ids
    if groups > 1:                                                                       # a group whose sum is largest but whose best is not
        z[5] = -9.0
        z[5, E - E // groups:] = 2.0
        z[5, :E - E // groups:E // groups] = 2.5
    wide = torch.cat([torch.full((30, 3), 99.0), z, torch.full((30, 2), 99.0)], 1).to(device)[:, 3:3 + E]
    spec = moe_ops.RouterSpec(E, k, router="softmax_grouped", router_n_group=groups, router_topk_group=keep, router_renormalize=False, router_scaling=1.7)
    w, idx = moe_ops.route(wide, spec)
    for t in range(30):
        ids, want = po.route(z[t].double(), {"experts": E, "top": k, "scale": 1.7, "groups": {"count": groups, "keep": keep}})
        got = dict(zip(idx[t].tolist(), w[t].tolist()))
        assert sorted(got) == sorted(ids), t
        assert max(abs(got[e] - float(x)) for e, x in zip(ids, want)) < 2e-6


def test_router_groups_go_by_their_best_expert():
    """Two good experts do not outweigh one better one."""
    z = torch.tensor([2.0, 2.0, 2.1, -5.0])
    r = {"experts": 4, "top": 1, "groups": {"count": 2, "keep": 1}}
    assert po.route(z, r)[0] == [2]
    w, idx = moe_ops.route(z[None], moe_ops.RouterSpec(4, 1, router="softmax_grouped", router_n_group=2, router_topk_group=1, router_renormalize=False))
    assert idx.tolist() == [[2]] and abs(float(w) - float(torch.softmax(z, 0)[2])) < 1e-6


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", DTYPES)
@pytest.mark.parametrize("T,W,E,top,ff,groups,shared", [(1, 64, 6, 2, 64, (3, 2), 40), (50, 100, 5, 2, 18, (1, 1), 26), (50, 96, 9, 4, 40, (3, 2), None),
                                                        (300, 128, 4, 1, 96, (2, 1), 64), (150, 44, 3, 3, 10, (1, 1), 12)])
def test_mixture_of_experts(device, fmt, T, W, E, top, ff, groups, shared):
    """Stacked, padded experts with their own limit, beside a gated shared one with another, through the streams' sum."""
    from metrale_inference_alpha_b200.models.decoder import Decoder
    from metrale_inference_alpha_b200.models.hyper import gated_moe
    from metrale_inference_alpha_b200.weights.loader import Loader
    mlp = pc.moe(E, top, ff, groups, shared, 1.6, 0.9, 0.3)
    cfg = pc.config([pc.normed(1, 1, 8, 8, 4, 1, mlp)], W, streams=1)
    t = pc.weights(cfg, seed=4, calm=True)
    m = {k[len("l0.mlp."):]: v.double() for k, v in t.items() if k.startswith("l0.mlp.")}

    class Source:
        has, get, names = (lambda s, n: n in t), (lambda s, n: t[n]), (lambda s: list(t))

    mc = pc.model_config(cfg, fmt)
    mw = Loader(mc, Source(), torch.device(device), 0, 1, 0, 1).load()
    h = gen(T, W, seed=5).to(dt(fmt))
    out = gated_moe(Decoder(mc, mw, device=device), mx.act_of(h.to(device), fmt), mw.layers[0].ffn)
    one = torch.ones(1, device=device)
    got = mx.stream_hyper(torch.zeros(T, W, device=device), 1, fmt, pending=out, hc=mx.HyperW(one, one, one.view(1, 1)), w_in=one, out_f32=True)[1]
    close(got, po.mixture(h.double(), m, mlp), 2e-5 if fmt == "fp32" else 2e-2)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", DTYPES)
@pytest.mark.parametrize("M,ff,W", [(1, 15, 20), (19, 128, 64), (70, 17, 33), (300, 320, 128)])
def test_clamped_glu(device, fmt, M, ff, W):
    from metrale_inference_alpha_b200.ops import QuantWeight
    h = gen(M, W, seed=1).to(dt(fmt))
    t = {n: (gen(*s, seed=i) * 2 * s[1] ** -0.5).to(dt(fmt)) for i, (n, s) in enumerate({"gate": (ff, W), "up": (ff, W)}.items(), 2)}
    gu = ops.interleave_gate_up(t["gate"], t["up"]).to(device)
    for limit in (0.4, 7.0):
        got = ops.linear(mx.act_of(h.to(device), fmt), QuantWeight(fmt, 2 * ff, W, gu), clamp_glu=(1.702, limit))
        eye = {**{k: v.double() for k, v in t.items()}, "down": torch.eye(ff, dtype=torch.float64)}
        close(got, po.feed_forward(h.double(), eye, limit), 1e-5 if fmt == "fp32" else 1e-2)


# ------------------------------------------------------------------ whole models
_ORACLE = {}


def oracle(name, n, seed=0, calm=False):
    """(tokens, logits [n, vocab]) of one sequence of a configuration, computed once."""
    key = name, n, seed, calm
    if key not in _ORACLE:
        cfg = pc.CONFIGS[name]
        toks = pc.tokens(cfg, n, seed)
        _ORACLE[key] = toks, po.forward(cfg, pc.weights(cfg, calm=calm), toks)
    return _ORACLE[key]


def replay(tmp_path, name, dtype, device, max_tokens=192, **kw):
    """A bf16 model has routers without close calls (rounding would decide those)."""
    d = tmp_path / name
    path = str(d) if d.exists() else pc.checkpoint(pc.CONFIGS[name], pc.weights(pc.CONFIGS[name], calm=dtype == "bf16"), d)
    return TraceReplay(path, dtype, max_tokens, device, **kw)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(pc.CONFIGS))
def test_model_whole_portions_and_decoding(tmp_path, device, dtype, name):
    """A prompt at once, in portions down to two tokens, and token by token, all through one engine (so pages are used
    again): each against the plain model."""
    toks, want = oracle(name, 75, calm=dtype == "bf16")
    r = replay(tmp_path, name, dtype, device)
    for cuts in ([75], [2], [1], [33, 2, 17, 3, 1], [16, 15, 17, 1]):
        assert near(pc.feed(r, "a", toks, cuts), want, dtype), cuts
    for rid, n in (("one", 1), ("two", 2)):                             # the first tokens of a sequence
        assert near(pc.feed(r, rid, toks[:n], [n]), want[:n], dtype)
    assert r.engine.scheduler.num_active == 0 and r.engine.runner.kv.allocator.num_used == 0


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["ragged", "tiles"])
def test_model_mixed_batches(tmp_path, device, dtype, name):
    """Portions beside single tokens, requests that pause, end and make room: against each alone."""
    seqs = {rid: oracle(name, n, seed, dtype == "bf16") for rid, n, seed in (("a", 75, 0), ("b", 40, 1), ("c", 3, 2), ("d", 58, 3), ("e", 21, 4))}
    r = replay(tmp_path, name, dtype, device, max_tokens=208)
    at, got = {k: 0 for k in seqs}, {k: [] for k in seqs}
    plan = [{"a": 20, "b": 2}, {"b": 17, "c": 1}, {"a": 1, "b": 1, "c": 2, "d": 30}, {"a": 2, "d": 2}, {"d": 1, "a": 1, "b": 1},
            {"a": 9, "b": 19, "d": 1}, {"a": 1, "d": 1, "e": 16}, {"a": 31, "e": 1}, {"d": 23, "e": 4, "a": 1}, {"a": 9}]
    for step in plan:
        entries = [{"id": k, "tokens": seqs[k][0][at[k]:at[k] + n], "want": list(range(n))} for k, n in step.items()]
        for k, n in step.items():
            at[k] += n
        out = r.step(entries, [k for k in step if at[k] == len(seqs[k][0])])
        i = 0
        for k, n in step.items():
            got[k].append(out[i:i + n])
            i += n
    for k, (toks, want) in seqs.items():
        assert at[k] == len(toks) and near(torch.cat(got[k]), want, dtype), k


@pytest.mark.parametrize("device", DEVICES)
def test_shared_tensors_have_caches_of_their_own(device):
    cfg = pc.model_config(pc.CONFIGS["ragged"])
    assert [cfg.layer_owner(i) for i in range(6)] == [0, 1, 2, 0, 5, 5]
    eng = LLMEngine(EngineArgs(model=cfg, device=device, max_num_seqs=2, max_model_len=64, num_kv_blocks=16))
    kv, L = eng.runner.kv, eng.weights.layers
    assert L[3] is L[0] and L[4] is L[5] and len({id(x) for x in L}) == 4
    assert len(kv.k) == 6 and len({t.data_ptr() for t in kv.k + kv.v}) == 12 and eng.runner.pool is None
    assert cfg.scaled(weight_format="fp32").kv_layer_dims() == [(1, 22, 30), (2, 36, 26), (2, 18, 14), (1, 22, 30), (1, 10, 50), (1, 10, 50)]


@pytest.mark.parametrize("device", DEVICES)
def test_long_decoding(tmp_path, device):
    """Windows that pass over many decoded tokens (32-bit)."""
    toks, want = oracle("ragged", 180, 9)
    r = replay(tmp_path, "ragged", "fp32", device)
    assert pc.error(pc.feed(r, "x", toks, [5, 1]), want) < TOL


@pytest.mark.gpu
@pytest.mark.parametrize("name", ["wide", "tiles"])
def test_long_prompts(tmp_path, name):
    """Prompts over many tiles and windows, then single tokens."""
    toks, want = oracle(name, 330, 5, True)
    r = replay(tmp_path, name, "bf16", "cuda", max_tokens=352)
    for cuts in ([330], [150, 129, 50, 1], [300, 1]):
        assert near(pc.feed(r, "a", toks, cuts), want, "bf16"), cuts
    ops.check_status("cuda")


@pytest.mark.parametrize("device", DEVICES)
def test_wanted_rows_and_steps_without(tmp_path, device):
    toks, want = oracle("ones", 30)
    r = replay(tmp_path, "ones", "fp32", device)
    assert r.step([{"id": "q", "tokens": toks[:7], "want": []}], []) is None
    got = r.step([{"id": "q", "tokens": toks[7:20], "want": [0, 5, 12]}], [])
    assert pc.error(got, want[[7, 12, 19]]) < TOL
    assert r.step([{"id": "q", "tokens": toks[20:21], "want": []}], []) is None
    assert pc.error(r.step([{"id": "q", "tokens": toks[21:22], "want": [0]}], ["q"]), want[21:22]) < TOL


def greedy_reference(name, prompt, n):
    cfg, t = pc.CONFIGS[name], pc.weights(pc.CONFIGS[name])
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(po.forward(cfg, t, toks)[-1].argmax()))
    return toks[len(prompt):]


@pytest.mark.parametrize("device", DEVICES)
def test_greedy_generation_scheduler_and_speculation(tmp_path, device):
    """generate() on a queue longer than the batch, with chunked prompts; with n-gram speculation, swapping and predicted
    outputs: the same tokens."""
    path = pc.checkpoint(pc.CONFIGS["ragged"], pc.weights(pc.CONFIGS["ragged"]), tmp_path / "m")
    prompts = [pc.tokens(pc.CONFIGS["ragged"], n, 50 + n) for n in (19, 1, 33)]
    want = [greedy_reference("ragged", p, 10) for p in prompts]
    kw = dict(model=path, device=device, dtype="fp32", max_num_seqs=2, max_model_len=96, max_prefill_tokens=13, num_kv_blocks=24)
    for extra in ({}, {"speculative": "ngram", "mtp_gate": False}, {"preempt_mode": "swap", "num_kv_blocks": 5}):
        eng = LLMEngine(EngineArgs(**{**kw, **extra}))
        outs = eng.generate(prompts, SamplingParams(max_tokens=10, temperature=0.0))
        assert [o.output_ids for o in outs] == want, extra
    guess = [w[:5] + [(w[5] + 1) % 150] + w[6:] for w in want]          # right, then wrong once, then right again
    eng = LLMEngine(EngineArgs(**kw))
    outs = eng.generate(prompts, [SamplingParams(max_tokens=10, temperature=0.0, prediction_ids=g) for g in guess])
    assert [o.output_ids for o in outs] == want
    assert any(o.accepted_draft_tokens for o in outs)


@pytest.mark.parametrize("device", DEVICES)
def test_prefix_cache(tmp_path, device):
    path = pc.checkpoint(pc.CONFIGS["ragged"], pc.weights(pc.CONFIGS["ragged"]), tmp_path / "m")
    eng = LLMEngine(EngineArgs(model=path, device=device, dtype="fp32", max_num_seqs=2, max_model_len=400, num_kv_blocks=80))
    p = pc.tokens(pc.CONFIGS["ragged"], 300, 5)
    sp = SamplingParams(max_tokens=5, temperature=0.0)
    a, b = (eng.generate([p], sp)[0] for _ in range(2))
    assert a.output_ids == b.output_ids and b.cached_tokens >= 256


def test_sampled_rows_take_the_models_distribution(tmp_path):
    path = pc.checkpoint(pc.CONFIGS["ones"], pc.weights(pc.CONFIGS["ones"]), tmp_path / "m")
    toks, want = oracle("ones", 30)
    eng = LLMEngine(EngineArgs(model=path, device="cpu", dtype="fp32", max_num_seqs=8, max_model_len=64, num_kv_blocks=64))
    top = set(want[-1].topk(3).indices.tolist())
    outs = eng.generate([toks] * 8, [SamplingParams(max_tokens=1, temperature=1.0, top_k=3, seed=s) for s in range(8)])
    assert {o.output_ids[0] for o in outs} <= top


def test_positions_end_with_the_table(tmp_path):
    """A sequence never grows past the learned positions."""
    cfg = pc.config([pc.normed(1, 1, 8, 8, 4, 1)], 32, positions=24)
    eng = LLMEngine(EngineArgs(model=pc.checkpoint(cfg, pc.weights(cfg), tmp_path / "m"), dtype="fp32", max_num_seqs=2, max_model_len=64, num_kv_blocks=16))
    out = eng.generate([pc.tokens(cfg, 20, 1)], SamplingParams(max_tokens=40, temperature=0.0))[0]
    assert eng.sched_cfg.max_model_len == 24 and 0 < len(out.output_ids) <= 5


# ------------------------------------------------------------------ configuration, weights, command line
def test_configuration_and_checkpoint(tmp_path):
    cfg = pc.CONFIGS["ragged"]
    c = from_hf_config(json.loads(json.dumps(cfg)))
    assert c.arch == "pivipel" and c.layer_types == ["gated"] * 6 and c.attention_layers() == list(range(6)) and c.streams == 3
    assert c.ffn_types == ["moe", "dense", "none", "moe", "moe", "moe"] and c.max_position == 400
    assert type(c).from_json(c.to_json()).to_json() == c.to_json()
    assert c.kv_bytes_per_token() == 2 * 128 * (1 + 2 + 2 + 1 + 1 + 1)
    from metrale_inference_alpha_b200.weights.checkpoint import open_checkpoint
    from metrale_inference_alpha_b200.weights.preflight import preflight
    t = pc.weights(cfg)
    assert not any(n.startswith(("l3.", "l4.")) for n in t)
    c2, src = open_checkpoint(pc.checkpoint(cfg, t, tmp_path / "ok"))
    assert preflight(c2, src).ok
    del t["l1.hc2.mix"]
    c3, src = open_checkpoint(pc.checkpoint(cfg, t, tmp_path / "bad"))
    assert preflight(c3, src, check_shapes=False).missing == ["l1.hc2.mix"]

    def broken(change, match):
        bad = json.loads(json.dumps(cfg))
        change(bad)
        with pytest.raises(ValueError, match=match):
            from_pivipel_config(bad)

    broken(lambda b: b["layers"][0].update(type="other"), "unknown mixer")
    broken(lambda b: b["layers"][0]["mlp"].update(kind="other"), "unknown feed-forward")
    broken(lambda b: b["layers"][0]["mixer"]["rot"].update(dims=24), "do not fit")
    broken(lambda b: b["layers"][1]["mixer"]["mask"].update(size=0), "window")
    broken(lambda b: b["layers"][0]["mlp"]["router"].update(top=5), "experts per token")
    broken(lambda b: b["layers"][0]["mlp"]["router"]["groups"].update(count=4), "groups")
    broken(lambda b: b["layers"][3].update(weights_of=6), "no tensors")
    broken(lambda b: b["layers"][3].update(weights_of=1), "not like layer")
    broken(lambda b: b["layers"][0].update(weights_of=3), "by way of others")
    broken(lambda b: b.update(streams=0), "streams")


def test_unserved_combinations_are_refused():
    with pytest.raises(ValueError):
        LLMEngine(EngineArgs(model="tiny-pivipel", dtype="int8", max_model_len=64, num_kv_blocks=16))
    for kw in (dict(kv_cache_dtype="fp8"), dict(speculative="dflash"), dict(speculative="mtp"), dict(expert_arena_slots=4)):
        with pytest.raises(NotImplementedError):
            LLMEngine(EngineArgs(model="tiny-pivipel", max_model_len=64, num_kv_blocks=16, **kw))


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
def test_preset_runs_from_synthetic_weights(device, dtype):
    eng = LLMEngine(EngineArgs(model=preset("tiny-pivipel"), device=device, dtype=dtype, max_num_seqs=2, max_model_len=64, num_kv_blocks=16))
    outs = eng.generate([[1, 2, 3], [9, 8, 7, 6]], SamplingParams(max_tokens=4))
    assert all(len(o.output_ids) == 4 for o in outs)
    if device != "cpu":
        ops.check_status(device)


def test_replay_command(tmp_path, capsys):
    import numpy as np
    from metrale_inference_alpha_b200.server import cli
    cfg = pc.CONFIGS["ones"]
    path = pc.checkpoint(cfg, pc.weights(cfg), tmp_path / "m")
    toks, want = oracle("ones", 30)
    ns = cli.build_parser().parse_args(["replay", "--model", path, "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "64",
                                        "--device", "cpu"])
    from metrale_inference_alpha_b200.engine.replay import run
    lines = [json.dumps({"step": 0, "entries": [{"id": "a", "tokens": toks[:9], "want": []}], "end": []}),
             json.dumps({"step": 1, "entries": [{"id": "a", "tokens": toks[9:30], "want": [20]}], "end": ["a"]})]
    assert run(ns, lines) == 0
    assert [x for x in capsys.readouterr().out.splitlines() if x.startswith("done")] == ["done 0", "done 1"]
    got = torch.from_numpy(np.fromfile(tmp_path / "1.f32", dtype="<f4")).view(1, -1)
    assert pc.error(got, want[29:30]) < 1e-5 and not (tmp_path / "0.f32").exists()
