"""The Fabulix decoder against a plain restatement (fabulix_oracle.py): every mechanism alone, then whole
models through the engine's own entry points. The CPU runs cover the engine's host logic and its op
restatements, the GPU runs the kernels."""
import json

import pytest
import torch

import fabulix_cases as fc
import fabulix_oracle as fo
from metrale_inference_alpha_b200 import ops
from metrale_inference_alpha_b200.config.model_config import from_fabulix_config, from_hf_config, preset
from metrale_inference_alpha_b200.engine.llm_engine import EngineArgs, LLMEngine
from metrale_inference_alpha_b200.engine.replay import TraceReplay
from metrale_inference_alpha_b200.ops import QuantWeight, mixers as mx
from metrale_inference_alpha_b200.sampling.params import SamplingParams

DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]
DTYPES = ["fp32", "bf16"]
TOL = {"fp32": 2e-5, "bf16": 0.04}          # of the logits' rms
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


# ------------------------------------------------------------------ mechanisms
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", DTYPES)
@pytest.mark.parametrize("W", [37, 96])
def test_stream_norm(device, fmt, W):
    T = 21
    x, y = gen(T, W, seed=1), gen(T, W, seed=2).to(dt(fmt))
    post = mx.DytNorm(0.7, b16(gen(W, seed=3)), b16(gen(W, seed=4)))
    pre = mx.DytNorm(0.4, b16(gen(W, seed=5)), b16(gen(W, seed=6)))
    rmsw = mx.RmsNorm(b16(gen(W, seed=7)), 1e-3)
    to = lambda n: mx.DytNorm(n.alpha, n.w.to(device), n.b.to(device)) if isinstance(n, mx.DytNorm) else mx.RmsNorm(n.w.to(device), n.eps)
    f = lambda t: t.double()
    tol = 1e-5 if fmt == "fp32" else 6e-3
    for p in (post, rmsw):
        add = fo.dyt(f(y), p.alpha, f(p.w), f(p.b)) if isinstance(p, mx.DytNorm) else fo.rms(f(y), 1e-3) * f(p.w)
        want = f(x) + add
        x1, h, _, _ = mx.stream_norm(x.to(device), fmt, y=y.to(device), post=to(p), pre=to(pre))
        close(x1, want, 1e-5)                                        # the stream itself is 32-bit in both formats
        close(h, fo.dyt(want, 0.4, f(pre.w), f(pre.b)), tol)
        close(mx.stream_norm(x.to(device), fmt, y=y.to(device), post=to(p), raw=True)[1], want, tol)
    close(mx.stream_norm(x.to(device), fmt, pre=to(pre))[1], fo.dyt(f(x), 0.4, f(pre.w), f(pre.b)), tol)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", DTYPES)
def test_token_shift_over_portions(device, fmt):
    """Mixes of a sequence do not depend on where its portions are cut; the state ends at the last row; the
    first token's neighbour is zero; sequences of one batch do not see each other."""
    W, mu = 44, b16(torch.rand(5, 44, generator=torch.Generator().manual_seed(3)))
    pre = mx.DytNorm(0.5, b16(gen(W, seed=5)).to(device), b16(gen(W, seed=6)).to(device))
    post = mx.RmsNorm(b16(gen(W, seed=7)).to(device), 1e-5)
    xs, ys = [gen(n, W, seed=20 + n) for n in (9, 14)], [gen(n, W, seed=40 + n).to(dt(fmt)) for n in (9, 14)]
    state = torch.full((4, W), 7.0, device=device)                    # stale content of reused slots
    got = [[], []]
    for cuts in ((1, 2), (2, 1), (3, 10), (3, 1)):
        at = [sum(g.shape[1] for g in got[s]) for s in (0, 1)]
        b = fc.batch(list(cuts), [at[0] + cuts[0], at[1] + cuts[1]], [2, 3], device=device)
        x = torch.cat([xs[s][at[s]:at[s] + cuts[s]] for s in (0, 1)]).to(device)
        y = torch.cat([ys[s][at[s]:at[s] + cuts[s]] for s in (0, 1)]).to(device)
        keep = state.clone()
        mx.stream_norm(x, fmt, y=y, post=post, pre=pre, mu=mu.to(device), state=state, batch=b, write_state=False)
        assert torch.equal(state, keep)                               # verify steps leave it alone
        m = mx.stream_norm(x, fmt, y=y, post=post, pre=pre, mu=mu.to(device), state=state, batch=b)[2]
        got[0].append(m[:, :cuts[0]])
        got[1].append(m[:, cuts[0]:])
    for s in (0, 1):
        xx = xs[s].double() + fo.rms(ys[s].double(), 1e-5) * post.w.cpu().double()
        h = fo.dyt(xx, 0.5, pre.w.cpu().double(), pre.b.cpu().double())
        prev = torch.cat([torch.zeros(1, W, dtype=h.dtype), h[:-1]])
        want = h + (prev - h) * mu.double()[:, None, :]
        close(torch.cat(got[s], 1), want, 1e-5 if fmt == "fp32" else 6e-3)
        close(state[2 + s], h[-1], 1e-5)


def run_attention(device, fmt, q, k, v, scale, sink, cuts, dims, pages=None, kernel="auto", out_scale=1.0, rot=0, base=100.0, block=16):
    """q [n, H, dk], k [n, G, dk], v [n, G, dv] of one sequence, fed in portions through the paged cache, beside
    a short second sequence that shares every batch. Returns [n, H, dv]."""
    H, G, dk, dv = dims
    n = q.shape[0]
    dkp, dvp = mx.padded_head_dims(dk, dv, fmt)
    nb = (n + block - 1) // block
    kc = torch.full((2 * nb + 8, block, G, dkp), float("nan"), dtype=dt(fmt), device=device)      # unwritten slots must not matter
    vc = torch.full((2 * nb + 8, block, G, dvp), float("nan"), dtype=dt(fmt), device=device)
    pages = pages or list(range(nb + 4, 4, -1))                       # descending: pages are not in order
    cos = sin = None
    if rot:
        from metrale_inference_alpha_b200.ops import reference as ref
        cos, sin = ref.rope_tables(4096, rot, base, device=device)
    outs, at, i = [], 0, 0
    other = torch.cat([q[:, :H].reshape(n, -1), k.reshape(n, -1), v.reshape(n, -1)], 1)
    while at < n:
        m = min(cuts[min(i, len(cuts) - 1)], n - at)
        o1 = min(at, 15)                                              # the neighbour's position this step
        b = fc.batch([m, 1], [at + m, o1 + 1], device=device, block=block, pages=[pages[:(at + m + block - 1) // block], [1]])
        qkv = torch.cat([other[at:at + m], other[o1:o1 + 1]]).to(dt(fmt)).to(device)
        qq = mx.rope_dims(qkv, Hq=H, Hkv=G, dk=dk, dv=dv, positions=b.positions, slots=b.slot_mapping, k_cache=kc, v_cache=vc, cos=cos,
                          sin=sin, fmt=fmt)
        wide = torch.full((m + 1, H * dv + 8), 5.0, dtype=dt(fmt), device=device)
        mx.attention_dims(qq, kc, vc, b, dk=dk, dv=dv, scale=scale, sink=sink, fmt=fmt, out=wide[:, 8:], out_scale=out_scale, kernel=kernel)
        assert bool((wide[:, :8] == 5.0).all())
        outs.append(wide[:m, 8:])
        at, i = at + m, i + 1
    return torch.cat(outs).view(n, H, dv).float().cpu()


def plain_attention(q, k, v, scale, sink, rot=0, base=100.0):
    q, k, v = q.double(), k.double(), v.double()
    n, H, G = q.shape[0], q.shape[1], k.shape[1]
    if rot:
        q = torch.stack([fo.rotate(q[p], p, base, rot) for p in range(n)])
        k = torch.stack([fo.rotate(k[p], p, base, rot) for p in range(n)])
    out = torch.zeros(n, H, v.shape[2], dtype=torch.float64)
    for h in range(H):
        for i in range(n):
            s = (k[:i + 1, h // (H // G)] @ q[i, h]) * scale
            w = fo.sink_softmax(s) if sink else torch.softmax(s, 0)
            out[i, h] = w @ v[:i + 1, h // (H // G)]
    return out


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", DTYPES)
@pytest.mark.parametrize("dims", [(4, 2, 30, 44), (2, 2, 64, 90), (3, 1, 72, 40), (4, 4, 16, 16)])
@pytest.mark.parametrize("cuts", [[70], [33, 1], [2], [31, 17, 2, 1]])
def test_attention_with_sink(device, fmt, dims, cuts):
    H, G, dk, dv = dims
    n = 70
    q, k, v = (gen(n, h, d, seed=s).to(dt(fmt)) for h, d, s in ((H, dk, 1), (G, dk, 2), (G, dv, 3)))
    # single keys that stand out: for the first tokens, at page borders and far away
    for i, j in ((0, 0), (15, 0), (16, 15), (17, 16), (32, 31), (33, 32), (47, 1), (48, 0), (63, 48), (69, 0), (69, 16)):
        q[i] = 0
        q[i, :, :8] = 2.0
        k[j, :, :8] += 3.0
    rot = dk // 2 // 2 * 2
    want = plain_attention(q, k, v, 0.3, True)
    close(run_attention(device, fmt, q, k, v, 0.3, True, cuts, dims), want, 1e-5 if fmt == "fp32" else 8e-3)
    close(run_attention(device, fmt, q, k, v, 0.3, True, cuts, dims, rot=rot, out_scale=0.5),
          0.5 * plain_attention(q, k, v, 0.3, True, rot=rot), 1e-5 if fmt == "fp32" else 2e-2)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", DTYPES)
def test_sink_takes_its_share(device, fmt):
    """Scores far below zero: nearly all weight is the sink's. Far above: it vanishes. One key of score 0: half."""
    n, dims = 40, (2, 1, 16, 16)
    v = gen(n, 1, 16, seed=3).to(dt(fmt))
    for level in (-60.0, -4.0, 0.0, 60.0):
        q = torch.zeros(n, 2, 16)
        q[..., 0] = 1.0
        k = torch.zeros(n, 1, 16)
        k[..., 0] = level
        got = run_attention(device, fmt, q, k, v, 1.0, True, [17, 1], dims)
        want = plain_attention(q, k, v, 1.0, True)
        assert float((got.double() - want).abs().max()) < (1e-5 if fmt == "fp32" else 2e-2) * max(1e-3, float(want.abs().max()))
        if level == 0.0:
            close(got[0], 0.5 * v[0].expand(2, 16).double(), 1e-2)
        if level == -60.0:
            assert float(got.abs().max()) < 1e-20


@pytest.mark.gpu
@pytest.mark.parametrize("kernel,dims", [("tc", (4, 2, 128, 128)), ("mma", (4, 2, 128, 128)), ("mma", (4, 2, 128, 64)), ("mma", (2, 2, 50, 100)),
                                         ("tc", (2, 1, 256, 256)), ("auto", (2, 1, 200, 130)), ("simt", (2, 2, 50, 100)), ("mma", (8, 1, 64, 64))])
def test_attention_kernels_long(kernel, dims):
    """Long contexts: tiles of every kernel, several split-KV partitions (decode past 512 and 1024 keys), far keys."""
    H, G, dk, dv = dims
    n = 1250
    q, k, v = (b16(gen(n, h, d, seed=s)) for h, d, s in ((H, dk, 1), (G, dk, 2), (G, dv, 3)))
    for i, j in ((700, 0), (1199, 511), (1210, 512), (1211, 1023), (1212, 1024), (1240, 3), (1249, 1248)):
        q[i] = 0
        q[i, :, :8] = 3.0
        k[j, :, :8] += 2.0
    f = torch.float64
    s = torch.einsum("ihd,jhd->hij", q.to(f), k.to(f).repeat_interleave(H // G, 1)) * 0.2
    s.masked_fill_(torch.ones(n, n, dtype=torch.bool).triu(1), float("-inf"))
    m = s.amax(-1, keepdim=True).clamp(min=0)
    e = torch.exp(s - m)
    want = torch.einsum("hij,jhd->ihd", e / (e.sum(-1, keepdim=True) + torch.exp(-m)), v.to(f).repeat_interleave(H // G, 1))
    got = run_attention("cuda", "bf16", q, k, v, 0.2, True, [n] if kernel == "tc" else [n - 60, 1], dims, kernel=kernel)
    close(got, want, 5e-3)
    if kernel != "tc":
        close(run_attention("cuda", "bf16", q[:40], k[:40], v[:40], 0.2, True, [7, 3], dims, kernel=kernel), want[:40], 5e-3)
    ops.check_status("cuda")


# ------------------------------------------------------------------ recurrences
def plain_linear(q, k, v, w, u):
    """q, k [n, H, dk], v [n, H, dv], w [n, H, dk] decays; u [H, dk] or None. Outputs [n, H, dv] and the final state."""
    q, k, v, w = (t.double() for t in (q, k, v, w))
    n, H, dk = q.shape
    out, S = torch.zeros(n, H, v.shape[2], dtype=torch.float64), torch.zeros(H, dk, v.shape[2], dtype=torch.float64)
    for t in range(n):
        kv = k[t][:, :, None] * v[t][:, None, :]
        read = S + u.double()[:, :, None] * kv if u is not None else None
        S = w[t][:, :, None] * S + kv
        out[t] = ((read if u is not None else S) * q[t][:, :, None]).sum(1)
    return out, S


def run_linear(device, fmt, qkv, log_w, decay, u, dims, cuts, slots, kernel="auto"):
    """Several sequences fed in portions (cuts[i][s] rows of sequence s in step i; 0 = left out), interleaved
    rows as the engine lays them out; returns per-sequence outputs and the state pool."""
    H, dk, dv = dims
    state = torch.full((max(slots) + 2, H, dk, dv), 9.0, device=device)       # stale content of reused slots
    S, at, outs = len(qkv), [0] * len(qkv), [[] for _ in qkv]
    for step in cuts:
        live = [s for s in range(S) if step[s]]
        b = fc.batch([step[s] for s in live], [at[s] + step[s] for s in live], [slots[s] for s in live], device=device)
        cat = lambda f: torch.cat([f(s)[at[s]:at[s] + step[s]] for s in live]).to(device)
        rows = torch.cat([cat(lambda s, i=i: qkv[s][i].reshape(qkv[s][i].shape[0], -1)) for i in range(3)], 1).to(dt(fmt))
        lw = cat(lambda s: log_w[s].reshape(log_w[s].shape[0], -1)).float() if log_w is not None else None
        kw = dict(heads=H, dk=dk, dv=dv, fmt=fmt, log_w=lw, decay=None if decay is None else decay.to(device),
                  u=None if u is None else u.to(device), kernel=kernel)
        q, k, v = rows[:, :H * dk], rows[:, H * dk:2 * H * dk], rows[:, 2 * H * dk:]
        keep = state.clone()
        mx.linear_attention(q, k, v, state, b, write_state=False, **kw)
        assert torch.equal(keep, state)
        y = mx.linear_attention(q, k, v, state, b, **kw)
        # a commit pass over the same rows leaves the same state, and writes nothing else
        again = keep.clone()
        mx.linear_attention(q, k, v, again, b, write_out=False, **kw)
        assert float((again - state).abs().max()) <= 1e-4 * float(state.abs().max())
        r = 0
        for s in live:
            outs[s].append(y[r:r + step[s]].view(step[s], H, dv).cpu())
            r += step[s]
            at[s] += step[s]
    return [torch.cat(o) for o in outs], state.cpu()


LIN_DIMS = [(3, 20, 28), (2, 64, 64), (1, 16, 7), (2, 40, 96), (1, 128, 128), (2, 32, 32)]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", DTYPES)
@pytest.mark.parametrize("dims", LIN_DIMS)
@pytest.mark.parametrize("mode", ["head", "channel+bonus"])
def test_linear_attention(device, fmt, dims, mode):
    """Ragged batches in portions; the first token of every sequence; decays from almost 1 (a far key that
    stands out must still be read at the end) down to exp(-30) (underflow inside a chunk must not matter)."""
    H, dk, dv = dims
    lens = (150, 83, 1)
    qkv = [[gen(n, H, d, seed=10 * i + n).to(dt(fmt)) for i, d in enumerate((dk, dk, dv))] for n in lens]
    for q, k, v in qkv[:2]:
        k[3] *= 20                                                     # one key among many
        q[-1] = k[3]
    log_w = decay = u = None
    if mode == "head":
        decay = torch.tensor([0.999, 0.6, 0.93][:H])
        ws = [decay.view(1, H, 1).expand(n, H, dk) for n in lens]
    else:
        log_w = [-torch.exp(gen(n, H, dk, seed=77 + n, std=2.0, mean=-3.0)).clamp(max=30.0) for n in lens]
        for lw in log_w:
            lw[..., 0] = -1e-4
            lw[5:9, :, 1] = -30.0
        u = gen(H, dk, seed=5)
        ws = [torch.exp(lw.double()) for lw in log_w]
    cuts = [(64, 2, 1), (1, 0, 0), (2, 64, 0), (70, 1, 0), (13, 16, 0)]
    outs, state = run_linear(device, fmt, qkv, log_w, decay, u, dims, cuts, [3, 1, 2])
    whole, state2 = run_linear(device, fmt, qkv, log_w, decay, u, dims, [lens], [1, 2, 3])
    for s, n in enumerate(lens):
        want, S = plain_linear(*qkv[s], ws[s], u)
        for got in (outs[s], whole[s]):
            assert float((got.double() - want).abs().amax((1, 2)).div(want.abs().amax((1, 2)).clamp(min=0.05 * float(want.abs().max()))).max()) < 2e-4
        close(state[[3, 1, 2][s]], S, 2e-4)
        close(state2[[1, 2, 3][s]], S, 2e-4)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", DTYPES)
@pytest.mark.parametrize("dims", [(3, 20, 28), (2, 64, 64), (2, 40, 96), (1, 128, 128), (2, 200, 160), (2, 16, 7)])
@pytest.mark.parametrize("n", [1, 3])
def test_linear_attention_with_its_norm(device, fmt, dims, n):
    """The head norm, gate and scale behind the recurrence (inside the decode kernel for single rows): as separate steps."""
    H, dk, dv = dims
    T = 3 * n
    q, k, v = (gen(T, H * d, seed=s).to(dt(fmt)).to(device) for d, s in ((dk, 1), (dk, 2), (dv, 3)))
    lw, u = -torch.exp(gen(T, H * dk, seed=4)).to(device), gen(H, dk, seed=5).to(device)
    gate, w = gen(T, H * dv, seed=6).to(dt(fmt)).to(device), b16(gen(H * dv, seed=7)).to(device)
    b = fc.batch([n] * 3, [n, n + 4, n + 20], [2, 1, 3], device=device)
    init = gen(4, H, dk, dv, seed=8).to(device)
    init[2] = float("nan")                                             # a fresh sequence reads nothing from its slot
    kw = dict(heads=H, dk=dk, dv=dv, fmt=fmt, log_w=lw, u=u)
    s1, s2 = init.clone(), init.clone()
    core = mx.linear_attention(q, k, v, s1, b, kernel="seq", **kw)
    want = mx.gated_norm(core, w, gate, fmt, group=dv, gate_act="silu", eps=1e-5, scale=0.65)
    out = torch.full((T, H * dv + 8), 3.0, dtype=dt(fmt), device=device)
    mx.linear_attention(q, k, v, s2, b, norm=dict(w=w, gate=gate, gate_act="silu", eps=1e-5, scale=0.65, out=out[:, 8:]), **kw)
    close(out[:, 8:], want.double().cpu(), 1e-5 if fmt == "fp32" else 8e-3)
    assert bool((out[:, :8] == 3.0).all())
    close(s2[1:], s1[1:].double().cpu(), 1e-5)
    kw = dict(heads=H, dk=dk, dv=dv, fmt=fmt, decay=torch.full((H,), 0.9, device=device))      # no norm, read after the update
    a, b2 = (mx.linear_attention(q, k, v, init.clone(), b, kernel=x, **kw) for x in ("seq", "auto"))
    close(b2, a.double().cpu(), 1e-5)


@pytest.mark.gpu
@pytest.mark.parametrize("dims", [(2, 64, 64), (3, 64, 128), (2, 128, 64), (5, 128, 128)])
@pytest.mark.parametrize("mode", ["head", "channel+bonus"])
def test_chunked_linear_attention(dims, mode):
    """Chunk edges in every position, ragged batches, a state handed from chunk to chunk and portion to portion,
    strong decays, keys that stand out just before and after chunk and sub-block edges."""
    H, dk, dv = dims
    lens = (333, 64, 65, 1, 16, 200)
    qkv = [[b16(gen(n, H, d, seed=10 * i + n)) for i, d in enumerate((dk, dk, dv))] for n in lens]
    q, k, v = qkv[0]
    for i, j in ((64, 63), (63, 62), (128, 127), (129, 64), (80, 79), (79, 64), (17, 15), (332, 63), (331, 331), (200, 0)):
        k[j] *= 6
        q[i] = k[j]
    decay = log_w = u = None
    if mode == "head":
        decay = torch.tensor([0.9995, 0.5, 0.97, 0.0, 1.0][:H])
        ws = [decay.view(1, H, 1).expand(n, H, dk) for n in lens]
    else:
        log_w = [-torch.exp(gen(n, H, dk, seed=77 + n, std=2.0, mean=-3.0)).clamp(max=200.0) for n in lens]
        for lw in log_w:
            lw[..., 0], lw[..., 1] = -1e-4, -90.0
            lw[30:90, :, 2] = -25.0
        u = gen(H, dk, seed=5)
        ws = [torch.exp(lw.double()) for lw in log_w]
    cuts = [(100, 64, 65, 1, 0, 0), (64, 0, 0, 0, 16, 63), (1, 0, 0, 0, 0, 0), (168, 0, 0, 0, 0, 137)]
    slots = [3, 1, 2, 6, 5, 4]
    outs, state = run_linear("cuda", "bf16", qkv, log_w, decay, u, dims, cuts, slots, kernel="chunked")
    for s, n in enumerate(lens):
        want, S = plain_linear(*qkv[s], ws[s], u)
        err = (outs[s].double() - want).abs().amax(2) / want.abs().amax(2).clamp(min=0.02 * float(want.abs().max()))
        assert float(err.max()) < 3e-4, (s, float(err.max()), int(err.amax(1).argmax()))
        close(state[slots[s]], S, 1e-4)
    ops.check_status("cuda")


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", DTYPES)
@pytest.mark.parametrize("group,act", [(24, "silu"), (72, "sigmoid"), (9, "silu")])
def test_gated_norm(device, fmt, group, act):
    x, w, g = gen(5, 72, seed=1), b16(gen(72, seed=2)), gen(5, 80, seed=3).to(dt(fmt))
    x[2] *= 1e-3                                                       # eps matters here
    n = fo.rms(x.double().view(5, -1, group), 1e-4).reshape(5, 72)
    gate = g[:, 4:76].double()
    want = n * w.double() * (fo.silu(gate) if act == "silu" else torch.sigmoid(gate)) * 0.65
    out = torch.zeros(5, 100, dtype=dt(fmt), device=device)
    mx.gated_norm(x.to(device), w.to(device), g.to(device)[:, 4:76], fmt, group=group, gate_act=act, eps=1e-4, scale=0.65, out=out[:, 20:92])
    close(out[:, 20:92], want, 1e-5 if fmt == "fp32" else 5e-3)
    assert float(out[:, :20].abs().max()) == 0.0 == float(out[:, 92:].abs().max())


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", DTYPES)
@pytest.mark.parametrize("M,N,K", [(1, 30, 20), (19, 256, 64), (70, 34, 33), (300, 640, 128)])
def test_linear_epilogues(device, fmt, M, N, K):
    x, w = gen(M, K, seed=1).to(dt(fmt)), (gen(N, K, seed=2) * K ** -0.5 * 3).to(dt(fmt))
    act = mx.act_of(x.to(device), fmt)
    W = QuantWeight(fmt, N, K, w.to(device))
    y = x.double() @ w.double().T
    tol = 1e-5 if fmt == "fp32" else 1e-2
    close(ops.linear(act, W), y, tol)
    close(ops.linear(act, W, out_f32=True), y, 1e-5)
    g, u = y[:, 0::2].clamp(max=1.5), y[:, 1::2].clamp(-1.5, 1.5)      # many values beyond the limit
    close(ops.linear(act, W, clamp_glu=(1.702, 1.5)), g * torch.sigmoid(1.702 * g) * (u + 1), tol)
    n = N // 3
    close(ops.linear(act, W, silu_cols=n), torch.cat([fo.silu(y[:, :n]), y[:, n:]], 1), tol)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", DTYPES)
def test_small_ops(device, fmt):
    z, w2, w0 = gen(9, 14, seed=1), b16(gen(50, 14, seed=2)), gen(50, seed=3, mean=-1)
    want = -torch.exp(torch.tanh(z.double()) @ w2.double().T + w0.double())
    close(mx.log_decay(z.to(device), w2.to(device), w0.to(device)), want, 1e-5)
    z, w2 = gen(300, 16, seed=1), b16(gen(136, 16, seed=2))
    w0 = gen(136, seed=3, mean=-1)
    want = -torch.exp(torch.tanh(z.double()) @ w2.double().T + w0.double())
    got = mx.log_decay(z.to(device), w2.to(device), w0.to(device), QuantWeight("bf16", 136, 32, torch.cat([w2, w2], 1).to(device)))
    assert float(((got.double().cpu() - want) / want).abs().max()) < 1e-4
    tab, ids = b16(gen(20, 36, seed=4)), torch.tensor([3, 19, 0, 7], dtype=torch.int32)
    zz = gen(4, 12, seed=5, std=2.0)
    close(mx.side_gate(zz.to(device), ids.to(device), tab.to(device), 24, fmt), fo.gelu_tanh(zz.double()) * tab[ids.long(), 24:].double(),
          1e-5 if fmt == "fp32" else 5e-3)
    close(mx.embed_scaled(ids.to(device), tab.to(device), 2.5), tab[ids.long()].double() * 2.5, 1e-6)
    mixes, r = gen(5, 300, 64, seed=6).to(dt(fmt)), [gen(128, 64, seed=7 + i).to(dt(fmt)) for i in range(4)]
    from metrale_inference_alpha_b200.weights.loader import TimeMixW
    for T in (1, 20, 130, 300):
        m = mixes[:, :T].contiguous().to(device)
        sep = TimeMixW(rkvg=[QuantWeight(fmt, 128, 64, w.to(device)) for w in r])
        both = [sep]
        if fmt == "bf16" and device == "cuda":
            both.append(TimeMixW(rkvg_stack=QuantWeight(fmt, 512, 64, torch.cat(r).to(device))))
        for tw in both:
            for s, y in enumerate(mx.mix_projections(m, tw, fmt)):
                close(y, mixes[s, :T].double() @ r[s].double().T, 1e-5 if fmt == "fp32" else 1e-2)


# ------------------------------------------------------------------ whole models
_ORACLE = {}


def oracle(name, n, seed=0):
    """(tokens, logits [n, vocab]) of one sequence of a configuration, computed once."""
    if (name, n, seed) not in _ORACLE:
        cfg = fc.CONFIGS[name]
        toks = fc.tokens(cfg, n, seed)
        _ORACLE[name, n, seed] = toks, fo.forward(cfg, fc.weights(cfg), toks)
    return _ORACLE[name, n, seed]


def replay(tmp_path, name, dtype, device, max_tokens=192, **kw):
    d = tmp_path / name
    path = str(d) if d.exists() else fc.checkpoint(fc.CONFIGS[name], fc.weights(fc.CONFIGS[name]), d)
    return TraceReplay(path, dtype, max_tokens, device, **kw)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(fc.CONFIGS))
def test_model_whole_portions_and_decoding(tmp_path, device, dtype, name):
    """A prompt at once, in portions down to two tokens, and token by token, all through one engine (so pages
    and slots are used again): each against the plain model."""
    toks, want = oracle(name, 75)
    r = replay(tmp_path, name, dtype, device)
    for cuts in ([75], [2], [1], [33, 2, 17, 3, 1], [16, 15, 17, 1]):
        assert fc.error(fc.feed(r, "a", toks, cuts), want) < TOL[dtype], cuts
    for rid, n in (("one", 1), ("two", 2)):                             # the first tokens of a sequence
        assert fc.error(fc.feed(r, rid, toks[:n], [n]), want[:n]) < TOL[dtype]
    assert r.engine.scheduler.num_active == 0 and r.engine.runner.kv.allocator.num_used == 0 and r.engine.runner.pool.num_free == 4


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["ragged", "equal"])
def test_model_mixed_batches(tmp_path, device, dtype, name):
    """Portions beside single tokens, requests that pause, end and make room: against each alone."""
    seqs = {rid: oracle(name, n, seed) for rid, n, seed in (("a", 75, 0), ("b", 40, 1), ("c", 3, 2), ("d", 58, 3), ("e", 21, 4))}
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
        assert at[k] == len(toks) and fc.error(torch.cat(got[k]), want) < TOL[dtype], k


@pytest.mark.parametrize("device", DEVICES)
def test_long_decoding(tmp_path, device):
    """The state neither drifts nor loses anything over many single steps (32-bit)."""
    toks, want = oracle("ragged", 180, 9)
    r = replay(tmp_path, "ragged", "fp32", device)
    assert fc.error(fc.feed(r, "x", toks, [5, 1]), want) < TOL["fp32"]


@pytest.mark.parametrize("device", DEVICES)
def test_wanted_rows_and_steps_without(tmp_path, device):
    toks, want = oracle("linear", 30)
    r = replay(tmp_path, "linear", "fp32", device)
    assert r.step([{"id": "q", "tokens": toks[:7], "want": []}], []) is None
    got = r.step([{"id": "q", "tokens": toks[7:20], "want": [0, 5, 12]}], [])
    assert fc.error(got, want[[7, 12, 19]]) < TOL["fp32"]
    assert r.step([{"id": "q", "tokens": toks[20:21], "want": []}], []) is None
    assert fc.error(r.step([{"id": "q", "tokens": toks[21:22], "want": [0]}], ["q"]), want[21:22]) < TOL["fp32"]


def greedy_reference(name, prompt, n):
    cfg, t = fc.CONFIGS[name], fc.weights(fc.CONFIGS[name])
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(fo.forward(cfg, t, toks)[-1].argmax()))
    return toks[len(prompt):]


@pytest.mark.parametrize("device", DEVICES)
def test_greedy_generation_scheduler_and_speculation(tmp_path, device):
    """generate() on a queue longer than the batch, with chunked prompts; then with n-gram speculation and
    predicted outputs (verify steps leave the state alone, accepted tokens are committed): the same tokens."""
    path = fc.checkpoint(fc.CONFIGS["ragged"], fc.weights(fc.CONFIGS["ragged"]), tmp_path / "m")
    prompts = [fc.tokens(fc.CONFIGS["ragged"], n, 50 + n) for n in (19, 1, 33)]
    want = [greedy_reference("ragged", p, 12) for p in prompts]
    kw = dict(model=path, device=device, dtype="fp32", max_num_seqs=2, max_model_len=96, max_prefill_tokens=13, num_kv_blocks=24)
    for extra in ({}, {"speculative": "ngram", "mtp_gate": False}):
        eng = LLMEngine(EngineArgs(**kw, **extra))
        outs = eng.generate(prompts, SamplingParams(max_tokens=12, temperature=0.0))
        assert [o.output_ids for o in outs] == want, extra
    guess = [w[:5] + [(w[5] + 1) % 150] + w[6:] for w in want]          # right, then wrong once, then right again
    eng = LLMEngine(EngineArgs(**kw))
    outs = eng.generate(prompts, [SamplingParams(max_tokens=12, temperature=0.0, prediction_ids=g) for g in guess])
    assert [o.output_ids for o in outs] == want
    assert any(o.accepted_draft_tokens for o in outs)


@pytest.mark.parametrize("device", DEVICES)
def test_prefix_cache_resumes_from_state_snapshots(tmp_path, device):
    path = fc.checkpoint(fc.CONFIGS["linear"], fc.weights(fc.CONFIGS["linear"]), tmp_path / "m")
    eng = LLMEngine(EngineArgs(model=path, device=device, dtype="fp32", max_num_seqs=2, max_model_len=400, num_kv_blocks=80))
    p = fc.tokens(fc.CONFIGS["linear"], 300, 5)
    sp = SamplingParams(max_tokens=5, temperature=0.0)
    a = eng.generate([p], sp)[0]
    b = eng.generate([p], sp)[0]
    assert a.output_ids == b.output_ids and b.cached_tokens >= 256


def test_sampled_rows_take_the_models_distribution(tmp_path):
    """Sampling runs on this model's logits: temperature 1 over many seeds visits only the likely tokens."""
    path = fc.checkpoint(fc.CONFIGS["linear"], fc.weights(fc.CONFIGS["linear"]), tmp_path / "m")
    toks, want = oracle("linear", 30)
    eng = LLMEngine(EngineArgs(model=path, device="cpu", dtype="fp32", max_num_seqs=8, max_model_len=64, num_kv_blocks=64))
    top = set(want[-1].topk(3).indices.tolist())
    outs = eng.generate([toks] * 8, [SamplingParams(max_tokens=1, temperature=1.0, top_k=3, seed=s) for s in range(8)])
    assert {o.output_ids[0] for o in outs} <= top


# ------------------------------------------------------------------ configuration, weights, command line
def test_configuration_and_checkpoint(tmp_path):
    cfg = fc.CONFIGS["ragged"]
    c = from_hf_config(json.loads(json.dumps(cfg)))
    assert c.arch == "fabulix" and c.layer_types == ["parallel", "lightning", "parallel", "lightning"]
    assert c.ffn_types == ["dense", "none", "none", "dense"] and c.attention_layers() == [0, 2]
    assert c.kv_layer_dims() == [(2, 64, 64), (1, 64, 64)]
    assert c.scaled(weight_format="fp32").kv_layer_dims() == [(2, 30, 44), (1, 24, 26)]
    assert type(c).from_json(c.to_json()).to_json() == c.to_json()
    from metrale_inference_alpha_b200.weights.checkpoint import open_checkpoint
    from metrale_inference_alpha_b200.weights.preflight import preflight
    t = fc.weights(cfg)
    c2, src = open_checkpoint(fc.checkpoint(cfg, t, tmp_path / "ok"))
    assert preflight(c2, src, check_shapes=False).ok
    del t["l2.mix.right.u"]
    c3, src = open_checkpoint(fc.checkpoint(cfg, t, tmp_path / "bad"))
    assert preflight(c3, src, check_shapes=False).missing == ["l2.mix.right.u"]
    bad = json.loads(json.dumps(cfg))
    bad["layers"][0]["type"] = "other"
    with pytest.raises(ValueError, match="unknown mixer"):
        from_fabulix_config(bad)
    bad = json.loads(json.dumps(cfg))
    bad["layers"][1]["mixer"]["decay"] = [0.5]
    with pytest.raises(ValueError, match="decays"):
        from_fabulix_config(bad)


def test_unserved_combinations_are_refused():
    for kw in (dict(model="tiny-dense", dtype="fp32"), dict(model="tiny-fabulix", dtype="int8")):
        with pytest.raises(ValueError):
            LLMEngine(EngineArgs(max_model_len=64, num_kv_blocks=16, **kw))
    for kw in (dict(kv_cache_dtype="fp8"), dict(speculative="dflash")):
        with pytest.raises(NotImplementedError):
            LLMEngine(EngineArgs(model="tiny-fabulix", max_model_len=64, num_kv_blocks=16, **kw))


@pytest.mark.parametrize("device", DEVICES)
def test_preset_runs_from_synthetic_weights(device):
    eng = LLMEngine(EngineArgs(model=preset("tiny-fabulix", num_layers=3), device=device, max_num_seqs=2, max_model_len=64, num_kv_blocks=16))
    outs = eng.generate([[1, 2, 3], [9, 8, 7, 6]], SamplingParams(max_tokens=4))
    assert all(len(o.output_ids) == 4 for o in outs)
    if device != "cpu":
        ops.check_status(device)


def test_replay_command(tmp_path, capsys):
    import numpy as np
    from metrale_inference_alpha_b200.server import cli
    cfg = fc.CONFIGS["linear"]
    path = fc.checkpoint(cfg, fc.weights(cfg), tmp_path / "m")
    toks, want = oracle("linear", 30)
    ns = cli.build_parser().parse_args(["replay", "--model", path, "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "64",
                                        "--device", "cpu"])
    from metrale_inference_alpha_b200.engine.replay import run
    lines = [json.dumps({"step": 0, "entries": [{"id": "a", "tokens": toks[:9], "want": []}], "end": []}),
             json.dumps({"step": 1, "entries": [{"id": "a", "tokens": toks[9:30], "want": [20]}], "end": ["a"]})]
    assert run(ns, lines) == 0
    assert [x for x in capsys.readouterr().out.splitlines() if x.startswith("done")] == ["done 0", "done 1"]
    got = torch.from_numpy(np.fromfile(tmp_path / "1.f32", dtype="<f4")).view(1, -1)
    assert fc.error(got, want[29:30]) < 1e-5 and not (tmp_path / "0.f32").exists()
