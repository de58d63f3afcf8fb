"""The Ledinex decoder against a plain restatement (ledinex_oracle.py): every mechanism alone, then whole models through
the engine's own entry points. The CPU runs cover the engine's host logic and its op restatements, the GPU runs the
kernels."""
import json
import math

import pytest
import torch

import ledinex_cases as lc
import ledinex_oracle as lo
from metrale_inference_alpha_b200 import ops
from metrale_inference_alpha_b200.config.model_config import from_hf_config, from_ledinex_config, preset
from metrale_inference_alpha_b200.engine.llm_engine import EngineArgs, LLMEngine
from metrale_inference_alpha_b200.engine.replay import TraceReplay
from metrale_inference_alpha_b200.ops import QuantWeight, canon, delta as dl, mixers as mx, moe as moe_ops, reference as ref
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


def portions(n, cuts):
    at, i = 0, 0
    while at < n:
        m = min(cuts[min(i, len(cuts) - 1)], n - at)
        yield at, m
        at, i = at + m, i + 1


# ------------------------------------------------------------------ convolutions
def run_stream(device, fmt, x, y, routed_of, norm, filt, cuts, slots=4, verify=()):
    """Two sequences side by side, x and y [2, n, W]: the first in portions of `cuts`, the second lagging behind by its own.
    Portions whose index is in `verify` leave the window alone and commit only part of their rows (and are fed again)."""
    n, W = x.shape[1:]
    taps = filt.shape[0]
    rows = torch.full((slots, 5 + (taps - 1) * W), 7.0, device=device)
    win = canon.Window(rows, 5, W)
    got = torch.zeros(2, n, W, dtype=torch.float64), torch.zeros(2, n, W, dtype=torch.float64)
    at, i = [0, 0], 0
    while min(at) < n:
        lens = [min(cuts[min(i, len(cuts) - 1)], n - at[0]), min(3 + i % 2 * 5, n - at[1])]
        b = lc.batch(lens, [at[s] + lens[s] for s in range(2)], slots=[3, 1], device=device)
        live = [slice(at[s], at[s] + lens[s]) for s in range(2)]
        cat = lambda z: torch.cat([z[s, live[s]] for s in range(2)]).to(device).contiguous()
        out = None if y is None else mx.SublayerOut(cat(y).to(dt(fmt)), None, routed_of and routed_of(cat(routed_of.rows)))
        v = i in verify
        x1, h = canon.stream_canon(cat(x), fmt, pending=out, norm=norm, filt=filt, window=win, batch=b, write_state=not v)
        if v:
            lens = [(m + 1) // 2 for m in lens]
            import dataclasses
            canon.canon_commit(x1, taps, win, dataclasses.replace(b, q_len=torch.tensor(lens, dtype=torch.int32, device=device)))
        r = 0
        for s in range(2):
            m = live[s].stop - live[s].start
            got[0][s, live[s]], got[1][s, live[s]] = x1[r:r + m].double().cpu(), h[r:r + m].double().cpu()
            r += m
            at[s] += lens[s]
        i += 1
    assert bool((rows[:, :5] == 7.0).all()) and bool((rows[[0, 2]] == 7.0).all())
    return got


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", DTYPES)
@pytest.mark.parametrize("W,taps", [(37, 3), (100, 1), (96, 2), (1100, 5), (52, 12), (8, 20)])
@pytest.mark.parametrize("plus", [True, False])
def test_stream_joins_and_convolves(device, fmt, W, taps, plus):
    """Pending output (alone, with expert rows, only expert rows, none), portions of many lengths beside another sequence,
    windows carried from portion to portion, verify steps that keep part of their rows."""
    n, K, eps = 130 if W <= 100 else 100, 3, 1e-3
    x, y, e = gen(2, n, W, seed=1, std=2.0), gen(2, n, W, seed=2).to(dt(fmt)).float(), gen(2, n, W, seed=3)
    w, filt = b16(gen(W, seed=4, std=0.4)), b16(gen(W, taps, seed=5, std=0.5))
    norm, f = mx.RmsNorm(w.to(device), eps, plus_one=plus), filt.t().contiguous().to(device)

    def routed(rows):                                                # K places per token, one of them empty, in no order
        T = len(rows)
        if device == "cpu":
            return mx.Routed(rows, None, None)
        place = torch.randperm(T * K, generator=torch.Generator().manual_seed(T)).int().to(device)
        ye, pw = torch.zeros(T * K, W + 4, device=device), torch.rand(T, K, device=device) + 0.5
        p = place.view(T, K)
        p[:, 1] = -1
        ye[p[:, 0].long(), :W], ye[p[:, 2].long(), :W] = rows * 0.25 / pw[:, :1], rows * 0.75 / pw[:, 2:]
        return mx.Routed(ye, place, pw)

    routed.rows = e
    wd = w.double() + (1.0 if plus else 0.0)
    for what, Y in (("y", y.double()), ("both", y.double() + e.double()), ("none", None)):
        X = x.double() if Y is None else x.double() + lo.unit_rms(Y, eps) * wd
        H = torch.stack([X[s] + lo.short_conv(X[s], filt.double()) for s in range(2)])
        for cuts in ([n], [2], [17, 1, 9, 8, 4], [3, 97, 1]):
            x1, h = run_stream(device, fmt, x, None if Y is None else y, routed if what == "both" else None, norm, f, cuts,
                               verify=(0, 2) if cuts[0] == 17 else ())
            close(x1, X, 3e-6)                                       # the stream is 32-bit in both formats
            close(h, H, 1e-5 if fmt == "fp32" else 6e-3)
    one = mx.SublayerOut(routed=routed(e[0].to(device)))
    x1, h = canon.stream_canon(x[0].to(device), fmt, pending=one, norm=norm)           # no filter: the stream alone
    assert h is None
    close(x1, x[0].double() + lo.unit_rms(e[0].double(), eps) * wd, 3e-6)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", DTYPES)
@pytest.mark.parametrize("C,taps", [(37, 3), (64, 4), (256, 2), (12, 1), (20, 9), (33, 17)])
def test_short_convolution(device, fmt, C, taps):
    n = 70
    x = gen(n, C + 8, seed=1).to(dt(fmt))
    filt = gen(C, taps, seed=2, std=0.6)
    want = lo.silu(lo.short_conv(x[:, 8:].double()[:, :C], filt.double()))
    f, tol = filt.t().contiguous().to(device), 1e-5 if fmt == "fp32" else 6e-3
    for cuts in ([n], [2], [1], [33, 1, 16, 17], [15, 3, 1]):
        rows = torch.full((3, 2 + (taps - 1) * C), 7.0, device=device)
        win = canon.Window(rows, 2, C)
        outs = []
        for i, (at, m) in enumerate(portions(n, cuts)):
            b = lc.batch([m, 1], [at + m, 1], slots=[2, 1], device=device)
            z = torch.cat([x[at:at + m], x[:1]]).to(device)
            y = canon.short_conv(z[:, 8:], f, win, b, fmt, write_state=i != 1)
            if i == 1:                                               # a verify step: outputs first, the window afterwards
                canon.short_conv(z[:, 8:], f, win, b, fmt, write_out=False)
            outs.append(y[:m])
            close(y[m:], want[:1], tol)
        close(torch.cat(outs), want, tol)
        assert bool((rows[0] == 7.0).all()) and bool((rows[:, :2] == 7.0).all())


# ------------------------------------------------------------------ rows of an attention layer
def test_scaled_frequencies():
    """Linear and blended scaling: every band, ramps of no width, ramps that end outside the dimensions."""
    kinds = set()
    for base, dims, s in ((1e4, 32, (4.0, 2048, 32.0, 1.0)), (900.0, 20, (5.0, 64, 4.0, 0.5)), (50.0, 6, (2.0, 1000000, 32.0, 1.0)),
                          (1e4, 16, (8.0, 4, 32.0, 1.0)), (1e4, 24, (0.5, 300, 2.0, 2.0)), (1e4, 2, (1.0, 1, 1.0, 1.0))):
        sc = dict(zip(("factor", "original", "fast", "slow"), s))
        want, gain = lo.frequencies({"base": base, "dims": dims, "scaling": sc})
        hf = {"rope_type": "yarn", "factor": s[0], "original_max_position_embeddings": s[1], "beta_fast": s[2], "beta_slow": s[3],
              "attention_factor": 0.1 * math.log(s[0]) + 1}
        got, att = ref.rope_inv_freq(dims, base, hf)
        assert float((got / torch.tensor(want, dtype=torch.float64) - 1).abs().max()) < 1e-12 and abs(att - gain) < 1e-12
        plain = lo.frequencies({"base": base, "dims": dims})[0]
        kinds |= {0 if a == b else 1 if abs(a * s[0] / b - 1) < 1e-12 else 2 for a, b in zip(want, plain)}
    assert kinds == {0, 1, 2}
    got, att = ref.rope_inv_freq(10, 700.0, {"rope_type": "linear", "factor": 3.0})
    assert att == 1.0 and torch.allclose(got, torch.tensor(lo.frequencies({"base": 700.0, "dims": 10, "scaling": {"factor": 3.0}})[0], dtype=torch.float64))


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", DTYPES)
@pytest.mark.parametrize("H,G,dk,dv,rot", [(4, 2, 64, 64, 64), (3, 1, 22, 30, 10), (6, 2, 128, 40, 32), (2, 1, 264, 12, 0), (1, 1, 2, 2, 2)])
@pytest.mark.parametrize("values", ["plain", "turned", "keys"])
def test_attention_rows(device, fmt, H, G, dk, dv, rot, values):
    """Norms over the whole projection, partial rotation, values as they are, turned by their position, or the raw keys;
    then an output turned back."""
    T, eps, block = 7, 1e-2, 16
    dv = dk if values == "keys" else dv
    cols = (3, 3 + H * dk + 5, 3 + H * dk + 5 if values == "keys" else 3 + (H + G) * dk + 8)
    x = gen(T, (H + G) * dk + G * dv + 16, seed=1).to(dt(fmt))
    pos = torch.tensor([0, 1, 15, 16, 17, 900, 3], dtype=torch.int32)
    slots = torch.tensor([40, 3, 17, 16, -1, 79, 47], dtype=torch.int64)
    qn, kn = b16(gen(H * dk, seed=2, std=0.3, mean=1.0)), b16(gen(G * dk, seed=3, std=0.3, mean=1.0))
    dkp, dvp = mx.padded_head_dims(dk, dv, fmt)
    kc, vc = (torch.full((5, block, G, d), 9.0, dtype=dt(fmt), device=device) for d in (dkp, dvp))
    tables = lambda d: ref.rope_tables(1000, d, 700.0, device=device)
    turn = tables(dv) if values == "turned" else None
    q = mx.attention_rows(x.to(device), cols=cols, Hq=H, Hkv=G, dk=dk, dv=dv, positions=pos.to(device), slots=slots.to(device), k_cache=kc,
                          v_cache=vc, rot=tables(rot) if rot else None, fmt=fmt, q_norm=mx.RmsNorm(qn.to(device), eps),
                          k_norm=mx.RmsNorm(kn.to(device), eps), v_rot=turn)
    part = lambda at, n: x[:, at:at + n].double()
    rotated = lambda t, d: torch.stack([lo.turn(t[i], [int(pos[i]) * 700.0 ** (-2.0 * j / d) for j in range(d // 2)]) for i in range(T)])
    qw = rotated((lo.unit_rms(part(cols[0], H * dk), eps) * qn.double()).view(T, H, dk), rot or 1)
    kw = rotated((lo.unit_rms(part(cols[1], G * dk), eps) * kn.double()).view(T, G, dk), rot or 1)
    vw = part(cols[2], G * dv).view(T, G, dv)
    vw = rotated(vw, dv) if turn else vw
    tol = 1e-5 if fmt == "fp32" else 6e-3
    close(q[..., :dk], qw, tol)
    kc, vc, live = kc.cpu().view(-1, G, dkp), vc.cpu().view(-1, G, dvp), slots >= 0
    close(kc[slots[live], :, :dk], kw[live], tol)
    close(vc[slots[live], :, :dv], vw[live], tol if turn else 1e-9)
    assert bool((q[..., dk:] == 0).all()) and bool((kc[slots[live], :, dk:] == 0).all()) and bool((vc[slots[live], :, dv:] == 0).all())
    untouched = [s for s in range(80) if s not in slots.tolist()]
    assert bool((kc[untouched] == 9).all()) and bool((vc[untouched] == 9).all())
    if turn:
        o = gen(T, H * dv + 8, seed=5).to(dt(fmt))
        got = o.to(device, copy=True)
        mx.turn_rows(got[:, 8:], H, dv, pos.to(device), turn, fmt)
        back = torch.stack([lo.turn(o[i, 8:].double().view(H, dv), [-int(pos[i]) * 700.0 ** (-2.0 * j / dv) for j in range(dv // 2)]) for i in range(T)])
        close(got[:, 8:], back.reshape(T, -1), tol)
        assert torch.equal(got[:, :8].cpu(), o[:, :8])


# H, G, dk, dv: the 64-, 128- and 256-wide tiles (equal and not), past them, away from whole vectors
ATT = {"t64": (4, 2, 64, 64), "t64/128": (4, 4, 40, 128), "t128": (6, 2, 128, 128), "t128/64": (3, 1, 100, 48), "t96": (4, 2, 96, 96),
       "t256": (2, 1, 200, 72), "t256 full": (4, 2, 256, 256), "past": (2, 1, 264, 20), "odd": (3, 1, 22, 30)}


def run_attention(device, fmt, q, k, v, dims, cuts, scale, window, softcap, kernel="auto", block=16, turn=None):
    """One sequence fed in portions through the paged cache (pages not in order, unwritten slots NaN); [n, H, dv]. `turn`:
    values are cached turned by their position, outputs turned back."""
    H, G, dk, dv = dims
    n = q.shape[0]
    dkp, dvp = mx.padded_head_dims(dk, dv, fmt)
    nb = (n + block - 1) // block
    kc, vc = (torch.full((nb + 8, block, G, d), float("nan"), dtype=dt(fmt), device=device) for d in (dkp, dvp))
    pages = list(range(nb + 4, 4, -1))
    rows = torch.cat([q.reshape(n, -1), k.reshape(n, -1), v.reshape(n, -1)], 1)
    outs = []
    for at, m in portions(n, cuts):
        b = lc.batch([m], [at + m], device=device, block=block, pages=[pages[:(at + m + block - 1) // block]])
        qq = mx.attention_rows(rows[at:at + m].to(device), cols=(0, H * dk, (H + G) * dk), Hq=H, Hkv=G, dk=dk, dv=dv, positions=b.positions,
                               slots=b.slot_mapping, k_cache=kc, v_cache=vc, rot=None, fmt=fmt, v_rot=turn)
        out = torch.empty(m, H * dv, dtype=dt(fmt), device=device)
        kern = kernel if kernel != "tc" or m >= 2 else "auto"
        outs.append(mx.attention_dims(qq, kc, vc, b, dk=dk, dv=dv, scale=scale, sink=False, fmt=fmt, out=out, window=window, softcap=softcap, kernel=kern,
                                      turn_back=turn))
    return torch.cat(outs).view(n, H, dv)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", DTYPES)
@pytest.mark.parametrize("name", list(ATT))
@pytest.mark.parametrize("window,softcap", [(0, 2.0), (19, 0.0), (0, 30.0), (1, 1.5), (33, 5.0)])
def test_capped_and_windowed_attention(device, fmt, name, window, softcap):
    """Scores far past the cap, keys that stand out at page borders and far away: without the cap (or with another one) the
    weights would differ by orders of magnitude."""
    dims, n, scale = ATT[name], 70, 0.5
    H, G, dk, dv = dims
    q, k, v = gen(n, H, dk, seed=1), gen(n, G, dk, seed=2), gen(n, G, dv, seed=3)
    for i, j in ((0, 0), (16, 15), (17, 16), (33, 32), (47, 1), (48, 0), (63, 48), (69, 0), (69, 16), (50, 33), (51, 32), (60, 42), (61, 42)):
        q[i] = k[j].repeat_interleave(H // G, 0)
    q, k, v = (t.to(dt(fmt)) for t in (q, k, v))
    want = lo.attend(q.double(), k.double(), v.double(), scale, window or None, softcap or None)
    for cuts in ([n], [2], [33, 1], [1]):
        close(run_attention(device, fmt, q, k, v, dims, cuts, scale, window, softcap), want, 2e-5 if fmt == "fp32" else 8e-3)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", DTYPES)
@pytest.mark.parametrize("name", list(ATT))
def test_rotated_values(device, fmt, name):
    """Values turned by their position and outputs turned back: what reaches a query is turned by the distance alone."""
    dims, n, scale, base = ATT[name], 150, 0.2, 50.0
    H, G, dk, dv = dims
    q, k, v = (gen(n, h, d, seed=s).to(dt(fmt)) for h, d, s in ((H, dk, 1), (G, dk, 2), (G, dv, 3)))
    turn = ref.rope_tables(200, dv, base, device=device)
    vt = lo.turn_values(v.double(), base, 1)
    s = torch.einsum("ihd,jhd->hij", q.double(), k.double().repeat_interleave(H // G, 1)) * scale
    p = torch.softmax(s.masked_fill(torch.arange(n)[None] > torch.arange(n)[:, None], float("-inf")), -1)
    want = lo.turn_values(torch.einsum("hij,jhd->ihd", p, vt.repeat_interleave(H // G, 1)), base, -1)
    for cuts in ([n], [7], [130, 1], [1]):
        close(run_attention(device, fmt, q, k, v, dims, cuts, scale, 0, 0.0, turn=turn), want, 2e-5 if fmt == "fp32" else 1e-2)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", DTYPES)
@pytest.mark.parametrize("window", [1, 16, 17, 64])
def test_single_keys_at_the_windows_edge(device, fmt, window):
    """One key outshines all others: the last query that sees it returns its value, the next one does not."""
    dims, n, scale = (2, 1, 16, 16), 100, 4.0
    q, k, v = gen(n, 2, 16, seed=1, std=0.05), gen(n, 1, 16, seed=2, std=0.05), gen(n, 1, 16, seed=3)
    q[..., 0] = 4.0
    for j in (0, 1, 15, 16, 33):
        kj = k.clone()
        kj[j, 0, 0] = 4.0
        a = tuple(t.to(dt(fmt)) for t in (q, kj, v))
        for cuts in ([n], [17, 16, 2, 1]):
            got = run_attention(device, fmt, *a, dims, cuts, scale, window, 0.0).double().cpu()
            for i in range(j, n):
                hit = float((got[i] - a[2][j].double()).abs().max()) < 2e-2
                assert hit == (i - j < window), (i, j)


@pytest.mark.gpu
@pytest.mark.parametrize("kernel,name", [("mma", "t64"), ("mma", "t128"), ("tc", "t128"), ("auto", "t256"), ("tc", "t256 full"), ("mma", "t128/64"),
                                         ("simt", "t64"), ("auto", "t96")])
@pytest.mark.parametrize("softcap", [30.0, 3.0])
def test_capped_attention_long(kernel, name, softcap):
    """Many tiles and several partitions, far keys whose scores lie past the cap."""
    dims, n, scale = ATT[name], 1250, 0.12
    H, G, dk, dv = dims
    q, k, v = (b16(gen(n, h, d, seed=s)) for h, d, s in ((H, dk, 1), (G, dk, 2), (G, dv, 3)))
    for i, j in ((700, 3), (1199, 64), (1210, 0), (1249, 511), (1249, 1023), (900, 899)):
        k[j] = k[j] * 2
        q[i] = k[j].repeat_interleave(H // G, 0)
    s = torch.einsum("ihd,jhd->hij", q.double(), k.double().repeat_interleave(H // G, 1)) * scale
    s = softcap * torch.tanh(s / softcap)
    s.masked_fill_(torch.arange(n)[None] > torch.arange(n)[:, None], float("-inf"))
    want = torch.einsum("hij,jhd->ihd", torch.softmax(s, -1), v.double().repeat_interleave(H // G, 1))
    for cuts in ([1250], [1000, 200, 7, 1]):
        got = run_attention("cuda", "bf16", q, k, v, dims, cuts, scale, 0, softcap, kernel=kernel if kernel != "mma" else "auto" if dk > 128 else "mma")
        close(got, want, 1e-2)
    ops.check_status("cuda")


# ------------------------------------------------------------------ recurrences
def rule_case(general, H, HK, dk, dv, n, fmt, strong=False):
    """(rows q | k | v | gate logits in the activation type, spans, oracle inputs) of one sequence."""
    nk = HK * dk
    x = {"q": gen(n, nk, seed=1), "k": gen(n, nk, seed=2, std=1.5), "v": gen(n, H * dv, seed=3)}
    if general:
        x["a"], lw = gen(n, H * dk, seed=4, std=2.0), -0.6 * torch.sigmoid(gen(n, H * dk, seed=5, std=3.0, mean=-1.0))
        bound = -math.inf if strong else -0.6
        if strong:
            lw = lw * 40
    else:
        x["a"], x["b"] = gen(n, H, seed=4, std=2.0), gen(n, H, seed=5, std=2.0)
        A, bias = gen(H, seed=6, std=1.0, mean=3.0 if strong else -1.0), gen(H, seed=7)
    x = {k: t.to(dt(fmt)) for k, t in x.items()}
    d = {k: t.double() for k, t in x.items()}
    heads = lambda t, h, e: t.view(n, h, e)
    if general:
        want = lo.general_delta_recurrence(heads(d["q"], H, dk), heads(d["k"], H, dk), heads(d["v"], H, dv), heads(torch.exp(lw.double()), H, dk),
                                           heads(lo.sigmoid(d["a"]), H, dk))
        return x, dict(lw=lw, bound=bound), want.reshape(n, -1)
    g = torch.exp(-torch.exp(A.double()) * lo.softplus(d["a"] + bias.double()))
    want = lo.gated_delta_recurrence(heads(d["q"], HK, dk), heads(d["k"], HK, dk), heads(d["v"], H, dv), g, lo.sigmoid(d["b"]))
    return x, dict(A=A, bias=bias), want.reshape(n, -1)


def run_rule(device, fmt, case, general, H, HK, dk, dv, cuts, kernel="auto", verify=(), norm=None):
    x, c, want = case
    n = len(want)
    state = torch.full((4, H, dk, dv), 5.0, device=device)
    cat = torch.cat([x["q"], x["k"], x["v"], x["a"]] + ([] if general else [x["b"]]), 1)
    wide = torch.cat([cat, cat.new_zeros(n, 8 + -cat.shape[1] % 8)], 1)
    spans, at = [], 0
    for t in (x["q"], x["k"], x["v"], x["a"], x["a"] if general else x["b"]):
        spans.append((at, t.shape[1]))
        at += t.shape[1]
    outs = []
    import dataclasses
    for i, (lo_, m) in enumerate(portions(n, cuts)):
        b = lc.batch([m, 1], [lo_ + m, 1], slots=[2, 1], device=device)
        z = torch.cat([wide[lo_:lo_ + m], wide[:1]]).to(device)
        q, k, v, a, bb = (z[:, s:s + w] for s, w in spans)
        rows = torch.cat([torch.arange(lo_, lo_ + m), torch.zeros(1, dtype=torch.long)])
        rule = dl.GeneralRule(a, c["lw"][rows].to(device).contiguous(), c["bound"]) if general else dl.GatedRule(a, bb, c["A"].to(device), c["bias"].to(device))
        kw = dict(heads=H, key_heads=HK, dk=dk, dv=dv, fmt=fmt)
        if norm is not None:
            gate = torch.cat([norm["gate"][lo_:lo_ + m], norm["gate"][:1]]).to(device)
            o = torch.zeros(m + 1, H * dv + 8, dtype=dt(fmt), device=device)
            dl.delta_attention(q, k, v, rule, state, b, kernel=kernel, **kw,
                               norm=dict(w=norm["w"].to(device), gate=gate, gate_act=norm["act"], eps=1e-3, scale=0.8, out=o[:, 8:]))
            outs.append(o[:m, 8:])
            continue
        y = dl.delta_attention(q, k, v, rule, state, b, write_state=i not in verify, kernel=kernel, **kw)
        if i in verify:
            dl.delta_attention(q, k, v, rule, state, b, write_out=False, kernel="seq", **kw)
        outs.append(y[:m])
    assert bool((state[[0, 3]] == 5.0).all())
    return torch.cat(outs)


RULES = [(False, 4, 2, 64, 64), (False, 6, 2, 18, 22), (False, 2, 1, 136, 264), (False, 3, 3, 32, 4), (False, 2, 2, 128, 128), (False, 2, 1, 64, 128),
         (True, 3, 3, 64, 64), (True, 2, 2, 128, 128), (True, 5, 5, 28, 28), (True, 1, 1, 200, 200), (True, 1, 1, 10, 10), (False, 1, 1, 256, 256)]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", DTYPES)
@pytest.mark.parametrize("general,H,HK,dk,dv", RULES)
@pytest.mark.parametrize("strong", [False, True])
def test_delta_rules(device, fmt, general, H, HK, dk, dv, strong):
    """Whole, token by token, in portions, and after steps that commit later; mild and strong decays."""
    n = 70
    case = rule_case(general, H, HK, dk, dv, n, fmt, strong)
    for cuts, verify in (([n], ()), ([1], ()), ([33, 1, 2, 17], ()), ([16, 5, 5, 40], (1, 2))):
        close(run_rule(device, fmt, case, general, H, HK, dk, dv, cuts, verify=verify), case[2], 1e-5 if fmt == "fp32" else 3e-5)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", DTYPES)
@pytest.mark.parametrize("general,H,HK,dk,dv", [(False, 4, 2, 32, 64), (True, 3, 3, 64, 64), (False, 2, 1, 18, 22), (True, 2, 2, 128, 128)])
def test_delta_rules_with_head_norm(device, fmt, general, H, HK, dk, dv):
    n = 40
    case = rule_case(general, H, HK, dk, dv, n, fmt)
    act = "sigmoid" if general else "silu"
    norm = dict(w=b16(gen(H * dv, seed=9, mean=1.0)), gate=gen(n, H * dv, seed=10).to(dt(fmt)), act=act)
    z = norm["gate"].double()
    want = 0.8 * (lo.unit_rms(case[2].view(n, H, dv), 1e-3).reshape(n, -1) * norm["w"].double() * (lo.sigmoid(z) if general else lo.silu(z)))
    for cuts in ([n], [1], [20, 1]):
        close(run_rule(device, fmt, case, general, H, HK, dk, dv, cuts, norm=norm), want, 1e-4 if fmt == "fp32" else 8e-3)


@pytest.mark.gpu
@pytest.mark.parametrize("general,H,HK,dk,dv", [(False, 4, 2, 64, 64), (False, 2, 1, 64, 128), (False, 2, 2, 128, 64), (False, 3, 1, 128, 128),
                                                (True, 3, 3, 64, 64), (True, 2, 2, 128, 128)])
@pytest.mark.parametrize("norm", [False, True])
@pytest.mark.parametrize("strong", [False, True])
def test_chunked_delta_rules(general, H, HK, dk, dv, norm, strong):
    """Several chunks, ragged ends, a carried state, a second sequence of one token beside it; the head norm inside."""
    if general and strong:
        pytest.skip("decays past the chunked kernels' range are served token by token")
    n = 250
    case = rule_case(general, H, HK, dk, dv, n, "bf16", strong)
    nm, want, tol = None, case[2], 4e-5
    if norm:
        nm = dict(w=b16(gen(H * dv, seed=9, mean=1.0)), gate=b16(gen(n, H * dv, seed=10)), act="sigmoid" if general else "silu")
        z = nm["gate"].double()
        want = 0.8 * (lo.unit_rms(want.view(n, H, dv), 1e-3).reshape(n, -1) * nm["w"].double() * (lo.sigmoid(z) if general else lo.silu(z)))
        tol = 8e-3
    for cuts in ([n], [64, 186], [1, 65, 63, 100], [130, 1]):
        got = run_rule("cuda", "bf16", case, general, H, HK, dk, dv, cuts, kernel="chunked", norm=nm)
        close(got, want, tol)
    ops.check_status("cuda")


@pytest.mark.gpu
@pytest.mark.parametrize("general", [False, True])
def test_chunked_rule_with_repeated_keys(general):
    """The hardest systems of a chunk: the same key in every row, full step sizes and removal rates, hardly any decay."""
    n, H, d = 200, 2, 64
    x, c, _ = rule_case(general, H, H, d, d, n, "bf16")
    x["k"][:] = x["k"][:1] * 0.5
    x["a"][:] = 6.0 if general else -9.0
    dbl = {k: t.double().view(n, H, -1) for k, t in x.items()}
    if general:
        c["lw"][:] = -1e-3
        want = lo.general_delta_recurrence(dbl["q"], dbl["k"], dbl["v"], torch.exp(c["lw"].double()).view(n, H, d), lo.sigmoid(dbl["a"]))
    else:
        x["b"][:] = 6.0
        g = torch.exp(-torch.exp(c["A"].double()) * lo.softplus(x["a"].double() + c["bias"].double()))
        want = lo.gated_delta_recurrence(dbl["q"], dbl["k"], dbl["v"], g, lo.sigmoid(x["b"].double()))
    case = x, c, want.reshape(n, -1)
    for kernel in ("chunked", "seq"):
        close(run_rule("cuda", "bf16", case, general, H, H, d, d, [n], kernel=kernel), case[2], 5e-4 if kernel == "chunked" else 1e-5)


def test_the_general_rule_reads_the_old_state_and_writes_the_key_itself():
    """Hand-made: what the decay keeps, what the rate removes along the unit key, what the key's own length writes."""
    r, k, v = torch.zeros(2, 1, 2), torch.zeros(2, 1, 2), torch.zeros(2, 1, 2)
    k[0, 0, 0], v[0, 0] = 2.0, torch.tensor([3.0, 0.0])                  # S = [[6, 0], [0, 0]]
    k[1, 0, 0], v[1, 0], r[1, 0, 0] = 5.0, torch.tensor([0.0, 1.0]), 1.0
    w, a = torch.full((2, 1, 2), 0.5), torch.full((2, 1, 2), 0.25)
    o = lo.general_delta_recurrence(r.double(), k.double(), v.double(), w.double(), a.double())
    assert torch.allclose(o[1, 0], torch.tensor([0.5 * 6 - 0.25 * 6, 5.0], dtype=torch.float64), atol=1e-5)
    state = torch.zeros(2, 1, 2, 2)
    got = dl.delta_attention(r.view(2, 2), k.view(2, 2), v.view(2, 2), dl.GeneralRule(torch.logit(a.view(2, 2)), torch.log(w.view(2, 2))), state,
                             lc.batch([2]), heads=1, dk=2, dv=2, fmt="fp32")
    assert torch.allclose(got.double(), o.view(2, 2), atol=1e-5)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", DTYPES)
@pytest.mark.parametrize("T,rank,n", [(1, 16, 40), (7, 9, 33), (300, 16, 256), (300, 12, 70), (5, 72, 64), (270, 1, 16)])
def test_bounded_decays(device, fmt, T, rank, n):
    """Low-rank logits through tanh: alone (CUDA cores and tensor cores) and inside the decode kernel."""
    z, w2, w0 = gen(T, rank + 8, seed=1, std=1.5).to(dt(fmt)), b16(gen(n, rank, seed=2)), gen(n, seed=3, std=2.0)
    want = -math.exp(-0.5) * lo.sigmoid(torch.tanh(z[:, 8:].double()) @ w2.double().t() + w0.double())
    twice = QuantWeight("bf16", n, 2 * rank, torch.cat([w2, w2], 1).contiguous().to(device)) if fmt == "bf16" and rank % 4 == 0 else None
    d = dl.BoundedDecay(z.to(device)[:, 8:], w2.to(device), w0.to(device), -math.exp(-0.5), twice)
    close(d.log(), want, 1e-5)
    if T < 10:
        q, k, v, a = (gen(T, n, seed=s).to(dt(fmt)).to(device) for s in (4, 5, 6, 7))
        st = [gen(T + 1, 1, n, n, seed=8).to(device) for _ in range(2)]
        b = lc.batch([1] * T, [9] * T, device=device)
        kw = dict(heads=1, dk=n, dv=n, fmt=fmt)
        got = dl.delta_attention(q, k, v, dl.GeneralRule(a, d), st[0], b, **kw)
        same = dl.delta_attention(q, k, v, dl.GeneralRule(a, want.float().to(device).contiguous()), st[1], b, **kw)
        close(got, same.cpu(), 1e-5)
        close(st[0], st[1].cpu(), 1e-5)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", DTYPES)
def test_decays_do_not_lose_a_far_token(device, fmt):
    """A head that hardly decays still finds a key written hundreds of tokens ago; one that decays fast does not."""
    n, H, d = 400, 2, 32
    q, k, v = (torch.zeros(n, H, d) for _ in range(3))
    k[5, :, 3], v[5], q[n - 1, :, 3] = 1.0, 1.0, 1.0
    k[6:, :, 7:9] = 0.3 * gen(n - 6, H, 2, seed=1)                        # other keys, none along the first one
    a = torch.stack([torch.full((n,), -12.0), torch.full((n,), 2.0)], 1)
    flat = [t.reshape(n, -1).to(dt(fmt)).to(device) for t in (q, k, v)]
    rule = dl.GatedRule(a.to(dt(fmt)).to(device), torch.full((n, H), 4.0).to(dt(fmt)).to(device), torch.zeros(H, device=device), torch.zeros(H, device=device))
    st = torch.zeros(2, H, d, d, device=device)
    o = dl.delta_attention(*flat, rule, st, lc.batch([n], device=device), heads=H, dk=d, dv=d, fmt=fmt).view(n, H, d)[-1].double().cpu()
    assert float((o[0] / (lo.sigmoid(torch.tensor(4.0)) * d ** -0.5) - 1).abs().max()) < 0.02 and float(o[1].abs().max()) < 1e-20


# ------------------------------------------------------------------ feed-forward
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", DTYPES)
@pytest.mark.parametrize("M,N,K", [(1, 15, 20), (19, 128, 64), (70, 17, 33), (300, 320, 128), (128, 20000, 64)])
def test_epilogues(device, fmt, M, N, K):
    h, w, b = gen(M, K, seed=1).to(dt(fmt)), gen(N, K, seed=2, std=K ** -0.5).to(dt(fmt)), gen(N, seed=3)
    y, W = h.double() @ w.double().t(), QuantWeight(fmt, N, K, w.to(device))
    a, tol = mx.act_of(h.to(device), fmt), 1e-5 if fmt == "fp32" else 6e-3
    close(ops.linear(a, W, relu2=True), torch.relu(y) ** 2, tol)
    close(ops.linear(a, W, sigmoid=(b.to(device), -0.3), out_f32=True), -0.3 * lo.sigmoid(y + b.double()), 1e-5 if fmt == "fp32" else 2e-5)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("E,k", [(6, 2), (40, 8), (1, 1), (64, 6), (3, 3), (130, 5)])
def test_router(device, E, k):
    z = gen(30, E, seed=1, std=2.0)
    z[3] *= 40
    z[4] = 0.5                                                           # all equal: the lowest ids
    wide = torch.cat([torch.full((30, 3), 99.0), z, torch.full((30, 2), 99.0)], 1).to(device)[:, 3:3 + E]
    w, idx = moe_ops.route(wide, moe_ops.RouterSpec(E, k, router="softmax", ffn_act="relu2"))
    for t in range(30):
        ids, want = lo.route(z[t].double(), k)
        got = dict(zip(idx[t].tolist(), w[t].tolist()))
        assert sorted(got) == sorted(ids), t
        assert max(abs(got[e] - float(x)) for e, x in zip(ids, want)) < 2e-6


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", DTYPES)
@pytest.mark.parametrize("T,W,E,top,ff,shared", [(1, 64, 6, 2, 64, 40), (50, 100, 5, 2, 18, 26), (50, 96, 9, 4, 40, None), (300, 128, 4, 1, 96, 64), (150, 44, 3, 3, 10, 12)])
def test_mixture_of_experts(device, fmt, T, W, E, top, ff, shared):
    """Stacked, padded squared-ReLU experts beside a shared one, through the stream's sum."""
    from metrale_inference_alpha_b200.models.canon import relu2_moe
    from metrale_inference_alpha_b200.models.decoder import Decoder
    from metrale_inference_alpha_b200.weights.loader import Loader
    mlp = lc.moe(E, top, ff, shared)
    cfg = lc.config([lc.delta(1, 1, 8, 8, 2, mlp)], W)
    t = lc.weights(cfg, seed=4, calm=True)
    m = {k[len("l0.mlp."):]: v.double() for k, v in t.items() if k.startswith("l0.mlp.")}

    class Source:
        has, get, names = (lambda s, n: n in t), (lambda s, n: t[n]), (lambda s: list(t))

    mc = lc.model_config(cfg, fmt)
    mw = Loader(mc, Source(), torch.device(device), 0, 1, 0, 1).load()
    h = gen(T, W, seed=5)
    h[:, 0] = 2.0
    h = h.to(dt(fmt))
    out = relu2_moe(Decoder(mc, mw, device=device), mx.act_of(h.to(device), fmt), mw.layers[0].ffn)
    one = mx.RmsNorm(torch.ones(W, dtype=torch.bfloat16, device=device), 1e-5)
    got = canon.stream_canon(torch.zeros(T, W, device=device), fmt, pending=out, norm=one)[0]
    close(got, lo.unit_rms(lo.mixture(h.double(), m, mlp), 1e-5), 2e-5 if fmt == "fp32" else 2e-2)


# ------------------------------------------------------------------ whole models
_ORACLE = {}


def oracle(name, n, seed=0, calm=False):
    """(tokens, logits [n, vocab]) of one sequence of a configuration, computed once."""
    key = name, n, seed, calm
    if key not in _ORACLE:
        cfg = lc.CONFIGS[name]
        toks = lc.tokens(cfg, n, seed)
        _ORACLE[key] = toks, lo.forward(cfg, lc.weights(cfg, calm=calm), toks)
    return _ORACLE[key]


def replay(tmp_path, name, dtype, device, max_tokens=192, **kw):
    """A bf16 model has routers without close calls (rounding would decide those)."""
    d = tmp_path / name
    path = str(d) if d.exists() else lc.checkpoint(lc.CONFIGS[name], lc.weights(lc.CONFIGS[name], calm=dtype == "bf16"), d)
    return TraceReplay(path, dtype, max_tokens, device, **kw)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(lc.CONFIGS))
def test_model_whole_portions_and_decoding(tmp_path, device, dtype, name):
    """A prompt at once, in portions down to two tokens, and token by token, all through one engine (so pages and slots are
    used again): each against the plain model."""
    toks, want = oracle(name, 75, calm=dtype == "bf16")
    r = replay(tmp_path, name, dtype, device)
    for cuts in ([75], [2], [1], [33, 2, 17, 3, 1], [16, 15, 17, 1]):
        assert near(lc.feed(r, "a", toks, cuts), want, dtype), cuts
    for rid, n in (("one", 1), ("two", 2)):                             # the first tokens of a sequence
        assert near(lc.feed(r, rid, toks[:n], [n]), want[:n], dtype)
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
def test_long_decoding(tmp_path, device):
    """Windows and filters that pass over many decoded tokens (32-bit)."""
    toks, want = oracle("ragged", 150, 9)
    r = replay(tmp_path, "ragged", "fp32", device)
    assert lc.error(lc.feed(r, "x", toks, [5, 1]), want) < TOL


@pytest.mark.gpu
@pytest.mark.parametrize("name", ["wide", "tiles"])
def test_long_prompts(tmp_path, name):
    """Prompts over many tiles, windows and chunks, then single tokens."""
    toks, want = oracle(name, 260, 5, True)
    r = replay(tmp_path, name, "bf16", "cuda", max_tokens=288)
    for cuts in ([260], [150, 64, 45, 1], [255, 1]):
        assert near(lc.feed(r, "a", toks, cuts), want, "bf16"), cuts
    ops.check_status("cuda")


@pytest.mark.parametrize("device", DEVICES)
def test_wanted_rows_and_steps_without(tmp_path, device):
    toks, want = oracle("ones", 30)
    r = replay(tmp_path, "ones", "fp32", device)
    assert r.step([{"id": "q", "tokens": toks[:7], "want": []}], []) is None
    got = r.step([{"id": "q", "tokens": toks[7:20], "want": [0, 5, 12]}], [])
    assert lc.error(got, want[[7, 12, 19]]) < TOL
    assert r.step([{"id": "q", "tokens": toks[20:21], "want": []}], []) is None
    assert lc.error(r.step([{"id": "q", "tokens": toks[21:22], "want": [0]}], ["q"]), want[21:22]) < TOL


_GREEDY = {}


def greedy_reference(name, prompt, n):
    key = name, tuple(prompt), n
    if key not in _GREEDY:
        cfg, t = lc.CONFIGS[name], lc.weights(lc.CONFIGS[name])
        toks = list(prompt)
        for _ in range(n):
            toks.append(int(lo.forward(cfg, t, toks)[-1].argmax()))
        _GREEDY[key] = toks[len(prompt):]
    return _GREEDY[key]


@pytest.mark.parametrize("device", DEVICES)
def test_greedy_generation_scheduler_and_speculation(tmp_path, device):
    """generate() on a queue longer than the batch, with chunked prompts; with n-gram speculation, swapping and predicted
    outputs: the same tokens."""
    path = lc.checkpoint(lc.CONFIGS["ragged"], lc.weights(lc.CONFIGS["ragged"]), tmp_path / "m")
    prompts = [lc.tokens(lc.CONFIGS["ragged"], n, 50 + n) for n in (19, 1, 27)]
    want = [greedy_reference("ragged", p, 8) for p in prompts]
    kw = dict(model=path, device=device, dtype="fp32", max_num_seqs=2, max_model_len=96, max_prefill_tokens=13, num_kv_blocks=24)
    for extra in ({}, {"speculative": "ngram", "mtp_gate": False}, {"preempt_mode": "swap", "num_kv_blocks": 5}):
        eng = LLMEngine(EngineArgs(**{**kw, **extra}))
        outs = eng.generate(prompts, SamplingParams(max_tokens=8, temperature=0.0))
        assert [o.output_ids for o in outs] == want, extra
    guess = [w[:4] + [(w[4] + 1) % 150] + w[5:] for w in want]          # right, then wrong once, then right again
    eng = LLMEngine(EngineArgs(**kw))
    outs = eng.generate(prompts, [SamplingParams(max_tokens=8, temperature=0.0, prediction_ids=g) for g in guess])
    assert [o.output_ids for o in outs] == want
    assert any(o.accepted_draft_tokens for o in outs)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("name", ["ragged", "ones"])
def test_verify_steps_of_one_request(tmp_path, device, name):
    """A request alone whose predicted output is right, wrong, right again: every verify step has as many drafts (on the GPU
    they replay one graph), and accepts all, some or none of them."""
    path = lc.checkpoint(lc.CONFIGS[name], lc.weights(lc.CONFIGS[name]), tmp_path / "m")
    prompt = lc.tokens(lc.CONFIGS[name], 7, 3)
    want = greedy_reference(name, prompt, 24)
    guess = [(w + 1) % 150 if i in (5, 6, 13) else w for i, w in enumerate(want)]
    eng = LLMEngine(EngineArgs(model=path, device=device, dtype="fp32", max_num_seqs=2, max_model_len=96, num_kv_blocks=24))
    for _ in range(2):
        out = eng.generate([prompt], SamplingParams(max_tokens=24, temperature=0.0, prediction_ids=guess))[0]
        assert out.output_ids == want and out.accepted_draft_tokens > 8
    assert device == "cpu" or any(k[0] == "verify" for k in eng.runner.graphs)


@pytest.mark.parametrize("device", DEVICES)
def test_prefix_cache(tmp_path, device):
    path = lc.checkpoint(lc.CONFIGS["ragged"], lc.weights(lc.CONFIGS["ragged"]), tmp_path / "m")
    eng = LLMEngine(EngineArgs(model=path, device=device, dtype="fp32", max_num_seqs=2, max_model_len=400, num_kv_blocks=80))
    p = lc.tokens(lc.CONFIGS["ragged"], 300, 5)
    sp = SamplingParams(max_tokens=5, temperature=0.0)
    a, b = (eng.generate([p], sp)[0] for _ in range(2))
    assert a.output_ids == b.output_ids and b.cached_tokens >= 256


def test_sampled_rows_take_the_models_distribution(tmp_path):
    path = lc.checkpoint(lc.CONFIGS["ones"], lc.weights(lc.CONFIGS["ones"]), tmp_path / "m")
    toks, want = oracle("ones", 30)
    eng = LLMEngine(EngineArgs(model=path, device="cpu", dtype="fp32", max_num_seqs=8, max_model_len=64, num_kv_blocks=64))
    top = set(want[-1].topk(3).indices.tolist())
    outs = eng.generate([toks] * 8, [SamplingParams(max_tokens=1, temperature=1.0, top_k=3, seed=s) for s in range(8)])
    assert {o.output_ids[0] for o in outs} <= top


# ------------------------------------------------------------------ configuration, weights, command line
def test_configuration_and_checkpoint(tmp_path):
    cfg = lc.CONFIGS["ragged"]
    c = from_hf_config(json.loads(json.dumps(cfg)))
    assert c.arch == "ledinex" and c.layer_types == ["delta", "twin", "twin", "delta", "twin"] and c.attention_layers() == [1, 2, 4]
    assert c.ffn_types == ["moe", "moe", "moe", "none", "none"] and c.canon_taps == 4
    assert c.scaled(weight_format="fp32").kv_layer_dims() == [(1, 22, 30), (2, 36, 36), (1, 14, 14)]
    assert type(c).from_json(c.to_json()).to_json() == c.to_json()
    from metrale_inference_alpha_b200.weights.checkpoint import open_checkpoint
    from metrale_inference_alpha_b200.weights.preflight import preflight
    t = lc.weights(cfg)
    c2, src = open_checkpoint(lc.checkpoint(cfg, t, tmp_path / "ok"))
    assert preflight(c2, src, check_shapes=False).ok
    del t["l2.mix.right.a.b"]
    c3, src = open_checkpoint(lc.checkpoint(cfg, t, tmp_path / "bad"))
    assert preflight(c3, src, check_shapes=False).missing == ["l2.mix.right.a.b"]

    def broken(change, match):
        bad = json.loads(json.dumps(cfg))
        change(bad)
        with pytest.raises(ValueError, match=match):
            from_ledinex_config(bad)

    broken(lambda b: b["layers"][0].update(type="other"), "unknown mixer")
    broken(lambda b: b["layers"][0]["mlp"].update(kind="dense"), "unknown feed-forward")
    broken(lambda b: b["layers"][0]["mixer"].update(heads=4), "does not serve")
    broken(lambda b: b["layers"][1]["mixer"]["left"]["rot"].update(dims=24), "do not fit")
    broken(lambda b: b["layers"][1]["mixer"]["right"]["decay"].pop(), "do not fit")
    broken(lambda b: b["layers"][2]["mixer"]["left"]["mask"].update(size=0), "window")
    broken(lambda b: b["layers"][2]["mixer"]["left"].update(vdim=20), "have their size")
    broken(lambda b: b["layers"][0]["mlp"]["router"].update(top=7), "experts per token")
    broken(lambda b: b["canon"].update(taps=0), "taps")


def test_state_rows_hold_every_window():
    cfg = lc.model_config(lc.CONFIGS["ragged"])
    eng = LLMEngine(EngineArgs(model=cfg, max_num_seqs=2, max_model_len=64, num_kv_blocks=16))
    W, C = 100, 2 * 3 * 18 + 6 * 22
    assert [t.shape[1] for t in eng.runner.pool.conv] == [6 * W + C, 6 * W, 6 * W, 3 * W + 4 * (2 * 3 * 10 + 3 * 6), 3 * W]
    assert [tuple(t.shape[1:]) for t in eng.runner.pool.ssm] == [(6, 18, 22), (3, 20, 26), (5, 28, 28), (3, 10, 6), (1, 10, 10)]


def test_unserved_combinations_are_refused():
    with pytest.raises(ValueError):
        LLMEngine(EngineArgs(model="tiny-ledinex", dtype="int8", max_model_len=64, num_kv_blocks=16))
    for kw in (dict(kv_cache_dtype="fp8"), dict(speculative="dflash"), dict(speculative="mtp"), dict(expert_arena_slots=4)):
        with pytest.raises(NotImplementedError):
            LLMEngine(EngineArgs(model="tiny-ledinex", max_model_len=64, num_kv_blocks=16, **kw))


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
def test_preset_runs_from_synthetic_weights(device, dtype):
    eng = LLMEngine(EngineArgs(model=preset("tiny-ledinex"), device=device, dtype=dtype, max_num_seqs=2, max_model_len=64, num_kv_blocks=16))
    outs = eng.generate([[1, 2, 3], [9, 8, 7, 6]], SamplingParams(max_tokens=4))
    assert all(len(o.output_ids) == 4 for o in outs)
    if device != "cpu":
        ops.check_status(device)


def test_replay_command(tmp_path, capsys):
    import numpy as np
    from metrale_inference_alpha_b200.server import cli
    cfg = lc.CONFIGS["ones"]
    path = lc.checkpoint(cfg, lc.weights(cfg), tmp_path / "m")
    toks, want = oracle("ones", 30)
    ns = cli.build_parser().parse_args(["replay", "--model", path, "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "64",
                                        "--device", "cpu"])
    from metrale_inference_alpha_b200.engine.replay import run
    lines = [json.dumps({"step": 0, "entries": [{"id": "a", "tokens": toks[:9], "want": []}], "end": []}),
             json.dumps({"step": 1, "entries": [{"id": "a", "tokens": toks[9:30], "want": [20]}], "end": ["a"]})]
    assert run(ns, lines) == 0
    assert [x for x in capsys.readouterr().out.splitlines() if x.startswith("done")] == ["done 0", "done 1"]
    got = torch.from_numpy(np.fromfile(tmp_path / "1.f32", dtype="<f4")).view(1, -1)
    assert lc.error(got, want[29:30]) < 1e-5 and not (tmp_path / "0.f32").exists()
