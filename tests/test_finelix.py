"""The Finelix decoder against a plain restatement (finelix_oracle.py): every mechanism alone, then whole models
through the engine's own entry points. The CPU runs cover the engine's host logic and its op restatements, the GPU
runs the kernels."""
import json

import pytest
import torch

import finelix_cases as fc
import finelix_oracle as fo
from metrale_inference_alpha_b200 import ops
from metrale_inference_alpha_b200.config.model_config import from_finelix_config, from_hf_config, preset
from metrale_inference_alpha_b200.engine.llm_engine import EngineArgs, LLMEngine
from metrale_inference_alpha_b200.engine.replay import TraceReplay
from metrale_inference_alpha_b200.ops import QuantWeight, latent as lt, mixers as mx, moe as moe_ops, reference as ref
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


# ------------------------------------------------------------------ the stream
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", DTYPES)
@pytest.mark.parametrize("W", [37, 96, 2560, 5000])
def test_stream_add_and_norm(device, fmt, W):
    T, K = 11, 3
    x, y = gen(T, W, seed=1, std=3.0), gen(T, W, seed=2).to(dt(fmt))
    pre = mx.RmsNorm(b16(gen(W, seed=5)).to(device), 1e-2)
    ye, pw = gen(T * K, W + 4, seed=3), gen(T, K, seed=4).abs()
    place = torch.randperm(T * K, generator=torch.Generator().manual_seed(1)).int()
    place[4] = place[20] = -1                                        # pairs that no row stands for
    esum = torch.zeros(T, W, dtype=torch.float64)
    for t in range(T):
        for j in range(K):
            if place[t * K + j] >= 0:
                esum[t] += pw[t, j].double() * ye[int(place[t * K + j]), :W].double()
    routed = mx.Routed(esum.float(), None, None) if device == "cpu" else mx.Routed(ye.to(device), place.to(device), pw.to(device))
    tol = 1e-5 if fmt == "fp32" else 6e-3
    w = pre.w.cpu().double()
    for yy, rr in ((None, None), (y, None), (y, routed), (None, routed)):
        want = x.double() + (0 if yy is None else y.double()) + (0 if rr is None else esum)
        kw = dict(y=None if yy is None else y.to(device), routed=rr)
        x1, h = mx.stream_rms(x.to(device), fmt, pre=pre, **kw)
        close(x1, want, 1e-6)                                        # the stream itself is 32-bit in both formats
        close(h, fo.rms_norm(want, w, 1e-2), tol)
        assert mx.stream_rms(x.to(device), fmt, **kw)[1] is None
        wide = torch.full((T, W + 8), 7.0, dtype=dt(fmt), device=device)
        mx.stream_rms(x.to(device), fmt, raw=True, out=wide[:, 8:], **kw)
        close(wide[:, 8:], want, tol)
        assert bool((wide[:, :8] == 7.0).all())


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", DTYPES)
@pytest.mark.parametrize("W", [52, 128])
def test_entry_of_a_pass(device, fmt, W):
    """What a looped range starts from: the projection of [stream | embedding output] and the pass's own vector, with
    the last sublayer's output still pending."""
    from metrale_inference_alpha_b200.models.stream import ResidualStream
    T = 9
    table, ids = b16(gen(30, W, seed=1)), torch.tensor([3, 29, 0, 7, 7, 1, 2, 11, 5], dtype=torch.int32)
    pair = torch.zeros(T, 2 * W, dtype=dt(fmt), device=device)
    x0 = mx.embed_scaled(ids.to(device), table.to(device), 2.5, pair[:, W:])
    want0 = table[ids.long()].double() * 2.5
    close(x0, want0, 1e-6)
    w, step = gen(W, 2 * W, seed=2, std=W ** -0.5).to(dt(fmt)), gen(2, W, seed=3)
    s = ResidualStream(x0, fmt, pair)
    t = {"loop.in": w.double(), "loop.step": step.double()}
    want = want0
    for p in range(2):
        y = gen(T, W, seed=4 + p).to(dt(fmt))
        s.add(y.to(device))
        s.enter_pass(QuantWeight(fmt, W, 2 * W, w.to(device)), step[p].to(device))
        want = fo.enter_pass(want + y.double(), want0, t, p)
        close(s.resolve(), want, 1e-5 if fmt == "fp32" else 1e-2)


# ------------------------------------------------------------------ latent attention
# heads, dim, rot, vdim, latent: the 64-, 128- and 256-wide tiles, the 576-wide kernels (with and without padding), past them
LAT = {"t64": (4, 16, 8, 24, 40), "t128": (3, 20, 32, 22, 96), "t256": (2, 36, 16, 30, 200), "t256 full": (5, 8, 32, 16, 224),
       "mla": (3, 24, 16, 28, 264), "mla full": (17, 16, 64, 16, 512), "past": (2, 12, 66, 10, 270), "odd": (3, 7, 2, 5, 11)}


def run_latent(device, fmt, x, w, dims, scale, cuts, kernel="auto", base=50.0, block=16, q_rank=12, eps=1e-4):
    """x [n, q_rank + L + R] of one sequence, fed in portions through the paged cache beside a short second sequence;
    w: the layer's remaining tensors. Returns [n, H, vdim]."""
    H, dim, R, dv, L = dims
    n = x.shape[0]
    lay = lt.latent_row(L, R, fmt)
    nb = (n + block - 1) // block
    cache = torch.full((2 * nb + 8, block, 1, lay.row), float("nan"), dtype=dt(fmt), device=device)   # unwritten slots must not matter
    pages = list(range(nb + 4, 4, -1))                                # descending: pages are not in order
    cos, sin = ref.rope_tables(4096, R, base, device=device)
    dev = {k: v.to(device) for k, v in w.items()}
    outs, at, i = [], 0, 0
    while at < n:
        m = min(cuts[min(i, len(cuts) - 1)], n - at)
        o1 = min(at, 15)                                              # the neighbour's position this step
        b = fc.batch([m, 1], [at + m, o1 + 1], device=device, block=block, pages=[pages[:(at + m + block - 1) // block], [1]])
        xx = torch.cat([x[at:at + m], x[o1:o1 + 1]]).to(device)
        cq = lt.norm_and_cache(xx, fmt, q_rank=q_rank, L=L, R=R, q_w=dev["dq.norm"], kv_w=dev["dkv.norm"], eps=eps, cos=cos, sin=sin,
                               positions=b.positions, slots=b.slot_mapping, cache=cache, lay=lay)
        q = ops.linear(mx.act_of(cq, fmt), QuantWeight(fmt, H * (dim + R), q_rank, dev["uq"]))
        qq = lt.absorbed_query(q, dev["uk"].view(H, dim, L), fmt, H=H, dim=dim, R=R, cos=cos, sin=sin, positions=b.positions, lay=lay)
        wide = torch.full((m + 1, H * dv + 8), 5.0, dtype=dt(fmt), device=device)
        lt.attention(qq, cache, b, dev["uv"].view(H, dv, L), scale, fmt, lay, wide[:, 8:], kernel=kernel)
        assert bool((wide[:, :8] == 5.0).all())
        outs.append(wide[:m, 8:])
        at, i = at + m, i + 1
    return torch.cat(outs).view(n, H, dv).float().cpu()


def plain_latent(x, w, dims, scale, q_rank=12, eps=1e-4, base=50.0):
    """The oracle's layer, its input projections and output projection replaced by the identity."""
    H, dim, R, dv, L = dims
    d = {k: v.double() for k, v in w.items()}
    n = x.shape[1]
    d["dq"], d["dkv"] = torch.eye(n, dtype=torch.float64)[:q_rank], torch.eye(n, dtype=torch.float64)[q_rank:]
    d["o"] = torch.eye(H * dv, dtype=torch.float64)
    m = {"heads": H, "dim": dim, "rot_dim": R, "vdim": dv, "kv_rank": L, "scale": scale, "rot": {"base": base}}
    return fo.latent_attention(x.double(), d, m, eps).view(x.shape[0], H, dv)


def latent_inputs(dims, n, fmt, far=(), seed=0, q_rank=12):
    H, dim, R, dv, L = dims
    x = gen(n, q_rank + L + R, seed=seed)
    for i, j in far:                                                  # key j stands out for query i, by one rotated pair of its own
        x[i, :q_rank] = 0
        x[i, 0] = 4.0
        x[j, q_rank + L + R // 2 - 1] = x[j, q_rank + L + R - 1] = 12.0
    w = {"dq.norm": gen(q_rank, seed=seed + 1, std=0.2, mean=1.0), "dkv.norm": gen(L, seed=seed + 2, std=0.2, mean=1.0),
         "uq": gen(H * (dim + R), q_rank, seed=seed + 3, std=0.5), "uk": gen(H * dim, L, seed=seed + 4, std=L ** -0.5),
         "uv": gen(H * dv, L, seed=seed + 5, std=L ** -0.5)}
    return x, {k: b16(v).to(torch.bfloat16 if "norm" in k else dt(fmt)) for k, v in w.items()}


FAR = ((0, 0), (15, 0), (16, 15), (17, 16), (32, 31), (33, 32), (47, 1), (48, 0), (63, 48), (69, 0), (69, 16))


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", DTYPES)
@pytest.mark.parametrize("name", list(LAT))
@pytest.mark.parametrize("cuts", [[70], [33, 1], [2], [31, 17, 2, 1]])
def test_latent_attention(device, fmt, name, cuts):
    dims = LAT[name]
    x, w = latent_inputs(dims, 70, fmt, FAR)
    want = plain_latent(x, w, dims, 0.21)
    close(run_latent(device, fmt, x, w, dims, 0.21, cuts), want, 2e-5 if fmt == "fp32" else 2.5e-2)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", DTYPES)
def test_latent_attention_reads_single_keys(device, fmt):
    """With scores far apart a query returns one key's value: the right position, before and behind page borders."""
    dims = (2, 8, 4, 6, 20)
    H, dim, R, dv, L = dims
    n = 50
    x, w = latent_inputs(dims, n, fmt, seed=3)
    w["uq"].zero_()
    w["uq"].view(H, dim + R, 12)[:, 0, 0] = 8.0                       # the unrotated query: its first coordinate, large
    w["uk"].zero_()
    w["uk"].view(H, dim, L)[:, 0, 0] = 1.0                            # the key's first coordinate is the latent's
    x[:, 12:12 + L] = gen(n, L, seed=9, std=0.05)
    for j in (0, 15, 16, 31, 32, 49):
        xj = x.clone()
        xj[j, 12] = 9.0
        got = run_latent(device, fmt, xj, w, dims, 3.0, [17, 16, 1])
        want = plain_latent(xj, w, dims, 3.0)
        close(got, want, 1e-4 if fmt == "fp32" else 2.5e-2)
        c = fo.rms_norm(xj[j, 12:12 + L].double(), w["dkv.norm"].double(), 1e-4)
        v = (w["uv"].double() @ c).view(H, dv)
        seen = [i for i in range(j, n) if float(xj[i, 0]) > 0.8]       # queries of the right sign that see it
        assert seen or j == 49
        for i in seen:
            close(got[i], v, 3e-2)


@pytest.mark.gpu
@pytest.mark.parametrize("kernel,name", [("mma", "t64"), ("mma", "t128"), ("auto", "t256"), ("simt", "t256"), ("mma", "mla"), ("mma", "mla full"), ("auto", "mla"),
                                         ("tc", "mla"), ("tc", "mla full"), ("auto", "mla full"), ("simt", "mla"), ("auto", "past")])
def test_latent_attention_kernels_long(kernel, name):
    """Long contexts: tiles of every kernel, several partitions of the context (decode past 256, 512 and 1024 keys),
    far keys. Queries and cache rows are rounded to bf16 on both sides, so only the attention itself is compared."""
    H, dim, R, dv, L = LAT[name]
    lay, n, fmt = lt.latent_row(L, R, "bf16"), 1250, "bf16"
    q, row = torch.zeros(n, H, lay.row), torch.zeros(n, lay.row)
    for t, k in ((q, 1), (row, 2)):
        t[..., :L], t[..., lay.rope_at:lay.rope_at + R] = gen(*t.shape[:-1], L, seed=k), gen(*t.shape[:-1], R, seed=k + 5)
    q *= 0.5
    for i, j in ((700, 0), (1199, 511), (1210, 512), (1211, 1023), (1212, 1024), (1240, 3), (1248, 255), (1249, 1248)):
        q[i] = 0
        q[i, :, :4], q[i, :, lay.rope_at] = 3.0, 2.0
        row[j, :4] += 2.0
        row[j, lay.rope_at] += 2.0
    q, row = b16(q), b16(row)
    scale = 2.0 * (L + R) ** -0.5
    s = torch.einsum("ihd,jd->hij", q.double(), row.double()) * scale
    s.masked_fill_(torch.ones(n, n, dtype=torch.bool).triu(1), float("-inf"))
    o = torch.einsum("hij,jl->ihl", torch.softmax(s, -1), row[:, :L].double())
    uv = gen(H, dv, L, seed=8, std=L ** -0.5)
    want = torch.einsum("ihl,hvl->ihv", o, b16(uv).double())
    nb = n // 16 + 2
    cache = torch.full((nb + 9, 16, 1, lay.row), float("nan"), dtype=torch.bfloat16)
    pages = list(range(nb + 7, 7, -1))
    idx = torch.tensor([pages[i // 16] * 16 + i % 16 for i in range(n)])
    cache.view(-1, lay.row)[idx] = row
    cache, qd, uvd = cache.cuda(), q.cuda(), b16(uv).cuda()
    cuts = [(i, i + 1) for i in range(1190, 1250)] + [(0, 256), (512, 513), (256, 257), (257, 258), (0, 1190), (1000, 1007), (630, 800)]
    got, ref_rows = [], []
    for lo, hi in cuts:
        b = fc.batch([hi - lo], [hi], pages=[pages[:(hi + 15) // 16]], device="cuda")
        out = torch.empty(hi - lo, H * dv, dtype=torch.bfloat16, device="cuda")
        lt.attention(qd[lo:hi].contiguous(), cache, b, uvd, scale, fmt, lay, out, kernel=kernel)
        got.append(out.view(-1, H, dv).cpu())
        ref_rows.append(want[lo:hi])
    close(torch.cat(got), torch.cat(ref_rows), 1e-2)
    ops.check_status("cuda")


@pytest.mark.gpu
@pytest.mark.parametrize("impl", [1, 2])
def test_latent_weights_keep_32_bits(impl):
    """Softmax weights enter the product with the values as two bf16 terms: the error is that of 16 bits, not of 8."""
    from metrale_inference_alpha_b200.ops import mla_cuda
    H, n = 32, 300
    q, row = b16(gen(1, H, 576, seed=1, std=0.2)), b16(gen(n, 576, seed=2))
    s = torch.einsum("hd,jd->hj", q[0].double(), row.double()) * 0.05
    want = torch.softmax(s, -1) @ row[:, :512].double()
    cache = torch.zeros(n // 16 + 2, 16, 1, 576, dtype=torch.bfloat16)
    cache.view(-1, 576)[16:16 + n] = row
    b = fc.batch([1], [n], pages=[list(range(1, n // 16 + 2))], device="cuda")
    err = []
    for split in (False, True):
        o = mla_cuda.mla_attention(q.cuda(), cache.cuda(), b.block_table, b.q_start, b.q_len, b.ctx_len, max_q_len=1, max_ctx=n, scale=0.05,
                                   impl=impl, split_p=split)
        err.append(float((o[0].double().cpu() - want).abs().max()))
    assert err[1] < 3e-5 and err[1] < 0.1 * err[0], err


# ------------------------------------------------------------------ gated linear attention
def plain_gla(q, k, v, w):
    """q, k [n, H, dk], v [n, H, dv], w [n, H, dk] decays. Outputs [n, H, dv] and the final state."""
    q, k, v, w = (t.double() for t in (q, k, v, w))
    n, H, dk = q.shape
    out, S = torch.zeros(n, H, v.shape[2], dtype=torch.float64), torch.zeros(H, dk, v.shape[2], dtype=torch.float64)
    for t in range(n):
        S = w[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out, S


def run_gla(device, fmt, qkv, a1, a2, bias, c, dims, cuts, slots, kernel="auto"):
    """Several sequences fed in portions (cuts[i][s] rows of sequence s in step i; 0 = left out); per-sequence outputs
    and the state pool. The decays come from their low-rank projection; every step is repeated as a commit pass."""
    H, dk, dv = dims
    state = torch.full((max(slots) + 2, H, dk, dv), 9.0, device=device)       # stale content of reused slots
    S, at, outs = len(qkv), [0] * len(qkv), [[] for _ in qkv]
    a2q = QuantWeight("bf16", a2.shape[0], a2.shape[1], a2.to(device)) if a2.shape[1] % 8 == 0 and fmt == "bf16" else None
    for step in cuts:
        live = [s for s in range(S) if step[s]]
        b = fc.batch([step[s] for s in live], [at[s] + step[s] for s in live], [slots[s] for s in live], device=device)
        cat = lambda f: torch.cat([f(s)[at[s]:at[s] + step[s]] for s in live]).to(device)
        rows = torch.cat([cat(lambda s, i=i: qkv[s][i].reshape(qkv[s][i].shape[0], -1)) for i in range(3)] + [cat(lambda s: a1[s])], 1)
        rows = torch.cat([rows, rows.new_zeros(rows.shape[0], -rows.shape[1] % 8)], 1).to(dt(fmt))
        q, k, v = rows[:, :H * dk], rows[:, H * dk:2 * H * dk], rows[:, 2 * H * dk:2 * H * dk + H * dv]
        lr = mx.LowRankDecay(rows[:, 2 * H * dk + H * dv:][:, :a2.shape[1]], a2.to(device), bias.to(device), c, a2q)
        kw = dict(heads=H, dk=dk, dv=dv, fmt=fmt, kernel=kernel)
        keep = state.clone()
        mx.linear_attention(q, k, v, state, b, write_state=False, low_rank=lr, **kw)
        assert torch.equal(keep, state)
        y = mx.linear_attention(q, k, v, state, b, low_rank=lr, **kw)
        again = keep.clone()
        mx.linear_attention(q, k, v, again, b, write_out=False, log_w=lr.log(), **kw)
        assert float((again - state).abs().max()) <= 1e-4 * float(state.abs().max())
        r = 0
        for s in live:
            outs[s].append(y[r:r + step[s]].view(step[s], H, dv).cpu())
            r += step[s]
            at[s] += step[s]
    return [torch.cat(o) for o in outs], state.cpu()


def gla_inputs(fmt, dims, lens, rank, far=()):
    H, dk, dv = dims
    qkv = [[gen(n, H, d, seed=10 * i + n).to(dt(fmt)) for i, d in enumerate((dk, dk, dv))] for n in lens]
    q, k, _ = qkv[0]
    for i, j in far:                                                          # one key among many
        k[j] *= 6
        q[i] = k[j]
    a1 = [gen(n, rank, seed=50 + n).to(dt(fmt)) for n in lens]
    a2, bias = b16(gen(H * dk, rank, seed=6, std=0.5)), gen(H * dk, seed=7, std=2.0, mean=2.0)
    bias.view(H, dk)[:, 0], bias.view(H, dk)[:, 1] = 40.0, -60.0              # channels that keep everything, and nothing
    a2.view(H, dk, rank)[:, :2] = 0
    return qkv, a1, a2, bias


def gla_decays(a1, a2, bias, c, H):
    z = a1.double() @ a2.double().T + bias.double()
    return torch.sigmoid(z).pow(c).view(a1.shape[0], H, -1)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", DTYPES)
@pytest.mark.parametrize("dims,rank,tau", [((3, 20, 28), 14, 16.0), ((2, 64, 64), 16, 16.0), ((1, 16, 7), 3, 1.0), ((2, 40, 96), 8, 4.0),
                                           ((1, 128, 128), 16, 16.0), ((2, 200, 36), 24, 9.0)])
def test_gated_linear_attention(device, fmt, dims, rank, tau):
    """Ragged batches in portions, single rows among them (decays computed inside the decode kernel), fresh and reused
    slots, a far key that must still be read at the end, decays that forget at once."""
    lens = (150, 83, 1)
    qkv, a1, a2, bias = gla_inputs(fmt, dims, lens, rank, ((149, 3), (64, 63), (65, 63), (2, 0)))
    cuts = [(64, 2, 1), (1, 1, 0), (1, 0, 0), (2, 64, 0), (70, 1, 0), (12, 15, 0)]
    outs, state = run_gla(device, fmt, qkv, a1, a2, bias, 1 / tau, dims, cuts, [3, 1, 2])
    whole, state2 = run_gla(device, fmt, qkv, a1, a2, bias, 1 / tau, dims, [lens], [1, 2, 3])
    for s, n in enumerate(lens):
        want, S = plain_gla(*qkv[s], gla_decays(a1[s], a2, bias, 1 / tau, dims[0]))
        for got in (outs[s], whole[s]):
            err = (got.double() - want).abs().amax((1, 2)) / want.abs().amax((1, 2)).clamp(min=0.05 * float(want.abs().max()))
            assert float(err.max()) < 2e-4, (s, float(err.max()), int(err.argmax()))
        close(state[[3, 1, 2][s]], S, 2e-4)
        close(state2[[1, 2, 3][s]], S, 2e-4)


@pytest.mark.gpu
@pytest.mark.parametrize("dims", [(2, 64, 64), (3, 64, 128), (2, 128, 64), (5, 128, 128)])
@pytest.mark.parametrize("tau", [16.0, 0.5])
def test_chunked_gated_linear_attention(dims, tau):
    """Chunk and sub-block edges in every position, ragged batches, a state handed from chunk to chunk and portion to
    portion, decays down to nothing inside a chunk."""
    lens = (333, 64, 65, 1, 16, 200)
    far = ((64, 63), (63, 62), (128, 127), (129, 64), (80, 79), (79, 64), (17, 15), (332, 63), (331, 331), (200, 0), (16, 15), (15, 15))
    qkv, a1, a2, bias = gla_inputs("bf16", dims, lens, 16, far)
    cuts = [(100, 64, 65, 1, 0, 0), (64, 0, 0, 0, 16, 63), (1, 0, 0, 0, 0, 0), (168, 0, 0, 0, 0, 137)]
    slots = [3, 1, 2, 6, 5, 4]
    outs, state = run_gla("cuda", "bf16", qkv, a1, a2, bias, 1 / tau, dims, cuts, slots, kernel="chunked")
    for s, n in enumerate(lens):
        want, S = plain_gla(*qkv[s], gla_decays(a1[s], a2, bias, 1 / tau, dims[0]))
        err = (outs[s].double() - want).abs().amax(2) / want.abs().amax(2).clamp(min=0.02 * float(want.abs().max()))
        assert float(err.max()) < 4e-4, (s, float(err.max()), int(err.amax(1).argmax()))
        close(state[slots[s]], S, 2e-4)
    ops.check_status("cuda")


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", DTYPES)
@pytest.mark.parametrize("T,rank", [(5, 14), (300, 16), (300, 9)])
def test_low_rank_decay(device, fmt, T, rank):
    """Logarithms of decays from far below zero to just under it, relative accuracy on both sides."""
    a1, a2 = gen(T, rank, seed=1, std=2.0).to(dt(fmt)), b16(gen(136, rank, seed=2, std=3.0))
    bias = gen(136, seed=3, std=8.0)
    q = QuantWeight("bf16", 136, rank, a2.to(device)) if rank % 8 == 0 and fmt == "bf16" else None
    wide = torch.cat([torch.full((T, 8), 9.0).to(dt(fmt)), a1, torch.full((T, 32 - rank), 9.0).to(dt(fmt))], 1).to(device)     # a column range
    got = mx.LowRankDecay(wide[:, 8:8 + rank], a2.to(device), bias.to(device), 1 / 16.0, q).log()
    z = a1.double() @ a2.double().T + bias.double()
    want = (z.clamp(max=0) - torch.log1p(torch.exp(-z.abs()))) / 16.0
    dz = 2e-6 * (a1.double().abs() @ a2.double().T.abs() + bias.double().abs())          # what 32-bit sums may be off by
    assert bool(((got.double().cpu() - want).abs() <= 2e-6 * want.abs() + dz * torch.sigmoid(-z) / 16.0 + 1e-30).all())


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", DTYPES)
@pytest.mark.parametrize("n", [1, 3])
def test_head_norm_with_the_query_factor(device, fmt, n):
    """The factor dim^-1/2 on the queries stands in front of the head norm: an eps dim times the size. Outputs small
    enough that eps matters."""
    H, dk, dv, eps = 2, 20, 24, 1e-3
    T = 3 * n
    q, k, v = (gen(T, H * d, seed=s, std=0.3).to(dt(fmt)).to(device) for d, s in ((dk, 1), (dk, 2), (dv, 3)))
    lr = mx.LowRankDecay(gen(T, 6, seed=4).to(dt(fmt)).to(device), b16(gen(H * dk, 6, seed=5)).to(device), gen(H * dk, seed=6).to(device), 0.25)
    gate, w = gen(T, H * dv, seed=7).to(dt(fmt)).to(device), b16(gen(dv, seed=8)).repeat(H).to(device)
    b = fc.batch([n] * 3, [n, n, n], [2, 1, 3], device=device)
    out = torch.full((T, H * dv + 8), 3.0, dtype=dt(fmt), device=device)
    mx.linear_attention(q, k, v, torch.zeros(4, H, dk, dv, device=device), b, heads=H, dk=dk, dv=dv, fmt=fmt, low_rank=lr,
                        norm=dict(w=w, gate=gate, gate_act="silu", eps=eps * dk, scale=1.0, out=out[:, 8:]))
    cpu = lambda t: t.cpu().double()
    decay = gla_decays(lr.a1.cpu(), lr.a2.cpu(), lr.bias.cpu(), 0.25, H)
    for s in range(3):
        r = slice(s * n, (s + 1) * n)
        o, _ = plain_gla(cpu(q[r]).view(n, H, dk) * dk ** -0.5, cpu(k[r]).view(n, H, dk), cpu(v[r]).view(n, H, dv), decay[r])
        want = fo.rms_norm(o, cpu(w[:dv]), eps).reshape(n, -1) * fo.silu(cpu(gate[r]))
        close(out[r, 8:], want, 2e-5 if fmt == "fp32" else 8e-3)
    assert bool((out[:, :8] == 3.0).all())


# ------------------------------------------------------------------ feed-forwards
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", DTYPES)
@pytest.mark.parametrize("M,N,K", [(1, 30, 20), (19, 256, 64), (70, 34, 33), (300, 640, 128), (130, 40000, 64)])
def test_linear_epilogues(device, fmt, M, N, K):
    if N > 1000 and device == "cpu":
        pytest.skip("more tiles than SMs: the persistent GEMM")
    x, w = gen(M, K, seed=1).to(dt(fmt)), (gen(N, K, seed=2) * K ** -0.5 * 3).to(dt(fmt))
    act, W = mx.act_of(x.to(device), fmt), QuantWeight(fmt, N, K, w.to(device))
    y = x.double() @ w.double().T
    tol = 1e-5 if fmt == "fp32" else 1e-2
    close(ops.linear(act, W, geglu=True), fo.gelu_tanh(y[:, 0::2]) * y[:, 1::2], tol)
    close(ops.linear(act, W, swiglu=True), fo.silu(y[:, 0::2]) * y[:, 1::2], tol)
    bias = gen(N, seed=3, std=5.0)
    close(ops.linear(act, W, out_f32=True, bias=bias.to(device)), y + bias.double(), 1e-5)
    got = ops.linear(act, W, out_f32=True, log_sigmoid=(bias.to(device), 0.3))
    close(got, -0.3 * torch.nn.functional.softplus(-(y + bias.double())), 1e-5)
    wide = torch.full((M, N // 2 + 8), 2.0, dtype=dt(fmt), device=device)                # a column range of a wider matrix
    ops.linear(act, W, geglu=True, out=wide[:, 8:])
    close(wide[:, 8:], fo.gelu_tanh(y[:, 0::2]) * y[:, 1::2], tol)
    assert bool((wide[:, :8] == 2.0).all())
    rows = torch.cat([x, x], 1).to(device)[:, K:] if K % 8 == 0 else x.to(device)        # and operands from one
    close(ops.linear(mx.act_of(rows, fmt), W), y, tol)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("E,k", [(5, 2), (40, 8), (1, 1), (64, 64 // 2)])
def test_router(device, E, k):
    """The largest biased logits, a softmax over those alone: biases that decide, far-apart logits, ties."""
    z, bias = gen(30, E, seed=1, std=2.0), gen(E, seed=2, std=2.0)
    z[3] *= 60
    z[4] = -bias                                                                         # all equal after the bias: the lowest ids
    spec = moe_ops.RouterSpec(E, k)
    wide = torch.cat([torch.full((30, 3), 99.0), z], 1).to(device)[:, 3:]                # logits are a column range
    w, idx = moe_ops.route(wide, spec, bias.to(device))
    picked = fo.route(z.double(), {"router": torch.eye(E, dtype=torch.float64), "router.b": bias.double()}, k)
    for t, (ids, want) in enumerate(picked):
        got = dict(zip(idx[t].tolist(), w[t].tolist()))
        assert sorted(got) == sorted(ids), t
        assert max(abs(got[e] - float(x)) for e, x in zip(ids, want)) < 2e-6


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", DTYPES)
@pytest.mark.parametrize("T,W,E,top,ff", [(1, 64, 6, 2, 64), (50, 100, 5, 2, 18), (50, 96, 9, 4, 40), (300, 128, 4, 1, 96), (150, 44, 3, 3, 10)])
def test_mixture_of_experts(device, fmt, T, W, E, top, ff):
    """Stacked, padded experts through the routing, the grouped products and the stream's sum: uneven loads, an expert
    that nobody takes, rows that are not whole vectors."""
    from metrale_inference_alpha_b200.weights.loader import Loader
    cfg = fc.config([fc.gla(1, 8, 8, 2.0, fc.moe(E, top, ff))], W)
    t = fc.weights(cfg, seed=4)
    if E > top:
        t["l0.mlp.router.b"][E - 1] = -50.0
    m = {k[len("l0.mlp."):]: v.double() for k, v in t.items() if k.startswith("l0.mlp.")}

    class Source:
        has, get, names = (lambda s, n: n in t), (lambda s, n: t[n]), (lambda s: list(t))

    lw = Loader(fc.model_config(cfg, fmt), Source(), torch.device(device), 0, 1, 0, 1).load().layers[0]
    h, x = gen(T, W, seed=5).to(dt(fmt)), gen(T, W, seed=6)
    from metrale_inference_alpha_b200.models.moe import routed_rows

    class Dec:
        cfg = fc.model_config(fc.config([fc.gla(1, 8, 8)], W))

    act = mx.act_of(h.to(device), fmt)
    routed = routed_rows(Dec, act, ops.linear(act, lw.ffn.router, out_f32=True), lw.ffn)
    got = mx.stream_rms(x.to(device), fmt, routed=routed)[0]
    want = fo.mixture(h.double(), m, {"router": {"top": top}})
    close(got.cpu().double() - x.double(), want, 2e-5 if fmt == "fp32" else 2e-2)


# ------------------------------------------------------------------ whole models
_ORACLE = {}


def oracle(name, n, seed=0, calm=False):
    """(tokens, logits [n, vocab]) of one sequence of a configuration, computed once."""
    key = name, n, seed, calm
    if key not in _ORACLE:
        cfg = fc.CONFIGS[name]
        toks = fc.tokens(cfg, n, seed)
        _ORACLE[key] = toks, fo.forward(cfg, fc.weights(cfg, calm=calm), toks)
    return _ORACLE[key]


def replay(tmp_path, name, dtype, device, max_tokens=192, **kw):
    """A bf16 model has routers without close calls (rounding would decide those)."""
    d = tmp_path / name
    path = str(d) if d.exists() else fc.checkpoint(fc.CONFIGS[name], fc.weights(fc.CONFIGS[name], calm=dtype == "bf16"), d)
    return TraceReplay(path, dtype, max_tokens, device, **kw)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(fc.CONFIGS))
def test_model_whole_portions_and_decoding(tmp_path, device, dtype, name):
    """A prompt at once, in portions down to two tokens, and token by token, all through one engine (so pages
    and slots are used again): each against the plain model."""
    toks, want = oracle(name, 75, calm=dtype == "bf16")
    r = replay(tmp_path, name, dtype, device)
    for cuts in ([75], [2], [1], [33, 2, 17, 3, 1], [16, 15, 17, 1]):
        assert near(fc.feed(r, "a", toks, cuts), want, dtype), cuts
    for rid, n in (("one", 1), ("two", 2)):                             # the first tokens of a sequence
        assert near(fc.feed(r, rid, toks[:n], [n]), want[:n], dtype)
    assert r.engine.scheduler.num_active == 0 and r.engine.runner.kv.allocator.num_used == 0 and r.engine.runner.pool.num_free == 4


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
def test_passes_have_caches_and_states_of_their_own(device):
    """Every pass of a looped layer owns a pool: as many as layer runs, none shared."""
    cfg = fc.model_config(fc.CONFIGS["ragged"])
    runs = cfg.layer_runs()
    assert [i for i, _ in runs] == [0, 1, 2, 3, 1, 2, 3, 4, 5] and [t for _, t in runs] == [None, 0, None, None, 1, None, None, None, None]
    eng = LLMEngine(EngineArgs(model=cfg, device=device, max_num_seqs=2, max_model_len=64, num_kv_blocks=16))
    kv, pool = eng.runner.kv, eng.runner.pool
    assert len(kv.k) == 5 and len(pool.ssm) == 4 and kv.v == [None] * 5
    assert len({t.data_ptr() for t in kv.k}) == 5 and len({t.data_ptr() for t in pool.ssm}) == 4
    assert [t.shape[-1] for t in kv.k] == [64, 64, 64, 64, 64] and pool.ssm[1].shape[1:] == (2, 36, 18)
    assert cfg.scaled(weight_format="fp32").kv_layer_dims() == [(1, 44, 0), (1, 60, 0), (1, 44, 0), (1, 60, 0), (1, 25, 0)]
    assert fc.model_config(fc.CONFIGS["linear"]).layer_runs() == [(0, None), (1, None)]
    assert [t for _, t in fc.model_config(fc.CONFIGS["ones"]).layer_runs()] == [0, None]


@pytest.mark.parametrize("device", DEVICES)
def test_long_decoding(tmp_path, device):
    """The state neither drifts nor loses anything over many single steps (32-bit)."""
    toks, want = oracle("ragged", 180, 9)
    r = replay(tmp_path, "ragged", "fp32", device)
    assert fc.error(fc.feed(r, "x", toks, [5, 1]), want) < TOL


@pytest.mark.gpu
@pytest.mark.parametrize("name", ["wide", "tiles"])
def test_long_prompts(tmp_path, name):
    """Prompts over many chunks and tiles, then single tokens: the chunked recurrence and the wide attention kernels
    inside whole models."""
    toks, want = oracle(name, 330, 5, True)
    r = replay(tmp_path, name, "bf16", "cuda", max_tokens=352)
    for cuts in ([330], [150, 129, 50, 1], [300, 1]):
        assert near(fc.feed(r, "a", toks, cuts), want, "bf16"), cuts
    ops.check_status("cuda")


@pytest.mark.parametrize("device", DEVICES)
def test_wanted_rows_and_steps_without(tmp_path, device):
    toks, want = oracle("ones", 30)
    r = replay(tmp_path, "ones", "fp32", device)
    assert r.step([{"id": "q", "tokens": toks[:7], "want": []}], []) is None
    got = r.step([{"id": "q", "tokens": toks[7:20], "want": [0, 5, 12]}], [])
    assert fc.error(got, want[[7, 12, 19]]) < TOL
    assert r.step([{"id": "q", "tokens": toks[20:21], "want": []}], []) is None
    assert fc.error(r.step([{"id": "q", "tokens": toks[21:22], "want": [0]}], ["q"]), want[21:22]) < TOL


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
    for extra in ({}, {"speculative": "ngram", "mtp_gate": False}, {"preempt_mode": "swap", "num_kv_blocks": 5}):
        eng = LLMEngine(EngineArgs(**{**kw, **extra}))
        outs = eng.generate(prompts, SamplingParams(max_tokens=12, temperature=0.0))
        assert [o.output_ids for o in outs] == want, extra
    guess = [w[:5] + [(w[5] + 1) % 150] + w[6:] for w in want]          # right, then wrong once, then right again
    eng = LLMEngine(EngineArgs(**kw))
    outs = eng.generate(prompts, [SamplingParams(max_tokens=12, temperature=0.0, prediction_ids=g) for g in guess])
    assert [o.output_ids for o in outs] == want
    assert any(o.accepted_draft_tokens for o in outs)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("name", ["linear", "ones"])
def test_prefix_cache_resumes_from_state_snapshots(tmp_path, device, name):
    path = fc.checkpoint(fc.CONFIGS[name], fc.weights(fc.CONFIGS[name]), tmp_path / "m")
    eng = LLMEngine(EngineArgs(model=path, device=device, dtype="fp32", max_num_seqs=2, max_model_len=400, num_kv_blocks=80))
    p = fc.tokens(fc.CONFIGS[name], 300, 5)
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
    assert c.arch == "finelix" and c.layer_types == ["gla", "latent", "gla", "latent", "gla", "latent"]
    assert c.ffn_types == ["dense", "moe", "moe", "dense", "none", "none"] and c.attention_layers() == [1, 3, 5]
    assert c.loop == {"start": 1, "stop": 4, "times": 2} and type(c).from_json(c.to_json()).to_json() == c.to_json()
    assert c.kv_bytes_per_token() == 5 * 64 * 2
    from metrale_inference_alpha_b200.weights.checkpoint import open_checkpoint
    from metrale_inference_alpha_b200.weights.preflight import preflight
    t = fc.weights(cfg)
    c2, src = open_checkpoint(fc.checkpoint(cfg, t, tmp_path / "ok"))
    assert preflight(c2, src, check_shapes=False).ok
    del t["l1.mlp.e3.down"]
    c3, src = open_checkpoint(fc.checkpoint(cfg, t, tmp_path / "bad"))
    assert preflight(c3, src, check_shapes=False).missing == ["l1.mlp.e3.down"]

    def broken(change, match):
        bad = json.loads(json.dumps(cfg))
        change(bad)
        with pytest.raises(ValueError, match=match):
            from_finelix_config(bad)

    broken(lambda b: b["layers"][0].update(type="other"), "unknown mixer")
    broken(lambda b: b["layers"][0]["mlp"].update(kind="other"), "unknown feed-forward")
    broken(lambda b: b["layers"][1]["mixer"]["rot"].update(dims=4), "rotary")
    broken(lambda b: b["layers"][1]["mlp"]["router"].update(top=9), "experts per token")
    broken(lambda b: b["loop"].update(stop=7), "loop")


def test_unserved_combinations_are_refused():
    with pytest.raises(ValueError):
        LLMEngine(EngineArgs(model="tiny-finelix", dtype="int8", max_model_len=64, num_kv_blocks=16))
    for kw in (dict(kv_cache_dtype="fp8"), dict(speculative="dflash"), dict(speculative="mtp"), dict(expert_arena_slots=4)):
        with pytest.raises(NotImplementedError):
            LLMEngine(EngineArgs(model="tiny-finelix", max_model_len=64, num_kv_blocks=16, **kw))


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
def test_preset_runs_from_synthetic_weights(device, dtype):
    eng = LLMEngine(EngineArgs(model=preset("tiny-finelix", num_layers=4), device=device, dtype=dtype, max_num_seqs=2, max_model_len=64,
                               num_kv_blocks=16))
    outs = eng.generate([[1, 2, 3], [9, 8, 7, 6]], SamplingParams(max_tokens=4))
    assert all(len(o.output_ids) == 4 for o in outs)
    if device != "cpu":
        ops.check_status(device)


def test_replay_command(tmp_path, capsys):
    import numpy as np
    from metrale_inference_alpha_b200.server import cli
    cfg = fc.CONFIGS["ones"]
    path = fc.checkpoint(cfg, fc.weights(cfg), tmp_path / "m")
    toks, want = oracle("ones", 30)
    ns = cli.build_parser().parse_args(["replay", "--model", path, "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "64",
                                        "--device", "cpu"])
    from metrale_inference_alpha_b200.engine.replay import run
    lines = [json.dumps({"step": 0, "entries": [{"id": "a", "tokens": toks[:9], "want": []}], "end": []}),
             json.dumps({"step": 1, "entries": [{"id": "a", "tokens": toks[9:30], "want": [20]}], "end": ["a"]})]
    assert run(ns, lines) == 0
    assert [x for x in capsys.readouterr().out.splitlines() if x.startswith("done")] == ["done 0", "done 1"]
    got = torch.from_numpy(np.fromfile(tmp_path / "1.f32", dtype="<f4")).view(1, -1)
    assert fc.error(got, want[29:30]) < 1e-5 and not (tmp_path / "0.f32").exists()
