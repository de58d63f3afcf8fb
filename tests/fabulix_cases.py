"""Small Fabulix configurations with random weights, and helpers that drive them through the engine."""
import json

import torch
from safetensors.torch import save_file

from metrale_inference_alpha_b200.config.model_config import from_fabulix_config
from metrale_inference_alpha_b200.engine.batch import ForwardBatch


def parallel(width, heads, kv, dim, vdim, rot, rheads, rdim, ff=None, scale=None, ls=0.8, rs=0.65, base=3000.0, limit=1.5):
    return {"type": "parallel", "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit},
            "mixer": {"left": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale,
                               "rot": {"base": base, "dims": rot}},
                      "right": {"heads": rheads, "dim": rdim}, "left_scale": ls, "right_scale": rs}}


def lightning(heads, dim, vdim, ff=None, decay=None, limit=2.5):
    return {"type": "lightning", "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit},
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim,
                      "decay": decay or [1 - 2.0 ** -(1 + 1.7 * h) for h in range(heads)]}}


def config(layers, width, vocab=150, side=12, scale=3.0, eps=1e-5):
    c = {"architecture": "Fabulix", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps}, "layers": layers}
    if side:
        c["token_side"] = {"dim": side}
    return c


# ragged sizes (rows that are not whole 16-byte vectors, head sizes away from every tile), grouped heads, partial
# rotation, layers that differ from one another; everything equal / 1; no attention at all; large tiles
CONFIGS = {
    "ragged": config([parallel(100, 4, 2, 30, 44, 12, 3, 20, ff=70), lightning(3, 36, 22), parallel(100, 3, 1, 24, 26, 24, 2, 36),
                      lightning(2, 18, 50, ff=44)], 100, side=10),
    "equal": config([lightning(2, 64, 64, ff=128), parallel(128, 4, 1, 64, 64, 64, 2, 64, ff=128, ls=1.0, rs=1.0, scale=1.0)], 128, side=16,
                    scale=1.0, vocab=128),
    "linear": config([lightning(1, 16, 16), lightning(4, 24, 40, ff=64)], 64, side=0),
    "wide": config([parallel(256, 4, 2, 128, 128, 96, 2, 128, ff=192), lightning(2, 128, 128), parallel(256, 2, 2, 112, 72, 32, 3, 64)], 256, side=24),
}


def weights(cfg, seed=0, rank=14):
    """Random bf16 tensors of a configuration under their checkpoint names."""
    g = torch.Generator().manual_seed(seed)
    W, t = cfg["width"], {}
    rnd = lambda *s, std=1.0, mean=0.0: (torch.randn(*s, generator=g) * std + mean)

    def lin(name, n, k, gain=1.0):
        t[name] = rnd(n, k, std=gain * k ** -0.5)

    def norm(name):
        t[name], t[name + ".b"], t[name + ".alpha"] = rnd(W, std=0.3, mean=1.0), rnd(W, std=0.2), rnd(1, std=0.1, mean=0.6)[0]

    t["embed"] = rnd(cfg["vocab"], W, std=1.2 / cfg["embedding"]["scale"])
    side = (cfg.get("token_side") or {}).get("dim", 0)
    if side:
        t["side.embed"] = rnd(cfg["vocab"], len(cfg["layers"]) * side)
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}", L["mixer"]
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if L["mlp"] else ()):
            norm(f"{p}.{n}")
        if L["type"] == "parallel":
            a, r = m["left"], m["right"]
            lin(f"{p}.mix.left.q", a["heads"] * a["dim"], W, 2.0)
            lin(f"{p}.mix.left.k", a["kv_heads"] * a["dim"], W, 2.0)
            lin(f"{p}.mix.left.v", a["kv_heads"] * a["vdim"], W)
            lin(f"{p}.mix.left.o", W, a["heads"] * a["vdim"], 1.5)
            hd, q = r["heads"] * r["dim"], f"{p}.mix.right"
            for n in "rkvgw":
                t[f"{q}.mu.{n}"] = torch.rand(W, generator=g)
            for n in "rkvg":
                lin(f"{q}.{n}", hd, W)
            lin(f"{q}.w1", rank, W)
            lin(f"{q}.w2", hd, rank)
            t[f"{q}.w0"], t[f"{q}.u"], t[f"{q}.norm"] = rnd(hd, std=1.5, mean=-2.0), rnd(r["heads"], r["dim"], std=0.5, mean=0.5), rnd(hd, std=0.3, mean=1)
            lin(f"{q}.o", W, hd, 1.5)
        else:
            q, dk, dv = f"{p}.mix", m["heads"] * m["dim"], m["heads"] * m["vdim"]
            for n, rows in (("q", dk), ("k", dk), ("v", dv), ("g", dv)):
                lin(f"{q}.{n}", rows, W)
            lin(f"{q}.o", W, dv, 1.5)
            t[f"{q}.norm"] = rnd(dv, std=0.3, mean=1)
        if L["mlp"]:
            ff = L["mlp"]["ff"]
            lin(f"{p}.mlp.gate", ff, W, 1.5)
            lin(f"{p}.mlp.up", ff, W, 1.5)
            lin(f"{p}.mlp.down", W, ff)
        if side:
            lin(f"{p}.side.gate", side, W)
            lin(f"{p}.side.proj", W, side)
            t[f"{p}.side.norm"] = rnd(W, std=0.3, mean=0.7)
    norm("final.norm")
    return {k: v.to(torch.bfloat16).contiguous() for k, v in t.items()}


def checkpoint(cfg, tensors, path):
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    save_file(tensors, str(path / "model.safetensors"))
    return str(path)


def model_config(cfg, dtype="bf16"):
    return from_fabulix_config(cfg).scaled(weight_format=dtype, kv_dtype=dtype)


def tokens(cfg, n, seed):
    g = torch.Generator().manual_seed(1000 + seed)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()


def feed(replay, rid, toks, cuts):
    """Feed `toks` alone in portions of the given sizes (the last size repeats); all logits [n, vocab]."""
    out, at, i = [], 0, 0
    while at < len(toks):
        n = min(cuts[min(i, len(cuts) - 1)], len(toks) - at)
        out.append(replay.step([{"id": rid, "tokens": toks[at:at + n], "want": list(range(n))}], [rid] if at + n == len(toks) else []))
        at, i = at + n, i + 1
    return torch.cat(out)


def error(got, want):
    """Largest rms difference of a row of logits (mean removed), relative to the logits' own rms."""
    d = got.double() - want.double()
    d = d - d.mean(-1, keepdim=True)
    return float(d.pow(2).mean(-1).sqrt().max() / want.double().pow(2).mean().sqrt())


def batch(lens, ctx=None, slots=None, device="cpu", block=16, pages=None):
    """A ForwardBatch of sequences with `lens[s]` new rows that end at context `ctx[s]`; token ids are zeros."""
    ctx = ctx or list(lens)
    seqs, nxt = [], 1
    for s, n in enumerate(lens):
        nb = (ctx[s] + block - 1) // block
        blocks = pages[s] if pages else list(range(nxt, nxt + nb))
        nxt += nb
        seqs.append(dict(tokens=[0] * n, start_pos=ctx[s] - n, blocks=blocks, state_slot=slots[s] if slots else s + 1, logits="all"))
    return ForwardBatch.build(seqs, block, device=device)
