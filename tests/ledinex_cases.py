"""Small Ledinex configurations with random weights. How they are driven through the engine is shared with the other
32-bit-stream decoders' cases."""
import torch

from fabulix_cases import batch, checkpoint, error, feed, tokens  # noqa: F401  (the tests' helpers)
from metrale_inference_alpha_b200.config.model_config import from_ledinex_config


def moe(experts, top, ff, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def delta(heads, kv, dim, vdim, conv, mlp=None):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": mlp}


def capped(left, right, mlp=None, softcap=9.0, base=900.0, factor=3.0, scales=(0.7, 0.9), scale=None):
    """left (heads, kv heads, dim, vdim, rotated dims), right (heads, dim, vdim)."""
    H, G, dk, dv, rot = left
    decay = [1.0 - 0.6 * 0.3 ** h for h in range(right[0])]
    a = {"heads": H, "kv_heads": G, "dim": dk, "vdim": dv, "scale": dk ** -0.5 if scale is None else scale, "softcap": softcap,
         "rot": {"base": base, "dims": rot, "scaling": {"factor": factor}}}
    return {"type": "parallel", "mlp": mlp, "mixer": {"left": a, "right": dict(zip(("heads", "dim", "vdim"), right), decay=decay),
                                                       "left_scale": scales[0], "right_scale": scales[1]}}


def windowed(left, right, mlp=None, base=900.0, scaling=(5.0, 64, 4.0, 0.5), scales=(1.2, 0.6), scale=None):
    """left (heads, kv heads, dim, rotated dims, window), right (heads, dim)."""
    H, G, dk, rot, size = left
    a = {"heads": H, "kv_heads": G, "dim": dk, "vdim": dk, "scale": dk ** -0.5 if scale is None else scale, "mask": {"size": size},
         "rot": {"base": base, "dims": rot, "scaling": dict(zip(("factor", "original", "fast", "slow"), scaling))}}
    return {"type": "parallel_2", "mlp": mlp, "mixer": {"left": a, "right": {"heads": right[0], "dim": right[1]}, "left_scale": scales[0],
                                                         "right_scale": scales[1]}}


def config(layers, width, taps=3, vocab=150, eps=1e-5, embed=2.0, logit=0.7):
    return {"architecture": "Ledinex", "vocab": vocab, "width": width, "embedding": {"scale": embed}, "logit_scale": logit,
            "canon": {"taps": taps}, "norm": {"eps": eps}, "layers": layers}


# ragged: rows that are not whole 16-byte vectors, head sizes away from every tile, a layer without feed-forward, a mixture
#   without shared expert, several value heads to a key head, a large eps
# tiles: aligned sizes, the chunked kernels' head sizes, unequal key and value sizes
# ones: single heads, experts and taps (and a short convolution of three beside inputs without one), a window of one, factors of one
# wide: heads past 128 (and past 256 values), filters longer than a run of tokens is short, a rank past what decode computes
CONFIGS = {
    "ragged": config([delta(6, 3, 18, 22, 2, moe(6, 2, 18, 26)), capped((3, 1, 22, 30, 10), (3, 20, 26), moe(5, 3, 22)),
                      windowed((6, 2, 36, 20, 19), (5, 28), moe(7, 2, 34, 12)), delta(3, 3, 10, 6, 5), windowed((2, 1, 14, 14, 4), (1, 10))],
                     100, taps=4, eps=1e-2),
    "tiles": config([windowed((4, 2, 64, 64, 33), (2, 64), moe(8, 3, 64, 64)), delta(4, 2, 64, 128, 4, moe(6, 2, 128)),
                     capped((4, 4, 128, 64, 64), (2, 128, 64), moe(4, 2, 40, 128)), delta(2, 2, 128, 64, 3, moe(3, 1, 32, 32))], 128, taps=2, vocab=128),
    "ones": config([capped((1, 1, 16, 16, 2), (1, 16, 16), moe(1, 1, 32, 32), softcap=1.0, factor=1.0, scales=(1.0, 1.0), scale=1.0),
                    windowed((1, 1, 16, 2, 1), (1, 16), moe(2, 1, 32), scaling=(1.0, 1, 1.0, 1.0), scales=(1.0, 1.0), scale=1.0),
                    delta(1, 1, 16, 16, 1, moe(1, 1, 16, 16)), delta(1, 1, 16, 16, 3)], 64, taps=1, embed=1.0, logit=1.0),
    "wide": config([delta(2, 1, 136, 264, 7, moe(4, 2, 96, 160)), capped((2, 1, 200, 72, 96), (2, 130, 12), moe(5, 2, 64)),
                    windowed((3, 1, 264, 40, 70), (1, 200), moe(3, 3, 40, 8)), capped((4, 2, 128, 128, 128), (3, 64, 128))], 256, taps=12),
}
RANKS = {"ragged": 9, "tiles": 16, "ones": 1, "wide": 72}


def weights(cfg, seed=0, calm=False, rank=None):
    """Random bf16 tensors of a configuration under their checkpoint names. `calm`: routers whose choice rests on a constant
    feature of their input, away from close calls, which rounding to bf16 would flip."""
    g = torch.Generator().manual_seed(seed)
    W, taps, t = cfg["width"], cfg["canon"]["taps"], {}
    rank = rank or next((RANKS[n] for n, c in CONFIGS.items() if c is cfg), 16)
    rnd = lambda *s, std=1.0, mean=0.0: (torch.randn(*s, generator=g) * std + mean)

    def lin(name, n, k, gain=1.0):
        t[name] = rnd(n, k, std=gain * k ** -0.5)

    t["embed"] = rnd(cfg["vocab"], W, std=0.8)
    for i, L in enumerate(cfg["layers"]):
        p, q, m, mlp = f"l{i}", f"l{i}.mix", L["mixer"], L["mlp"]
        for n in "12" if mlp else "1":
            t[f"{p}.norm{n}"], t[f"{p}.canon{n}"] = rnd(W, std=0.3), rnd(W, taps, std=0.4)
            if calm:
                t[f"{p}.norm{n}"][0], t[f"{p}.canon{n}"][0] = -1.0, 0.0
        if L["type"] == "delta":
            H, nk, nv = m["heads"], m["kv_heads"] * m["dim"], m["heads"] * m["vdim"]
            for n, rows in (("q", nk), ("k", nk), ("v", nv)):
                lin(f"{q}.{n}", rows, W)
                t[f"{q}.{n}.conv"] = rnd(rows, m["conv"], std=0.5, mean=0.2)
            lin(f"{q}.a", H, W, 0.7)
            lin(f"{q}.b", H, W, 0.7)
            lin(f"{q}.g", nv, W)
            lin(f"{q}.o", W, nv)
            t[f"{q}.A_log"], t[f"{q}.dt_bias"], t[f"{q}.norm"] = rnd(H, std=0.7, mean=-1.5), rnd(H, mean=-1.0), rnd(m["vdim"], std=0.3, mean=1)
        else:
            a, r = m["left"], m["right"]
            H, G = a["heads"], a["kv_heads"]
            lin(f"{q}.left.q", H * a["dim"], W)
            lin(f"{q}.left.k", G * a["dim"], W)
            t[f"{q}.left.q.norm"], t[f"{q}.left.k.norm"] = rnd(H * a["dim"], std=0.4, mean=1.6), rnd(G * a["dim"], std=0.4, mean=1.6)
            dk = r["heads"] * r["dim"]
            if L["type"] == "parallel":
                lin(f"{q}.left.v", G * a["vdim"], W)
                lin(f"{q}.left.o", W, H * a["vdim"])
                dv = r["heads"] * r["vdim"]
                rows = (("q", dk), ("k", dk), ("v", dv), ("g", dv))
            else:
                t[f"{q}.left.q.b"], t[f"{q}.left.k.b"] = rnd(H * a["dim"]), rnd(G * a["dim"])
                lin(f"{q}.left.o", W, H * a["dim"])
                dv, rows = dk, (("r", dk), ("k", dk), ("v", dk), ("g", dk), ("a", dk), ("w1", rank))
                lin(f"{q}.right.w2", dk, rank, 2.0)
                t[f"{q}.right.w0"], t[f"{q}.right.a.b"] = rnd(dk, std=2.0, mean=-2.0), rnd(dk)
            for n, k in rows:
                lin(f"{q}.right.{n}", k, W)
            t[f"{q}.right.norm"] = rnd(dv, std=0.3, mean=1)
            lin(f"{q}.right.o", W, dv)
        if mlp is None:
            continue
        E = mlp["router"]["experts"]
        for n, ff in [(f"e{e}", mlp["expert"]["ff"]) for e in range(E)] + ([("shared", mlp["shared"]["ff"])] if mlp.get("shared") else []):
            lin(f"{p}.mlp.{n}.up", ff, W)
            lin(f"{p}.mlp.{n}.down", W, ff)
        lin(f"{p}.mlp.router", E, W, 0.04 if calm else 0.7)
        if calm:                                         # channel 0 of the stream stays embedding.scale
            t[f"{p}.mlp.router"][:, 0] = torch.randperm(E, generator=g) * 1.0 / cfg["embedding"]["scale"]
    t["final.norm"] = rnd(W, std=0.3)
    if calm:
        t["embed"][:, 0] = 1.0
    return {k: v.to(torch.bfloat16).contiguous() for k, v in t.items()}


def model_config(cfg, dtype="bf16"):
    return from_ledinex_config(cfg).scaled(weight_format=dtype, kv_dtype=dtype)
