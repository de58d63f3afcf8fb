"""Small Pivipel configurations with random weights. How they are driven through the engine is shared with the other
32-bit-stream decoders' cases."""
import torch

from fabulix_cases import batch, checkpoint, error, feed, tokens  # noqa: F401  (the tests' helpers)
from metrale_inference_alpha_b200.config.model_config import from_pivipel_config


def rotated(heads, kv, dim, vdim, rot, window, mlp=None, scale=None, base=3000.0, scaling=(6.0, 1.0, 3.0, 96)):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale, "mask": {"size": window},
         "rot": {"base": base, "dims": rot}}
    if scaling:
        m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return {"type": "attention", "mixer": m, "mlp": mlp}


def normed(heads, kv, dim, vdim, window, keep, mlp=None, scale=None):
    return {"type": "attention_2", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale,
                      "mask": {"size": window, "keep_first": keep}}}


def dense(ff, limit=1.4):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(experts, top, ff, groups=(1, 1), shared=None, scale=1.0, limit=1.3, shared_limit=0.7):
    m = {"kind": "moe", "expert": {"ff": ff, "limit": limit},
         "router": {"experts": experts, "top": top, "scale": scale, "groups": dict(zip(("count", "keep"), groups))}}
    if shared:
        m["shared"] = {"ff": shared, "limit": shared_limit}
    return m


def same(layer, of):
    return {**layer, "weights_of": of}


def config(layers, width, streams=2, vocab=150, eps=1e-5, positions=400):
    return {"architecture": "Pivipel", "vocab": vocab, "width": width, "streams": streams, "max_positions": positions, "norm": {"eps": eps},
            "layers": layers}


_a = rotated(3, 1, 22, 30, 10, 7, moe(6, 2, 18, (3, 2), 26, 1.7))
_b = normed(6, 2, 36, 26, 19, 5, dense(44, 2.0), scale=0.31)
_t = rotated(8, 2, 64, 64, 64, 33, moe(8, 3, 64, (4, 2), 64, 0.8, 1.1, 1.9), scaling=None)
# ragged: rows that are not whole 16-byte vectors, head sizes away from every tile, three streams, layers that use
#   another one's tensors (an earlier and a later one's), a layer without feed-forward
# tiles: aligned sizes, one stream per token and kernel registers to spare (four), unequal value heads
# ones: single heads, experts, groups and streams, windows and kept runs of one, factors of one
# wide: tiles past 128, more streams than the kernel holds in registers, windows longer than a tile, many kept tokens
CONFIGS = {
    "ragged": config([_a, _b, rotated(2, 2, 18, 14, 18, 40, None, base=200.0, scaling=(3.0, 0.5, 8.0, 30)), same(_a, 0), same(normed(4, 1, 10, 50, 3, 2, moe(5, 2, 22)), 5),
                      normed(4, 1, 10, 50, 3, 2, moe(5, 2, 22))], 100, streams=3, eps=1e-2),
    "tiles": config([_t, normed(4, 4, 64, 128, 20, 3, moe(6, 2, 40, (2, 1), None, 1.4)), rotated(4, 1, 128, 64, 32, 48, dense(96, 0.6)), same(_t, 0)], 128,
                    streams=4, vocab=128),
    "ones": config([rotated(1, 1, 16, 16, 2, 1, dense(32, 1.0), scale=1.0), normed(1, 1, 16, 16, 1, 1, moe(1, 1, 32, (1, 1), 32, 1.0, 1.0, 1.0), scale=1.0)],
                   64, streams=1),
    "wide": config([rotated(4, 2, 128, 128, 96, 100, dense(192)), normed(6, 1, 128, 128, 70, 66, moe(10, 4, 96, (5, 3), 160, 2.0)),
                    normed(2, 1, 200, 72, 130, 20, dense(64)), rotated(2, 1, 264, 40, 264, 90)], 256, streams=6),
}


def weights(cfg, seed=0, calm=False):
    """Random bf16 tensors of a configuration under their checkpoint names. `calm`: routers whose choice rests on a constant
    feature of their input, far from close calls, which rounding to bf16 would flip."""
    g = torch.Generator().manual_seed(seed)
    W, S, t = cfg["width"], cfg["streams"], {}
    rnd = lambda *s, std=1.0, mean=0.0: (torch.randn(*s, generator=g) * std + mean)

    def lin(name, n, k, gain=1.0):
        t[name] = rnd(n, k, std=gain * k ** -0.5)

    def norm(name):
        t[name], t[name + ".b"], t[name + ".alpha"] = rnd(W, std=0.3, mean=1.0), rnd(W, std=0.2), rnd(1, std=0.1, mean=0.6)[0]

    def hyper(name):
        t[name + ".in"], t[name + ".out"] = rnd(S, std=0.4, mean=1.0 / S), rnd(S, std=0.4, mean=0.8)
        t[name + ".mix"] = rnd(S, S, std=0.25) + 0.7 * torch.eye(S)

    def ffn(name, ff):
        lin(f"{name}.gate", ff, W, 1.5)
        lin(f"{name}.up", ff, W, 1.5)
        lin(f"{name}.down", W, ff)

    t["embed"], t["pos"] = rnd(cfg["vocab"], W, std=1.2), rnd(cfg["max_positions"], W, std=0.8)
    norm("embed.norm")
    for i, L in enumerate(cfg["layers"]):
        if L.get("weights_of") is not None:
            continue
        p, q, m, mlp = f"l{i}", f"l{i}.mix", L["mixer"], L["mlp"]
        H, G = m["heads"], m["kv_heads"]
        norm(f"{p}.norm1")
        hyper(f"{p}.hc1")
        lin(f"{q}.q", H * m["dim"], W, 2.0)
        lin(f"{q}.k", G * m["dim"], W, 2.0)
        lin(f"{q}.v", G * m["vdim"], W)
        lin(f"{q}.o", W, H * m["vdim"], 2.0)
        lin(f"{q}.g", H if L["type"] == "attention" else H * m["vdim"], W, 2.0)
        if L["type"] == "attention":
            t[f"{q}.sink"] = rnd(H, std=1.0, mean=0.5)
        else:
            t[f"{q}.q.norm"], t[f"{q}.k.norm"] = rnd(m["dim"], std=0.3, mean=1.3), rnd(m["dim"], std=0.3, mean=1.3)
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
        lin(f"{p}.mlp.router", E, W, 0.3 if calm else 2.0)
        if calm:                                         # feature 0 is 1 after the norm: it carries a ladder of scores
            t[f"{p}.norm2"][0], t[f"{p}.norm2.b"][0] = 0.0, 1.0
            t[f"{p}.mlp.router"][:, 0] = torch.randperm(E, generator=g) * 2.0
        if mlp.get("shared"):
            ffn(f"{p}.mlp.shared", mlp["shared"]["ff"])
            lin(f"{p}.mlp.shared.sg", 1, W, 2.0)
    norm("final.norm")
    return {k: v.to(torch.bfloat16).contiguous() for k, v in t.items()}


def model_config(cfg, dtype="bf16"):
    return from_pivipel_config(cfg).scaled(weight_format=dtype, kv_dtype=dtype)
