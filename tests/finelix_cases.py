"""Small Finelix configurations with random weights. How they are driven through the engine is shared with the
other 32-bit-stream decoder's cases."""
import torch

from fabulix_cases import batch, checkpoint, error, feed, tokens  # noqa: F401  (the tests' helpers)
from metrale_inference_alpha_b200.config.model_config import from_finelix_config


def latent(heads, dim, rot, vdim, rank, q_rank, mlp=None, scale=None, base=3000.0):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "q_rank": q_rank,
                      "scale": (dim + rot) ** -0.5 if scale is None else scale, "rot": {"base": base, "dims": rot}}}


def gla(heads, dim, vdim, tau=16.0, mlp=None, name="gla"):
    return {"type": name, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=None):
    m = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def config(layers, width, vocab=150, scale=3.0, eps=1e-5, loop=None):
    c = {"architecture": "Finelix", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps}, "layers": layers}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


# ragged: rows that are not whole 16-byte vectors, head sizes away from every tile, a loop in the middle, layers that
#   differ from one another, every mixer beside every feed-forward and beside none
# tiles: aligned sizes, everything inside one loop
# ones: single heads, experts and passes, factors of one
# wide: rows past the 256-wide attention tiles (few heads and many), chunked recurrences, value sizes away from key sizes
CONFIGS = {
    "ragged": config([gla(3, 20, 28, 7.0, dense(70)), latent(3, 20, 6, 22, 38, 30, moe(5, 2, 18, 26)), gla(2, 36, 18, 16.0, moe(4, 3, 22), "gla_2"),
                      latent(2, 14, 10, 30, 50, 44, dense(44), scale=0.31, base=500.0), gla(1, 18, 50, 3.0), latent(5, 8, 4, 12, 21, 13)],
                     100, loop=(1, 4, 2)),
    "tiles": config([latent(4, 32, 32, 48, 96, 64, moe(6, 3, 64, 96)), gla(2, 64, 64, 16.0, dense(96), "gla_2"), latent(8, 24, 16, 32, 200, 72, dense(64)),
                     gla(3, 64, 128, 11.0, moe(9, 4, 40))], 128, loop=(0, 4, 2), scale=2.0, vocab=128),
    "ones": config([gla(1, 16, 16, 1.0, dense(32)), latent(1, 16, 2, 16, 16, 16, moe(1, 1, 32, 32), scale=1.0)], 64, loop=(0, 1, 1), scale=1.0),
    "wide": config([gla(2, 128, 64, 16.0, dense(192)), latent(16, 48, 32, 40, 264, 96, moe(8, 2, 96, 160)), gla(1, 64, 128, 5.0),
                    latent(3, 40, 48, 56, 320, 80)], 256, loop=(1, 2, 2)),
    "linear": config([gla(2, 24, 40, 16.0, dense(64)), gla(3, 16, 16, 2.0, moe(4, 2, 24, 40), "gla_2")], 64),
}


def weights(cfg, seed=0, rank=14, calm=False):
    """Random bf16 tensors of a configuration under their checkpoint names. `calm`: router biases keep the choice of
    experts far from close calls, which rounding to bf16 would flip."""
    g = torch.Generator().manual_seed(seed)
    W, t = cfg["width"], {}
    rnd = lambda *s, std=1.0, mean=0.0: (torch.randn(*s, generator=g) * std + mean)

    def lin(name, n, k, gain=1.0):
        t[name] = rnd(n, k, std=gain * k ** -0.5)

    def ffn(name, ff):
        lin(f"{name}.gate", ff, W, 1.5)
        lin(f"{name}.up", ff, W, 1.5)
        lin(f"{name}.down", W, ff)

    t["embed"] = rnd(cfg["vocab"], W, std=1.2 / cfg["embedding"]["scale"])
    if cfg.get("loop"):
        lin("loop.in", W, 2 * W)
        t["loop.step"] = rnd(cfg["loop"]["times"], W, std=0.5)
    for i, L in enumerate(cfg["layers"]):
        p, q, m, mlp = f"l{i}", f"l{i}.mix", L["mixer"], L["mlp"]
        H = m["heads"]
        t[f"{p}.norm1"] = rnd(W, std=0.3, mean=1.0)
        if L["type"] == "latent_attention":
            rank_, R = m["kv_rank"], m["rot_dim"]
            lin(f"{q}.dq", m["q_rank"], W)
            t[f"{q}.dq.norm"] = rnd(m["q_rank"], std=0.3, mean=1.0)
            lin(f"{q}.uq", H * (m["dim"] + R), m["q_rank"], 2.0)
            lin(f"{q}.dkv", rank_ + R, W, 1.5)
            t[f"{q}.dkv.norm"] = rnd(rank_, std=0.3, mean=1.0)
            lin(f"{q}.uk", H * m["dim"], rank_, 1.5)
            lin(f"{q}.uv", H * m["vdim"], rank_)
            lin(f"{q}.o", W, H * m["vdim"], 1.5)
        else:
            dk, dv = H * m["dim"], H * m["vdim"]
            for n, rows in (("q", dk), ("k", dk), ("v", dv), ("g", dv)):
                lin(f"{q}.{n}", rows, W)
            lin(f"{q}.o", W, dv, 1.5)
            t[f"{q}.norm"] = rnd(m["vdim"], std=0.3, mean=1.0)
            lin(f"{q}.a1", rank, W)
            lin(f"{q}.a2", dk, rank, 2.0)
            t[f"{q}.a2.b"] = rnd(dk, std=2.0, mean=1.0)
        if mlp is None:
            continue
        if mlp["kind"] == "dense":
            ffn(f"{p}.mlp", mlp["ff"])
            continue
        E = mlp["router"]["experts"]
        for e in range(E):
            ffn(f"{p}.mlp.e{e}", mlp["expert"]["ff"])
        lin(f"{p}.mlp.router", E, W, 0.7 if calm else 2.0)
        t[f"{p}.mlp.router.b"] = rnd(E, std=0.7)
        if calm:
            t[f"{p}.mlp.router.b"] = torch.where(torch.randperm(E, generator=g) < mlp["router"]["top"], 3.0, -3.0)
        if mlp.get("shared"):
            ffn(f"{p}.mlp.shared", mlp["shared"]["ff"])
    t["final.norm"] = rnd(W, std=0.3, mean=1.0)
    lin("head", cfg["vocab"], W, 1.3)
    return {k: v.to(torch.bfloat16).contiguous() for k, v in t.items()}


def model_config(cfg, dtype="bf16"):
    return from_finelix_config(cfg).scaled(weight_format=dtype, kv_dtype=dtype)
