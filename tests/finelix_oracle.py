"""Plain, slow restatement of the Finelix decoder, one function per mechanism, written from the equations
alone. It shares no code with the package: every sequence is processed whole, with explicit loops over heads,
tokens and keys, in the dtype of the inputs (float64 unless a test asks otherwise).

Shapes: a sequence's hidden rows are [n, width]; weights are [out, in].
"""
import math

import torch


# ------------------------------------------------------------------ pieces
def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def silu(z):
    return z / (1 + torch.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def rotate(x, pos, base):
    """Rotary positions on vectors [..., d] at position `pos`: coordinate i is paired with i + d / 2."""
    y, d = x.clone(), x.shape[-1]
    for i in range(d // 2):
        a = pos * base ** (-2.0 * i / d)
        u, v = x[..., i], x[..., i + d // 2]
        y[..., i] = u * math.cos(a) - v * math.sin(a)
        y[..., i + d // 2] = v * math.cos(a) + u * math.sin(a)
    return y


def latent_attention(h, t, m, eps):
    """Keys and values are linear in a normed latent per token; one rotated key part serves all heads. The keys and
    values are written out here (nothing is absorbed). h [n, width] -> [n, width]."""
    H, dim, rot, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    n = h.shape[0]
    q = (rms_norm(h @ t["dq"].T, t["dq.norm"], eps) @ t["uq"].T).view(n, H, dim + rot)
    kv = h @ t["dkv"].T
    c = rms_norm(kv[:, :rank], t["dkv.norm"], eps)
    k = (c @ t["uk"].T).view(n, H, dim)
    v = (c @ t["uv"].T).view(n, H, dv)
    k_rot = torch.stack([rotate(kv[p, rank:], p, m["rot"]["base"]) for p in range(n)])
    q_rot = torch.stack([rotate(q[p, :, dim:], p, m["rot"]["base"]) for p in range(n)])
    out = torch.zeros(n, H, dv, dtype=h.dtype)
    for head in range(H):
        for i in range(n):
            s = (k[:i + 1, head] @ q[i, head, :dim] + k_rot[:i + 1] @ q_rot[i, head]) * m["scale"]
            w = torch.exp(s - s.max())
            out[i, head] = (w / w.sum()) @ v[:i + 1, head]
    return out.reshape(n, H * dv) @ t["o"].T


def gated_linear_attention(h, t, m, eps):
    """A matrix state per head whose key channels decay by sigmoid(z)^(1 / tau), read after the update."""
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    n = h.shape[0]
    q = (h @ t["q"].T * dk ** -0.5).view(n, H, dk)
    k = (h @ t["k"].T).view(n, H, dk)
    v = (h @ t["v"].T).view(n, H, dv)
    z = h @ t["a1"].T @ t["a2"].T + t["a2.b"]
    alpha = torch.sigmoid(z).pow(1 / m["tau"]).view(n, H, dk)
    out = torch.zeros(n, H, dv, dtype=h.dtype)
    for head in range(H):
        S = torch.zeros(dk, dv, dtype=h.dtype)
        for i in range(n):
            S = alpha[i, head][:, None] * S + torch.outer(k[i, head], v[i, head])
            out[i, head] = S.T @ q[i, head]
    out = rms_norm(out, t["norm"], eps).reshape(n, H * dv)
    return (out * silu(h @ t["g"].T)) @ t["o"].T


def feed_forward(h, t, act):
    return (act(h @ t["gate"].T) * (h @ t["up"].T)) @ t["down"].T


def route(h, t, top):
    """(expert ids, weights) per token: the largest biased logits, a softmax over those alone."""
    z = h @ t["router"].T + t["router.b"]
    picked = []
    for row in z:
        ids = sorted(range(len(row)), key=lambda e: (-float(row[e]), e))[:top]
        w = torch.exp(row[ids] - row[ids].max())
        picked.append((ids, w / w.sum()))
    return picked


def mixture(h, t, mlp):
    out = torch.zeros_like(h)
    for i, (ids, w) in enumerate(route(h, t, mlp["router"]["top"])):
        for e, we in zip(ids, w):
            out[i] += we * feed_forward(h[i], _sub(t, f"e{e}."), silu)
    if mlp.get("shared"):
        out = out + feed_forward(h, _sub(t, "shared."), silu)
    return out


def enter_pass(x, x0, t, step):
    """What stands before a pass of the looped layers."""
    return torch.cat([x, x0], 1) @ t["loop.in"].T + t["loop.step"][step]


# ------------------------------------------------------------------ the model
MIXERS = {"latent_attention": latent_attention, "gla": gated_linear_attention, "gla_2": gated_linear_attention}


def _sub(tensors, prefix):
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


def layer(x, t, L, eps):
    """Both sublayers read one norm and join the stream together."""
    h = rms_norm(x, t["norm1"], eps)
    y = MIXERS[L["type"]](h, _sub(t, "mix."), L["mixer"], eps)
    if L["mlp"] is not None:
        mt = _sub(t, "mlp.")
        y = y + (mixture(h, mt, L["mlp"]) if L["mlp"]["kind"] == "moe" else feed_forward(h, mt, gelu_tanh))
    return x + y


def forward(cfg, tensors, tokens, dtype=torch.float64, layers=False):
    """Logits [n, vocab] of one whole sequence (and, with `layers`, the residual stream after every layer run)."""
    t = {k: v.to(dtype) for k, v in tensors.items()}
    eps, L = cfg["norm"]["eps"], cfg["layers"]
    loop = cfg.get("loop") or {"start": 0, "stop": 0, "times": 0}
    x0 = t["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    x, trace = x0, []

    def run(i):
        nonlocal x
        x = layer(x, _sub(t, f"l{i}."), L[i], eps)
        trace.append(x)

    for i in range(loop["start"]):
        run(i)
    for p in range(loop["times"]):
        x = enter_pass(x, x0, t, p)
        for i in range(loop["start"], loop["stop"]):
            run(i)
    for i in range(loop["stop"] if loop["times"] else loop["start"], len(L)):
        run(i)
    logits = rms_norm(x, t["final.norm"], eps) @ t["head"].T
    return (logits, torch.stack(trace)) if layers else logits
