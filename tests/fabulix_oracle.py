"""Plain, slow restatement of the Fabulix decoder, one function per mechanism, written from the
equations alone. It shares no code with the package: every sequence is processed token by token with
explicit loops over keys and channels, in the dtype of the inputs (float64 unless a test asks otherwise).

Shapes: a sequence's hidden rows are [n, width]; weights are [out, in].
"""
import math

import torch


# ------------------------------------------------------------------ pieces
def dyt(x, alpha, w, b):
    """Dynamic Tanh: tanh(alpha x) w + b."""
    return torch.tanh(alpha * x) * w + b


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def rotate(x, pos, base, dims):
    """Rotary positions on one head vector [d] at position `pos`: coordinate i is paired with i + dims / 2."""
    y = x.clone()
    half = dims // 2
    for i in range(half):
        a = pos * base ** (-2.0 * i / dims)
        c, s = math.cos(a), math.sin(a)
        u, v = x[..., i], x[..., i + half]
        y[..., i] = u * c - v * s
        y[..., i + half] = v * c + u * s
    return y


def sink_softmax(scores):
    """exp(s_j) / (1 + sum exp(s)): a phantom score of 0 without a value."""
    m = torch.clamp(scores.max(), min=0.0)
    e = torch.exp(scores - m)
    return e / (torch.exp(-m) + e.sum())


def attention(h, t, mix):
    """Causal grouped-query attention with the sink. h [n, width] -> [n, width]."""
    H, G, dk, dv, rot = mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"], mix["rot"]
    n = h.shape[0]
    q = (h @ t["q"].T).view(n, H, dk)
    k = (h @ t["k"].T).view(n, G, dk)
    v = (h @ t["v"].T).view(n, G, dv)
    q = torch.stack([rotate(q[p], p, rot["base"], rot["dims"]) for p in range(n)])
    k = torch.stack([rotate(k[p], p, rot["base"], rot["dims"]) for p in range(n)])
    out = torch.zeros(n, H, dv, dtype=h.dtype)
    for head in range(H):
        g = head // (H // G)
        for i in range(n):
            s = (k[:i + 1, g] @ q[i, head]) * mix["scale"]
            out[i, head] = sink_softmax(s) @ v[:i + 1, g]
    return out.reshape(n, H * dv) @ t["o"].T


def time_mix(h, t, mix, eps):
    """RWKV-style time mixing: token shift, per-channel data-dependent decay, bonus for the current token."""
    H, D = mix["heads"], mix["dim"]
    n, W = h.shape
    prev = torch.cat([torch.zeros(1, W, dtype=h.dtype), h[:-1]])
    m = {s: h + (prev - h) * t["mu." + s] for s in "rkvgw"}
    r, k, v = ((m[s] @ t[s].T).view(n, H, D) for s in "rkv")
    gate = silu(m["g"] @ t["g"].T)
    w = torch.exp(-torch.exp(torch.tanh(m["w"] @ t["w1"].T) @ t["w2"].T + t["w0"])).view(n, H, D)
    out = torch.zeros(n, H, D, dtype=h.dtype)
    for head in range(H):
        S = torch.zeros(D, D, dtype=h.dtype)
        for i in range(n):
            kv = torch.outer(k[i, head], v[i, head])
            out[i, head] = (S + t["u"][head][:, None] * kv).T @ r[i, head]
            S = w[i, head][:, None] * S + kv
    out = rms(out, eps).reshape(n, H * D) * t["norm"] * gate
    return out @ t["o"].T


def lightning(h, t, mix, eps):
    """Linear attention with one fixed decay per head, read after the update."""
    H, dk, dv = mix["heads"], mix["dim"], mix["vdim"]
    n = h.shape[0]
    q = silu(h @ t["q"].T).view(n, H, dk)
    k = silu(h @ t["k"].T).view(n, H, dk)
    v = silu(h @ t["v"].T).view(n, H, dv)
    out = torch.zeros(n, H, dv, dtype=h.dtype)
    for head in range(H):
        S = torch.zeros(dk, dv, dtype=h.dtype)
        for i in range(n):
            S = mix["decay"][head] * S + torch.outer(k[i, head], v[i, head])
            out[i, head] = S.T @ q[i, head]
    out = rms(out.reshape(n, H * dv), eps) * t["norm"] * torch.sigmoid(h @ t["g"].T)
    return out @ t["o"].T


def clamped_glu(h, t, limit):
    g = torch.clamp(h @ t["gate"].T, max=limit)
    u = torch.clamp(h @ t["up"].T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ t["down"].T


def token_side(x, tokens, t, table, layer, dim, eps):
    """The per-layer token input: a gated slice of a second embedding, projected, normalised and added."""
    e = table[tokens][:, layer * dim:(layer + 1) * dim]
    y = (gelu_tanh(x @ t["gate"].T) * e) @ t["proj"].T
    return x + rms(y, eps) * t["norm"]


# ------------------------------------------------------------------ the model
def _sub(tensors, prefix):
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


def forward(cfg, tensors, tokens, dtype=torch.float64, layers=False):
    """Logits [n, vocab] of one whole sequence (and, with `layers`, the residual stream after every layer)."""
    t = {k: v.to(dtype) for k, v in tensors.items()}
    eps = cfg["norm"]["eps"]
    tok = torch.as_tensor(tokens, dtype=torch.long)

    def norm(x, name):
        return dyt(x, t[name + ".alpha"], t[name], t[name + ".b"])

    x = t["embed"][tok] * cfg["embedding"]["scale"]
    trace = []
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        mt, m = _sub(t, p + "mix."), L["mixer"]
        h = norm(x, p + "norm1")
        if L["type"] == "parallel":
            y = (m["left_scale"] * attention(h, _sub(mt, "left."), m["left"])
                 + m["right_scale"] * time_mix(h, _sub(mt, "right."), m["right"], eps))
        else:
            y = lightning(h, mt, m, eps)
        x = x + norm(y, p + "norm1b")
        if L["mlp"] is not None:
            x = x + norm(clamped_glu(norm(x, p + "norm2"), _sub(t, p + "mlp."), L["mlp"]["limit"]), p + "norm2b")
        if cfg.get("token_side"):
            x = token_side(x, tok, _sub(t, p + "side."), t["side.embed"], i, cfg["token_side"]["dim"], eps)
        trace.append(x)
    logits = norm(x, "final.norm") @ t["embed"].T
    return (logits, torch.stack(trace)) if layers else logits
