"""Plain, slow restatement of the Ledinex decoder, one function per mechanism, written from the equations alone. It
shares no code with the package: every sequence is processed whole, with explicit loops over heads, positions and
experts, in the dtype of the inputs (float64 unless a caller asks otherwise).

Shapes: a sequence's hidden rows are [n, width]; weights are [out, in].
"""
import math

import torch


# ------------------------------------------------------------------ pieces
def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def unit_length(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def short_conv(x, w):
    """Causal convolution over time, one filter per channel: x [n, C], w [C, taps], the last column the current row's."""
    taps = w.shape[1]
    out = torch.zeros_like(x)
    for t in range(len(x)):
        for j in range(taps):
            if t - taps + 1 + j >= 0:
                out[t] += w[:, j] * x[t - taps + 1 + j]
    return out


# ------------------------------------------------------------------ positions
def frequencies(rot):
    """(rotary frequencies, factor on cos and sin) of a layer: plain, all divided by a factor, or blended (YaRN)."""
    n, base, s = rot["dims"], rot["base"], rot.get("scaling")
    f = [base ** (-2.0 * i / n) for i in range(n // 2)]
    if not s:
        return f, 1.0
    if "original" not in s:
        return [x / s["factor"] for x in f], 1.0

    def dim(turns):
        return n * math.log(s["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

    lo, hi = max(math.floor(dim(s["fast"])), 0), min(math.ceil(dim(s["slow"])), n - 1)
    out = []
    for i, x in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(x / s["factor"] * ramp + x * (1 - ramp))
    return out, 0.1 * math.log(s["factor"]) + 1


def turn(x, angles, gain=1.0):
    """x [..., dim]: coordinate i turns with i + len(angles) by angles[i]; those past the pairs stay."""
    y, half = x.clone(), len(angles)
    for i, a in enumerate(angles):
        c, s = math.cos(a) * gain, math.sin(a) * gain
        y[..., i] = x[..., i] * c - x[..., i + half] * s
        y[..., i + half] = x[..., i + half] * c + x[..., i] * s
    return y


def rotate(x, rot):
    """Rows x [n, heads, dim] at positions 0 .. n - 1."""
    f, gain = frequencies(rot)
    return torch.stack([turn(x[p], [p * w for w in f], gain) for p in range(len(x))])


def turn_values(x, base, sign):
    """Rows x [n, heads, vdim], row p turned by sign * p over all of vdim, with the unscaled frequencies."""
    dv = x.shape[-1]
    return torch.stack([turn(x[p], [sign * p * base ** (-2.0 * m / dv) for m in range(dv // 2)]) for p in range(len(x))])


# ------------------------------------------------------------------ attention
def attend(q, k, v, scale, window=None, softcap=None):
    """q [n, H, dk], k [n, G, dk], v [n, G, dv] -> [n, H, dv]; head h reads key/value head h // (H / G)."""
    n, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = torch.zeros(n, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        for i in range(n):
            lo = 0 if window is None else max(0, i - window + 1)
            s = k[lo:i + 1, g] @ q[i, h] * scale
            if softcap is not None:
                s = softcap * torch.tanh(s / softcap)
            e = torch.exp(s - s.max())
            out[i, h] = (e / e.sum()) @ v[lo:i + 1, g]
    return out


def rotated_attention(h, t, m, eps):
    """Queries and keys normed over all heads at once, then rotated; values rotated by their position and the output
    turned back; capped scores."""
    n, H, G = len(h), m["heads"], m["kv_heads"]
    q = (unit_rms(h @ t["q"].T, eps) * t["q.norm"]).view(n, H, m["dim"])
    k = (unit_rms(h @ t["k"].T, eps) * t["k.norm"]).view(n, G, m["dim"])
    v = turn_values((h @ t["v"].T).view(n, G, m["vdim"]), m["rot"]["base"], 1)
    o = attend(rotate(q, m["rot"]), rotate(k, m["rot"]), v, m["scale"], softcap=m["softcap"])
    return turn_values(o, m["rot"]["base"], -1).reshape(n, -1) @ t["o"].T


def key_value_attention(h, t, m, eps):
    """The values are the keys as projected (with their bias); a window."""
    n, H, G = len(h), m["heads"], m["kv_heads"]
    q, v = h @ t["q"].T + t["q.b"], h @ t["k"].T + t["k.b"]
    k = (unit_rms(v, eps) * t["k.norm"]).view(n, G, m["dim"])
    q = (unit_rms(q, eps) * t["q.norm"]).view(n, H, m["dim"])
    o = attend(rotate(q, m["rot"]), rotate(k, m["rot"]), v.view(n, G, m["dim"]), m["scale"], window=m["mask"]["size"])
    return o.reshape(n, -1) @ t["o"].T


# ------------------------------------------------------------------ recurrences
def lightning_recurrence(q, k, v, decay):
    """q, k [n, H, dk], v [n, H, dv], decay [H] -> [n, H, dv]."""
    n, H = q.shape[:2]
    out = torch.zeros_like(v)
    for h in range(H):
        S = torch.zeros(q.shape[2], v.shape[2], dtype=q.dtype)
        for t in range(n):
            S = decay[h] * S + torch.outer(k[t, h], v[t, h])
            out[t, h] = S.T @ q[t, h]
    return out


def lightning(h, t, m, eps):
    n, H = len(h), m["heads"]
    q, k, v = (silu(h @ t[x].T).view(n, H, d) for x, d in (("q", m["dim"]), ("k", m["dim"]), ("v", m["vdim"])))
    o = lightning_recurrence(q, k, v, m["decay"]).reshape(n, -1)
    return (unit_rms(o, eps) * t["norm"] * sigmoid(h @ t["g"].T)) @ t["o"].T


def general_delta_recurrence(r, k, v, w, a):
    """All [n, H, d]; w the decays, a the removal rates of the key channels -> [n, H, d]."""
    n, H, d = r.shape
    out = torch.zeros_like(v)
    for h in range(H):
        S = torch.zeros(d, v.shape[2], dtype=r.dtype)
        for t in range(n):
            u = unit_length(k[t, h])
            S = w[t, h][:, None] * S - torch.outer(a[t, h] * u, S.T @ u) + torch.outer(k[t, h], v[t, h])
            out[t, h] = S.T @ r[t, h]
    return out


def general_delta_decay(h, t):
    return torch.exp(-math.exp(-0.5) * sigmoid(torch.tanh(h @ t["w1"].T) @ t["w2"].T + t["w0"]))


def general_delta(h, t, m, eps):
    n, H, d = len(h), m["heads"], m["dim"]
    r, k, v = ((h @ t[x].T).view(n, H, d) for x in "rkv")
    w, a = general_delta_decay(h, t).view(n, H, d), sigmoid(h @ t["a"].T + t["a.b"]).view(n, H, d)
    o = unit_rms(general_delta_recurrence(r, k, v, w, a), eps).reshape(n, -1)
    return (o * t["norm"] * sigmoid(h @ t["g"].T)) @ t["o"].T


def gated_delta_recurrence(q, k, v, g, beta):
    """q, k [n, G, dk] (as convolved), v [n, H, dv], g, beta [n, H] -> [n, H, dv]."""
    n, G, dk = q.shape
    H = v.shape[1]
    out = torch.zeros_like(v)
    for h in range(H):
        S, j = torch.zeros(dk, v.shape[2], dtype=q.dtype), h // (H // G)
        for t in range(n):
            kt, qt = unit_length(k[t, j]), unit_length(q[t, j]) * dk ** -0.5
            S = g[t, h] * S
            S = S + torch.outer(kt, beta[t, h] * (v[t, h] - S.T @ kt))
            out[t, h] = S.T @ qt
    return out


def gated_delta(h, t, m, eps):
    n, H, G = len(h), m["heads"], m["kv_heads"]
    q, k, v = (silu(short_conv(h @ t[x].T, t[f"{x}.conv"])) for x in "qkv")
    g = torch.exp(-torch.exp(t["A_log"]) * softplus(h @ t["a"].T + t["dt_bias"]))
    o = gated_delta_recurrence(q.view(n, G, m["dim"]), k.view(n, G, m["dim"]), v.view(n, H, m["vdim"]), g, sigmoid(h @ t["b"].T))
    o = unit_rms(o, eps) * t["norm"] * silu(h @ t["g"].T).view(n, H, m["vdim"])
    return o.reshape(n, -1) @ t["o"].T


# ------------------------------------------------------------------ mixers and feed-forward
def parallel(h, t, m, eps):
    return m["left_scale"] * rotated_attention(h, sub(t, "left."), m["left"], eps) + m["right_scale"] * lightning(h, sub(t, "right."), m["right"], eps)


def parallel_2(h, t, m, eps):
    return m["left_scale"] * key_value_attention(h, sub(t, "left."), m["left"], eps) + m["right_scale"] * general_delta(h, sub(t, "right."), m["right"], eps)


def feed_forward(h, t):
    return torch.clamp(h @ t["up"].T, min=0) ** 2 @ t["down"].T


def route(z, top):
    """(expert ids, weights) of one token from its router logits z [E]."""
    s = torch.exp(z - z.max())
    s = s / s.sum()
    ids = sorted(range(len(z)), key=lambda e: (-float(s[e]), e))[:top]
    return ids, s[ids] / (s[ids].sum() + 1e-20)


def mixture(h, t, mlp):
    out = torch.zeros_like(h)
    z = h @ t["router"].T
    for i in range(len(h)):
        for e, w in zip(*route(z[i], mlp["router"]["top"])):
            out[i] += w * feed_forward(h[i], sub(t, f"e{e}."))
    return out + feed_forward(h, sub(t, "shared.")) if mlp.get("shared") else out


# ------------------------------------------------------------------ the model
MIXERS = {"parallel": parallel, "parallel_2": parallel_2, "delta": gated_delta}


def sub(tensors, prefix):
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


def layer(x, t, L, eps):
    def sublayer(x, q, f):
        y = f(x + short_conv(x, t[f"canon{q}"]))
        return x + unit_rms(y, eps) * (1 + t[f"norm{q}"])

    x = sublayer(x, 1, lambda h: MIXERS[L["type"]](h, sub(t, "mix."), L["mixer"], eps))
    return x if L["mlp"] is None else sublayer(x, 2, lambda h: mixture(h, sub(t, "mlp."), L["mlp"]))


def forward(cfg, tensors, tokens, dtype=torch.float64, layers=False):
    """Logits [n, vocab] of one whole sequence (and, with `layers`, the stream after every layer)."""
    t = {k: v.to(dtype) for k, v in tensors.items()}
    eps, trace = cfg["norm"]["eps"], []
    x = t["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    for i, L in enumerate(cfg["layers"]):
        x = layer(x, sub(t, f"l{i}."), L, eps)
        trace.append(x)
    logits = unit_rms(x, eps) * (1 + t["final.norm"]) @ t["embed"].T * cfg["logit_scale"]
    return (logits, torch.stack(trace)) if layers else logits
