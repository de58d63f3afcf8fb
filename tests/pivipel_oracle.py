"""Plain, slow restatement of the Pivipel decoder, one function per mechanism, written from the equations alone. It
shares no code with the package: every sequence is processed whole, with explicit loops over heads, queries and
experts, in the dtype of the inputs (float64 unless a caller asks otherwise).

Shapes: a sequence's hidden rows are [n, width], its streams [streams, n, width]; weights are [out, in].
"""
import math

import torch


# ------------------------------------------------------------------ pieces
def dynamic_tanh(x, alpha, w, b):
    return torch.tanh(alpha * x) * w + b


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def frequencies(rot):
    """The rotary frequencies of a layer: slow ones divided by the factor, a linear blend between the two wavelengths."""
    out, s = [], rot.get("scaling")
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        if s:
            wave = 2 * math.pi / f
            if wave > s["original"] / s["low"]:
                f = f / s["factor"]
            elif not wave < s["original"] / s["high"]:
                blend = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
                f = (1 - blend) * f / s["factor"] + blend * f
        out.append(f)
    return out


def rotate(x, pos, rot):
    """x [..., dim] at position `pos`: coordinate i turns with i + dims / 2, those from dims on stay."""
    y, half = x.clone(), rot["dims"] // 2
    for i, f in enumerate(frequencies(rot)):
        c, s = math.cos(pos * f), math.sin(pos * f)
        y[..., i] = x[..., i] * c - x[..., i + half] * s
        y[..., i + half] = x[..., i + half] * c + x[..., i] * s
    return y


def visible(i, mask):
    """The positions that position i sees."""
    size, keep = mask.get("size"), mask.get("keep_first", 0)
    return [j for j in range(i + 1) if size is None or i - j < size or j < keep]


def attend(q, k, v, mask, scale, sink=None):
    """q [n, H, dk], k [n, G, dk], v [n, G, dv] -> [n, H, dv]; head h reads key/value head h // (H / G)."""
    n, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = torch.zeros(n, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        for i in range(n):
            js = visible(i, mask)
            s = k[js, g] @ q[i, h] * scale
            top = s.max() if sink is None else torch.maximum(s.max(), sink[h])
            e = torch.exp(s - top)
            out[i, h] = (e / (e.sum() + (0 if sink is None else torch.exp(sink[h] - top)))) @ v[js, g]
    return out


def heads_of(h, t, m):
    n = h.shape[0]
    return ((h @ t["q"].T).view(n, m["heads"], m["dim"]), (h @ t["k"].T).view(n, m["kv_heads"], m["dim"]),
            (h @ t["v"].T).view(n, m["kv_heads"], m["vdim"]))


def sink_attention(h, t, m, eps):
    """Rotated queries and keys, a window, a learned sink per head, one gate per head."""
    n = h.shape[0]
    q, k, v = heads_of(h, t, m)
    if m.get("rot"):
        q, k = (torch.stack([rotate(x[p], p, m["rot"]) for p in range(n)]) for x in (q, k))
    o = attend(q, k, v, m.get("mask") or {}, m["scale"], t["sink"])
    return (o * sigmoid(h @ t["g"].T)[:, :, None]).reshape(n, -1) @ t["o"].T


def normed_attention(h, t, m, eps):
    """Queries and keys normed per head, no positions, a window beside kept first tokens, a gate per element."""
    n = h.shape[0]
    q, k, v = heads_of(h, t, m)
    o = attend(rms_norm(q, t["q.norm"], eps), rms_norm(k, t["k.norm"], eps), v, m.get("mask") or {}, m["scale"])
    return (o.reshape(n, -1) * sigmoid(h @ t["g"].T)) @ t["o"].T


def feed_forward(h, t, limit):
    g = (h @ t["gate"].T).clamp(max=limit)
    u = (h @ t["up"].T).clamp(-limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ t["down"].T


def route(z, r):
    """(expert ids, weights) of one token from its router logits z [E]."""
    E, n = r["experts"], (r.get("groups") or {}).get("count", 1)
    s = torch.exp(z - z.max())
    s = s / s.sum()
    size, keep = E // n, (r.get("groups") or {}).get("keep", 1)
    best = sorted(range(n), key=lambda g: (-float(s[g * size:(g + 1) * size].max()), g))[:keep]
    ids = [e for e in range(E) if e // size in best]
    ids = sorted(ids, key=lambda e: (-float(s[e]), e))[:r["top"]]
    return ids, s[ids] * r.get("scale", 1.0)


def mixture(h, t, mlp):
    out = torch.zeros_like(h)
    z = h @ t["router"].T
    for i in range(len(h)):
        ids, w = route(z[i], mlp["router"])
        for e, we in zip(ids, w):
            out[i] += we * feed_forward(h[i], sub(t, f"e{e}."), mlp["expert"]["limit"])
    if mlp.get("shared"):
        out = out + feed_forward(h, sub(t, "shared."), mlp["shared"]["limit"]) * sigmoid(h @ t["shared.sg"].T)
    return out


def read_streams(xs, w_in):
    return sum(w_in[s] * xs[s] for s in range(len(xs)))


def write_streams(xs, y, w_mix, w_out):
    """Every stream anew from all the old ones (w_mix is [from, to]) and the sublayer's output."""
    return torch.stack([sum(w_mix[s, t] * xs[s] for s in range(len(xs))) + w_out[t] * y for t in range(len(xs))])


# ------------------------------------------------------------------ the model
MIXERS = {"attention": sink_attention, "attention_2": normed_attention}


def sub(tensors, prefix):
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


def norm(x, t, name):
    return dynamic_tanh(x, t[f"{name}.alpha"], t[name], t[f"{name}.b"])


def layer(xs, t, L, eps):
    def sublayer(xs, q, f):
        hc = sub(t, f"hc{q}.")
        y = f(norm(read_streams(xs, hc["in"]), t, f"norm{q}"))
        return write_streams(xs, y, hc["mix"], hc["out"])

    xs = sublayer(xs, 1, lambda h: MIXERS[L["type"]](h, sub(t, "mix."), L["mixer"], eps))
    mlp, mt = L["mlp"], sub(t, "mlp.")
    if mlp is None:
        return xs
    if mlp["kind"] == "moe":
        return sublayer(xs, 2, lambda h: mixture(h, mt, mlp))
    return sublayer(xs, 2, lambda h: feed_forward(h, mt, mlp["limit"]))


def owner(layers, i):
    """The layer whose tensors layer i uses."""
    while layers[i].get("weights_of") is not None:
        i = layers[i]["weights_of"]
    return i


def forward(cfg, tensors, tokens, dtype=torch.float64, layers=False):
    """Logits [n, vocab] of one whole sequence (and, with `layers`, the summed streams after every layer)."""
    t = {k: v.to(dtype) for k, v in tensors.items()}
    n, L = len(tokens), cfg["layers"]
    x = norm(t["embed"][torch.as_tensor(tokens, dtype=torch.long)] + t["pos"][:n], t, "embed.norm")
    xs, trace = torch.stack([x] * cfg["streams"]), []
    for i in range(len(L)):
        xs = layer(xs, sub(t, f"l{owner(L, i)}."), L[i], cfg["norm"]["eps"])
        trace.append(xs.sum(0))
    logits = norm(xs.sum(0), t, "final.norm") @ t["embed"].T
    return (logits, torch.stack(trace)) if layers else logits
