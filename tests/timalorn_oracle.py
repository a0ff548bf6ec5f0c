"""Plain, slow statement of the Timalorn decoder in fp64: one function per mechanism, whole sequences, no caches.

`cfg` is the dictionary of a config.json, `w` maps checkpoint names to tensors.  Nothing here is shared with the package."""
import math

import torch

F64 = torch.float64


def layer_norm(x, weight, eps):
    mean = x.mean(-1, keepdim=True)
    var = ((x - mean) ** 2).mean(-1, keepdim=True)
    return (x - mean) / torch.sqrt(var + eps) * weight


def pair_frequencies(rot):
    """Radians per position of every rotated pair, and the factor on cos and sin."""
    dims, base, sc = rot["dims"], rot["base"], rot.get("scaling")
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if sc is None:
        return f, 1.0
    def dim_of(turns):
        return dims * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    low, high = max(math.floor(dim_of(sc["fast"])), 0), min(math.ceil(dim_of(sc["slow"])), dims - 1)
    out = []
    for i, x in enumerate(f):
        ramp = min(1.0, max(0.0, (i - low) / max(high - low, 0.001)))
        out.append((x / sc["factor"]) * ramp + x * (1 - ramp))
    return out, 0.1 * math.log(sc["factor"]) + 1


def rotate(vec, position, rot):
    """vec [heads, D] at one position."""
    if rot is None:
        return vec
    freq, mag = pair_frequencies(rot)
    half = rot["dims"] // 2
    out = vec.clone()
    for i in range(half):
        c, s = math.cos(position * freq[i]) * mag, math.sin(position * freq[i]) * mag
        u, v = vec[:, i], vec[:, i + half]
        out[:, i] = u * c - v * s
        out[:, i + half] = v * c + u * s
    return out


def attention_scores(q, keys, scale, softcap):
    """q [D], keys [n, D]."""
    s = (keys @ q) * scale
    return softcap * torch.tanh(s / softcap) if softcap else s


def sink_softmax(s, sink):
    """Weights of the keys when exp(sink) is part of the denominator."""
    top = max(float(s.max()), float(sink))
    e = torch.exp(s - top)
    return e / (e.sum() + math.exp(float(sink) - top))


def attention(h, w, p, m):
    T, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = (h @ w[p + "q"].T).reshape(T, H, D)
    v = (h @ w[p + "k"].T).reshape(T, G, D)
    rot = m.get("rot")
    k = torch.stack([rotate(v[t], t, rot) for t in range(T)])
    q = torch.stack([rotate(q[t], t, rot) for t in range(T)])
    out = torch.zeros(T, H, D, dtype=F64)
    for t in range(T):
        lo = max(0, t - m["mask"]["size"] + 1)
        for i in range(H):
            g = i // (H // G)
            weights = sink_softmax(attention_scores(q[t, i], k[lo:t + 1, g], m["scale"], m.get("softcap")), w[p + "sink"][i])
            out[t, i] = weights @ v[lo:t + 1, g]
    return out.reshape(T, H * D) @ w[p + "o"].T


def log_gates(h, w, p, cap):
    i = cap * torch.tanh((h @ w[p + "i"].T + w[p + "i.b"]) / cap)
    f = cap * torch.tanh((h @ w[p + "f"].T + w[p + "f.b"]) / cap)
    return i, -torch.log1p(torch.exp(-f))


def mlstm_recurrence(q, k, v, i, f):
    """q, k [T, H, D], v [T, H, V], log gates [T, H] -> read-outs [T, H, V]."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=F64)
    n = torch.zeros(H, D, dtype=F64)
    m = torch.zeros(H, dtype=F64)
    out = []
    for t in range(T):
        top = torch.maximum(f[t] + m, i[t])
        keep, add = torch.exp(f[t] + m - top), torch.exp(i[t] - top)
        m = top
        for a in range(H):
            S[a] = keep[a] * S[a] + add[a] * torch.outer(k[t, a], v[t, a])
            n[a] = keep[a] * n[a] + add[a] * k[t, a]
        row = []
        for a in range(H):
            floor = max(abs(float(n[a] @ q[t, a])), math.exp(-float(m[a])))
            row.append((S[a].T @ q[t, a]) / (floor + 1e-6))
        out.append(torch.stack(row))
    return torch.stack(out)


def head_rms_norm(o, eps):
    return o / torch.sqrt((o * o).mean(-1, keepdim=True) + eps)


def mlstm(h, w, p, m, eps):
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).reshape(T, H, D) / math.sqrt(D)
    k = (h @ w[p + "k"].T).reshape(T, H, D)
    v = (h @ w[p + "v"].T).reshape(T, H, V)
    i, f = log_gates(h, w, p, m["gate_cap"])
    o = head_rms_norm(mlstm_recurrence(q, k, v, i, f), eps).reshape(T, H * V)
    gate = 1 / (1 + torch.exp(-(h @ w[p + "g"].T)))
    return (o * w[p + "norm"] * gate) @ w[p + "o"].T


def feed_forward(h, w, p):
    g = h @ w[p + "gate"].T
    return (g / (1 + torch.exp(-g)) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def hidden_states(cfg, w, tokens):
    """Residual stream after every layer."""
    w = {k: t.to(F64) for k, t in w.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    out = []
    for n, layer in enumerate(cfg["layers"]):
        src = n
        while cfg["layers"][src].get("weights_of") is not None:
            src = cfg["layers"][src]["weights_of"]
        p = f"l{src}."
        h = layer_norm(x, w[p + "norm1"], eps)
        y = attention(h, w, p + "mix.", layer["mixer"]) if layer["type"] == "attention" else \
            mlstm(h, w, p + "mix.", layer["mixer"], eps)
        if layer["mlp"] is not None:
            y = y + feed_forward(h, w, p + "mlp.")
        x = x + y
        out.append(x)
    return out


def logits(cfg, w, tokens):
    x = hidden_states(cfg, w, tokens)[-1]
    return layer_norm(x, w["final.norm"].to(F64), cfg["norm"]["eps"]) @ w["head"].to(F64).T


def greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(logits(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]
