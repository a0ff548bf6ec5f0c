"""Plain, slow statement of the Domilix decoder in fp64: one function per mechanism, whole sequences, no caches.

`cfg` is the dictionary of a config.json, `w` maps checkpoint names to tensors.  Nothing here is shared with the package."""
import math

import torch

F64 = torch.float64


def rms(v, eps):
    return v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)


def rotate_pairs(vec, position, rot):
    """vec [..., D] at one position: neighbours (2i, 2i + 1) of the first rot.dims values turn by position * base^(-2i/dims)."""
    out = vec.clone()
    for i in range(rot["dims"] // 2 if rot else 0):
        a = position * rot["base"] ** (-2.0 * i / rot["dims"])
        c, s = math.cos(a), math.sin(a)
        u, v = vec[..., 2 * i], vec[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def queries(h, w, p, m, eps):
    """-> (content part [T, H, dim], rotated part [T, H, rot_dim])."""
    T, H, D, R = h.shape[0], m["heads"], m["dim"], m["rot_dim"]
    low = rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]
    q = (low @ w[p + "uq"].T).reshape(T, H, D + R)
    turned = torch.stack([rotate_pairs(q[t, :, D:], t, m.get("rot")) for t in range(T)])
    return q[:, :, :D], turned


def latents(h, w, p, m, eps):
    """What a layer caches: (latent [T, kv_rank], rotated key part [T, rot_dim] common to all heads)."""
    C = m["kv_rank"]
    z = h @ w[p + "dkv"].T
    c = rms(z[:, :C], eps) * w[p + "dkv.norm"]
    return c, torch.stack([rotate_pairs(z[t, C:], t, m.get("rot")) for t in range(z.shape[0])])


def softmax_row(s):
    e = torch.exp(s - s.max())
    return e / e.sum()


def latent_attention(h, c, kr, w, p, m, eps):
    """Heads' outputs before the output projection, with latent c and rotated key part kr (this layer's or another one's)."""
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    qc, qr = queries(h, w, p, m, eps)
    k = (c @ w[p + "uk"].T).reshape(T, H, D)
    v = (c @ w[p + "uv"].T).reshape(T, H, V)
    gate = 1.0 / (1.0 + torch.exp(-(h @ w[p + "g"].T)))
    out = torch.zeros(T, H, V, dtype=F64)
    for i in range(H):
        s = (qc[:, i] @ k[:, i].T + qr[:, i] @ kr.T) * m["scale"]
        for t in range(T):
            out[t, i] = gate[t, i] * (softmax_row(s[t, :t + 1]) @ v[:t + 1, i])
    return out.reshape(T, H * V)


def relu(z):
    return torch.clamp(z, min=0.0)


def dense_mlp(h, w, p):
    return (relu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(z, top):
    """Router logits of one token -> (chosen experts, their weights)."""
    chosen = sorted(range(len(z)), key=lambda e: -float(z[e]))[:top]
    return chosen, softmax_row(z[chosen])


def expert(h, w, p):
    return (relu(h @ w[p + "up"].T) ** 2) @ w[p + "down"].T


def mixture(h, w, p, mlp):
    z = h @ w[p + "router"].T + w[p + "router.b"]
    out = torch.zeros_like(h)
    share = torch.zeros(h.shape[0], mlp["router"]["experts"], dtype=F64)
    for t in range(h.shape[0]):
        chosen, weight = route(z[t], mlp["router"]["top"])
        share[t, chosen] = weight
    for e in range(mlp["router"]["experts"]):
        at = (share[:, e] > 0).nonzero().flatten()
        if len(at):
            out[at] += share[at, e, None] * expert(h[at], w, f"{p}e{e}.")
    return out


def hidden_states(cfg, w, tokens):
    """Residual stream after every layer."""
    w = {k: t.to(F64) for k, t in w.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    out, kept = [], {}
    for n, layer in enumerate(cfg["layers"]):
        p, m = f"l{n}.", layer["mixer"]
        src = m.get("kv_from")
        if src is None:
            kept[n] = latents(x, w, p + "mix.", m, eps)
        c, kr = kept[n if src is None else src]
        y = latent_attention(x, c, kr, w, p + "mix.", m, eps) @ w[p + "mix.o"].T
        x = x + rms(y, eps) * w[p + "norm1"]
        if layer["mlp"] is not None:
            y = dense_mlp(x, w, p + "mlp.") if layer["mlp"]["kind"] == "dense" else mixture(x, w, p + "mlp.", layer["mlp"])
            x = x + rms(y, eps) * w[p + "norm2"]
        out.append(x)
    return out


def logits(cfg, w, tokens):
    x = hidden_states(cfg, w, tokens)[-1]
    return rms(x, cfg["norm"]["eps"]) * w["final.norm"].to(F64) @ w["head"].to(F64).T


def greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(logits(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]
