"""Plain, slow statement of the Fogizen decoder in fp64: one function per mechanism, whole sequences, no caches.

`cfg` is the dictionary of a config.json, `w` maps checkpoint names to tensors.  Nothing here is shared with the package."""
import math

import torch

F64 = torch.float64


def rms(v, eps):
    return v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def before(h):
    """The previous token's row, zeros for the first token."""
    return torch.cat([torch.zeros_like(h[:1]), h[:-1]])


def blend(h, mu):
    """Between a token's row (mu 0) and the previous token's (mu 1), element by element."""
    return h + (before(h) - h) * mu


# ---- embedding -------------------------------------------------------------------------------------------
def bigram_rows(tokens, b):
    rows, last = [], None
    for t in tokens:
        rows.append(b["buckets"] if last is None else (last * b["mul_prev"] + t * b["mul_cur"]) % b["buckets"])
        last = t
    return rows


def embedding(cfg, w, tokens):
    return w["embed"][torch.tensor(tokens)] + w["bigram"][torch.tensor(bigram_rows(tokens, cfg["embedding"]["bigram"]))]


# ---- softmax attention -----------------------------------------------------------------------------------
def rotate(vec, position, rot):
    """vec [..., D] at one position: of the first rot.dims values 2i turns with 2i + 1."""
    out, n = vec.clone(), rot["dims"]
    for i in range(n // 2):
        a = position * rot["base"] ** (-2.0 * i / n) / rot["scaling"]["factor"]
        u, v = vec[..., 2 * i], vec[..., 2 * i + 1]
        out[..., 2 * i] = u * math.cos(a) - v * math.sin(a)
        out[..., 2 * i + 1] = v * math.cos(a) + u * math.sin(a)
    return out


def sink_softmax(s, sink):
    """exp(s_j) / (exp(sink) + sum exp(s_j))."""
    top = max(float(s.max()), float(sink))
    e = torch.exp(s - top)
    return e / (math.exp(float(sink) - top) + e.sum())


def attention_heads(q, k, v, m, q_norm, k_norm, talk, sink, eps):
    """q [T, H, D], k [T, G, D], v [T, G, V] as projected (biases included) -> heads' outputs [T, H, V] before the gate."""
    T, H, G = q.shape[0], m["heads"], m["kv_heads"]
    q, k = rms(q, eps) * q_norm, rms(k, eps) * k_norm
    q = torch.stack([rotate(q[t], t, m["rot"]) for t in range(T)])
    k = torch.stack([rotate(k[t], t, m["rot"]) for t in range(T)])
    raw = torch.stack([q[:, g] @ k[:, g // (H // G)].T for g in range(H)]) * m["scale"]
    out = torch.zeros(T, H, v.shape[-1], dtype=F64)
    for h in range(H):
        s = sum(talk[h, g] * raw[g] for g in range(H))
        for t in range(T):
            lo = t // m["mask"]["size"] * m["mask"]["size"]
            out[t, h] = sink_softmax(s[t, lo:t + 1], sink[h]) @ v[lo:t + 1, h // (H // G)]
    return out


def attention(h, w, p, m, eps):
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T + w[p + "q.b"]).reshape(T, H, D)
    k = (h @ w[p + "k"].T + w[p + "k.b"]).reshape(T, G, D)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).reshape(T, G, V)
    o = attention_heads(q, k, v, m, w[p + "q.norm"], w[p + "k.norm"], w[p + "talk"], w[p + "sink"], eps)
    return (o * sigmoid(h @ w[p + "g"].T)[:, :, None]).reshape(T, -1) @ w[p + "o"].T


# ---- time mixing -----------------------------------------------------------------------------------------
def decay_of(x, w, p):
    return torch.exp(-torch.exp(torch.tanh(x @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"]))


def bonus_scan(r, k, v, decay, u):
    """o_t = (S + diag(u) k_t v_t^T)^T r_t, S <- diag(decay_t) S + k_t v_t^T per head: r, k, v, decay [T, H, D], u [H, D]."""
    S = torch.zeros(r.shape[1], r.shape[2], v.shape[2], dtype=F64)
    out = []
    for t in range(r.shape[0]):
        new = k[t][:, :, None] * v[t][:, None, :]
        out.append(((S + u[:, :, None] * new) * r[t][:, :, None]).sum(1))
        S = decay[t][:, :, None] * S + new
    return torch.stack(out)


def time_mixing(h, w, p, m, eps):
    T, shape = h.shape[0], (h.shape[0], m["heads"], m["dim"])
    r, k, v = ((blend(h, w[f"{p}mu.{n}"]) @ w[p + n].T).reshape(shape) for n in "rkv")
    gate = silu(blend(h, w[p + "mu.g"]) @ w[p + "g"].T)
    decay = decay_of(blend(h, w[p + "mu.w"]), w, p).reshape(shape)
    o = rms(bonus_scan(r, k, v, decay, w[p + "u"]), eps).reshape(T, -1)
    return (o * w[p + "norm"] * gate) @ w[p + "o"].T


def mixer(h, w, p, m, eps):
    left = rms(attention(h, w, p + "left.", m["left"], eps), eps) * w[p + "left.out"]
    right = rms(time_mixing(h, w, p + "right.", m["right"], eps), eps) * w[p + "right.out"]
    return 0.5 * (left + right)


# ---- feed-forward ----------------------------------------------------------------------------------------
def xielu(z, p, q):
    return torch.where(z > 0, softplus(p) * z * z, (0.5 + softplus(q)) * (torch.expm1(z) - z)) + 0.5 * z


def dense(h, w, p):
    return xielu(h @ w[p + "up"].T, w[p + "act"][0], w[p + "act"][1]) @ w[p + "down"].T


def route(z, correction, r):
    """Router logits of one token -> (chosen experts, their weights)."""
    s = sigmoid(z)
    c = s + correction
    n = len(z) // r["groups"]["count"]
    score = [float(c[g * n:(g + 1) * n].sort(descending=True).values[:2].sum()) for g in range(r["groups"]["count"])]
    best = sorted(range(len(score)), key=lambda g: -score[g])[:r["groups"]["keep"]]
    open_ = [e for e in range(len(z)) if e // n in best]
    chosen = sorted(open_, key=lambda e: -float(c[e]))[:r["top"]]
    return chosen, s[chosen] / (s[chosen].sum() + 1e-20) * r["scale"]


def expert(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def mixture(h, w, p, mlp):
    z, out = h @ w[p + "router"].T, torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, weight in zip(*route(z[t], w[p + "correction"], mlp["router"])):
            out[t] += weight * expert(h[t:t + 1], w, f"{p}e{e}.")[0]
    return out


def feed_forward(h, w, p, mlp):
    if mlp is None:
        return 0.0
    return dense(h, w, p) if mlp["kind"] == "dense" else mixture(h, w, p, mlp)


# ---- model -----------------------------------------------------------------------------------------------
def hidden_states(cfg, w, tokens):
    """Residual after every layer."""
    w = {k: t.to(F64) for k, t in w.items()}
    eps = cfg["norm"]["eps"]
    x = embedding(cfg, w, tokens)
    out = []
    for n, layer in enumerate(cfg["layers"]):
        p = f"l{n}."
        h = rms(x, eps) * w[p + "norm1"]
        x = x + mixer(blend(h, w[p + "shift"]), w, p + "mix.", layer["mixer"], eps) + feed_forward(h, w, p + "mlp.", layer["mlp"])
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
