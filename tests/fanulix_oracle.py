"""Plain, slow statement of the Fanulix decoder in fp64: one function per mechanism, whole sequences, no caches.

`cfg` is the dictionary of a config.json, `w` maps checkpoint names to tensors.  Nothing here is shared with the package."""
import math

import torch

F64 = torch.float64


def rms(v, eps):
    return v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)


def layer_norm(v, weight, bias, eps):
    d = v - v.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * weight + bias


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def rotate(vec, position, rot):
    """vec [..., D] at one position: value i of the first rot.dims turns with value i + dims/2."""
    out, n = vec.clone(), rot["dims"]
    for i in range(n // 2):
        a = position * rot["base"] ** (-2.0 * i / n)
        u, v = vec[..., i], vec[..., i + n // 2]
        out[..., i] = u * math.cos(a) - v * math.sin(a)
        out[..., i + n // 2] = v * math.cos(a) + u * math.sin(a)
    return out


# ---- softmax attention ---------------------------------------------------------------------------------
def temperature(position, q_temp):
    return 1.0 + q_temp["coef"] * math.log(math.floor((position + 1) / q_temp["every"]) + 1.0)


def sink_softmax(s):
    """exp(s_j) / (1 + sum exp(s_j))."""
    top = max(float(s.max()), 0.0)
    e = torch.exp(s - top)
    return e / (math.exp(-top) + e.sum())


def attention_heads(q, k, v, m, eps):
    """q [T, H, D], k [T, G, D], v [T, G, V] as projected (biases included) -> heads' outputs [T, H * V] before the gate."""
    T, H, G = q.shape[0], m["heads"], m["kv_heads"]
    q = rms(q, eps) * torch.tensor([temperature(p, m["q_temp"]) for p in range(T)], dtype=F64)[:, None, None]
    k = rms(k, eps)
    out = torch.zeros(T, H, v.shape[-1], dtype=F64)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * m["scale"]
        for t in range(T):
            out[t, h] = sink_softmax(s[t, :t + 1]) @ v[:t + 1, g]
    return out.reshape(T, -1)


def attention(h, w, p, m, eps):
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T + w[p + "q.b"]).reshape(T, H, D)
    k = (h @ w[p + "k"].T + w[p + "k.b"]).reshape(T, G, D)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).reshape(T, G, V)
    return (attention_heads(q, k, v, m, eps) * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


# ---- recurrences -----------------------------------------------------------------------------------------
def linear_scan(q, k, v, decay):
    """S <- decay_t S + k_t v_t^T, o_t = S^T q_t per head: q, k [T, H, N], v [T, H, V], decay [T, H]."""
    S = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=F64)
    out = []
    for t in range(q.shape[0]):
        S = decay[t][:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out)


def retention_heads(q, k, v, m):
    """q, k [T, H, D], v [T, H, V] as projected -> heads' read-outs [T, H, V] before their norm."""
    T = q.shape[0]
    q = torch.stack([rotate(q[t], t, m["rot"]) for t in range(T)])
    k = torch.stack([rotate(k[t], t, m["rot"]) for t in range(T)]) * m["dim"] ** -0.5
    return linear_scan(q, k, v, torch.tensor(m["decay"], dtype=F64).expand(T, -1))


def retention(h, w, p, m, eps):
    T, H = h.shape[0], m["heads"]
    q, k, v = ((h @ w[p + n].T).reshape(T, H, -1) for n in ("q", "k", "v"))
    o = rms(retention_heads(q, k, v, m), eps).reshape(T, -1)
    return (o * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def causal_conv(x, taps, bias):
    """x [T, C], taps [C, n]: channel c of token t is bias + sum_j taps[c, n - 1 - j] x[t - j], zeros before the start."""
    n = taps.shape[1]
    past = torch.cat([torch.zeros(n - 1, x.shape[1], dtype=F64), x])
    return sum(past[n - 1 - j:past.shape[0] - j] * taps[:, n - 1 - j] for j in range(n)) + bias


def mamba2_heads(x, B, C, dt, a_log, d, m):
    """x [T, H, V], B and C [T, G, N], dt [T, H] after the softplus -> y [T, H, V]."""
    of = [h // (m["heads"] // m["groups"]) for h in range(m["heads"])]
    decay = torch.exp(-torch.exp(a_log) * dt)
    return linear_scan(C[:, of], dt[:, :, None] * B[:, of], x, decay) + d[:, None] * x


def mamba2_gate_norm(y, z, weight, m, eps):
    g = y * silu(z)
    return rms(g.reshape(g.shape[0], m["norm_groups"], -1), eps).reshape(g.shape) * weight


def mamba2(h, w, p, m, eps):
    T, H, G, N, V = h.shape[0], m["heads"], m["groups"], m["state"], m["vdim"]
    inner = H * V
    z, xbc, dt = (h @ w[p + "in"].T).split([inner, inner + 2 * G * N, H], -1)
    x, B, C = silu(causal_conv(xbc, w[p + "conv"], w[p + "conv.b"])).split([inner, G * N, G * N], -1)
    y = mamba2_heads(x.reshape(T, H, V), B.reshape(T, G, N), C.reshape(T, G, N), softplus(dt + w[p + "dt_bias"]), w[p + "A_log"],
                     w[p + "D"], m)
    return mamba2_gate_norm(y.reshape(T, inner), z, w[p + "norm"], m, eps) @ w[p + "o"].T


def mixer(kind, h, w, p, m, eps):
    if kind == "mamba2":
        return mamba2(h, w, p, m, eps)
    return (m["left_scale"] * attention(h, w, p + "left.", m["left"], eps)
            + m["right_scale"] * retention(h, w, p + "right.", m["right"], eps))


# ---- feed-forward ------------------------------------------------------------------------------------------
def route(z, top):
    """Router logits of one token -> (chosen experts, their weights)."""
    s = torch.exp(z - z.max())
    s = s / s.sum()
    chosen = sorted(range(len(z)), key=lambda e: -float(s[e]))[:top]
    return chosen, s[chosen] / (s[chosen].sum() + 1e-20)


def expert(h, w, p):
    return gelu(h @ w[p + "up"].T) @ w[p + "down"].T


def mixture(h, w, p, mlp):
    z = h @ w[p + "router"].T
    out = expert(h, w, p + "shared.")
    share = torch.zeros(h.shape[0], mlp["router"]["experts"], dtype=F64)
    for t in range(h.shape[0]):
        chosen, weight = route(z[t], mlp["router"]["top"])
        share[t, chosen] = weight
    for e in range(mlp["router"]["experts"]):
        at = (share[:, e] > 0).nonzero().flatten()
        if len(at):
            out[at] += share[at, e, None] * expert(h[at], w, f"{p}e{e}.")
    return out


# ---- streams -------------------------------------------------------------------------------------------------
def sublayer(xs, w, p, q, f, eps):
    """xs [s, T, W]: one sublayer's input from all streams, its output back into all of them."""
    u = torch.einsum("s,stw->tw", w[f"{p}hc{q}.in"], xs)
    y = f(layer_norm(u, w[f"{p}norm{q}"], w[f"{p}norm{q}.b"], eps))
    return torch.einsum("sr,stw->rtw", w[f"{p}hc{q}.mix"], xs) + w[f"{p}hc{q}.out"][:, None, None] * y


def hidden_states(cfg, w, tokens):
    """Sum of the streams after every layer."""
    w = {k: t.to(F64) for k, t in w.items()}
    eps = cfg["norm"]["eps"]
    xs = w["embed"][torch.tensor(tokens)].expand(cfg["streams"], -1, -1)
    out = []
    for n, layer in enumerate(cfg["layers"]):
        p = f"l{n}."
        xs = sublayer(xs, w, p, 1, lambda h: mixer(layer["type"], h, w, p + "mix.", layer["mixer"], eps), eps)
        if layer["mlp"] is not None:
            xs = sublayer(xs, w, p, 2, lambda h: mixture(h, w, p + "mlp.", layer["mlp"]), eps)
        out.append(xs.sum(0))
    return out


def logits(cfg, w, tokens):
    x = hidden_states(cfg, w, tokens)[-1]
    h = layer_norm(x, w["final.norm"].to(F64), w["final.norm.b"].to(F64), cfg["norm"]["eps"])
    return h @ w["embed"].to(F64).T * cfg["logit_scale"]


def greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(logits(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]
