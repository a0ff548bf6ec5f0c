"""Mechanisms of the latent-attention decoder, each alone, against the plain oracle: query and key/value latents, paged attention in
latent space and over expanded keys, ungated experts and their router, post-norm residual.  CPU statements and, marked `gpu`, the
kernels in both compute types."""
import math

import pytest
import torch

import domilix_oracle as O
from stkernel_b200.config import HybridConfig, HybridLayer, LatentAttentionMixer, RotaryConfig
from stkernel_b200.models.hybrid import build_latent
from stkernel_b200.ops import functional as Fn
from stkernel_b200.ops import hybrid as HB
from stkernel_b200.ops import latent as LA
from stkernel_b200.ops import moe as MO
from stkernel_b200.ops import reference as R

CPU = pytest.param(("cpu", torch.float32), id="cpu")
G32 = pytest.param(("cuda:0", torch.float32), id="gpu-f32", marks=pytest.mark.gpu)
G16 = pytest.param(("cuda:0", torch.bfloat16), id="gpu-bf16", marks=pytest.mark.gpu)
ALL = pytest.mark.parametrize("where", [CPU, G32, G16])
GPU = pytest.mark.parametrize("where", [G32, G16])
F64 = torch.float64
PAGE = 64


def rel(got, ref):
    got, ref = got.double().cpu(), ref.double()
    return ((got - ref).norm() / ref.norm().clamp(min=1e-30)).item()


def worst_row(got, ref):
    """Largest relative error over the leading dimension."""
    got, ref = got.double().cpu().flatten(1), ref.double().flatten(1)
    return ((got - ref).norm(dim=1) / ref.norm(dim=1).clamp(min=1e-30)).max().item()


def rand(*shape, seed, scale=1.0, dtype=torch.bfloat16):
    """Random values that bf16 represents exactly, as fp64."""
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * scale).to(dtype).double()


def mixer(heads=4, dim=24, rot=8, vdim=20, q_rank=40, kv_rank=36, scale=None, base=500.0):
    return LatentAttentionMixer(heads, dim, rot, vdim, q_rank, kv_rank, scale or (dim + rot) ** -0.5,
                                RotaryConfig(base, rot, interleaved=True) if rot else None)


def rot_of(m):
    return {"base": m.rotary.base if m.rotary else 1.0, "dims": m.rot_dim}


def params(m, where, seed=0, eps=1e-5):
    dev, dt = where
    w = {"mix.uq": rand(m.heads * (m.dim + m.rot_dim), m.q_rank, seed=seed, scale=m.q_rank ** -0.5),
         "mix.uk": rand(m.heads * m.dim, m.kv_rank, seed=seed + 1, scale=m.kv_rank ** -0.5),
         "mix.uv": rand(m.heads * m.vdim, m.kv_rank, seed=seed + 2, scale=m.kv_rank ** -0.5),
         "mix.dq.norm": 1 + rand(m.q_rank, seed=seed + 3, scale=0.2), "mix.dkv.norm": 1 + rand(m.kv_rank, seed=seed + 4, scale=0.2)}
    cfg = HybridConfig(64, 32, (HybridLayer(m),), eps, block="post_norm", dtype="float32" if dt == torch.float32 else "bfloat16")
    cfg.validate()
    return build_latent(cfg, lambda n: w[n].to(torch.float32).to(dev), m, dt, dev), w


def step(spans, dev, rows):
    """Meta of one step over (start, tokens) spans; rows: request row of each."""
    T = sum(n for _, n in spans)
    tok = torch.cat([torch.full((n,), r, dtype=torch.int32) for r, (_, n) in zip(rows, spans)])
    pos = torch.cat([torch.arange(s, s + n) for s, n in spans])
    first = torch.cat([torch.full((n,), s, dtype=torch.int32) for s, n in spans])
    last = torch.cat([torch.full((n,), s + n - 1, dtype=torch.int32) for s, n in spans])
    qs = torch.tensor([0] + list(torch.tensor([n for _, n in spans]).cumsum(0)), dtype=torch.int32)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
    ns = [n for _, n in spans]
    return HB.HybridMeta(torch.zeros(T, dtype=torch.int64, device=dev), tok.to(dev), pos.to(dev), first.to(dev), last.to(dev),
                         qs.to(dev), i32(rows), i32([s for s, _ in spans]), len(spans), max(ns), max(ns) == 1, min(ns),
                         tuple(spans), max_context=max(s + n for s, n in spans))


def paged(m, where, contexts, seed, rows=None, spread=1.0):
    """A cache holding random latents and key parts for every request, in scattered pages; everything else is NaN."""
    dev, dt = where
    row, off = LA.latent_row(m.kv_rank, m.rot_dim)
    rows = rows or list(range(len(contexts)))
    need = [-(-c // PAGE) for c in contexts]
    order = torch.randperm(sum(need) + 3, generator=torch.Generator().manual_seed(seed)).tolist()
    cache = torch.full((sum(need) + 3, PAGE, row), float("nan"), dtype=torch.float32)
    table = torch.full((max(rows) + 1, max(need) + 2), -1, dtype=torch.int32)
    lat, key = [], []
    for i, c in enumerate(contexts):
        lat.append(rand(c, m.kv_rank, seed=seed + 10 * i, scale=spread))
        key.append(rand(c, m.rot_dim, seed=seed + 10 * i + 1, scale=spread))
        full = torch.zeros(c, row)
        full[:, :m.kv_rank], full[:, off:off + m.rot_dim] = lat[-1], key[-1]
        for p in range(need[i]):
            page = order.pop()
            table[rows[i], p] = page
            part = full[p * PAGE:(p + 1) * PAGE]
            cache[page, :len(part)] = part
    return cache.to(dt).to(dev), table.to(dev), lat, key


def attention_oracle(m, w, qc, qr, gate, lat, key, start, n):
    """One request: qc [n, H, dim], qr [n, H, rot] before rotation, at positions start .. start + n - 1."""
    H, D, V = m.heads, m.dim, m.vdim
    k = (lat @ w["mix.uk"].T).view(-1, H, D)
    v = (lat @ w["mix.uv"].T).view(-1, H, V)
    out = torch.zeros(n, H, V, dtype=F64)
    for t in range(n):
        p = start + t
        q = O.rotate_pairs(qr[t], p, rot_of(m))
        for i in range(H):
            s = (k[:p + 1, i] @ qc[t, i] + key[:p + 1] @ q[i]) * m.scale
            out[t, i] = torch.sigmoid(gate[t, i]) * (O.softmax_row(s) @ v[:p + 1, i])
    return out


def run_attention(m, where, spans, seed=0, sharp=2.0, gated=True):
    dev, dt = where
    a, w = params(m, where, seed)
    T = sum(n for _, n in spans)
    rows = [2 * i + 1 for i in range(len(spans))][::-1]
    cache, table, lat, key = paged(m, where, [s + n for s, n in spans], seed + 100, rows)
    qc, qr = rand(T, m.heads, m.dim, seed=seed + 7, scale=sharp), rand(T, m.heads, m.rot_dim, seed=seed + 8, scale=sharp)
    gate = rand(T, m.heads, seed=seed + 9)
    q = torch.zeros(T, a.w_uq.out_features)
    q[:, :m.heads * a.dp].view(T, m.heads, a.dp)[:, :, :m.dim] = qc
    q[:, m.heads * a.dp:m.heads * a.dp + m.heads * m.rot_dim] = qr.reshape(T, -1)
    got = LA.latent_attention(q.to(dt).to(dev), gate.float().to(dev) if gated else None, a, step(spans, dev, rows), table, cache)
    got = got.view(T, m.heads, a.vp)
    assert not got[:, :, m.vdim:].any()
    if not gated:
        gate = torch.full_like(gate, 60.0)
    ref, at = [], 0
    for i, (s, n) in enumerate(spans):
        ref.append(attention_oracle(m, w, qc[at:at + n], qr[at:at + n], gate[at:at + n], lat[i], key[i], s, n))
        at += n
    return got[:, :, :m.vdim], torch.cat(ref)


TOL = {torch.float32: 2e-5, torch.bfloat16: 3e-2}
SHAPES = {
    "small": dict(),
    "one_head": dict(heads=1, dim=16, rot=16, vdim=16, kv_rank=16),
    "odd": dict(heads=3, dim=23, rot=6, vdim=21, kv_rank=37),
    "no_rotation": dict(heads=2, dim=40, rot=0, vdim=40, kv_rank=64),
    "row_of_two_panels": dict(heads=6, dim=48, rot=24, vdim=40, kv_rank=72),
    "row_of_three_panels": dict(heads=8, dim=64, rot=64, vdim=64, kv_rank=128),
    "values_reach_the_odd_panel": dict(heads=2, dim=32, rot=10, vdim=32, kv_rank=150),
    "seventeen_heads": dict(heads=17, dim=32, rot=16, vdim=32, kv_rank=96),
    "two_head_groups": dict(heads=40, dim=16, rot=8, vdim=16, kv_rank=48),
    "large": dict(heads=16, dim=128, rot=64, vdim=128, kv_rank=512),
    "wide_rotation": dict(heads=2, dim=24, rot=72, vdim=130, kv_rank=40),
    "widest": dict(heads=2, dim=200, rot=128, vdim=256, kv_rank=600),
    "values_of_seventy": dict(heads=2, dim=70, rot=16, vdim=70, kv_rank=80),
}


@ALL
@pytest.mark.parametrize("shape", list(SHAPES))
def test_decode_rows(where, shape):
    """One token per request, at page and block borders and far from them."""
    spans = [(p, 1) for p in (0, 1, 62, 63, 64, 127, 128, 191, 300)]
    got, ref = run_attention(mixer(**SHAPES[shape]), where, spans, 3)
    assert worst_row(got, ref) < TOL[where[1]]


@GPU
def test_decode_rows_over_many_blocks_and_splits(where):
    got, ref = run_attention(mixer(heads=20, dim=32, rot=16, vdim=24, kv_rank=128), where, [(2047, 1), (1500, 1), (5, 1)], 4)
    assert worst_row(got, ref) < TOL[where[1]]
    got, ref = run_attention(mixer(heads=2), where, [(700 + i, 1) for i in range(40)], 5)
    assert worst_row(got, ref) < TOL[where[1]]


@ALL
@pytest.mark.parametrize("shape", ["small", "odd", "two_head_groups", "row_of_two_panels", "large", "seventeen_heads"])
def test_short_spans(where, shape):
    spans = [(0, 3), (61, 7), (126, 5), (200, 1), (0, 40)]
    if where[0] == "cpu":
        spans = spans[:4]
    got, ref = run_attention(mixer(**SHAPES[shape]), where, spans, 6)
    assert worst_row(got, ref) < TOL[where[1]]


@GPU
@pytest.mark.parametrize("shape", list(SHAPES))
@pytest.mark.parametrize("spans", [[(0, 130)], [(70, 64), (0, 257), (300, 100)], [(0, 64), (511, 1), (129, 300), (64, 9)]],
                         ids=["one", "three", "mixed"])
def test_long_spans(where, shape, spans):
    got, ref = run_attention(mixer(**SHAPES[shape]), where, spans, 8)
    assert worst_row(got, ref) < TOL[where[1]]


@GPU
def test_expanded_heads_in_groups(where, monkeypatch):
    """A bound on the expanded keys and values cuts the heads into several launches with the same result."""
    m = mixer(heads=5, dim=64, rot=32, vdim=64, kv_rank=64)
    whole, ref = run_attention(m, where, [(10, 200)], 11)
    monkeypatch.setattr(LA, "EXPANDED_BYTES", 2 * 256 * 128 * 2)
    parts, _ = run_attention(m, where, [(10, 200)], 11)
    assert torch.equal(whole, parts) and worst_row(parts, ref) < TOL[where[1]]


@ALL
@pytest.mark.parametrize("spans", [[(299, 1)], [(290, 10)], [(200, 100)]], ids=["decode", "short", "long"])
def test_far_key_stands_out(where, spans):
    """One key, at page and block borders, gets nearly all the weight of the last query: leaving it out changes everything."""
    m = mixer(heads=2, dim=32, rot=8, vdim=32, kv_rank=64)
    dev, dt = where
    a, w = params(m, where, 21)
    n = spans[0][1]
    for at in (0, 1, 63, 64, 127, 128, 255, 256, 298):
        cache, table, lat, key = paged(m, where, [300], 22, spread=0.3)
        # the query in latent space of head 0 is the key itself
        target = w["mix.uk"].view(2, 32, 64)[0]
        want = rand(32, seed=23)
        c = torch.linalg.lstsq(target, want).solution
        lat[0][at] = (c / c.norm() * 8).to(torch.bfloat16).double()
        cache[table[0, at // PAGE].long(), at % PAGE, :64] = lat[0][at].to(dt).to(dev)
        qc, qr = rand(n, 2, 32, seed=24, scale=0.1), rand(n, 2, 8, seed=25, scale=0.1)
        qc[-1, 0] = (want / want.norm() * 40).to(torch.bfloat16).double()
        q = torch.zeros(n, a.w_uq.out_features)
        q[:, :2 * a.dp].view(n, 2, a.dp)[:, :, :32] = qc
        q[:, 2 * a.dp:2 * a.dp + 16] = qr.reshape(n, -1)
        got = LA.latent_attention(q.to(dt).to(dev), None, a, step(spans, dev, [0]), table, cache).view(n, 2, a.vp)[-1, 0, :32]
        gate = torch.full((n, 2), 60.0, dtype=F64)
        ref = attention_oracle(m, w, qc, qr, gate, lat[0], key[0], 300 - n, n)[-1, 0]
        assert rel(got, ref) < TOL[dt]
        alone = lat[0][at] @ w["mix.uv"].view(2, 32, 64)[0].T
        assert rel(got, alone) < 0.2


@ALL
@pytest.mark.parametrize("m", [mixer(), mixer(q_rank=300, kv_rank=37, rot=6), mixer(q_rank=2500, kv_rank=520, rot=64, dim=32),
                               mixer(rot=0)], ids=["small", "odd", "large", "no_rotation"])
@pytest.mark.parametrize("own", [True, False])
def test_latents_are_normed_rotated_and_inserted(where, m, own):
    dev, dt = where
    a, w = params(m, where, 31, eps=0.3)
    spans, rows = [(60, 7), (0, 2), (100000, 1)], [1, 0, 2]
    T, off = 10, LA.latent_row(m.kv_rank, m.rot_dim)[1]
    p = rand(T, m.q_rank + m.kv_rank + m.rot_dim + 9, seed=32)
    cache = torch.full((9, PAGE, LA.latent_row(m.kv_rank, m.rot_dim)[0]), 7.0, dtype=dt, device=dev)
    table = torch.full((3, 100000 // PAGE + 1), -1, dtype=torch.int32, device=dev)
    table[1, 0], table[1, 1], table[0, 0], table[2, -1] = 5, 2, 7, 0
    meta = step(spans, dev, rows)
    cq = LA.latent_prep(p.float().to(dev), 4, m.q_rank + 5 if own else -1, a, meta, table, cache, dt)
    ref = O.rms(p[:, 4:4 + m.q_rank], 0.3) * w["mix.dq.norm"]
    assert worst_row(cq[:, :m.q_rank], ref) < TOL[dt] and not cq[:, m.q_rank:].any()
    if not own:
        assert (cache == 7).all()
        return
    z = p[:, m.q_rank + 5:m.q_rank + 5 + m.kv_rank + m.rot_dim]
    c = O.rms(z[:, :m.kv_rank], 0.3) * w["mix.dkv.norm"]
    pos = meta.positions.tolist()
    written = torch.zeros(9, PAGE, dtype=torch.bool)
    for t in range(T):
        page = int(table[int(meta.tok_req[t]), pos[t] // PAGE])
        row = cache[page, pos[t] % PAGE]
        written[page, pos[t] % PAGE] = True
        assert rel(row[:m.kv_rank], c[t]) < TOL[dt]
        if m.rot_dim:
            assert rel(row[off:off + m.rot_dim], O.rotate_pairs(z[t, m.kv_rank:], pos[t], rot_of(m))) < TOL[dt]
        assert not row[m.kv_rank:off].any() and not row[off + m.rot_dim:].any()
    assert (cache.cpu()[~written] == 7).all()


@ALL
def test_rotation_far_from_the_start(where):
    """The angle keeps 32-bit resolution at positions where position * frequency in fp32 alone does not."""
    m = mixer(rot=64, dim=8, base=1e6)
    a, _ = params(m, (where[0], torch.float32), 33)
    pos = 987654
    meta = step([(pos, 1)], where[0], [0])
    table = torch.full((1, pos // PAGE + 1), -1, dtype=torch.int32, device=where[0])
    table[0, -1] = 0
    cache = torch.zeros(1, PAGE, LA.latent_row(m.kv_rank, 64)[0], device=where[0])
    p = rand(1, m.q_rank + m.kv_rank + 64, seed=34)
    LA.latent_prep(p.float().to(where[0]), 0, m.q_rank, a, meta, table, cache, torch.float32)
    off = LA.latent_row(m.kv_rank, 64)[1]
    got = cache[0, pos % PAGE, off:off + 64]
    assert rel(got, O.rotate_pairs(p[0, m.q_rank + m.kv_rank:], pos, rot_of(m))) < 2e-6


# ---- experts ---------------------------------------------------------------------------------------------
def expert_weights(E, W, F, where, seed=41):
    dev, dt = where
    Wp, Fp = (W + 15) // 16 * 16, (F + 15) // 16 * 16
    up, down = rand(E, F, W, seed=seed, scale=W ** -0.5), rand(E, W, F, seed=seed + 1, scale=F ** -0.5)
    pu, pd = torch.zeros(E, Fp, Wp), torch.zeros(E, Wp, Fp)
    pu[:, :F, :W], pd[:, :W, :F] = up, down
    return MO.PlainExperts(pu.to(dt).to(dev), pd.to(dt).to(dev)), up, down, Wp


@ALL
@pytest.mark.parametrize("E,W,F,top,T", [(6, 40, 24, 2, 9), (12, 96, 48, 4, 40), (5, 72, 30, 5, 3), (1, 32, 16, 1, 4), (8, 128, 320, 2, 700),
                                         (64, 256, 128, 6, 300), (3, 200, 136, 1, 150), (512, 64, 16, 8, 70), (4, 88, 72, 3, 257)])
def test_experts_and_their_weighted_sum(where, E, W, F, top, T):
    dev, dt = where
    ex, up, down, Wp = expert_weights(E, W, F, where)
    g = torch.Generator().manual_seed(42)
    # a skewed choice: some experts get many tokens, some none
    score = torch.randn(T, E, generator=g) + torch.linspace(2, -2, E)
    ids = score.topk(top).indices.to(torch.int32)
    wts = torch.softmax(torch.randn(T, top, generator=g), -1)
    h = rand(T, W, seed=43)
    hp = torch.zeros(T, Wp)
    hp[:, :W] = h
    rows = MO.plain_experts(hp.to(dt).to(dev), ids.to(dev), wts.to(dev), ex)
    x = rand(T, W, seed=44).float().to(dev)
    norm = (1 + rand(W, seed=45, scale=0.3))
    out = HB.post_norm_add(x, rows, norm.float().to(dev), 1e-3, Wp, dt)
    ref = torch.zeros(T, W, dtype=F64)
    for t in range(T):
        for j in range(top):
            e = int(ids[t, j])
            ref[t] += wts[t, j].double() * (O.relu(h[t] @ up[e].T) ** 2 @ down[e].T)
    ref = rand(T, W, seed=44) + O.rms(ref, 1e-3) * norm
    assert worst_row(x, ref) < TOL[dt] and worst_row(out[:, :W], ref) < TOL[dt]
    assert not out[:, W:].any()


@ALL
@pytest.mark.parametrize("E,top,W,T", [(6, 2, 40, 5), (12, 4, 96, 8), (300, 8, 64, 4), (512, 32, 48, 33), (1, 1, 32, 3), (7, 7, 80, 130)])
def test_router_takes_the_softmax_over_the_chosen(where, E, top, W, T):
    dev, dt = where
    w, b = rand(E, W, seed=51, scale=W ** -0.5), rand(E, seed=52, scale=3.0)
    h = rand(T, W, seed=53, scale=4.0)
    lw = Fn.LinearWeight(w.to(dt).to(dev))
    hd, bias = h.to(dt).to(dev), b.float().to(dev)
    got = Fn.gate_route(hd, lw, bias, top, "softmax_topk", True, 1.0) if dev != "cpu" else None
    if got is None:
        got = MO.router(Fn.linear(hd, lw, out_dtype=torch.float32), bias, top, "softmax_topk", True, 1.0)
    for t in range(T):
        ids, wt = O.route(h[t] @ w.T + b, top)
        mine = dict(zip(got[0][t].tolist(), got[1][t].tolist()))
        assert set(mine) == set(ids) and all(abs(mine[e] - float(x)) < 1e-4 for e, x in zip(ids, wt))


# ---- residual --------------------------------------------------------------------------------------------
@ALL
@pytest.mark.parametrize("W", [40, 77, 2048, 5000])
def test_post_norm_add_and_final_norm(where, W):
    dev, dt = where
    T, Wp = 7, (W + 15) // 16 * 16
    x0, y, w = rand(T, W, seed=61), rand(T, W, seed=62, scale=0.01), rand(W, seed=63)
    x = x0.float().to(dev)
    h = HB.post_norm_add(x, y.float().to(dev), w.float().to(dev), 1e-4, Wp, dt)
    ref = x0 + O.rms(y, 1e-4) * w
    assert rel(x, ref) < 1e-6 and rel(h[:, :W], ref) < (1e-6 if dt == torch.float32 else 4e-3) and not h[:, W:].any()
    rows = torch.tensor([5, 0, 5], device=dev)
    f = HB.add_layer_norm(x, None, w.float().to(dev), 1e-4, Wp, dt, rows=rows, center=False)
    assert rel(f[:, :W], (O.rms(ref, 1e-4) * w)[[5, 0, 5]]) < (1e-5 if dt == torch.float32 else 4e-3)


@ALL
def test_embedding_leaves_the_compute_copy(where):
    dev, dt = where
    e = rand(30, 41, seed=71)
    ids = torch.tensor([3, 29, 0], device=dev)
    h = torch.full((3, 48), 9.0, dtype=dt, device=dev)
    x = HB.embed_scaled(ids, e.to(dt).to(dev), 0.37, h)
    assert rel(x, e[[3, 29, 0]] * 0.37) < 1e-6 and rel(h[:, :41], e[[3, 29, 0]] * 0.37) < 4e-3 and not h[:, 41:].any()


@ALL
def test_relu_gate(where):
    dev, dt = where
    p = rand(5, 80, seed=72)
    out = torch.full((5, 32), 9.0, dtype=dt, device=dev)
    HB.join_glu(p.to(dt).to(dev), out, 0, (0, 40, 30), "relu")
    assert rel(out[:, :30], O.relu(p[:, :30]) * p[:, 40:70]) < 4e-3 and not out[:, 30:].any()
