"""Mechanisms of the streams decoder, each alone, against the plain oracle: residual streams, grouped attention, retention, Mamba-2 and its
convolution, gelu experts with a shared one.  CPU statements and, marked `gpu`, the kernels in both compute types."""
import pytest
import torch

import fanulix_oracle as O
from stkernel_b200.ops import _lib
from stkernel_b200.ops import functional as Fn
from stkernel_b200.ops import grouped as GA
from stkernel_b200.ops import hybrid as HB
from stkernel_b200.ops import moe as MO
from stkernel_b200.ops import recurrence as RC
from stkernel_b200.ops.latent import split_frequencies
from test_latent_ops import rand, rel, step, worst_row

F32, F64, BF16 = torch.float32, torch.float64, torch.bfloat16
WHERE = pytest.mark.parametrize("where", [
    pytest.param(("cpu", F32), id="cpu"), pytest.param(("cuda:0", F32), id="gpu-f32", marks=pytest.mark.gpu),
    pytest.param(("cuda:0", BF16), id="gpu-bf16", marks=pytest.mark.gpu)])
ids = lambda c: "x".join(str(v) for v in c.values())
al = lambda n: (n + 15) // 16 * 16


def columns(parts, dt):
    """Parts [T, n] side by side on 16-column borders -> (matrix, first column of each)."""
    at, offs = 0, []
    for p in parts:
        offs.append(at)
        at += al(p.shape[1])
    m = torch.full((parts[0].shape[0], at), 7.0, dtype=dt)
    for o, p in zip(offs, parts):
        m[:, o:o + p.shape[1]] = p.to(dt)
    return m, offs


# ---- residual streams ----------------------------------------------------------------------------------
@WHERE
@pytest.mark.parametrize("s,W", [(1, 40), (2, 77), (3, 256), (4, 2048), (5, 36), (8, 4100)])
def test_streams_are_mixed_read_and_normed(where, s, W):
    dev, dt = where
    T, Wp = 6, al(W)
    x0, y = rand(T, s, W, seed=1), rand(T, W, seed=2) + 30.0              # a large mean: the deviations are what counts
    sw = HB.StreamWeights(*(rand(*n, seed=3 + i).float().to(dev) for i, n in enumerate(((s,), (s,), (s, s)))))
    read, w, b = rand(s, seed=7), rand(W, seed=8), rand(W, seed=9)
    mix, write = sw.mix.double().cpu(), sw.write.double().cpu()
    new = torch.einsum("sr,tsw->trw", mix, x0) + write[:, None] * y[:, None]
    args = (read.float().to(dev), w.float().to(dev), b.float().to(dev), 1e-3, Wp, dt)
    tol = 2e-5 if dt == F32 else 4e-3
    want = lambda z: O.layer_norm(torch.einsum("s,tsw->tw", read, z), w, b, 1e-3)
    x = x0.float().to(dev)
    rows = torch.tensor([4, 0, 5], device=dev)
    some = HB.stream_norm(x, y.float().to(dev), sw, *args, rows=rows)
    assert torch.equal(x.double().cpu(), x0) and rel(some[:, :W], want(new)[[4, 0, 5]]) < tol
    first = HB.stream_norm(x, None, None, *args)
    assert torch.equal(x.double().cpu(), x0) and rel(first[:, :W], want(x0)) < tol
    h = HB.stream_norm(x, y.float().to(dev), sw, *args)
    assert rel(x, new) < 1e-6 and rel(h[:, :W], want(new)) < tol and not h[:, W:].any()


@WHERE
@pytest.mark.parametrize("W,copies", [(41, 3), (64, 4), (64, 1)])
def test_embedding_fills_every_stream(where, W, copies):
    dev, dt = where
    e = rand(30, W, seed=11)
    x = HB.embed_scaled(torch.tensor([3, 29, 0], device=dev), e.to(dt).to(dev), 1.0, streams=copies)
    assert x.shape == (3, copies, W) and torch.equal(x.double().cpu(), e[[3, 29, 0], None].expand(-1, copies, -1))


# ---- experts ---------------------------------------------------------------------------------------------
MOE = [dict(E=6, top=2, W=40, F=24, shared=72, T=5), dict(E=4, top=4, W=96, F=32, shared=20, T=90), dict(E=9, top=1, W=64, F=16, shared=16, T=40),
       dict(E=3, top=3, W=48, F=8, shared=200, T=7), dict(E=16, top=5, W=128, F=64, shared=64, T=300)]


@WHERE
@pytest.mark.parametrize("c", MOE, ids=ids)
def test_experts_with_a_shared_one(where, c):
    """Router, gelu experts and the shared expert (of any width) as parts that every token takes, through the streams' update."""
    from stkernel_b200.config import MoeMlp
    from stkernel_b200.models.hybrid import BlockWeights, build_feed_forward
    dev, dt = where
    E, top, W, F, T = (c[k] for k in ("E", "top", "W", "F", "T"))
    mlp = MoeMlp(E, top, F, "gelu", False, c["shared"])
    w = {"mlp.router": rand(E, W, seed=20, scale=3 * W ** -0.5), "norm2": rand(W, seed=21)}
    for i, e in enumerate([f"e{i}" for i in range(E)] + ["shared"]):
        ff = c["shared"] if e == "shared" else F
        w[f"mlp.{e}.up"], w[f"mlp.{e}.down"] = rand(ff, W, seed=200 + i, scale=W ** -0.5), rand(W, ff, seed=300 + i, scale=ff ** -0.5)
    blk = BlockWeights(None, None, None, {})
    build_feed_forward(blk, mlp, lambda n: w[n].float().to(dev), W, dt, dev)
    assert blk.experts.num == E + mlp.shared_parts and mlp.expert_width * mlp.shared_parts >= c["shared"]
    h = rand(T, W, seed=22)
    hp = torch.zeros(T, al(W), dtype=dt)
    hp[:, :W] = h
    hp = hp.to(dev)
    routed = Fn.gate_route(hp, blk.router, None, top, "softmax_topk", True, 1.0, always=mlp.shared_parts) if dev != "cpu" else None
    if routed is None:
        routed = MO.router(Fn.linear(hp, blk.router, out_dtype=F32), None, top, "softmax_topk", True, 1.0, always=mlp.shared_parts)
    assert (routed[0][:, top:].cpu() == torch.arange(E, E + mlp.shared_parts)).all() and (routed[1][:, top:] == 1).all()
    y = MO.plain_experts(hp, *routed, blk.experts)
    x = torch.zeros(T, 1, W, device=dev)
    one, zero = torch.ones(1, device=dev), torch.zeros(W, device=dev)
    HB.stream_norm(x, y, HB.StreamWeights(one, one, one.view(1, 1)), one, torch.ones(W, device=dev), zero, 1e-5, al(W), dt)
    ref = O.mixture(h, {k[4:]: v for k, v in w.items()}, "", {"router": {"experts": E, "top": top}})
    assert worst_row(x[:, 0], ref) < (2e-5 if dt == F32 else 2e-2)


@pytest.mark.parametrize("experts,top,ff,shared,parts,width", [(8, 2, 64, 0, 0, 64), (8, 2, 64, 128, 2, 64), (8, 2, 64, 130, 3, 64),
                                                               (8, 2, 64, 40, 1, 64), (8, 2, 8, 200, 8, 25), (64, 30, 8, 200, 2, 100)])
def test_the_shared_expert_is_cut_into_parts(experts, top, ff, shared, parts, width):
    from stkernel_b200.config import MoeMlp
    m = MoeMlp(experts, top, ff, "gelu", False, shared)
    assert (m.shared_parts, m.expert_width) == (parts, width) and m.top + m.shared_parts <= 32


# ---- grouped attention -------------------------------------------------------------------------------------
ATT = [dict(H=4, G=2, D=24, V=40, bias=1), dict(H=3, G=1, D=64, V=64, bias=1), dict(H=2, G=2, D=17, V=21, bias=1), dict(H=8, G=1, D=128, V=128, bias=0),
       dict(H=20, G=1, D=16, V=8, bias=1), dict(H=2, G=1, D=72, V=136, bias=1), dict(H=1, G=1, D=300, V=24, bias=0), dict(H=4, G=4, D=48, V=16, bias=1)]


@WHERE
@pytest.mark.parametrize("c", ATT, ids=ids)
@pytest.mark.parametrize("coef,every,sink,gate", [(0.7, 13.0, True, True), (0.0, 1.0, False, False)])
def test_grouped_attention(where, c, coef, every, sink, gate):
    """Prompt, portions, a few tokens and one at a time, over scattered pages full of NaN where nothing was written."""
    dev, dt = where
    H, G, D, V, n, eps = c["H"], c["G"], c["D"], c["V"], 200, 1e-3
    q, k, v, g = (rand(n, k_, seed=30 + i) for i, k_ in enumerate((H * D, G * D, G * V, H * V)))
    bias = [rand(k_, seed=40 + i, scale=0.5) for i, k_ in enumerate((H * D, G * D, G * V))] if c["bias"] else None
    k[150] = 0.01 * k[150]                                    # eps matters to a small key
    proj, offs = columns((q, k, v, g), dt)
    full = [x + b for x, b in zip((q, k, v), bias)] if bias else [q, k, v]
    m = {"heads": H, "kv_heads": G, "scale": 1.3 * D ** -0.5, "q_temp": {"coef": coef, "every": every}}
    keep = O.sink_softmax
    try:
        if not sink:
            O.sink_softmax = lambda s: torch.softmax(s, -1)
        ref = O.attention_heads(*(x.reshape(n, hd, -1) for x, hd in zip(full, (H, G, G))), m, eps)
    finally:
        O.sink_softmax = keep
    ref = 0.6 * ref * (O.sigmoid(g) if gate else 1.0)
    a = GA.GroupedParams(H, G, D, V, m["scale"], torch.cat(bias).float().to(dev) if bias else None, eps, (coef, every),
                         torch.zeros(H, device=dev) if sink else None, gate, 0.6)
    plans = ([n], [130, 3, 2, 65], [198, 1, 1], [63, 1, 64, 72], [1] * 70 + [130])
    for cuts in plans if dev != "cpu" else plans[1:2]:
        cache = torch.full((12, G, 64, GA.grouped_row(D, V)[0]), float("nan"), dtype=dt, device=dev)
        table = torch.full((3, 8), -1, dtype=torch.int32)
        table[1, :4] = torch.tensor([9, 2, 11, 5], dtype=torch.int32)
        table = table.to(dev)
        out = torch.zeros(n, H * V + 5, dtype=dt, device=dev)
        at = 0
        for t in cuts:
            p, meta = proj[at:at + t].to(dev), step([(at, t)], dev, [1])
            qq = GA.grouped_prep(p, *offs[:3], a, meta, table, cache)
            GA.grouped_attention(p, qq, offs[3], a, meta, table, cache, out[at:at + t])
            at += t
        assert worst_row(out[:, :H * V], ref) < (2e-5 if dt == F32 else 2e-2), cuts
        assert not out[:, H * V:].any()


@WHERE
def test_query_temperature_steps_where_it_should(where):
    """The factor changes at the positions just before a multiple of `every`, far away too."""
    dev, dt = where
    a = GA.GroupedParams(1, 1, 16, 16, 1.0, None, None, (0.5, 256.0), None, False, 1.0)
    pos = [0, 254, 255, 256, 510, 511, 512, 256 * 4096 - 2, 256 * 4096 - 1, 256 * 4096]
    meta = step([(0, len(pos))], dev, [0])
    meta.positions = torch.tensor(pos, device=dev)
    q = GA.grouped_prep(torch.ones(len(pos), 48, dtype=dt, device=dev), 0, 16, 32, a, meta, torch.full((1, 1 << 15), -1, dtype=torch.int32, device=dev),
                        torch.zeros(1, 1, 64, 32, dtype=dt, device=dev))
    ref = torch.tensor([O.temperature(p, {"coef": 0.5, "every": 256}) for p in pos])
    assert rel(q.view(len(pos), -1)[:, 0], ref) < (1e-6 if dt == F32 else 4e-3)
    if dt == F32:
        f = q[:, 0].cpu()
        assert f[0] == f[1] == 1 and f[2] == f[3] == f[4] > 1 and f[5] == f[6] > f[4] and f[7] < f[8] == f[9]


LONG = [dict(H=8, G=2, D=128, V=128), dict(H=4, G=4, D=64, V=128), dict(H=6, G=2, D=96, V=80), dict(H=5, G=1, D=40, V=24), dict(H=130, G=1, D=32, V=16),
        dict(H=2, G=1, D=192, V=64), dict(H=3, G=3, D=200, V=200)]


@pytest.mark.gpu
@pytest.mark.parametrize("c", LONG, ids=ids)
def test_attention_kernels_agree_over_many_pages(c):
    """Several requests in one step (long portions that begin inside a page, short ones, a few tokens): the tensor-core kernels
    against the fp32 one."""
    dev = torch.device("cuda:0")
    H, G, D, V = c["H"], c["G"], c["D"], c["V"]
    g = torch.Generator(device=dev).manual_seed(1)
    spans, rows = [(0, 777), (500, 1), (1300, 333), (130, 40), (0, 3), (64, 64), (1001, 65)], [0, 3, 1, 2, 4, 5, 6]
    n = sum(s[1] for s in spans)
    meta = step(spans, dev, rows)
    pages, (row, k_col) = 27, GA.grouped_row(D, V)
    cache = torch.randn(7 * pages, G, 64, row, generator=g, device=dev).to(BF16)
    table = torch.randperm(7 * pages, generator=torch.Generator().manual_seed(2)).view(7, pages).to(torch.int32).to(dev)
    offs = [0, al(H * D), al(H * D) + al(G * D), al(H * D) + al(G * D) + al(G * V)]
    proj = torch.randn(n, offs[3] + al(H * V), generator=g, device=dev).to(BF16)
    a = GA.GroupedParams(H, G, D, V, 1.5 * D ** -0.5, torch.randn(H * D + G * (D + V), generator=g, device=dev), 1e-5, (0.3, 100.0),
                         torch.zeros(H, device=dev), True, 0.9)
    q = GA.grouped_prep(proj, *offs[:3], a, meta, table, cache)
    out = torch.full((n, al(H * V)), float("nan"), dtype=BF16, device=dev)
    GA.grouped_attention(proj, q, offs[3], a, meta, table, cache, out)
    ref = torch.empty_like(out)
    gate = proj[:, offs[3]:]
    _lib.call("stk_window_attention_simt", q, q.stride(0), 0, 0, meta.positions, meta.tok_req, table, table.stride(0), cache, row, None, 0,
              1.0, H, G, D, k_col, V, (D + 63) // 64 * 64, gate, gate.stride(0), 0.9, 1 << 30, a.scale, 0.0, a.sink, ref, ref.stride(0), 0, n,
              _lib.stream())
    x, y = out[:, :H * V].float(), ref[:, :H * V].float()
    assert torch.isfinite(x).all()
    err = ((x - y).norm(dim=-1) / y.norm(dim=-1)).cpu()
    assert err.max() < 1e-2, int(err.argmax())
    _lib.check_status()


# ---- recurrences ---------------------------------------------------------------------------------------------
PLANS = [[(170, 170)], [(64, 1), (64, 100), (42, 69)], [(23, 24), (2, 65), (145, 81)], [(63, 129), (65, 2), (42, 39)], [(1, 1)] * 30 + [(140, 140)],
         [(2, 3)] * 20 + [(130, 110)]]


def plans(dev):
    return PLANS if dev != "cpu" else PLANS[2:3]


def run_plan(plan, data, refs, state, call, width, tol, dev, dt):
    """Two requests in rows 2 and 0 advance together by the plan's portions; row 1 belongs to nobody."""
    at = [0, 0]
    for sizes in plan:
        meta = step([(at[r], sizes[r]) for r in range(2)], dev, [2, 0])
        p = torch.cat([data[r][at[r]:at[r] + sizes[r]] for r in range(2)]).to(dev)
        out = torch.full((sum(sizes), HB.out_offset(width)), 9.0, dtype=dt, device=dev)
        call(p, meta, state, out)
        for r in range(2):
            got = out[:sizes[0]] if r == 0 else out[sizes[0]:]
            ref = refs[r][at[r]:at[r] + sizes[r]]
            e = worst_row(got[:, :width], ref)
            assert e < tol and (sizes[r] == 1 or rel(got[:, :width], ref) < tol / 3), (plan[:4], sizes, r, e)
            at[r] += sizes[r]
        assert not out[:, width:].any()
    for s in state:
        assert torch.isnan(s[1]).all()


RET = [dict(H=2, D=16, V=24, R=16), dict(H=1, D=9, V=5, R=4), dict(H=3, D=64, V=64, R=32), dict(H=1, D=200, V=136, R=200), dict(H=1, D=256, V=72, R=64),
       dict(H=1, D=300, V=33, R=20), dict(H=2, D=128, V=256, R=128)]


@WHERE
@pytest.mark.parametrize("c", RET, ids=ids)
def test_retention(where, c):
    """Chunks of every size against the recurrence, state carried between steps; one head forgets at once, one hardly ever."""
    dev, dt = where
    H, D, V, R, n = c["H"], c["D"], c["V"], c["R"], 170
    decay = [0.9995, 0.3, 1.0][:H]
    m = {"heads": H, "dim": D, "decay": decay, "rot": {"base": 300.0, "dims": R}}
    freq = [300.0 ** (-2.0 * i / R) for i in range(R // 2)]
    a = RC.RetentionParams(H, D, V, torch.tensor(decay, dtype=F64).log().float().to(dev), split_frequencies(decay, dev),
                           split_frequencies(freq, dev), 1e-4, 0.7)
    data, refs = [], []
    for r in range(2):
        k = rand(n, H * D, seed=50 + r)
        q, v, g = (k + 0.5 * rand(n, H * D, seed=60 + r)).to(BF16).double(), rand(n, H * V, seed=70 + r), rand(n, H * V, seed=80 + r)
        p, offs = columns((q, k, v, g), dt)
        o = O.rms(O.retention_heads(*(x.reshape(n, H, -1) for x in (q, k, v)), m), 1e-4).reshape(n, -1)
        data.append(p)
        refs.append(0.7 * o * O.silu(g))
    for plan in plans(dev):
        state = (torch.full((3, H, D, V), float("nan"), device=dev),)
        run_plan(plan, data, refs, state, lambda p, meta, st, out: RC.retention(p, *offs, a, meta, st, out, 0), H * V,
                 1e-4 if dt == F32 else 2e-2, dev, dt)


SSM = [dict(H=4, V=24, N=16, G=2, taps=4, NG=2), dict(H=2, V=5, N=9, G=1, taps=3, NG=1), dict(H=3, V=64, N=64, G=3, taps=2, NG=1),
       dict(H=2, V=136, N=200, G=1, taps=4, NG=2), dict(H=1, V=40, N=300, G=1, taps=1, NG=1), dict(H=8, V=64, N=128, G=2, taps=4, NG=8),
       dict(H=2, V=16, N=24, G=2, taps=7, NG=4)]


def ssm_params(c, dev, seed=0, slow=0.0):
    H, V, N, G = c["H"], c["V"], c["N"], c["G"]
    cd = H * V + 2 * G * N
    w = {"conv": rand(cd, c["taps"], seed=seed + 1, scale=0.6), "bias": rand(cd, seed=seed + 2, scale=0.3), "dt": rand(H, seed=seed + 3) - 2.0,
         "a": rand(H, seed=seed + 4) - slow, "d": rand(H, seed=seed + 5), "norm": 1 + rand(H * V, seed=seed + 6, scale=0.2)}
    f = lambda x: x.float().contiguous().to(dev)
    a = RC.Mamba2Params(H, V, N, G, c["NG"], f(w["conv"].t()), f(w["bias"]), f(w["dt"]), f(-torch.exp(w["a"])), f(w["d"]), f(w["norm"]), 1e-4)
    return a, w


@WHERE
@pytest.mark.parametrize("c", SSM, ids=ids)
def test_mamba2(where, c):
    """Portions of every size (shorter than the convolution too) against the recurrence, state and inputs carried between steps."""
    dev, dt = where
    H, V, N, G, n = c["H"], c["V"], c["N"], c["G"], 170
    inner = H * V
    a, w = ssm_params(c, dev)
    w["a"][0] = 6.0                                           # one head whose decays differ by thousands
    a.neg_a[0] = -float(torch.exp(w["a"][0]))
    w["dt"][0] = -9.0
    a.dt_bias[0] = -9.0
    m = {"heads": H, "groups": G, "norm_groups": c["NG"]}
    data, refs = [], []
    for r in range(2):
        z, x, t = rand(n, inner, seed=90 + r), rand(n, inner + 2 * G * N, seed=94 + r), rand(n, H, seed=98 + r)
        t[11::37] += 30.0                                     # all but forgets what was before; its neighbours decay slowly
        t = t.to(BF16).double()
        p, offs = columns((z, x, t), dt)
        y = O.silu(O.causal_conv(x, w["conv"], w["bias"])).split([inner, G * N, G * N], -1)
        y = O.mamba2_heads(y[0].reshape(n, H, V), y[1].reshape(n, G, N), y[2].reshape(n, G, N), O.softplus(t + w["dt"]), w["a"], w["d"], m)
        data.append(p)
        refs.append(O.mamba2_gate_norm(y.reshape(n, inner), z, w["norm"], m, 1e-4))
    for plan in plans(dev):
        nan = lambda *s, d=F32: torch.full((3,) + s, float("nan"), dtype=d, device=dev)
        state = (nan(H, N, V), nan(c["taps"] - 1, inner + 2 * G * N, d=dt))
        run_plan(plan, data, refs, state, lambda p, meta, st, out: RC.mamba2(p, *offs, a, meta, st, out), inner,
                 1e-4 if dt == F32 else 0.1, dev, dt)


@WHERE
def test_the_convolution_sees_exactly_its_taps(where):
    """One spike: it counts for the next taps - 1 tokens, in a prompt, over the border of a portion and in decoding."""
    dev, dt = where
    c = dict(H=1, V=8, N=8, G=1, taps=4, NG=1)
    a, _ = ssm_params(c, dev)
    a.neg_a.fill_(-1e4)                                       # the state forgets at once: only the convolution carries anything
    for at in (0, 1, 29, 30, 31, 32) if dev != "cpu" else (0, 30):
        x = torch.zeros(60, 16 + 32 + 16, dtype=dt)
        x[:, :8] = 1
        quiet = x.clone()
        x[at, 16:16 + 24] = 5.0
        for cuts in ([60], [32, 28], [30, 2, 28], [31, 1, 1, 27], [1] * 60, [2] * 30):
            outs = []
            for p in (x, quiet):
                st = (torch.zeros(1, 1, 8, 8, device=dev), torch.full((1, 3, 24), 3.0, dtype=dt, device=dev))
                rows, pos = [], 0
                for n in cuts:
                    out = torch.empty(n, 16, dtype=dt, device=dev)
                    RC.mamba2(p[pos:pos + n].to(dev), 0, 16, 48, a, step([(pos, n)], dev, [0]), st, out)
                    rows.append(out[:, :8])
                    pos += n
                outs.append(torch.cat(rows).float().cpu())
            differs = (outs[0] - outs[1]).abs().amax(1) > 1e-3
            assert differs.nonzero().flatten().tolist() == list(range(at, min(60, at + 4))), (at, cuts)


@pytest.mark.gpu
@pytest.mark.parametrize("kind,c", [("ret", dict(H=2, D=64, V=128, R=64)), ("ret", dict(H=3, D=40, V=72, R=24)), ("ret", dict(H=1, D=256, V=320, R=256)),
                                    ("ret", dict(H=2, D=24, V=13, R=2)), ("ssm", dict(H=8, V=64, N=128, G=1, taps=4, NG=1)),
                                    ("ssm", dict(H=3, V=40, N=72, G=1, taps=4, NG=1)), ("ssm", dict(H=4, V=16, N=8, G=4, taps=3, NG=2))])
def test_chunks_agree_with_the_scan_over_many_chunks(kind, c):
    """Long spans from a carried state beside a fresh request and a decode row; slow decays."""
    dev = torch.device("cuda:0")
    g = torch.Generator(device=dev).manual_seed(3)
    meta = step([(5, 2300), (70, 1), (0, 130)], dev, [2, 0, 3])
    H, V, n = c["H"], c["V"], 2431
    rnd = lambda *s: torch.randn(*s, generator=g, device=dev)
    if kind == "ret":
        D = c["D"]
        decay = [0.999, 0.9, 0.5][:H]
        a = RC.RetentionParams(H, D, V, torch.tensor(decay, dtype=F64).log().float().to(dev), split_frequencies(decay, dev),
                               split_frequencies([0.3 ** i for i in range(c["R"] // 2)], dev), 1e-6, 1.0)
        offs = [0, al(H * D), 2 * al(H * D), 2 * al(H * D) + al(H * V)]
        p = rnd(n, offs[3] + al(H * V)).to(BF16)
        init = [rnd(4, H, D, V)]
        call = lambda st, out: RC.retention(p, *offs, a, meta, st, out, 0)
    else:
        a, _ = ssm_params(c, dev, slow=4.0)
        cd = H * V + 2 * c["G"] * c["N"]
        offs = [0, al(H * V), al(H * V) + al(cd)]
        p = rnd(n, offs[2] + al(H)).to(BF16)
        init = [rnd(4, H, c["N"], V), rnd(4, c["taps"] - 1, cd).to(BF16)]
        call = lambda st, out: RC.mamba2(p, *offs, a, meta, st, out)
    outs, states = [], []
    keep = RC.CHUNK_SPAN
    try:
        for span in (keep, 1 << 20):
            RC.CHUNK_SPAN = span
            st = [x.clone() for x in init]
            out = torch.zeros(n, HB.out_offset(H * V), dtype=BF16, device=dev)
            call(tuple(st), out)
            outs.append(out)
            states.append(st)
    finally:
        RC.CHUNK_SPAN = keep
    assert rel(outs[0], outs[1].cpu()) < 6e-3
    # the chunked form rounds the convolved operands of Mamba-2 to bf16, the scan does not
    assert rel(states[0][0], states[1][0].cpu()) < (2e-4 if kind == "ret" else 4e-3)
    assert torch.equal(states[0][0][1], init[0][1])
