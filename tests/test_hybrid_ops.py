"""Each mechanism of the hybrid decoder alone, against one plain function of the oracle: fp32 and (on a GPU) bf16 forms."""
import math

import pytest
import torch

import timalorn_oracle as O
from stkernel_b200.config import RotaryConfig, YarnScaling
from stkernel_b200.ops import functional as Fn
from stkernel_b200.ops import hybrid as HB
from stkernel_b200.ops.functional import LinearWeight

F32, F64, BF16 = torch.float32, torch.float64, torch.bfloat16
WHERE = pytest.mark.parametrize("where", [
    pytest.param(("cpu", F32), id="cpu"), pytest.param(("cuda:0", F32), id="gpu-f32", marks=pytest.mark.gpu),
    pytest.param(("cuda:0", BF16), id="gpu-bf16", marks=pytest.mark.gpu)])


def gen(seed):
    return torch.Generator().manual_seed(seed)


def rel(got, ref):
    return ((got.double().cpu() - ref).norm() / ref.norm()).item()


def one_request(n, start, row, dev, total=None, splits=None):
    """Step description of one request's span [start, start + n) (or of several: splits = [(n, start, row), ...])."""
    spans = splits or [(n, start, row)]
    pos = torch.cat([torch.arange(s, s + k) for k, s, _ in spans])
    i32 = lambda x: torch.as_tensor(x, dtype=torch.int32, device=dev)
    rep = lambda f: i32([v for k, s, r in spans for v in [f(k, s, r)] * k])
    q = [0]
    for k, _, _ in spans:
        q.append(q[-1] + k)
    sizes = [k for k, _, _ in spans]
    return HB.HybridMeta(torch.zeros(len(pos), dtype=torch.int64, device=dev), rep(lambda k, s, r: r), pos.to(dev),
                         rep(lambda k, s, r: s), rep(lambda k, s, r: s + k - 1), i32(q), i32([r for _, _, r in spans]),
                         i32([s for _, s, _ in spans]), len(spans), max(sizes), max(sizes) == 1, min(sizes))


# ---- residual, norms, feed-forward ----------------------------------------------------------------
@WHERE
@pytest.mark.parametrize("w_n", [8, 77, 256, 4100])
def test_embedding_and_layer_norm(where, w_n):
    dev, dt = where
    t = 9
    e = torch.randn(50, w_n, generator=gen(0)).to(dt)
    ids = torch.randint(0, 50, (t,), generator=gen(1))
    x = HB.embed_scaled(ids.to(dev), e.to(dev), 3.25)
    assert x.dtype == F32 and torch.equal(x.cpu(), e[ids].float() * 3.25)
    w = torch.randn(w_n, generator=gen(2))
    y = torch.randn(t, w_n, generator=gen(3)) + 40.0            # a large mean: the deviations are what counts
    width = (w_n + 15) // 16 * 16
    ref_x = x.double().cpu() + y.double()
    rows = torch.tensor([4, 0, 7])
    some = HB.add_layer_norm(x, y.to(dev), w.to(dev), 1e-3, width, dt, rows=rows.to(dev))
    h = HB.add_layer_norm(x, y.to(dev), w.to(dev), 1e-3, width, dt)
    ref = O.layer_norm(ref_x, w.double(), 1e-3)
    tol = 1e-5 if dt == F32 else 4e-3
    assert rel(x, ref_x) < 1e-6 and rel(h[:, :w_n], ref) < tol and not h[:, w_n:].any()
    assert rel(some[:, :w_n], ref[rows]) < tol
    assert rel(HB.add_layer_norm(x, None, w.to(dev), 1e-3, width, dt)[:, :w_n], ref) < tol


@pytest.mark.gpu
def test_unknown_token_is_reported():
    from stkernel_b200.ops import _lib
    x = HB.embed_scaled(torch.tensor([3, 99], device="cuda:0"), torch.ones(10, 16, device="cuda:0"), 1.0)
    torch.cuda.synchronize()
    assert not x[1].any()
    with pytest.raises(_lib.KernelError):
        _lib.check_status()


@WHERE
@pytest.mark.parametrize("mix,ff", [(24, 40), (16, 2100), (37, 5), (30, 0)])
def test_joined_feed_forward(where, mix, ff):
    dev, dt = where
    pad = (ff + 15) // 16 * 16
    p = torch.randn(5, 64 + 2 * pad, generator=gen(4)).to(dt)
    o0 = HB.out_offset(mix)
    out = torch.full((5, o0 + pad), 7.0, dtype=dt, device=dev)
    HB.join_glu(p.to(dev), out, mix, (64, 64 + pad, ff) if ff else None)
    out = out.double().cpu()
    assert (out[:, :mix] == 7).all() and not out[:, mix:o0].any() and not out[:, o0 + ff:].any()
    if ff:
        g, u = p[:, 64:64 + ff].double(), p[:, 64 + pad:64 + pad + ff].double()
        assert rel(out[:, o0:o0 + ff], g / (1 + torch.exp(-g)) * u) < (1e-6 if dt == F32 else 4e-3)


@pytest.mark.parametrize("dev", ["cpu", pytest.param("cuda:0", marks=pytest.mark.gpu)])
@pytest.mark.parametrize("t,n,k", [(1, 5, 7), (8, 130, 65), (9, 64, 64), (70, 200, 33), (200, 129, 256)])
def test_fp32_linear_is_fp32(dev, t, n, k):
    x, w = torch.randn(t, k, generator=gen(5)), torch.randn(n, k, generator=gen(6))
    y = Fn.linear(x.to(dev), LinearWeight(w.to(dev)))
    assert y.dtype == F32 and rel(y, x.double() @ w.double().T) < 1e-6


# ---- attention ----------------------------------------------------------------------------------------
def test_rotary_frequencies():
    for rot in (RotaryConfig(10000.0, 32), RotaryConfig(500.0, 24, YarnScaling(8.0, 256, 20.0, 1.5)),
                RotaryConfig(1e6, 64, YarnScaling(2.5, 4096, 32.0, 1.0)), RotaryConfig(100.0, 2, YarnScaling(4.0, 8, 9.0, 0.1))):
        d = {"base": rot.base, "dims": rot.dims}
        if rot.scaling:
            d["scaling"] = {"factor": rot.scaling.factor, "original": rot.scaling.original, "fast": rot.scaling.fast,
                            "slow": rot.scaling.slow}
        f, m = rot.frequencies()
        g, n = O.pair_frequencies(d)
        assert f == pytest.approx(g, rel=1e-12) and m == pytest.approx(n)
    f, m = RotaryConfig(10000.0, 64, YarnScaling(4.0, 2048, 32.0, 1.0)).frequencies()
    assert m == pytest.approx(1 + 0.1 * math.log(4.0)) and f[0] == 1.0 and f[-1] == pytest.approx(10000.0 ** (-62 / 64) / 4)


ATT = [dict(H=4, G=2, D=24, R=8, win=30), dict(H=8, G=1, D=64, R=64, win=64), dict(H=3, G=3, D=40, R=0, win=7),
       dict(H=34, G=2, D=16, R=4, win=65), dict(H=70, G=1, D=8, R=2, win=200), dict(H=2, G=1, D=128, R=64, win=129),
       dict(H=2, G=2, D=256, R=32, win=100), dict(H=1, G=1, D=300, R=20, win=50)]


@WHERE
@pytest.mark.parametrize("c", ATT, ids=lambda c: "x".join(str(v) for v in c.values()))
@pytest.mark.parametrize("cap,sink", [(5.0, True), (0.0, False)])
def test_window_attention(where, c, cap, sink):
    """Prompt portion, a few tokens, and one token at a time, over pages in scrambled order."""
    dev, dt = where
    H, G, D, R, win, n = c["H"], c["G"], c["D"], c["R"], c["win"], 200
    rot = RotaryConfig(400.0, R, YarnScaling(3.0, 64, 4.0, 0.5)) if R else None
    freq, mag = rot.frequencies() if rot else ([], 1.0)
    g = gen(7)
    k = torch.randn(n, G, D, generator=g).to(dt)
    q = torch.randn(n, H, D, generator=g).to(dt)
    q[::3] *= 3.0                                        # some queries pick out single keys
    s = torch.randn(H, generator=g) * 2 if sink else None
    qo, ko = 16, (16 + H * D + 15) // 16 * 16
    proj = torch.zeros(n, ko + (G * D + 15) // 16 * 16, dtype=dt)
    proj[:, qo:qo + H * D] = q.flatten(1)
    proj[:, ko:ko + G * D] = k.flatten(1)
    rd = {"base": 400.0, "dims": R, "scaling": {"factor": 3.0, "original": 64, "fast": 4.0, "slow": 0.5}} if R else None
    kd, qd, vd = (torch.stack([O.rotate(x[t].double(), t, rd) for t in range(n)]) for x in (k, q, k[:, :, :]))
    vd = k.double()
    if dt == BF16:
        kd, qd = kd.to(BF16).double(), qd.to(BF16).double()
    ref = torch.zeros(n, H, D, dtype=F64)
    for t in range(n):
        lo = max(0, t - win + 1)
        for h in range(H):
            j = h // (H // G)
            sc = O.attention_scores(qd[t, h], kd[lo:t + 1, j], D ** -0.5, cap)
            wts = O.sink_softmax(sc, s[h]) if sink else torch.softmax(sc, -1)
            ref[t, h] = wts @ vd[lo:t + 1, j]
    a = HB.AttentionParams(H, G, D, win, D ** -0.5, cap, torch.tensor(freq, dtype=F64).float().to(dev), mag,
                           s.to(dev) if sink else None)
    for cuts in ([n], [130, 3, 2, 65], [198, 1, 1], [1] * 70 + [130]):
        cache = torch.zeros(12, G, 64, (D + R + 7) // 8 * 8, dtype=dt, device=dev)
        table = torch.full((3, 8), -1, dtype=torch.int32)
        table[1, :4] = torch.tensor([9, 2, 11, 5], dtype=torch.int32)
        table = table.to(dev)
        out = torch.zeros(n, H * D + 5, dtype=dt, device=dev)
        at = 0
        for m in cuts:
            HB.window_attention(proj[at:at + m].to(dev), qo, ko, a, one_request(m, at, 1, dev), table, cache, out[at:at + m])
            at += m
        assert rel(out[:, :H * D], ref.flatten(1)) < (2e-5 if dt == F32 else 6e-3), cuts
        assert not out[:, H * D:].any()


# ---- mLSTM ----------------------------------------------------------------------------------------------
REC = [dict(H=2, D=16, V=24), dict(H=1, D=9, V=5), dict(H=3, D=64, V=64), dict(H=1, D=200, V=136), dict(H=1, D=256, V=72),
       dict(H=1, D=300, V=33)]


@WHERE
@pytest.mark.parametrize("c", REC, ids=lambda c: "x".join(str(v) for v in c.values()))
def test_mlstm(where, c):
    """Chunks of every size against the recurrence, two requests in different rows, state carried between steps."""
    dev, dt = where
    H, D, V, n, cap = c["H"], c["D"], c["V"], 170, 6.0
    al = lambda x: (x + 15) // 16 * 16
    offs = [0, al(H * D), 2 * al(H * D), 2 * al(H * D) + al(H * V)]
    p = HB.MlstmParams(H, D, V, cap, torch.randn(2 * H, generator=gen(8)).to(dev), (1 + 0.1 * torch.randn(H * V, generator=gen(9))).to(dev),
                       1e-5)
    data, refs = [], []
    for r in range(2):
        g = gen(10 + r)
        proj = torch.zeros(n, offs[3] + al(H * V), dtype=dt)
        k = torch.randn(n, H, D, generator=g).to(dt)
        q = (k.float() + 0.5 * torch.randn(n, H, D, generator=g)).to(dt)
        v = torch.randn(n, H, V, generator=g).to(dt)
        gate = torch.randn(n, H * V, generator=g).to(dt)
        for o, x in zip(offs, (q.flatten(1), k.flatten(1), v.flatten(1), gate)):
            proj[:, o:o + x.shape[1]] = x
        gates = torch.randn(n, 2 * H, generator=g) * 4
        pre = cap * torch.tanh((gates.double() + p.gate_bias.double().cpu()) / cap)
        o = O.mlstm_recurrence(q.double() / math.sqrt(D), k.double(), v.double(), pre[:, :H], -torch.log1p(torch.exp(-pre[:, H:])))
        ref = O.head_rms_norm(o, 1e-5).reshape(n, -1) * p.norm.double().cpu() / (1 + torch.exp(-gate.double()))
        data.append((proj, gates))
        refs.append(ref)
    for plan in ([(170, 170)], [(64, 1), (64, 100), (42, 69)], [(23, 24), (2, 65), (145, 81)], [(1, 1)] * 30 + [(140, 140)]):
        S = [torch.full((3, H) + s, float("nan"), device=dev) for s in ((D, V), (D,), ())]
        at = [0, 0]
        for sizes in plan:
            spans = [(sizes[r], at[r], (2, 0)[r]) for r in range(2)]
            proj = torch.cat([data[r][0][at[r]:at[r] + sizes[r]] for r in range(2)]).to(dev)
            gates = torch.cat([data[r][1][at[r]:at[r] + sizes[r]] for r in range(2)]).to(dev)
            out = torch.zeros(sum(sizes), HB.out_offset(H * V), dtype=dt, device=dev)
            HB.mlstm(proj, *offs, gates, p, one_request(0, 0, 0, dev, splits=spans), S, out, None)
            for r in range(2):
                got = out[:sizes[0]] if r == 0 else out[sizes[0]:]
                e = rel(got[:, :H * V], refs[r][at[r]:at[r] + sizes[r]])
                assert e < (2e-5 if dt == F32 else 5e-3), (plan, sizes, r, e)
                at[r] += sizes[r]
        assert all(torch.isnan(s[1]).all() for s in S)          # a row nobody owns is not touched


# ---- the kernels of one layer agree with one another at sizes the oracle is too slow for --------------------
LONG = [dict(H=8, G=2, D=128, R=64, win=300), dict(H=4, G=4, D=128, R=128, win=1000), dict(H=4, G=2, D=128, R=12, win=700),
        dict(H=3, G=1, D=128, R=120, win=200), dict(H=6, G=2, D=96, R=12, win=129),
        dict(H=16, G=1, D=64, R=16, win=64), dict(H=5, G=1, D=112, R=6, win=500), dict(H=40, G=2, D=16, R=16, win=257),
        dict(H=130, G=1, D=32, R=32, win=90), dict(H=4, G=2, D=72, R=8, win=400), dict(H=2, G=1, D=200, R=40, win=333)]


@pytest.mark.gpu
@pytest.mark.parametrize("c", LONG, ids=lambda c: "x".join(str(v) for v in c.values()))
@pytest.mark.parametrize("cap,sink", [(20.0, True), (0.0, False)])
def test_attention_kernels_agree_over_many_pages(c, cap, sink):
    """Three requests in one step (a long portion that begins inside a page, a short one, a few tokens): the tensor-core kernels
    against the fp32 one, over more pages than any ring of stages holds."""
    from stkernel_b200.ops import _lib
    dev = torch.device("cuda:0")
    H, G, D, R, win = c["H"], c["G"], c["D"], c["R"], c["win"]
    g = torch.Generator(device=dev).manual_seed(1)
    spans = [(777, 0, 0), (1, 500, 3), (333, 1300, 1), (40, 130, 2), (3, 0, 4), (64, 64, 5)]
    n = sum(s[0] for s in spans)
    meta = one_request(0, 0, 0, dev, splits=spans)
    pages = -(-1700 // 64)
    cache = torch.zeros(6 * pages, G, 64, (D + R + 7) // 8 * 8, dtype=BF16, device=dev)
    cache[..., :D + R] = torch.randn(6 * pages, G, 64, D + R, generator=g, device=dev)
    table = torch.randperm(6 * pages, generator=torch.Generator().manual_seed(2)).view(6, pages).to(torch.int32).to(dev)
    ko = (H * D + 15) // 16 * 16
    proj = torch.randn(n, ko + (G * D + 15) // 16 * 16, generator=g, device=dev).to(BF16)
    proj[::5, :H * D] *= 4
    sk = torch.randn(H, generator=g, device=dev) * 3 if sink else None
    freq = torch.rand(R // 2, generator=g, device=dev)
    a = HB.AttentionParams(H, G, D, win, D ** -0.5, cap, freq, 1.1, sk)
    out = torch.full((n, HB.out_offset(H * D)), float("nan"), dtype=BF16, device=dev)
    HB.window_attention(proj, 0, ko, a, meta, table, cache, out)
    ref = torch.empty_like(out)
    _lib.call("stk_window_attention_simt", proj, proj.stride(0), 0, ko, meta.positions, meta.tok_req, table, table.stride(0), cache,
              cache.shape[3], freq, R, 1.1, H, G, D, R, D, D, None, 0, 1.0, win, D ** -0.5, cap, sk, ref, ref.stride(0), 0, n, _lib.stream())
    x, y = out[:, :H * D].float(), ref[:, :H * D].float()
    assert torch.isfinite(x).all()
    err = ((x - y).view(n, H, D).norm(dim=-1) / y.view(n, H, D).norm(dim=-1).clamp(min=1e-3)).amax(1)
    # the tensor-core kernels round the rotated query and the row copy of it to bf16, the fp32 one only the row
    assert err.max() < 6e-2 and err.mean() < 1e-2, int(err.argmax())


@pytest.mark.gpu
@pytest.mark.parametrize("c", [dict(H=2, D=64, V=128), dict(H=3, D=40, V=72), dict(H=1, D=256, V=320), dict(H=2, D=24, V=13)],
                         ids=lambda c: "x".join(str(v) for v in c.values()))
def test_mlstm_chunks_agree_with_the_scan_over_many_chunks(c):
    """More chunks than one pass of the gate chain holds, from a carried state, beside a fresh request and a decode row."""
    dev = torch.device("cuda:0")
    H, D, V = c["H"], c["D"], c["V"]
    g = torch.Generator(device=dev).manual_seed(3)
    spans = [(2300, 5, 2), (1, 70, 0), (130, 0, 3)]
    n = sum(s[0] for s in spans)
    meta = one_request(0, 0, 0, dev, splits=spans)
    al = lambda x: (x + 15) // 16 * 16
    offs = [0, al(H * D), 2 * al(H * D), 2 * al(H * D) + al(H * V)]
    proj = torch.randn(n, offs[3] + al(H * V), generator=g, device=dev).to(BF16)
    proj[:, :H * D] = (proj[:, offs[1]:offs[1] + H * D].float() + 0.4 * proj[:, :H * D].float()).to(BF16)
    gates = torch.randn(n, 2 * H, generator=g, device=dev) * 3
    gates[:, H:] += 4
    p = HB.MlstmParams(H, D, V, 10.0, torch.zeros(2 * H, device=dev), torch.ones(H * V, device=dev), 1e-6)
    init = [torch.randn(4, H, D, V, generator=g, device=dev), torch.randn(4, H, D, generator=g, device=dev),
            torch.randn(4, H, generator=g, device=dev)]
    outs, states = [], []
    keep = HB.MLSTM_CHUNK_SPAN
    try:
        for span in (keep, 1 << 20):
            HB.MLSTM_CHUNK_SPAN = span
            st = [x.clone() for x in init]
            out = torch.zeros(n, HB.out_offset(H * V), dtype=BF16, device=dev)
            HB.mlstm(proj, *offs, gates, p, meta, st, out, None)
            outs.append(out.double().cpu())
            states.append([x.double().cpu() for x in st])
    finally:
        HB.MLSTM_CHUNK_SPAN = keep
    assert rel(outs[0], outs[1]) < 4e-3
    for x, y in zip(*states):
        assert rel(x, y) < 2e-4
    assert torch.equal(states[0][0][1], init[0][1].double().cpu())
