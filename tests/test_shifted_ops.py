"""Mechanisms of the shifted decoder, each alone, against the plain oracle: bigram embedding, token shift, talking-heads attention in chunks,
time mixing, xIELU, gated experts chosen in groups.  CPU statements and, marked `gpu`, the kernels in both compute types."""
import pytest
import torch

import fogizen_oracle as O
from stkernel_b200.config import BigramTable
from stkernel_b200.ops import _lib
from stkernel_b200.ops import functional as Fn
from stkernel_b200.ops import hybrid as HB
from stkernel_b200.ops import moe as MO
from stkernel_b200.ops import recurrence as RC
from stkernel_b200.ops import shifted as SH
from stkernel_b200.ops import talking as TK
from stkernel_b200.ops.functional import LinearWeight
from stkernel_b200.ops.latent import split_frequencies
from test_latent_ops import rand, rel, step, worst_row
from test_streams_ops import WHERE, al, columns, ids, plans, run_plan

F32, F64, BF16 = torch.float32, torch.float64, torch.bfloat16


# ---- bigram embedding ------------------------------------------------------------------------------------
@WHERE
@pytest.mark.parametrize("W,table", [(41, (50, 7, 3)), (64, (1, 5, 2)), (72, (997, 2147483647, 2147483646))])
def test_bigram_embedding(where, W, table):
    """Rows by the previous token: inside a span, over the border of a portion, for the first token; products beyond 32 bits."""
    dev, dt = where
    vocab, b = 200000, BigramTable(*table)
    e, t = rand(vocab, W, seed=1).float(), rand(b.buckets + 1, W, seed=2)
    ids_ = [[199999, 5, 5, 0, 199998, 77, 0], [3, 123456, 9]]
    cfg = {"embedding": {"bigram": {"buckets": table[0], "mul_prev": table[1], "mul_cur": table[2]}}}
    ref = [O.embedding(cfg, {"embed": e.double(), "bigram": t}, s) for s in ids_]
    for cuts in ([[4, 3], [1, 2]], [[1] * 7, [1] * 3], [[7], [3]]):
        st = SH.shift_state(1, 3, W, dev)
        st.token.fill_(-12345)
        at, got = [0, 0], [[], []]
        for k in range(max(len(c) for c in cuts)):
            part = [(r, cuts[r][k]) for r in range(2) if k < len(cuts[r])]
            meta = step([(at[r], n) for r, n in part], dev, [2 * r for r, _ in part])
            meta.token_ids = torch.tensor([x for r, n in part for x in ids_[r][at[r]:at[r] + n]], device=dev)
            x = SH.embed_bigram(meta, e.to(dt).to(dev), 1.0, t.to(dt).to(dev), b, st).double().cpu()
            SH.commit(st, meta)
            for r, n in part:
                got[r].append(x[:n])
                x, at[r] = x[n:], at[r] + n
        for r in range(2):
            assert rel(torch.cat(got[r]), ref[r]) < (1e-6 if dt == F32 else 4e-3), cuts
    assert rel(SH.embed_bigram(meta, e.to(dt).to(dev), 2.0, None, None, st), 2 * e[meta.token_ids.cpu()].double()) < (1e-6 if dt == F32 else 4e-3)


# ---- token shift -----------------------------------------------------------------------------------------
@WHERE
@pytest.mark.parametrize("W,blends,ff", [(41, 5, "rows"), (77, 0, None), (256, 2, "pairs"), (1000, 5, "pairs"), (2048, 5, "rows"), (4100, 1, "pairs")])
def test_shifted_norm(where, W, blends, ff):
    """Residual update, norm, shifted rows and blends: portions of every size, two requests side by side, carried states."""
    dev, dt = where
    n, eps, Wp = 90 if dev != "cpu" else 30, 1e-3, al(W)
    x0, y0, y1 = (rand(2, n, W, seed=10 + i) for i in range(3))
    y1 *= 0.02                                                              # eps matters to a small output
    w0, w1, norm, shift = (rand(W, seed=20 + i) for i in range(4))
    mu = rand(blends, W, seed=25) if blends else None
    fr = rand(2, n, W, seed=26) if ff == "rows" else torch.zeros(2, n, W, dtype=F64)
    top = 3
    rows, share = rand(2, n * top, W, seed=27), rand(2, n, top, seed=28)
    if ff == "pairs":
        rows = rows.to(dt).double()
        fr = (rows.view(2, n, top, W) * share.float().double()[..., None]).sum(2)
    new = x0 + 0.5 * O.rms(y0, eps) * w0 + 0.7 * O.rms(y1, eps) * w1 + fr
    h = O.rms(new, eps) * norm
    s = torch.stack([O.blend(h[r], shift) for r in range(2)])
    f = lambda v: v.float().contiguous().to(dev)
    tol = 3e-6 if dt == F32 else 4e-3
    for cuts in ([[n], [n]], [[1, 2, 40, n], [33, 1, n]], [[1] * 12 + [n], [2] * 20 + [n]]) if dev != "cpu" else ([[1, 2, 10, n], [13, 1, n]],):
        st = SH.shift_state(2, 3, W, dev)
        st.now.fill_(float("nan"))
        at = [0, 0]
        while at != [n, n]:
            part = []
            for r in range(2):
                c = cuts[r].pop(0) if cuts[r] else n
                if at[r] < n:
                    part.append((r, min(c, n - at[r])))
            meta = step([(at[r], k) for r, k in part], dev, [2 * r for r, _ in part])
            meta.pure_decode = all(k == 1 for _, k in part)
            take = lambda v: torch.cat([v[r, at[r]:at[r] + k] for r, k in part])
            tail = None
            if ff == "rows":
                tail = f(take(fr))
            elif ff == "pairs":
                tail = MO.ExpertRows(take(rows.view(2, n, top * W)).view(-1, W).to(dt).to(dev), None, f(take(share)))
            pend = SH.Pending([(f(take(y0)), f(w0), 0.5), (f(take(y1)), f(w1), 0.7)], tail)
            x, hh, ss, mix = SH.shifted_norm(f(take(x0)), pend, f(norm), eps, Wp, dt, f(shift), f(mu) if blends else None, st, 1, meta)
            assert rel(x, take(new)) < 2e-6 and rel(hh[:, :W], take(h)) < tol and rel(ss[:, :W], take(s)) < tol
            assert not hh[:, W:].any() and not ss[:, W:].any()
            for j in range(blends):
                ref = torch.stack([O.blend(s[r], mu[j]) for r in range(2)])
                assert worst_row(mix[:, j * Wp:j * Wp + W], take(ref)) < 4 * tol and not mix[:, j * Wp + W:(j + 1) * Wp].any()
            assert (mix is None) == (blends == 0)
            SH.commit(st, meta)
            for r, k in part:
                at[r] += k
        for r in range(2):
            assert rel(st.now[1, 2 * r], torch.stack([h[r, -1], s[r, -1]])) < 3e-6
        assert torch.isnan(st.now[:, 1]).all()
    pick = torch.tensor([4, 0, n - 1], device=dev)
    plain = SH.Pending([(f(y0[0]), None, 2.0)], f(fr[0]))
    some = SH.shifted_norm(f(x0[0]), plain, f(norm), eps, Wp, dt, rows=pick)[1]
    ref = O.rms(x0[0] + 2.0 * y0[0] + fr[0], eps) * norm
    assert rel(some[:, :W], ref[pick.cpu()]) < tol
    x, first, *_ = SH.shifted_norm(f(x0[0]), None, f(norm), eps, Wp, dt)
    assert rel(x, x0[0]) < 1e-6 and rel(first[:, :W], O.rms(x0[0], eps) * norm) < tol


# ---- talking-heads attention -----------------------------------------------------------------------------
ATT = [dict(H=4, G=2, D=24, V=40, R=16), dict(H=3, G=1, D=64, V=64, R=64), dict(H=2, G=2, D=17, V=21, R=6), dict(H=8, G=4, D=96, V=80, R=32),
       dict(H=20, G=2, D=16, V=8, R=2), dict(H=2, G=1, D=72, V=136, R=40), dict(H=6, G=6, D=128, V=128, R=128), dict(H=33, G=3, D=40, V=24, R=0),
       dict(H=16, G=8, D=64, V=128, R=64), dict(H=1, G=1, D=300, V=24, R=300)]


def talking(c, chunk, dev, sink=True, gate=True, bias=True, norm=True, seed=0, scale=None):
    """-> (parameters, the oracle's dictionary and tensors)."""
    H, G, D, V = c["H"], c["G"], c["D"], c["V"]
    rot = {"base": 300.0, "dims": c["R"], "scaling": {"factor": 2.5}}
    m = {"heads": H, "kv_heads": G, "scale": scale or 1.2 * D ** -0.5, "rot": rot, "mask": {"size": chunk or 1 << 30}}
    w = {"bias": rand(H * D + G * (D + V), seed=seed + 40, scale=0.5), "q": 1 + rand(D, seed=seed + 41, scale=0.3),
         "k": 1 + rand(D, seed=seed + 42, scale=0.3), "talk": torch.eye(H, dtype=F64) + rand(H, H, seed=seed + 43, scale=0.5 * H ** -0.5),
         "sink": rand(H, seed=seed + 44)}
    if not sink:
        w["sink"] -= 1e4
    if not bias:
        w["bias"] *= 0
    f = lambda v: v.float().contiguous().to(dev)
    freq = [300.0 ** (-2.0 * i / c["R"]) / 2.5 for i in range(c["R"] // 2)]
    a = TK.TalkingParams(H, G, D, V, m["scale"], chunk, 1e-3, f(w["bias"]) if bias else None, f(w["q"]) if norm else None,
                         f(w["k"]) if norm else None, split_frequencies(freq, dev), f(w["talk"]), f(w["sink"]) if sink else None, gate)
    return a, m, w


@WHERE
@pytest.mark.parametrize("c", ATT, ids=ids)
@pytest.mark.parametrize("chunk,sink,gate,bias,scale", [(0, True, True, True, None), (64, True, True, True, None), (50, False, False, False, -0.2),
                                                        (7, True, False, True, None), (150, True, True, True, None)])
def test_talking_attention(where, c, chunk, sink, gate, bias, scale):
    """Prompt, portions, a few tokens and one at a time, over scattered pages full of NaN where nothing was written."""
    dev, dt = where
    H, G, D, V, n = c["H"], c["G"], c["D"], c["V"], 200
    if dev == "cpu":
        n = 70
    q, k, v, g = (rand(n, k_, seed=30 + i) for i, k_ in enumerate((H * D, G * D, G * V, H)))
    proj, offs = columns((q, k, v, g), dt)
    a, m, w = talking(c, chunk, dev, sink, gate, bias, True, scale=scale)
    b = w["bias"].split([H * D, G * D, G * V])
    ref = O.attention_heads(*((x + y).reshape(n, hd, -1) for x, y, hd in zip((q, k, v), b, (H, G, G))), m, w["q"], w["k"], w["talk"], w["sink"], 1e-3)
    if gate:
        ref = ref * O.sigmoid(g)[..., None]
    ref = ref.reshape(n, -1)
    row = TK.talking_row(G, D, V)[0]
    for cuts in ([n], [130, 3, 2, 65], [198, 1, 1], [63, 1, 64, 72], [1] * 70 + [130]) if dev != "cpu" else ([40, 3, 2, 24, 1],):
        cache = torch.full((12, 64, row), float("nan"), dtype=dt, device=dev)
        table = torch.full((3, 8), -1, dtype=torch.int32)
        table[1, :4] = torch.tensor([9, 2, 11, 5], dtype=torch.int32)
        table = table.to(dev)
        out = torch.full((n, H * V + 5), 3.0, dtype=dt, device=dev)
        at = 0
        for t in cuts:
            p, meta = proj[at:at + t].to(dev), step([(at, t)], dev, [1])
            qq, gg = TK.talking_prep(p, *offs, a, meta, table, cache)
            TK.talking_attention(qq, gg, a, meta, table, cache, out[at:at + t])
            at += t
        assert worst_row(out[:, :H * V], ref) < (3e-5 if dt == F32 else 3e-2), cuts
        assert rel(out[:, :H * V], ref) < (1e-5 if dt == F32 else 1e-2) and not out[:, H * V:].any()
    if dev != "cpu":
        _lib.check_status()


@WHERE
def test_rotation_is_exact_far_away(where):
    """Angles of positions in the hundreds of thousands: the cached key is the fp64 rotation."""
    dev, dt = where
    a, m, w = talking(dict(H=2, G=1, D=32, V=16, R=32), 0, dev, bias=False)
    k = rand(3, 32, seed=5)
    proj, offs = columns((rand(3, 64, seed=4), k, rand(3, 16, seed=6), rand(3, 2, seed=7)), dt)
    for pos in (0, 1, 131071, 400001):
        meta = step([(pos, 3)], dev, [0])
        table = torch.full((1, (pos + 3) // 64 + 1), 0, dtype=torch.int32, device=dev)
        table[0, (pos + 2) // 64] = 1
        cache = torch.zeros(2, 64, TK.talking_row(1, 32, 16)[0], dtype=dt, device=dev)
        TK.talking_prep(proj.to(dev), *offs, a, meta, table, cache)
        for i in range(3):
            ref = O.rotate(O.rms(k[i], 1e-3) * w["k"], pos + i, m["rot"])
            got = cache[int(table[0, (pos + i) // 64]), (pos + i) % 64, 16:48]
            assert rel(got, ref) < (2e-6 if dt == F32 else 4e-3), pos


LONG = [dict(H=8, G=2, D=128, V=128, R=128), dict(H=4, G=4, D=64, V=128, R=32), dict(H=6, G=2, D=96, V=80, R=96), dict(H=5, G=1, D=40, V=24, R=8),
        dict(H=16, G=4, D=128, V=128, R=64), dict(H=40, G=8, D=128, V=64, R=128), dict(H=3, G=3, D=200, V=200, R=10)]


def kernels_agree(c, chunk, spans, rows):
    """The tensor-core kernels against the fp32 one over scattered pages."""
    dev = torch.device("cuda:0")
    H, G, D, V = c["H"], c["G"], c["D"], c["V"]
    g = torch.Generator(device=dev).manual_seed(1)
    n = sum(s[1] for s in spans)
    meta = step(spans, dev, rows)
    pages, (row, k_col, kp, vp) = 27, TK.talking_row(G, D, V)
    cache = torch.randn(8 * pages, 64, row, generator=g, device=dev).to(BF16)
    table = torch.randperm(8 * pages, generator=torch.Generator().manual_seed(2)).view(8, pages).to(torch.int32).to(dev)
    if chunk:                                                  # pages before the chunk have gone, and the first page is another's
        cache[0] = float("nan")
        for (start, _), r in zip(spans, rows):
            table[r, :start // chunk * chunk // 64] = -1
            table[table == 0] = 8 * pages - 1
    a, _, _ = talking(c, chunk, dev)
    proj = torch.randn(n, al(H * D) + al(G * D) + al(G * V) + al(H), generator=g, device=dev).to(BF16)
    offs = [0, al(H * D), al(H * D) + al(G * D), al(H * D) + al(G * D) + al(G * V)]
    q, gate = TK.talking_prep(proj, *offs, a, meta, table, cache)
    out = torch.full((n, al(H * V)), float("nan"), dtype=BF16, device=dev)
    TK.talking_attention(q, gate, a, meta, table, cache, out)
    ref = torch.empty_like(out)
    _lib.call("stk_talking_simt", q, gate, a.sink, meta.positions, meta.tok_req, table, table.stride(0), cache, row, k_col, kp, vp, H, G,
              V, chunk, a.scale, ref, ref.stride(0), ref.shape[1], 0, meta.first_pos, meta.last_pos, 1 << 30, n, _lib.stream())
    x, y = out[:, :H * V].float(), ref[:, :H * V].float()
    assert torch.isfinite(x).all()
    err = ((x - y).norm(dim=-1) / y.norm(dim=-1)).cpu()
    assert err.max() < 1e-2, int(err.argmax())
    _lib.check_status()


@pytest.mark.gpu
@pytest.mark.parametrize("c", LONG, ids=ids)
@pytest.mark.parametrize("chunk", [0, 256, 300, 77])
def test_attention_kernels_agree_over_many_pages(c, chunk):
    """Several requests in one step: long portions that begin inside a page and a chunk, short ones, single tokens."""
    kernels_agree(c, chunk, [(0, 777), (500, 1), (1300, 333), (130, 40), (0, 3), (64, 64), (1001, 65), (255, 2)], [0, 3, 1, 2, 4, 5, 6, 7])


@pytest.mark.gpu
@pytest.mark.parametrize("c", LONG, ids=ids)
@pytest.mark.parametrize("chunk", [0, 300])
@pytest.mark.parametrize("sms", [1, 148, 4000])
def test_decode_rows_agree_whatever_the_split(monkeypatch, c, chunk, sms):
    """One token per request: all heads in a CTA over the whole range, up to a CTA per key/value head and block of keys."""
    monkeypatch.setattr(_lib, "sm_count", lambda: sms)
    kernels_agree(c, chunk, [(1500, 1), (0, 1), (299, 1), (300, 1), (127, 1), (128, 1), (777, 1), (64, 1)], [0, 3, 1, 2, 4, 5, 6, 7])


# ---- time mixing -----------------------------------------------------------------------------------------
TM = [dict(H=2, D=16), dict(H=1, D=9), dict(H=3, D=64), dict(H=1, D=128), dict(H=1, D=200), dict(H=1, D=300), dict(H=4, D=40)]


def time_mix_params(c, dev, seed=0, slow=0.0):
    H, D = c["H"], c["D"]
    N = H * D
    w = {"w0": 1.5 * rand(N, seed=seed + 1) - 2.0 - slow, "u": rand(N, seed=seed + 2), "norm": 1 + rand(N, seed=seed + 3, scale=0.2)}
    f = lambda x: x.float().contiguous().to(dev)
    return RC.TimeMixParams(H, D, al(N), f(w["w0"]), f(w["u"]), f(w["norm"]), 1e-4), {k: v.float().double() for k, v in w.items()}


@WHERE
@pytest.mark.parametrize("c", TM, ids=ids)
def test_time_mixing(where, c):
    """Portions of every size against the recurrence, state carried between steps.  Some channels forget all at some tokens, some of
    their neighbours hardly anything."""
    dev, dt = where
    H, D, n = c["H"], c["D"], 170
    N = H * D
    a, w = time_mix_params(c, dev)
    w["w0"][0], w["w0"][1] = -30.0, 3.0                        # decays of 1 - 1e-13 and exp(-20)
    a.w0[:2] = torch.tensor([-30.0, 3.0])
    data, refs = [], []
    for r in range(2):
        rr, k, v, g, z = (rand(n, N, seed=50 + 7 * r + i) for i in range(5))
        rr = (k + 0.5 * rr).to(BF16).double()                 # read-outs that do not cancel
        z[11::37] += 9.0                                      # all but forgets what was before, by factors down to exp(-8000)
        p, _ = columns((rr, k, v, g), dt)
        z32 = z.float()
        decay = torch.exp(-torch.exp(z32.double() + w["w0"]))
        o = O.bonus_scan(*(x.reshape(n, H, D) for x in (rr, k, v, decay)), w["u"].view(H, D))
        data.append(torch.cat([p.float(), z32], 1))
        refs.append(O.rms(o, 1e-4).reshape(n, -1) * w["norm"] * O.silu(g))

    def call(p, meta, st, out):
        RC.time_mix(p[:, :4 * a.np].to(dt), p[:, 4 * a.np:].contiguous(), a, meta, st, out)

    for plan in plans(dev):
        state = (torch.full((3, H, D, D), float("nan"), device=dev),)
        run_plan(plan, data, refs, state, call, N, 1e-4 if dt == F32 else 3e-2, dev, dt)


@pytest.mark.gpu
@pytest.mark.parametrize("c", [dict(H=4, D=64), dict(H=3, D=40), dict(H=2, D=128), dict(H=2, D=13)], ids=ids)
@pytest.mark.parametrize("slow", [0.0, 4.0, -3.0])
def test_chunks_agree_with_the_scan_over_many_chunks(c, slow):
    """Long spans from a carried state beside a fresh request and a decode row; slow and very fast decays."""
    dev = torch.device("cuda:0")
    g = torch.Generator(device=dev).manual_seed(3)
    meta = step([(5, 2300), (70, 1), (0, 130)], dev, [2, 0, 3])
    H, D, n = c["H"], c["D"], 2431
    a, _ = time_mix_params(c, dev, slow=slow)
    rnd = lambda *s: torch.randn(*s, generator=g, device=dev)
    p, z = rnd(n, 4 * a.np).to(BF16), rnd(n, H * D)
    init = rnd(4, H, D, D)
    outs, states = [], []
    keep = RC.CHUNK_SPAN
    try:
        for span in (keep, 1 << 20):
            RC.CHUNK_SPAN = span
            st, out = init.clone(), torch.zeros(n, al(H * D), dtype=BF16, device=dev)
            RC.time_mix(p, z, a, meta, (st,), out)
            outs.append(out)
            states.append(st)
    finally:
        RC.CHUNK_SPAN = keep
    assert rel(outs[0], outs[1].cpu()) < 6e-3
    assert rel(states[0], states[1].cpu()) < 2e-4
    assert torch.equal(states[0][1], init[1])


@WHERE
def test_tanh_keeps_what_rounding_takes(where):
    dev, dt = where
    z = rand(7, 24, seed=1) * 2
    y = RC.tanh_rows(z.float().to(dev), dt).double().cpu()
    if dt == BF16:
        y = y[:, :24] + y[:, 24:]
    assert rel(y, torch.tanh(z)) < 1e-5


# ---- feed-forward ----------------------------------------------------------------------------------------
@WHERE
@pytest.mark.parametrize("T,ff,width", [(3, 37, 48), (300, 64, 64), (2, 9, 16)])
def test_xielu(where, T, ff, width):
    dev, dt = where
    z = rand(T, al(ff), seed=1) * 3
    z[0, :5] = torch.tensor([0.0, -30.0, 30.0, -1e-3, 1e-3])
    z = z.to(dt).double()
    p, q = torch.tensor(0.6, dtype=F64), torch.tensor(-1.1, dtype=F64)
    got = HB.xielu_rows(z.to(dt).to(dev), ff, (float(O.softplus(p)), float(O.softplus(q)) + 0.5), width)
    assert rel(got[:, :ff], O.xielu(z[:, :ff], p, q)) < (1e-6 if dt == F32 else 4e-3) and not got[:, ff:].any()


MOE = [dict(E=6, top=2, W=40, F=24, T=5, groups=3, keep=2), dict(E=4, top=4, W=96, F=32, T=90, groups=1, keep=1),
       dict(E=16, top=5, W=128, F=64, T=300, groups=4, keep=2), dict(E=64, top=6, W=64, F=40, T=40, groups=8, keep=3),
       dict(E=12, top=1, W=48, F=8, T=7, groups=6, keep=1), dict(E=6, top=3, W=72, F=200, T=700, groups=2, keep=1),
       dict(E=96, top=8, W=128, F=16, T=33, groups=32, keep=5)]


@WHERE
@pytest.mark.parametrize("c", MOE, ids=ids)
def test_gated_experts_chosen_in_groups(where, c):
    from stkernel_b200.config import MoeMlp
    from stkernel_b200.models.hybrid import BlockWeights, build_feed_forward
    dev, dt = where
    E, top, W, F, T = (c[k] for k in ("E", "top", "W", "F", "T"))
    mlp = MoeMlp(E, top, F, "silu", False, scoring="sigmoid", groups=c["groups"], keep=c["keep"], scale=1.7)
    w = {"mlp.router": rand(E, W, seed=20, scale=3 * W ** -0.5), "mlp.correction": rand(E, seed=21) - 1.0}
    for e in range(E):
        for i, (n, r, k) in enumerate((("gate", F, W), ("up", F, W), ("down", W, F))):
            w[f"mlp.e{e}.{n}"] = rand(r, k, seed=200 + 3 * e + i, scale=k ** -0.5)
    blk = BlockWeights(None, None, None, {})
    build_feed_forward(blk, mlp, lambda n: w[n].float().to(dev), W, dt, dev)
    h = rand(T, W, seed=22)
    hp = torch.zeros(T, al(W), dtype=dt)
    hp[:, :W] = h
    hp = hp.to(dev)
    how, kw = (blk.router_bias, top, "sigmoid", True, 1.7), dict(groups=c["groups"], keep=c["keep"])
    split = MO.router(Fn.linear(hp, blk.router, out_dtype=F32), *how, **kw)
    routed = (Fn.gate_route(hp, blk.router, *how, **kw) if dev != "cpu" else None) or split
    assert all(torch.equal(a.sort(1).values, b.sort(1).values) for a, b in zip(routed[:1], split[:1]))
    r = {"top": top, "scale": 1.7, "groups": {"count": c["groups"], "keep": c["keep"]}}
    z = h @ w["mlp.router"].T
    for t in range(T):
        chosen, share = O.route(z[t], w["mlp.correction"], r)
        at = [chosen.index(e) for e in routed[0][t].tolist()]           # the same experts, in any order
        assert torch.allclose(routed[1][t].double().cpu(), share[at], rtol=1e-4)
    y = MO.plain_experts(hp, *routed, blk.experts)
    x = torch.zeros(T, W, device=dev)
    got = SH.shifted_norm(x, SH.Pending([], y), torch.ones(W, device=dev), 1e-5, al(W), dt)[0]
    ref = O.mixture(h, {k[4:]: v for k, v in w.items()}, "", {"router": r})
    assert worst_row(got, ref) < (2e-5 if dt == F32 else 2e-2)


@WHERE
def test_closed_groups_stay_closed_where_every_choice_score_is_negative(where):
    """The corrections push every score below zero: an expert of a closed group must not win by a score of 0."""
    dev, _ = where
    z = torch.tensor([[1.0, 0.5, -2.0, -2.5, 3.0, -9.0]], device=dev)
    bias = torch.tensor([-2.0, -2.0, -1.5, -1.5, -4.0, -4.0], device=dev)
    ids_, w = MO.router(z, bias, 2, "sigmoid", True, 1.0, groups=3, keep=1)
    assert sorted(ids_[0].tolist()) == [0, 1] and abs(float(w.sum()) - 1) < 1e-6


@WHERE
@pytest.mark.parametrize("T,K,N", [(1, 48, 40), (5, 64, 128), (100, 128, 128), (200, 64, 256), (7, 80, 256)])
def test_products_of_a_few_large_blocks(where, T, K, N):
    dev, dt = where
    x, w = rand(T, 3 * K, seed=1), rand(3 * N, K, seed=2, scale=K ** -0.5)
    got = Fn.linear_blocks(x.to(dt).to(dev), LinearWeight(w.to(dt).to(dev)), 3)
    assert rel(got, torch.cat([x[:, g * K:(g + 1) * K] @ w[g * N:(g + 1) * N].T for g in range(3)], 1)) < (1e-5 if dt == F32 else 1e-2)
