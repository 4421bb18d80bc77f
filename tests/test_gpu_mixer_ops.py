"""GPU: every operator of libfa_b200_mixers and the row-wise operators that came with it against the plain restatement of its
mechanism (oracle/sabipel_oracle.py or the few lines here, float64).

In float32 the bound is rounding; in bfloat16 the inputs are the same bfloat16 numbers on both sides and the bound is a few
times the rounding of the result.  Errors are relative to the largest magnitude of the reference."""
import pytest
import torch

from oracle import sabipel_oracle as orc

pytestmark = pytest.mark.gpu
TOL = {torch.float32: 2e-5, torch.bfloat16: 1e-2}
TYPES = [torch.float32, torch.bfloat16]


def mops():
    from flash_attn_v100_b200 import mixer_ops
    return mixer_ops


def rops():
    from flash_attn_v100_b200 import row_ops
    return row_ops


def gen(seed):
    return torch.Generator().manual_seed(seed)


def rnd(g, *shape, dtype=torch.float32):
    return torch.randn(*shape, generator=g).to(dtype)


def i32(*v):
    return torch.tensor(v, dtype=torch.int32, device="cuda")


def status():
    return torch.zeros(1, dtype=torch.int32, device="cuda")


def close(got, ref, tol):
    got, ref = got.double().cpu(), ref.double()
    assert got.shape == ref.shape and torch.isfinite(got).all()
    err = (got - ref).abs().max() / ref.abs().max().clamp(min=1e-30)
    assert err < tol, float(err)


def strided(rows, cols, dtype, fill=7.0):
    """A [rows, cols] view inside wider rows, and the wide tensor."""
    wide = torch.full((rows, (cols + 15) // 8 * 8 + 8), fill, dtype=dtype, device="cuda")
    return wide[:, 8:8 + cols], wide


# ---- row-wise ------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("cols", [7, 64, 200, 1024, 4096, 9000])
def test_two_norms_and_summed_embeddings(cols, dtype):
    g = gen(cols)
    x, d, w1, w2 = rnd(g, 4, cols), *(rnd(g, *s, dtype=dtype) for s in ((4, cols), (cols,), (cols,)))
    xg = x.cuda()
    a, b = rops().residual_norm(xg, w1.cuda(), 1e-3, delta=d.cuda(), w2=w2.cuda())
    ref = x.double() + d.double()
    close(xg, ref, 2e-6)
    close(a, orc.rms_norm(ref, w1.double(), 1e-3), TOL[dtype])
    close(b, orc.rms_norm(ref, w2.double(), 1e-3), TOL[dtype])
    e, t2, t3 = rnd(g, 9, cols, dtype=dtype), rnd(g, 5, cols, dtype=dtype), rnd(g, 3, cols, dtype=dtype)
    tok, i2, i3 = torch.tensor([8, 0, 3, 3]), [4, 0, 2, 1], [0, 2, 1, 2]
    xg = torch.full((4, cols), float("nan"), device="cuda")
    a, b = rops().residual_norm(xg, w1.cuda(), 1e-3, embed=e.cuda(), tokens=tok.cuda(), init=True, embed_scale=5.5, w2=w2.cuda(),
                                more=[(t2.cuda(), i32(*i2)), (t3.cuda(), i32(*i3))])
    ref = e.double()[tok] * 5.5 + t2.double()[i2] + t3.double()[i3]
    close(xg, ref, 2e-6)
    close(b, orc.rms_norm(ref, w2.double(), 1e-3), TOL[dtype])


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("silu_first", [False, True])
@pytest.mark.parametrize("cols, group", [(96, 32), (96, 96), (120, 40), (1024, 128), (1536, 256), (3072, 1536), (33, 11), (16384, 8192),
                                         (20000, 20000), (640, 320)])
def test_gated_norm_of_parts(cols, group, silu_first, dtype):
    g = gen(cols + group)
    o, gate, w = (rnd(g, *s, dtype=dtype) for s in ((5, cols), (5, cols), (cols,)))
    gs, _ = strided(5, cols, dtype)
    gs.copy_(gate)
    out, wide = strided(5, cols, dtype)
    got = rops().gated_norm(o.cuda(), gs, w.cuda(), 1e-2, group=group, silu_first=silu_first, out=out)
    od, gd = o.double(), gate.double()
    y = (od * orc.silu(gd) if silu_first else od).view(5, -1, group)
    ref = orc.rms_scale(y, 1e-2).view(5, cols) * w.double()
    close(got, ref if silu_first else ref * orc.sigmoid(gd), TOL[dtype])
    assert (wide[:, :8] == 7).all() and (wide[:, 8 + cols:] == 7).all()


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("n", [5, 64, 1000])
def test_gelu(n, dtype):
    z = rnd(gen(n), 6, n, dtype=dtype) * 3
    out, wide = strided(6, n, dtype)
    close(rops().gelu(z.cuda(), out=out), orc.gelu_tanh(z.double()), TOL[dtype])
    assert (wide[:, :8] == 7).all() and (wide[:, 8 + n:] == 7).all()


def test_bigram_rows_remember_the_last_token():
    """Portions and single tokens give the rows of the whole sequence; a slot that is used again starts over."""
    buckets, mp, mc = 1000003, 8191, 131
    t = torch.randint(0, 100000, (700,), generator=gen(1)).tolist()
    want = orc.bigram_rows(t, buckets, mp, mc).tolist()
    last, st = torch.full((3,), 77, dtype=torch.int32, device="cuda"), status()

    def rows(parts, slots, starts, cu=True):
        flat = torch.tensor([x for p in parts for x in p], device="cuda")
        c = i32(0, *torch.tensor([len(p) for p in parts]).cumsum(0).tolist()) if cu else None
        return rops().bigram_rows(flat, i32(*starts), i32(*slots), last, buckets, mp, mc, st, cu_seqlens=c).tolist()
    for _ in range(2):
        got = rows([t[:600], t[:1], t[:2]], (2, 0, 1), (0, 0, 0))
        assert got == want[:600] + want[:1] + want[:2]
        got = rows([t[600:601], t[1:2], t[2:3]], (2, 0, 1), (600, 1, 2), cu=False)
        assert got == [want[600], want[1], want[2]]
        assert rows([t[3:650], t[601:]], (1, 2), (3, 601)) == want[3:650] + want[601:]
    assert int(st.item()) == 0
    rows([t[:1]], (3,), (0,), cu=False)
    assert int(st.item()) == 2


# ---- recurrences ----------------------------------------------------------------------------------------------------
def scan(q, k, v, la, b, floor=None, state=None, n=None, norm_eps=0.0, skip=None):
    """q, k [T, H, K], v [T, H, V], la, b, floor [H, T], float64."""
    T, H, K = q.shape
    S = torch.zeros(H, K, v.shape[-1], dtype=torch.float64) if state is None else state.clone()
    n = torch.zeros(H, K, dtype=torch.float64) if n is None else n.clone()
    out = torch.empty_like(v)
    for t in range(T):
        d, w = la[:, t].exp()[:, None], b[:, t][:, None]
        S = d[..., None] * S + w[..., None] * k[t][:, :, None] * v[t][:, None, :]
        n = d * n + w * k[t]
        o = torch.einsum("hkv,hk->hv", S, q[t])
        if floor is not None:
            o = o / (torch.maximum((n * q[t]).sum(-1).abs(), floor[:, t]) + norm_eps)[:, None]
        out[t] = o + (skip[:, None] * v[t] if skip is not None else 0)
    return out, S, n


def gates(g, H, T, strength):
    """Log decays and weights: mostly mild, some tokens that forget (nearly) everything, some that keep all."""
    la = -torch.rand(H, T, generator=g) * strength
    la[torch.rand(H, T, generator=g) < 0.03] = -40.0
    la[torch.rand(H, T, generator=g) < 0.2] = 0.0
    b = torch.rand(H, T, generator=g)
    b[torch.rand(H, T, generator=g) < 0.1] = 0.0
    return la, b


# (heads, groups, dk, dv): a pair of heads per CTA, odd numbers of heads per group, several column tiles, sizes of the general kernel
RECURRENCE_SIZES = [(4, 1, 32, 32), (6, 2, 128, 64), (2, 2, 128, 128), (3, 3, 48, 200), (4, 4, 16, 40), (8, 2, 64, 16), (3, 1, 9, 13), (2, 1, 136, 24)]


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("H, G, K, V", RECURRENCE_SIZES)
@pytest.mark.parametrize("normed", [False, True])
def test_recurrence_over_prompts(H, G, K, V, normed, dtype):
    """Packed sequences of lengths around the chunk, started afresh and continued."""
    lens, past = [1, 127, 128, 129, 2, 300], [0, 5, 0, 33, 64, 0]
    g, T, n_slots = gen(H * K + V), sum([1, 127, 128, 129, 2, 300]), 8
    pad = 8
    x = rnd(g, T, 2 * G * K + H * V + 3 * pad, dtype=dtype)
    x = x[:, :x.size(1) // 8 * 8].contiguous()
    oq, ok, ov = pad, pad + G * K, pad + 2 * G * K
    la, b = gates(g, H, T, 0.3)
    floor = 0.5 + torch.rand(H, T, generator=g) if normed else None
    skip = None if normed else rnd(g, H)
    state, norm, n0 = rnd(g, n_slots, H, K, V), rnd(g, n_slots, 2, H, K), rnd(g, len(lens), H, K)
    slots = [3, 0, 7, 1, 4, 2]
    cu = [0] + torch.tensor(lens).cumsum(0).tolist()
    sg, ng, st = state.cuda(), norm.cuda(), status()
    seqs = mops().Sequences(i32(*slots), i32(*past), i32(*cu), max(lens))
    kw = dict(floor=floor.cuda(), n0=n0.cuda(), norm=ng, norm_eps=1e-3) if normed else dict(skip=skip.cuda())
    got = mops().recurrence(x.cuda(), (oq, ok, ov), H, G, K, V, la.cuda(), b.cuda(), sg, seqs, st, q_scale=0.7, **kw)
    assert int(st.item()) == 0
    xd = x.double()
    rep = lambda off: xd[:, off:off + G * K].view(T, G, K).repeat_interleave(H // G, 1)
    q, k, v = 0.7 * rep(oq), rep(ok), xd[:, ov:ov + H * V].view(T, H, V)
    d = lambda t: None if t is None else t.double()
    outs = []
    for i, (a, e) in enumerate(zip(cu, cu[1:])):
        o, S, n = scan(q[a:e], k[a:e], v[a:e], d(la)[:, a:e], d(b)[:, a:e], d(floor)[:, a:e] if normed else None,
                       d(state[slots[i]]) if past[i] else None, d(n0[i]), 1e-3, d(skip))
        outs.append(o)
        close(sg[slots[i]], S, 2e-5)
        if normed:
            close(ng[slots[i], (past[i] + e - a - 1) & 1], n, 2e-5)
    close(got, torch.cat(outs).reshape(T, H * V), TOL[dtype])
    untouched = [s for s in range(n_slots) if s not in slots]
    assert torch.equal(sg[untouched].cpu(), state[untouched])


@pytest.mark.parametrize("H, G, K, V, normed", [(2, 1, 128, 64, False), (1, 1, 64, 128, True), (2, 2, 32, 16, True)])
def test_long_sequences_in_segments(H, G, K, V, normed):
    """Few heads and long sequences are cut into segments that run side by side."""
    lens, past = [2100, 513], [0, 7]
    g, T = gen(H * K + V), sum([2100, 513])
    x = rnd(g, T, 2 * G * K + H * V, dtype=torch.bfloat16)
    la, b = gates(g, H, T, 0.02)
    floor = 0.5 + torch.rand(H, T, generator=g) if normed else None
    state, norm, n0 = rnd(g, 2, H, K, V), rnd(g, 2, 2, H, K), rnd(g, 2, H, K)
    sg, ng, st = state.cuda(), norm.cuda(), status()
    seqs = mops().Sequences(i32(1, 0), i32(*past), i32(0, 2100, T), 2100)
    kw = dict(floor=floor.cuda(), n0=n0.cuda(), norm=ng, norm_eps=1e-3) if normed else {}
    got = mops().recurrence(x.cuda(), (0, G * K, 2 * G * K), H, G, K, V, la.cuda(), b.cuda(), sg, seqs, st, **kw)
    assert int(st.item()) == 0
    xd = x.double()
    rep = lambda off: xd[:, off:off + G * K].view(T, G, K).repeat_interleave(H // G, 1)
    q, k, v = rep(0), rep(G * K), xd[:, 2 * G * K:].view(T, H, V)
    for i, (a, e) in enumerate([(0, 2100), (2100, T)]):
        o, S, n = scan(q[a:e], k[a:e], v[a:e], la.double()[:, a:e], b.double()[:, a:e], floor.double()[:, a:e] if normed else None,
                       state[1 - i].double() if past[i] else None, n0[i].double(), 1e-3)
        close(got[a:e], o.reshape(e - a, H * V), TOL[torch.bfloat16])
        close(sg[1 - i], S, 2e-5)
        if normed:
            close(ng[1 - i, (past[i] + e - a - 1) & 1], n, 2e-5)


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("H, cap", [(3, 15.0), (1, 2.0), (40, 30.0)])
def test_max_gates(H, cap, dtype):
    """The running maximum over sequences longer than a tile of the scan, fresh and continued; large and small logits."""
    lens, past = [1, 2500, 70, 1024], [0, 0, 9, 4]
    g, T, K = gen(H), sum([1, 2500, 70, 1024]), 6
    x = rnd(g, T, 2 * H + 5, dtype=dtype) * 6
    bi, bf = rnd(g, H, dtype=dtype), rnd(g, H, dtype=dtype) + 2
    m, norm = rnd(g, 5, 2, H), rnd(g, 5, 2, H, K)
    slots, cu = [4, 1, 0, 2], [0] + torch.tensor(lens).cumsum(0).tolist()
    mg, st = m.cuda(), status()
    seqs = mops().Sequences(i32(*slots), i32(*past), i32(*cu), max(lens))
    la, b, floor, n0 = mops().max_gates(x.cuda(), 2, H + 3, bi.cuda(), bf.cuda(), cap, mg, norm.cuda(), seqs, st)
    i = orc.soft_cap(x.double()[:, 2:2 + H] + bi.double(), cap)
    f = orc.log_sigmoid(orc.soft_cap(x.double()[:, H + 3:2 * H + 3] + bf.double(), cap))
    for s, (a, e) in enumerate(zip(cu, cu[1:])):
        old = (past[s] - 1) & 1
        mt = m[slots[s], old].double() if past[s] else torch.zeros(H, dtype=torch.float64)
        assert torch.equal(n0[s].cpu(), norm[slots[s], old] if past[s] else torch.zeros(H, K))
        for t in range(a, e):
            mn = torch.maximum(f[t] + mt, i[t])
            if t % 97 == 0 or e - t < 3:
                for got, ref, atol in ((la, f[t] + mt - mn, 3e-5), (b, (i[t] - mn).exp(), 0.0), (floor, (-mn).exp(), 0.0)):
                    assert torch.allclose(got[:, t].double().cpu(), ref, rtol=1e-4, atol=atol)
            mt = mn
        assert torch.allclose(mg[slots[s], (past[s] + e - a - 1) & 1].double().cpu(), mt, atol=3e-5)
    assert int(st.item()) == 0


@pytest.mark.parametrize("dtype", TYPES)
def test_step_gates(dtype):
    g = gen(4)
    x, bias, a_log = rnd(g, 77, 45, dtype=dtype) * 8, rnd(g, 37), rnd(g, 37)
    la, b = mops().step_gates(x.cuda(), 5, bias.cuda(), a_log.cuda())
    dt = orc.softplus(x.double()[:, 5:42] + bias.double())
    assert torch.allclose(b.double().cpu(), dt.t(), rtol=1e-5) and torch.allclose(la.double().cpu(), (-a_log.double().exp() * dt).t(), rtol=1e-5)


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("channels, taps", [(64, 4), (40, 3), (24, 2), (16, 1), (56, 9), (13, 4)])
def test_convolution_in_portions(channels, taps, dtype):
    """One sequence in portions down to one token beside others, against the whole; ring slots that are used again."""
    g = gen(channels + taps)
    T, off = 60, 8
    x = rnd(g, T, channels + 16, dtype=dtype)
    w, b = rnd(g, channels, taps, dtype=dtype), rnd(g, channels, dtype=dtype)
    u = x.double()[:, off:off + channels]
    ref = orc.silu(orc.causal_conv(u, w.double(), b.double()))
    ring, st = torch.full((3, taps, channels), 9.0, dtype=dtype, device="cuda"), status()
    wt = w.t().contiguous().cuda()

    def run(parts, slots, decode=False):
        """parts: (first, stop) of the sequence for every slot."""
        rows = torch.cat([x[a:e] for a, e in parts]).cuda()
        cu = [0]
        for a, e in parts:
            cu.append(cu[-1] + e - a)
        pos = i32(*[p for a, e in parts for p in range(a, e)])
        seq = i32(*[i for i, (a, e) in enumerate(parts) for _ in range(a, e)])
        seqs = mops().Sequences(i32(*slots), i32(*[a for a, _ in parts]), None if decode else i32(*cu), max(e - a for a, e in parts))
        got = mops().conv_silu(rows, off, wt, b.cuda(), ring, seqs, seq, pos, st)
        close(got, torch.cat([ref[a:e] for a, e in parts]), TOL[dtype])
    for _ in range(2):
        run([(0, 2), (0, 40)], (1, 2))
        run([(2, 3), (40, 43)], (1, 2))
        run([(3, 4), (43, 44)], (1, 2), decode=True)
        run([(4, 60), (44, 45), (0, 1)], (1, 2, 0))
        run([(45, 60), (1, 20)], (2, 0))
    assert int(st.item()) == 0


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("H, K, V", [(4, 32, 48), (2, 128, 256), (3, 20, 12), (1, 300, 8), (5, 64, 64), (2, 9, 16), (640, 8, 8)])
def test_max_gate_step_equals_the_scan(H, K, V, dtype):
    """Decode steps in one kernel: many tokens one by one, from position 0 in slots with leftovers."""
    g, T, cap = gen(H * K), 12, 9.0
    stride = (2 * H * K + H * V + 2 * H + 7) // 8 * 8
    x = rnd(g, T, 2, stride, dtype=dtype)
    bi, bf = rnd(g, H, dtype=dtype), rnd(g, H, dtype=dtype) + 1
    state, norm, m = (rnd(g, 4, H, K, V).cuda(), rnd(g, 4, 2, H, K).cuda(), rnd(g, 4, 2, H).cuda())
    st = status()
    oi, of = 2 * H * K + H * V, 2 * H * K + H * V + H
    got = []
    for t in range(T):
        starts = i32(t, max(t - 3, 0))                        # the second sequence starts over until token 3
        got.append(mops().max_gate_step(x[t].contiguous().cuda(), (0, H * K, 2 * H * K), H, K, V, oi, of, bi.cuda(), bf.cuda(), cap, state, norm, m,
                                        mops().Sequences(i32(2, 1), starts), st, q_scale=K ** -0.5, norm_eps=1e-6).cpu())
    assert int(st.item()) == 0
    for s, first in ((0, 0), (1, 3)):
        xd = x[first:, s].double()
        n = xd.size(0)
        i = orc.soft_cap(xd[:, oi:oi + H] + bi.double(), cap)
        f = orc.log_sigmoid(orc.soft_cap(xd[:, of:of + H] + bf.double(), cap))
        ref, (S, nn, mm) = orc.mlstm_scan(xd[:, :H * K].view(n, H, K) * K ** -0.5, xd[:, H * K:2 * H * K].view(n, H, K),
                                          xd[:, 2 * H * K:oi].view(n, H, V), i, f)
        close(torch.stack([a[s] for a in got[first:]]), ref.reshape(n, H * V), TOL[dtype])
        slot, half = (2, 1)[s], (n - 1) & 1
        close(state[slot], S, 2e-5)
        close(norm[slot, half], nn, 2e-5)
        close(m[slot, half], mm, 2e-5)


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("H, G, N, V, taps", [(4, 2, 40, 32, 4), (6, 1, 128, 64, 4), (2, 2, 20, 12, 3), (3, 3, 64, 200, 2), (8, 2, 16, 16, 1), (4, 1, 9, 8, 6), (1280, 160, 8, 8, 4)])
def test_ssd_step_equals_the_scan(H, G, N, V, taps, dtype):
    g, T = gen(H * N), 11
    ch = H * V + 2 * G * N
    stride = (H * V + ch + H + 7) // 8 * 8
    x = rnd(g, T, 2, stride, dtype=dtype)
    w, b = rnd(g, ch, taps, dtype=dtype), rnd(g, ch, dtype=dtype)
    bias, a_log, D = rnd(g, H), rnd(g, H), rnd(g, H)
    state, ring, st = rnd(g, 3, H, N, V).cuda(), torch.full((3, taps, ch), 5.0, dtype=dtype, device="cuda"), status()
    got = [mops().ssd_step(x[t].contiguous().cuda(), H * V, H, G, N, V, H * V + ch, bias.cuda(), a_log.cuda(), D.cuda(), w.t().contiguous().cuda(), b.cuda(),
                           ring, state, mops().Sequences(i32(0, 2), i32(t, max(t - 2, 0))), st).cpu() for t in range(T)]
    assert int(st.item()) == 0
    for s, first in ((0, 0), (1, 2)):
        xd = x[first:, s].double()
        n = xd.size(0)
        u = orc.silu(orc.causal_conv(xd[:, H * V:H * V + ch], w.double(), b.double())).to(dtype).double()
        dt = orc.softplus(xd[:, H * V + ch:H * V + ch + H] + bias.double())
        ref, S = orc.ssd_scan(u[:, :H * V].reshape(n, H, V), u[:, H * V:H * V + G * N].reshape(n, G, N), u[:, H * V + G * N:].reshape(n, G, N), dt,
                              a_log.double(), D.double())
        tol = TOL[dtype] if dtype == torch.float32 else 2e-2        # (an activation may round the other way)
        close(torch.stack([a[s] for a in got[first:]]), ref.reshape(n, H * V), tol)
        close(state[(0, 2)[s]], S, 2e-5 if dtype == torch.float32 else 1e-2)


def test_bad_slots_are_reported_and_skipped():
    g = gen(0)
    x = rnd(g, 3, 64, dtype=torch.bfloat16).cuda()
    la, b = torch.zeros(1, 3, device="cuda"), torch.ones(1, 3, device="cuda")
    state = torch.zeros(2, 1, 16, 16, device="cuda")
    for seqs in (mops().Sequences(i32(5), i32(4), i32(0, 3), 3), mops().Sequences(i32(-1, 2, 0), i32(1, 1, 1))):
        st = status()
        mops().recurrence(x, (0, 16, 32), 1, 1, 16, 16, la, b, state, seqs, st)
        assert int(st.item()) == 2


# ---- attention -------------------------------------------------------------------------------------------------------
def paged(g, lens, G, K, V, dtype, extra=3):
    """Keys and values of sequences of the given lengths in shuffled pages; returns pools, table and the plain rows."""
    blocks = [(n + 15) // 16 for n in lens]
    order = torch.randperm(sum(blocks) + extra, generator=g).tolist()
    kp, vp = (torch.full((len(order), G, 16, d), 50.0).to(dtype) for d in (K, V))
    table = torch.full((len(lens), max(blocks)), -1, dtype=torch.int32)
    ks, vs = [], []
    for s, n in enumerate(lens):
        k, v = rnd(g, n, G, K, dtype=dtype), rnd(g, n, G, V, dtype=dtype)
        for j in range(blocks[s]):
            page = order.pop()
            table[s, j] = page
            c = min(16, n - j * 16)
            kp[page, :, :c], vp[page, :, :c] = k[j * 16:j * 16 + c].transpose(0, 1), v[j * 16:j * 16 + c].transpose(0, 1)
        ks.append(k)
        vs.append(v)
    return kp.cuda(), vp.cuda(), table.cuda(), ks, vs


def attend(q, k, v, pos, chunk, scale, slopes, gate):
    """One query row [H, K] at `pos` on k [n, G, K], v [n, G, V], float64."""
    H, rep = q.shape[0], q.shape[0] // k.shape[1]
    first = pos - pos % chunk if chunk else 0
    k, v = (t.double()[first:pos + 1].repeat_interleave(rep, 1) for t in (k, v))
    s = torch.einsum("hd,jhd->hj", q.double(), k) * scale - slopes.double()[:, None] * (pos - torch.arange(first, pos + 1)).double()
    o = torch.einsum("hj,jhd->hd", torch.softmax(s, -1), v).reshape(-1)
    return o * orc.sigmoid(gate.double()) if gate is not None else o


ATTENTION_SIZES = [(4, 1, 56, 32), (8, 2, 128, 128), (16, 1, 64, 64), (24, 1, 48, 72), (3, 3, 32, 128), (6, 2, 10, 14), (2, 1, 160, 24)]


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("H, G, K, V", ATTENTION_SIZES)
@pytest.mark.parametrize("chunk", [0, 48, 101])
def test_attention_rows_on_pages(H, G, K, V, chunk, dtype):
    """Rows at the edges of pages and chunks; a key that stands out is put just inside or just outside what a row sees."""
    g = gen(H * K + chunk)
    lens = [1, 17, 260, 700]
    rows = [(0, 0), (1, 16), (1, 15)] + [(2, p) for p in (47, 48, 49, 95, 96, 100, 101, 102, 201, 202, 259)] + [(3, p) for p in (303, 304, 511, 512, 699)]
    kp, vp, table, ks, vs = paged(g, lens, G, K, V, dtype)
    q = rnd(g, len(rows), H, K, dtype=dtype)
    for r, (s, p) in enumerate(rows):                        # a strong key just before the chunk, or at its start
        first = p - p % chunk if chunk else 0
        j = first - 1 if r % 2 and first > 0 else first
        strong = (q[r].double().view(G, H // G, K).sum(1) * 3).to(dtype)
        ks[s][j] = strong
        kp[table[s, j // 16].long(), :, j % 16] = strong.cuda()
    gate = rnd(g, len(rows), H * V, dtype=dtype)
    slopes = torch.tensor(orc.slopes(H, torch.float64).tolist())
    gs, _ = strided(len(rows), H * V, dtype)
    gs.copy_(gate)
    st = status()
    pages = mops().Pages(kp, vp, table, i32(*[s for s, _ in rows]), i32(*[p for _, p in rows]), st)
    out, wide = strided(len(rows), H * V, dtype)
    mops().kv_attention(pages, q.reshape(len(rows), -1).cuda(), H, chunk, K ** -0.5, slopes=slopes.cuda(), gate=gs, out=out)
    ref = torch.stack([attend(q[r], ks[s], vs[s], p, chunk, K ** -0.5, slopes, gate[r]) for r, (s, p) in enumerate(rows)])
    close(out, ref, TOL[dtype])
    assert (wide[:, :8] == 7).all() and (wide[:, 8 + H * V:] == 7).all() and int(st.item()) == 0
    plain = mops().kv_attention(pages, q.reshape(len(rows), -1).cuda(), H, chunk, K ** -0.5)
    ref = torch.stack([attend(q[r], ks[s], vs[s], p, chunk, K ** -0.5, torch.zeros(H), None) for r, (s, p) in enumerate(rows)])
    close(plain, ref, TOL[dtype])


def test_one_long_row_is_shared_by_several_blocks():
    g = gen(8)
    H, G, K, V, n = 8, 2, 128, 64, 3000
    kp, vp, table, ks, vs = paged(g, [n], G, K, V, torch.bfloat16)
    q = rnd(g, 1, H, K, dtype=torch.bfloat16)
    slopes = torch.full((H,), 0.001)
    for pos, chunk in ((2999, 0), (100, 0), (2999, 2048), (2048, 2048)):
        st = status()
        got = mops().kv_attention(mops().Pages(kp, vp, table, i32(0), i32(pos), st), q.reshape(1, -1).cuda(), H, chunk, 0.1, slopes=slopes.cuda())
        close(got[0], attend(q[0], ks[0], vs[0], pos, chunk, 0.1, slopes, None), TOL[torch.bfloat16])
        assert int(st.item()) == 0


@pytest.mark.parametrize("H, G, K, V", [(4, 1, 56, 32), (8, 2, 128, 128), (3, 3, 32, 128), (6, 2, 128, 64), (2, 1, 40, 24), (2, 1, 64, 48)])
def test_prompt_attention(H, G, K, V):
    """Pieces whose queries are all or only the last of their keys; a strong far key; steep and flat slopes."""
    g = gen(H * K)
    lens, klens = [1, 130, 257, 64, 300, 5], [1, 130, 400, 191, 300, 700]
    q, k, v = rnd(g, sum(lens), H, K, dtype=torch.bfloat16), rnd(g, sum(klens), G, K, dtype=torch.bfloat16), rnd(g, sum(klens), G, V, dtype=torch.bfloat16)
    cu, ck = ([0] + torch.tensor(x).cumsum(0).tolist() for x in (lens, klens))
    for i in range(len(lens)):
        k[ck[i]] = (q[cu[i + 1] - 1].double().view(G, H // G, K).sum(1) * 4).to(torch.bfloat16)
    gate = rnd(g, sum(lens), H * V, dtype=torch.bfloat16)
    for slopes in (orc.slopes(H, torch.float32), torch.full((H,), 1e-4), orc.slopes(H, torch.float32) * 3):
        st = status()
        out, wide = strided(sum(lens), H * V, torch.bfloat16)
        mops().kv_prefill(q.reshape(-1, H * K).cuda(), k.reshape(-1, G * K).cuda(), v.reshape(-1, G * V).cuda(), i32(*cu), i32(*ck), max(lens), H, G, K ** -0.5,
                          slopes.cuda(), st, gate=gate.cuda(), out=out)
        assert int(st.item()) == 0
        ref = torch.empty(sum(lens), H * V, dtype=torch.float64)
        for i, (n, kn) in enumerate(zip(lens, klens)):
            for r in range(n):
                row = cu[i] + r
                ref[row] = attend(q[row], k[ck[i]:ck[i + 1]], v[ck[i]:ck[i + 1]], kn - n + r, 0, K ** -0.5, slopes, gate[row])
        close(out, ref, TOL[torch.bfloat16])
        assert (wide[:, :8] == 7).all() and (wide[:, 8 + H * V:] == 7).all()


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("H, G, K, V", [(4, 2, 32, 16), (3, 1, 10, 7), (32, 8, 128, 128), (64, 64, 128, 8), (80, 1, 128, 128)])
def test_preparation_and_gather(H, G, K, V, dtype):
    g = gen(H + K)
    rows, eps = [(0, 3), (1, 16), (1, 17), (2, 0), (0, 4), (2, 31)], 1e-2
    T = len(rows)
    stride = (H * K + G * K + G * V + 8 + 7) // 8 * 8
    x, first = rnd(g, T, stride, dtype=dtype), rnd(g, T, G * V, dtype=dtype)
    wq, wk = rnd(g, H * K, dtype=dtype), rnd(g, G * K, dtype=dtype)
    table = torch.tensor([[4, -1], [0, 5], [1, 3]], dtype=torch.int32).cuda()
    kp, vp, st = torch.zeros(7, G, 16, K, dtype=dtype).cuda(), torch.zeros(7, G, 16, V, dtype=dtype).cuda(), status()
    pages = mops().Pages(kp, vp, table, i32(*[s for s, _ in rows]), i32(*[p for _, p in rows]), st)
    offs = (8, 8 + H * K, 8 + H * K + G * K)
    fs, _ = strided(T, G * V, dtype)
    fs.copy_(first)
    q, k, v = mops().kv_prep(pages, x.cuda(), offs, H, wq.cuda(), wk.cuda(), eps, v_first=fs, lam=0.3, contiguous_kv=True)
    xd = x.double()
    close(q, orc.rms_norm(xd[:, 8:8 + H * K], wq.double(), eps), TOL[dtype])
    close(k, orc.rms_norm(xd[:, offs[1]:offs[1] + G * K], wk.double(), eps), TOL[dtype])
    close(v, orc.mix_values(xd[:, offs[2]:offs[2] + G * V], first.double(), 0.3), TOL[dtype])
    for r, (s, p) in enumerate(rows):
        page = int(table[s, p // 16])
        assert torch.equal(kp[page, :, p % 16].reshape(-1), k[r]) and torch.equal(vp[page, :, p % 16].reshape(-1), v[r])
    assert int(kp.abs().sum(-1).ne(0).sum()) <= T * G
    got_k, got_v = mops().kv_gather(pages, H, i32(1, 0, 2), i32(16, 3, 31), i32(0, 2, 4, 5), 5)
    order = [1, 2, 0, 4, 5]
    assert torch.equal(got_k, k[order]) and torch.equal(got_v, v[order])
    _, k2, v2 = mops().kv_prep(pages, x.cuda(), offs, H, wq.cuda(), wk.cuda(), eps)
    assert k2 is None and v2 is None and int(st.item()) == 0
    plain = vp[4, :, 3].reshape(-1).double().cpu()
    close(plain, xd[0, offs[2]:offs[2] + G * V], TOL[dtype])
    mops().kv_gather(pages, H, i32(0), i32(16), i32(0, 1), 1)     # a page the sequence does not have
    assert int(st.item()) == 2
