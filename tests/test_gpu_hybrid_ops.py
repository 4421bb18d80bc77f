"""GPU: every operator of the hybrid decoder against the plain restatement of its mechanism (oracle/berilix_oracle.py, float64).

In float32 the bound is rounding; in bfloat16 the inputs are the same bfloat16 numbers on both sides and the bound is a few
times the rounding of the result.  Errors are relative to the largest magnitude of the reference."""
import pytest
import torch

from oracle import berilix_oracle as orc

pytestmark = pytest.mark.gpu
TOL = {torch.float32: 2e-5, torch.bfloat16: 1e-2}
TYPES = [torch.float32, torch.bfloat16]


def hops():
    from flash_attn_v100_b200 import hybrid_ops
    return hybrid_ops


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


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("cols", [7, 64, 200, 4096, 6000, 9000])
def test_residual_norm(cols, dtype):
    g = gen(cols)
    x, d, w, dw, e = rnd(g, 5, cols), *(rnd(g, *s, dtype=dtype) for s in ((5, cols), (cols,), (cols,), (9, cols)))
    tok = torch.tensor([3, 0, 8, 3, 5])
    c = lambda t: None if t is None else t.cuda()
    for delta, delta_w, emb, init, weight in [(None, None, None, False, w), (d, None, None, False, w), (d, dw, None, False, w),
                                              (d, dw, e, False, w), (None, None, e, True, w), (d, None, e, True, None)]:
        ref = (e.double()[tok] if init else x.double() + (e.double()[tok] if emb is not None else 0))
        if delta is not None:
            ref = ref + (orc.rms_norm(d.double(), dw.double(), 1e-3) if delta_w is not None else d.double())
        xg = x.cuda()
        out = hops().residual_norm(xg, c(weight), 1e-3, delta=c(delta), delta_w=c(delta_w), embed=c(emb), tokens=tok.cuda(), init=init)
        close(xg, ref, 2e-6)
        close(out, orc.rms_norm(ref, w.double(), 1e-3) if weight is not None else ref, TOL[dtype])
        if delta is not None:
            xg = x.cuda()
            assert hops().residual_norm(xg, None, 1e-3, delta=c(delta), delta_w=c(delta_w), embed=c(emb), tokens=tok.cuda(), init=init,
                                        out=False) is None
            close(xg, ref, 2e-6)


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("cols", [6, 64, 3000, 4096, 8192, 10240])
def test_gated_norm(cols, dtype):
    g = gen(cols)
    o, z, w = rnd(g, 3, cols, dtype=dtype), rnd(g, 3, 2 * cols + 8, dtype=dtype), rnd(g, cols, dtype=dtype)
    at = 8 if cols % 8 == 0 else 3
    out = hops().gated_norm(o.cuda(), z.cuda()[:, at:at + cols], w.cuda(), 1e-2)
    ref = orc.rms_norm(o.double(), w.double(), 1e-2) * orc.sigmoid(z.double()[:, at:at + cols])
    close(out, ref, TOL[dtype])


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("n,limit", [(5, 1.0), (64, 0.4), (200, 7.0)])
def test_clamped_glu(n, limit, dtype):
    z = 3 * rnd(gen(n), 9, 2 * n, dtype=dtype)
    eye = {"gate": torch.eye(2 * n)[:n], "up": torch.eye(2 * n)[n:], "down": torch.eye(n)}
    ref = orc.clamped_glu(z.double(), {k: v.double() for k, v in eye.items()}, "", limit)
    close(hops().clamped_glu(z.cuda(), limit, 1.702, 1.0), ref, TOL[dtype])
    alpha2 = hops().clamped_glu(z.cuda(), limit, 0.5, 0.25)          # the constants are parameters
    gg, uu = z.double()[:, :n].clamp(max=limit), z.double()[:, n:].clamp(-limit, limit)
    close(alpha2, gg * orc.sigmoid(0.5 * gg) * (uu + 0.25), TOL[dtype])


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("n,off,stride", [(5, 7, 20), (16, 32, 64), (24, 8, 40)])
def test_side_gate(n, off, stride, dtype):
    g = gen(n)
    z, e, tok = 2 * rnd(g, 6, n, dtype=dtype), rnd(g, 11, stride, dtype=dtype), torch.tensor([0, 10, 3, 3, 7, 1])
    out = hops().side_gate(z.cuda(), e.cuda(), tok.cuda(), off)
    close(out, orc.gelu_tanh(z.double()) * e.double()[tok, off:off + n], TOL[dtype])


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("q_rank,kv_rank,rot", [(7, 10, 6), (64, 48, 16), (24, 96, 2)])
def test_latent_prep_and_gather(q_rank, kv_rank, rot, dtype):
    """Rows of two sequences go to scattered pages at their positions, from the middle of a page on, and come back in order."""
    g, h = gen(rot), hops()
    cols = q_rank + kv_rank + rot + 3
    down, wq, wkv = rnd(g, 21, cols, dtype=dtype), rnd(g, q_rank, dtype=dtype), rnd(g, kv_rank, dtype=dtype)
    pos = list(range(9, 26)) + [0, 1, 2, 3]
    seq = [0] * 17 + [1] * 4
    stride = (kv_rank + rot + 7) // 8 * 8
    pool = torch.full((6, 16, stride), 9.0, dtype=dtype, device="cuda")
    table = torch.tensor([[5, 2], [0, -1]], dtype=torch.int32, device="cuda")
    f = 100.0 ** (-torch.arange(0, rot, 2, dtype=torch.float64) / rot)
    ang = torch.tensor(pos, dtype=torch.float64)[:, None] * f
    st = status()
    at = (0, q_rank, q_rank + kv_rank)
    cq, c, r = h.latent_prep(down.cuda(), at[0], q_rank, at[1], kv_rank, at[2], rot, wq.cuda(), wkv.cuda(), 1e-2, ang.cos().float().cuda(),
                             ang.sin().float().cuda(), pool, table, i32(*seq), i32(*pos), st, contiguous_kv=True)
    d = down.double()
    ref_c = orc.rms_norm(d[:, at[1]:at[2]], wkv.double(), 1e-2)
    ref_r = orc.rotate(d[:, at[2]:at[2] + rot], torch.tensor(pos), 100.0, rot)
    close(cq, orc.rms_norm(d[:, :q_rank], wq.double(), 1e-2), TOL[dtype])
    close(c, ref_c, TOL[dtype])
    close(r, ref_r, TOL[dtype])
    c2, r2 = h.latent_gather(pool, table, i32(0, 26, 30), 30, kv_rank, rot, st)
    assert torch.equal(c2[9:], c) and torch.equal(r2[9:], r)
    assert (pool[1] == 9).all() and (pool[3] == 9).all() and (pool[0, 4:] == 9).all() and int(st) == 0
    h.latent_gather(pool, table, i32(0, 26, 43), 43, kv_rank, rot, st)        # sequence 1 has no second page
    assert int(st) == 2


@pytest.mark.parametrize("dtype", TYPES)
def test_rotate_heads(dtype):
    g = gen(1)
    q, pos = rnd(g, 7, 3 * 20, dtype=dtype), torch.tensor([0, 1, 5, 63, 64, 1000, 3])
    f = 50.0 ** (-torch.arange(0, 12, 2, dtype=torch.float64) / 12)
    ang = pos.double()[:, None] * f
    out = hops().rotate_heads_(q.cuda(), ang.cos().float().cuda(), ang.sin().float().cuda(), 3, 20, 5, 12).view(7, 3, 20)
    ref = q.double().view(7, 3, 20).clone()
    ref[..., 5:17] = orc.rotate(ref[..., 5:17], pos, 50.0, 12)
    close(out, ref, TOL[dtype])
    assert torch.equal(out[..., :5].cpu(), q.view(7, 3, 20)[..., :5]) and torch.equal(out[0].cpu(), q.view(7, 3, 20)[0])


# ---- decayed linear attention ---------------------------------------------------------------------------------
def lightning_case(dtype, H, dk, dv, lens, starts, decay, seed=0, pad=0, z=None):
    g, h = gen(seed), hops()
    T, n = sum(lens), len(lens)
    cols = H * (2 * dk + dv)
    if z is None:
        z = rnd(g, T, cols + pad, dtype=dtype)
    at = (pad, pad + H * dk, pad + 2 * H * dk)
    dec = torch.tensor(decay, dtype=torch.float32)
    state = rnd(g, n + 3, H, dk, dv)
    before = state.clone()
    slots = [n + 2 - i for i in range(n)]
    cu = [0]
    for x in lens:
        cu.append(cu[-1] + x)
    st, sg = status(), state.cuda()
    prompt = any(x != 1 for x in lens)
    out = h.lightning(z.cuda(), at, H, dk, dv, dec.cuda(), sg, i32(*slots), i32(*starts), st, cu_seqlens=i32(*cu) if prompt else None,
                      max_len=max(lens))
    assert int(st) == 0
    for i in range(n):
        zz = z[cu[i]:cu[i + 1]].double()
        act = lambda a, w: orc.silu(zz[:, a:a + H * w]).to(dtype).double().view(-1, H, w)    # activations have the type of the model
        o, s = orc.linear_attention_scan(act(at[0], dk), act(at[1], dk), act(at[2], dv), dec.double(),
                                         None if starts[i] == 0 else before[slots[i]].double())
        close(out[cu[i]:cu[i + 1]], o.reshape(-1, H * dv), TOL[dtype])
        close(sg[slots[i]], s, 2e-5 if dtype == torch.float32 else 1e-3)      # fp32 state (activations may round the other way)
    keep = [i for i in range(n + 3) if i not in slots]
    assert torch.equal(sg[keep].cpu(), before[keep])
    return out, sg


DECAYS = [0.0, 0.3, 0.97, 0.9995, 1.0]


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("H,dk,dv", [(5, 64, 64), (5, 16, 24), (5, 40, 8), (5, 128, 128), (5, 96, 72), (5, 24, 136), (5, 9, 13), (5, 136, 8)])
def test_lightning_prompts(H, dk, dv, dtype):
    """Small heads (mma.sync chunks), large heads (tcgen05 chunks) and sizes only the token-by-token kernel takes; lengths
    around the chunks, fresh sequences and ones with a state, decays of 0 and 1."""
    lightning_case(dtype, H, dk, dv, [63, 2, 129, 64, 200], [0, 7, 0, 1, 64], DECAYS, pad=8)


@pytest.mark.parametrize("dk,dv", [(32, 64), (128, 64)])
def test_lightning_long_sequences_run_in_segments(dk, dv):
    lightning_case(torch.bfloat16, 2, dk, dv, [1700, 5, 513], [0, 3, 9], [0.999, 0.6])


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("H,dk,dv", [(5, 64, 64), (5, 9, 13), (5, 128, 200), (5, 20, 36)])
def test_lightning_decode(H, dk, dv, dtype):
    lightning_case(dtype, H, dk, dv, [1, 1, 1], [0, 4, 1000], DECAYS, pad=8)


@pytest.mark.parametrize("dk", [64, 128])
def test_lightning_one_far_token_shows(dk):
    """One token's key and value stand out; the last query of a prompt sees them through many chunks' decays."""
    H, dv, T, at = 1, 64, 300, 5
    z = torch.full((T, 2 * dk + dv), -30.0, dtype=torch.bfloat16)             # SiLU ~ 0
    z[at, dk:] = 2.0
    z[T - 1, :dk] = 1.0
    out, _ = lightning_case(torch.bfloat16, H, dk, dv, [T], [0], [0.99], z=z)
    q, kv = orc.silu(torch.tensor(1.0)), orc.silu(torch.tensor(2.0))
    assert abs(out[-1, 0].item() / (0.99 ** (T - 1 - at) * dk * q * kv * kv).item() - 1) < 0.02


def test_lightning_reports_a_bad_slot():
    h, st = hops(), status()
    z, state = torch.ones(4, 24, device="cuda").bfloat16(), torch.ones(2, 1, 8, 8, device="cuda")
    dec = torch.tensor([0.5], device="cuda")
    for cu, slots in ((None, [0, 5, -1, 1]), ([0, 2, 4], [7, 1])):
        st.zero_()
        h.lightning(z, (0, 8, 16), 1, 8, 8, dec, state, i32(*slots), i32(*[1] * len(slots)), st, cu_seqlens=i32(*cu) if cu else None, max_len=2)
        assert int(st) == 2


# ---- attention over latent rows ---------------------------------------------------------------------------------
def paged(rows, lens, seed):
    """Scatter [sum(lens), n] rows over shuffled pages; returns pool and table."""
    g = gen(seed)
    n_pages = sum((n + 15) // 16 for n in lens) + 2
    perm = torch.randperm(n_pages, generator=g)
    width = max((n + 15) // 16 for n in lens) + 1
    align = 8 if rows.dtype == torch.bfloat16 else 4
    stride = (rows.size(1) + align - 1) // align * align
    pool = torch.full((n_pages, 16, stride), 50.0, dtype=rows.dtype)          # what a freed page may hold
    pool[..., rows.size(1):] = 0
    table = torch.full((len(lens), width), -1, dtype=torch.int32)
    used = base = 0
    for i, n in enumerate(lens):
        for b in range((n + 15) // 16):
            page = int(perm[used])
            used += 1
            table[i, b] = page
            m = min(16, n - 16 * b)
            pool[page, :m, :rows.size(1)] = rows[base + 16 * b:base + 16 * b + m]
        base += n
    return pool.cuda(), table.cuda()


def latent_ref(q_abs, q_rot, rows, r, scale):
    """One query: q_abs [H, r], q_rot [H, rot] (rotated), rows [n, r + rot]."""
    s = (q_abs @ rows[:, :r].T + q_rot @ rows[:, r:].T) * scale
    s = torch.exp(s - s.max(-1, keepdim=True).values)
    return (s / s.sum(-1, keepdim=True)) @ rows[:, :r]


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("H,r,rot", [(3, 22, 6), (3, 48, 16), (16, 88, 40), (20, 184, 8), (33, 256, 64), (32, 512, 64), (2, 600, 8)])
def test_latent_attention(H, r, rot, dtype):
    """Rows of several sequences at positions around pages and key tiles, in the middle of their sequences and at the end; in every
    row one key, here and there, outweighs the others."""
    g, h = gen(H), hops()
    lens = [1, 15, 16, 17, 64, 65, 130, 700]
    where = [(0, 0), (1, 14), (2, 15), (3, 16), (4, 63), (5, 64), (6, 129), (6, 100), (6, 2), (7, 699), (7, 400)]
    total = sum(lens)
    rows = rnd(g, total, r + rot, dtype=dtype)
    off = [sum(lens[:i]) for i in range(len(lens))]
    T, qo = len(where), 5 * 8
    q_abs, q = rnd(g, T, H, r, dtype=dtype), rnd(g, T, H, qo + rot + 8, dtype=dtype)
    for t, (s, p) in enumerate(where):
        far = [0, p // 2, max(p - 1, 0), p][t % 4]
        q_abs[t, 0] = rows[off[s] + far, :r] * 3.0
    gate = rnd(g, T, H + 4, dtype=dtype)
    pool, table = paged(rows, lens, H)
    pos = torch.tensor([p for _, p in where])
    f = 30.0 ** (-torch.arange(0, rot, 2, dtype=torch.float64) / rot)
    ang = pos.double()[:, None] * f
    st, scale = status(), 1.5 * (r + rot) ** -0.5
    args = (q_abs.cuda(), q.cuda(), qo, ang.cos().float().cuda(), ang.sin().float().cuda(), pool, table, i32(*[s for s, _ in where]),
            i32(*pos.tolist()))
    qr = orc.rotate(q.double()[..., qo:qo + rot], pos, 30.0, rot).to(dtype).double()
    ref = torch.stack([latent_ref(q_abs[t].double(), qr[t], rows[off[s]:off[s] + p + 1].double(), r, scale)
                       for t, (s, p) in enumerate(where)])
    out = h.latent_attention(*args, gate.cuda()[:, 4:], r, rot, scale, st)
    close(out, ref * orc.sigmoid(gate.double()[:, 4:])[..., None], TOL[dtype])
    close(h.latent_attention(*args, None, r, rot, scale, st), ref, TOL[dtype])
    assert int(st) == 0


@pytest.mark.parametrize("dtype", TYPES)
def test_latent_attention_reports_pages_outside_the_pool(dtype):
    h, st = hops(), status()
    pool, table = paged(torch.randn(40, 24).to(dtype), [40], 0)
    bad = table.clone()
    bad[0, 1] = pool.size(0) + 3
    z = lambda *s: torch.randn(*s, device="cuda").to(dtype)
    ones = torch.ones(1, 4, device="cuda")
    h.latent_attention(z(1, 2, 16), z(1, 2, 8), 0, ones, ones, pool, bad, i32(0), i32(39), None, 16, 8, 1.0, st)
    assert int(st) == 2
    st.zero_()
    out = h.latent_attention(z(1, 2, 16), z(1, 2, 8), 0, ones, ones, pool, table, i32(0), i32(39), None, 16, 8, 1.0, st)
    assert int(st) == 0 and torch.isfinite(out).all()


@pytest.mark.parametrize("dim,rot,vdim", [(64, 40, 64), (128, 64, 128), (40, 16, 104), (72, 8, 24), (16, 64, 128), (8, 8, 8)])
def test_latent_prefill(dim, rot, vdim):
    """Packed prompts with and without earlier keys, lengths around the 128-row tiles; the last query of a sequence has one key
    (the first, or one at a tile's edge) that outweighs the others."""
    g, h, H = gen(dim), hops(), 3
    new, past = [130, 1, 300, 64, 128], [0, 17, 200, 128, 1]
    cu_q, cu_k = [0], [0]
    for a, b in zip(new, past):
        cu_q.append(cu_q[-1] + a)
        cu_k.append(cu_k[-1] + a + b)
    Tq, Tk, bf = cu_q[-1], cu_k[-1], torch.bfloat16
    q, kv, kr = rnd(g, Tq, H, dim + rot, dtype=bf), rnd(g, Tk, H * (dim + vdim), dtype=bf), rnd(g, Tk, rot, dtype=bf)
    for i, far in enumerate([0, 3, 128, 127, 64]):
        q[cu_q[i + 1] - 1, :, :dim] = kv[cu_k[i] + far, :H * dim].view(H, dim) * 4.0
    gate, scale, st = rnd(g, Tq, H + 5, dtype=bf), (dim + rot) ** -0.5, status()
    out = h.latent_prefill(q.view(Tq, -1).cuda(), kv.cuda(), kr.cuda(), gate.cuda()[:, :H], i32(*cu_q), i32(*cu_k), max(new), H, dim, vdim,
                           scale, st)
    for i, (a, b) in enumerate(zip(new, past)):
        ks = slice(cu_k[i], cu_k[i + 1])
        k = torch.cat([kv[ks, :H * dim].view(-1, H, dim), kr[ks, None].expand(-1, H, -1)], -1).double()
        v = kv[ks, H * dim:].view(-1, H, vdim).double()
        qq = torch.cat([torch.zeros(b, H, dim + rot, dtype=torch.float64), q[cu_q[i]:cu_q[i + 1]].double()])
        ref = orc.causal_attention(qq, k, v, scale)[b:] * orc.sigmoid(gate[cu_q[i]:cu_q[i + 1], :H].double())[..., None]
        close(out[cu_q[i]:cu_q[i + 1]], ref.reshape(a, -1), TOL[bf])
    assert int(st) == 0
