"""CPU: configuration, weights and cache bookkeeping of the Sabipel decoder, argument checks of its library, and properties of the
oracle that the GPU tests lean on."""
import ctypes
import json

import pytest
import torch

import sabipel_cases as sc
from flash_attn_v100_b200.engine import registry
from flash_attn_v100_b200.engine.config import ChunkedAttentionSpec, GeluSpec, Mamba2Spec, MlstmSpec, sabipel_config
from flash_attn_v100_b200.engine.hybrid import Step
from flash_attn_v100_b200.engine.weights import hybrid_tensor_shapes, hybrid_weights, random_hybrid_tensors
from flash_attn_v100_b200.kv_cache import HybridCache
from oracle import sabipel_oracle as orc


# ---- configuration and weights ----------------------------------------------------------------------------------------
def test_configuration_is_read_from_the_dictionary():
    cfg = sabipel_config(sc.small_config())
    a, m, s = (cfg.layers[i].mixer for i in (3, 1, 2))
    assert a == ChunkedAttentionSpec(4, 2, 24, 16, 24 ** -0.5, 50, (0.25, 0.0625, 2.0 ** -6, 2.0 ** -8), True)
    assert m == MlstmSpec(3, 32, 48, 10.0) and s == Mamba2Spec(4, 24, 40, 2, 4, 2) and s.channels == 96 + 160
    assert cfg.parallel and cfg.embed_scale == 3.0 and cfg.bigram.buckets == 101 and cfg.max_positions == 700
    assert cfg.layers[0].mlp == GeluSpec(80) and cfg.layers[2].mlp is None and not cfg.layers[0].mixer.v_mix
    assert sabipel_config(sc.config([(sc.attention(3, 1, 8, 8, 5), None)])).layers[0].mixer.slopes == pytest.approx(
        [2 ** (-8 / 3), 2 ** (-16 / 3), 2 ** -8])
    fam = registry.family_of(sc.small_config())
    assert fam.libraries == ("rows", "mixers") and torch.float32 in fam.dtypes


@pytest.mark.parametrize("change", [
    lambda d: d["layers"][0].update(type="lightning"), lambda d: d["layers"][0]["mlp"].update(kind="moe"),
    lambda d: d["layers"][0]["mixer"].update(kv_heads=4), lambda d: d["layers"][0]["mixer"]["mask"].update(size=0),
    lambda d: d["layers"][2]["mixer"].update(groups=3), lambda d: d["layers"][2]["mixer"].update(norm_groups=5),
    lambda d: d["layers"][1]["mixer"].update(gate_cap=0), lambda d: d["layers"][6]["mixer"].update(vdim=8),
    lambda d: d["embedding"]["bigram"].update(buckets=0), lambda d: d.update(layers=[])])
def test_configuration_errors_are_refused(change):
    d = sc.small_config()
    change(d)
    with pytest.raises(ValueError):
        sabipel_config(d)


def test_weights_in_the_layout_the_decoder_runs():
    d = sc.odd_config()
    cfg, w = sabipel_config(d), sc.weights(d)
    got = hybrid_weights(cfg, w, torch.float32, "cpu")
    l0, l1, l2, l3 = got["layers"][:4]
    assert l0["in_at"] == (0, 32, 64, 104, 144, 152) and l0["w_in"].shape == (160, 50)       # blocks padded to eight rows
    assert torch.equal(l0["w_in"][152:155], w["l0.mix.f"].float())
    assert l0["w_out"].shape == (50, 39 + 27)                                                # activations of mixer and feed-forward
    assert torch.equal(l0["w_out"][:, 39:], w["l0.mlp.down"].float()) and "w_down" not in l0
    assert l1["lambda"] == float(w["l1.mix.vmix"]) and l1["slopes"].tolist() == pytest.approx(cfg.layers[1].mixer.slopes)
    assert l2["conv_w"].shape == (1, 15 + 42) and l3["w_in"].shape[0] % 8 == 0
    assert got["pos"].shape == (700, 50) and got["bigram"].shape == (8, 50)
    for change in (lambda t: t.pop("l0.mix.i.b"), lambda t: t.update(extra=torch.zeros(1)), lambda t: t.update(bigram=torch.ones(7, 50))):
        t = dict(w)
        change(t)
        with pytest.raises(ValueError):
            hybrid_weights(cfg, t, torch.float32, "cpu")
    small, ws = sabipel_config(sc.small_config()), sc.weights(sc.small_config())
    got = hybrid_weights(small, dict(ws, **{"l0.mix.vmix": torch.tensor(0.5)}), torch.float32, "cpu")   # of a layer that does not mix: not used
    assert got["layers"][0]["lambda"] == 0.0 and got["layers"][6]["lambda"] > 0
    assert set(random_hybrid_tensors(cfg, 0)) == set(hybrid_tensor_shapes(cfg))


# ---- cache and batching -----------------------------------------------------------------------------------------------
def test_cache_gives_up_the_pages_of_past_chunks():
    c = HybridCache([("kv", 2, 8, 4, 64), ("slots", ((3,), torch.float32), ((), torch.int32)), ("kv", 1, 8, 8, 48)], 12, 2, 16, "cpu")
    assert [tuple(t.shape) for t in c.stores[0]] == [(12, 2, 16, 8), (12, 2, 16, 4)] and c.stores[1][1].shape == (2,)
    assert c.stores[1][0].dtype == torch.float32 and c.stores[0][0].dtype == torch.bfloat16 and not c.enable_prefix_cache
    c.allocate("a", 100)
    c.commit("a", 63)
    assert min(c.get_block_table("a")) >= 0                                  # position 63 still reads from 0 on
    c.commit("a", 17)                                                        # 80: chunks from 64 and from 48 on
    assert c.get_block_table("a")[:4] == [-1, -1, -1, c.get_block_table("a")[3]] and c.get_block_table("a")[3] >= 0
    c.commit("a", 20)                                                        # 100: from 64 and 96 on
    assert c.get_block_table("a")[3] == -1 and c.get_num_free_blocks() == 12 - 7 + 4
    assert c.block_table[c.row_of("a"), :4].tolist() == [-1] * 4
    c.release("a")
    assert c.get_num_free_blocks() == 12
    c = HybridCache([("kv", 1, 8, 8, 64), ("latent", 8)], 12, 1, 16, "cpu")  # one layer reads everything
    c.allocate("a", 100)
    c.commit("a", 100)
    assert min(c.get_block_table("a")) >= 0
    assert HybridCache([("kv", 1, 8, 8, 0)], 4, 1, 4, "cpu").enable_prefix_cache


@pytest.mark.parametrize("chunk", [1, 7, 16, 50, 1000])
def test_pieces_cover_the_pass_and_stay_inside_chunks(chunk):
    past, lens = [0, 13, 99, 50], [30, 2, 120, 50]
    T = sum(lens)
    step = Step(torch.zeros(T, dtype=torch.int64), None, None, None, None, None, None, lens, past, None, None)
    p = step.pieces(chunk)
    cq, ck, seq, key0 = (t.tolist() for t in (p.cu_q, p.cu_kv, p.seq, p.key0))
    pos = [(s, q) for s in range(4) for q in range(past[s], past[s] + lens[s])]
    assert cq[-1] == T and p.max_q == max(b - a for a, b in zip(cq, cq[1:])) and p.total_kv == ck[-1]
    for i in range(len(seq)):
        n, kn = cq[i + 1] - cq[i], ck[i + 1] - ck[i]
        for r in range(n):
            s, q = pos[cq[i] + r]
            at = key0[i] + kn - n + r                        # a piece's queries are its last keys
            assert s == seq[i] and q == at and key0[i] == q - q % chunk
    assert p.fresh == (cq == ck) and step.pieces(chunk) is p


# ---- library ------------------------------------------------------------------------------------------------------------
def test_calls_check_their_arguments_before_the_device():
    from flash_attn_v100_b200 import _lib
    from flash_attn_v100_b200.build import build
    build(library="mixers")
    lib = _lib.library("mixers")
    p = 256
    good = dict(x=p, stride=64, total=4, off_q=0, off_k=16, off_v=32, heads=2, groups=1, dk=16, dv=16, n_slots=1, n_seq=1, max_len=4, dtype=1, q_scale=1.0,
                state=p, slots=p, starts=p, cu_seqlens=p, out=p, status=p, la=p, b=p)
    call = lambda **kw: lib.fam_recurrence(ctypes.byref(_lib.Recurrence(**dict(good, **kw))), None)
    for bad in (dict(x=None), dict(groups=3), dict(dk=0), dict(dk=2000), dict(off_v=40), dict(total=0), dict(la=None), dict(floor=p), dict(dtype=4),
                dict(max_len=0)):
        assert call(**bad) == -1 and lib.fam_last_error()
    step = lambda **kw: lib.fam_max_gate_step(ctypes.byref(_lib.Recurrence(**dict(good, cu_seqlens=None, total=1, norm=p, **kw))), 0, 1, p, p, 5.0, p, None)
    assert step(dv=14) == -2 and b"not built" in lib.fam_last_error() and step(off_k=60) == -1
    ssd = lib.fam_ssd_step(ctypes.byref(_lib.Recurrence(**dict(good, cu_seqlens=None, total=1, skip=p))), 0, p, p, p, p, p, 4, None)
    assert ssd == -1 and b"adjacent" in lib.fam_last_error()
    assert [lib.fam_recurrence_step_supported(*s) for s in ((128, 64), (2000, 64), (16, 30))] == [1, 0, 0]
    pages = dict(k_pool=p, v_pool=p, block_table=p, tok_seq=p, positions=p, n_blocks=1, max_blocks=1, n_seq=1, heads=4, kv_heads=2, dim=16, vdim=8, dtype=1,
                 rows=1, status=p)
    attn = lambda stride=32, chunk=8, **kw: lib.fam_kv_attention(ctypes.byref(_lib.Pages(**dict(pages, **kw))), p, None, None, 0, chunk, 1.0, p, stride, None, 0, None)
    assert attn(kv_heads=3) == -1 and attn(stride=31) == -1 and attn(chunk=-1) == -1 and attn(n_blocks=0) == -1
    assert lib.fam_kv_prefill_supported(4, 2, 128, 64, 0.1, 1) == 1 and lib.fam_kv_prefill_supported(4, 2, 136, 64, 0.1, 1) == 0
    assert lib.fam_kv_prefill_supported(4, 2, 64, 64, -0.1, 1) == 0 and lib.fam_kv_prefill_supported(4, 2, 64, 64, 0.1, 0) == 0
    assert lib.fam_kv_prefill(p, p, p, p, p, 1, 1, 1, 1, 4, 2, 64, 64, 0.1, p, None, 0, p, 250, p, None) == -1
    assert lib.fam_conv_silu(p, 8, 4, 8, 2, p, p, p, 1, p, p, None, p, p, 1, 1, p, p, 1, None) == -1
    assert lib.fam_step_gates(p, 8, 4, 8, p, p, 1, p, p, 1, None) == -1


# ---- oracle ---------------------------------------------------------------------------------------------------------------
def test_oracle_matrix_memory_equals_its_closed_form():
    """With the normaliser undone, every output is a sum over the tokens so far weighted by the gates between them."""
    g = torch.Generator().manual_seed(0)
    T = 9
    q, k, v = (torch.randn(T, 2, n, generator=g, dtype=torch.float64) for n in (3, 3, 5))
    i, f = torch.randn(T, 2, generator=g, dtype=torch.float64) * 3, orc.log_sigmoid(torch.randn(T, 2, generator=g, dtype=torch.float64))
    o, (S, n, m) = orc.mlstm_scan(q, k, v, i, f)
    F = f.cumsum(0)
    for h in range(2):
        best = torch.stack([torch.cat([F[t, h][None], F[t, h] - F[:t + 1, h] + i[:t + 1, h]]).max() for t in range(T)])      # m_0 = 0
        for t in range(T):
            w = torch.exp(F[t, h] - F[:t + 1, h] + i[:t + 1, h] - best[t]) * (k[:t + 1, h] @ q[t, h])
            want = w @ v[:t + 1, h] / (torch.maximum(w.sum().abs(), torch.exp(-best[t])) + 1e-6)
            assert torch.allclose(o[t, h], want)
    o1, s1 = orc.mlstm_scan(q[:4], k[:4], v[:4], i[:4], f[:4])
    o2, s2 = orc.mlstm_scan(q[4:], k[4:], v[4:], i[4:], f[4:], s1)
    assert torch.allclose(torch.cat([o1, o2]), o) and all(torch.allclose(a, b) for a, b in zip(s2, (S, n, m)))


def test_oracle_state_space_scan_equals_its_closed_form():
    g = torch.Generator().manual_seed(1)
    T, H, G = 8, 4, 2
    x, B, C = (torch.randn(T, *s, generator=g, dtype=torch.float64) for s in ((H, 3), (G, 5), (G, 5)))
    dt = orc.softplus(torch.randn(T, H, generator=g, dtype=torch.float64))
    A_log, D = torch.randn(H, generator=g, dtype=torch.float64), torch.randn(H, generator=g, dtype=torch.float64)
    y, _ = orc.ssd_scan(x, B, C, dt, A_log, D)
    for h in range(H):
        L = (-A_log[h].exp() * dt[:, h]).cumsum(0)
        w = torch.tensor([[float(torch.exp(L[t] - L[s]) * dt[s, h] * (C[t, h // 2] @ B[s, h // 2])) if s <= t else 0.0 for s in range(T)] for t in range(T)],
                         dtype=torch.float64)
        assert torch.allclose(y[:, h], w @ x[:, h] + D[h] * x[:, h])


def test_oracle_convolution_and_chunks():
    u, w, b = torch.arange(10, dtype=torch.float64).view(5, 2), torch.tensor([[1.0, 10, 100], [0, 0, 1]], dtype=torch.float64), torch.tensor([0.5, 0.0])
    got = orc.causal_conv(u, w, b.double())
    assert got[:, 1].tolist() == u[:, 1].tolist() and got[:3, 0].tolist() == [0.5, 200.5, 420.5]
    assert torch.equal(orc.causal_conv(u[2:], w, b.double(), u[:2]), got[2:])
    m = orc.chunk_mask(7, 3)
    assert m.sum(1).tolist() == [1, 2, 3, 1, 2, 3, 1] and m[5, 3] and not m[5, 2] and not m[3, 5]


@pytest.mark.parametrize("name", ["small_config", "odd_config", "wide_config"])
def test_oracle_is_causal_and_reads_every_constant(name):
    """Later tokens change nothing; every number of the configuration changes something."""
    d = getattr(sc, name)()
    w, t = sc.weights(d), sc.tokens(d, 90)
    a = orc.forward(d, w, t)
    assert torch.allclose(orc.forward(d, w, t[:50]), a[:50], atol=1e-9)
    for change in (lambda c: c["embedding"].update(scale=2.5), lambda c: c["embedding"]["bigram"].update(mul_prev=4), lambda c: c["embedding"]["bigram"].update(mul_cur=9),
                   lambda c: c["norm"].update(eps=1e-2), *(lambda c, i=i: c["layers"][i]["mixer"].update(gate_cap=1.0) for i, l in enumerate(d["layers"])
                                                           if l["type"] == "mlstm"),
                   *(lambda c, i=i: c["layers"][i]["mixer"]["mask"].update(size=20) for i, l in enumerate(d["layers"]) if l["type"] == "attention")):
        c = json.loads(json.dumps(d))
        change(c)
        assert float((orc.forward(c, w, t) - a).abs().max()) > 1e-3
