"""CPU: configuration, registry, weight files, cache bookkeeping and request validation of the hybrid decoders; properties
of their oracle; the C ABI's symbols."""
import ctypes
import json
import os
import re
import struct

import pytest
import torch

import hybrid_cases as hc
from flash_attn_v100_b200.engine import registry, safetensors
from flash_attn_v100_b200.engine.config import HybridConfig, LatentAttentionSpec, LightningSpec, ModelConfig
from flash_attn_v100_b200.engine.runner import GenerationRunner
from flash_attn_v100_b200.engine.weights import hybrid_tensor_shapes, hybrid_weights
from flash_attn_v100_b200.kv_cache import HybridCache
from oracle import berilix_oracle as orc

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


# ---- configuration and registry --------------------------------------------------------------------
def test_config_reads_every_size_and_constant():
    cfg = HybridConfig.from_dict(hc.small_config())
    assert [type(l.mixer) for l in cfg.layers] == [LightningSpec, LatentAttentionSpec] * 2
    m = cfg.layers[1].mixer
    assert (m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, m.q_rank, m.rot_base) == (3, 40, 16, 56, 48, 64, 1000.0)
    assert m.scale == pytest.approx(56 ** -0.5)
    assert cfg.layers[1].mlp is None and cfg.layers[2].mlp.limit == 0.7
    assert (cfg.vocab_size, cfg.width, cfg.side_dim, cfg.norm_eps) == (160, 96, 8, 1e-5)
    assert len(cfg.layers[0].mixer.decay) == 3


@pytest.mark.parametrize("loop,want", [
    ((1, 3, 3), [(0, 0), (1, 0), (2, 0), (1, 1), (2, 0), (1, 1), (2, 0), (3, 0)]),
    ((0, 4, 2), [(0, 0), (1, 0), (2, 0), (3, 0), (0, 1), (1, 0), (2, 0), (3, 0)]),
    ((2, 3, 1), [(0, 0), (1, 0), (2, 0), (3, 0)]),
    (None, [(0, 0), (1, 0), (2, 0), (3, 0)])])
def test_layer_runs_of_a_loop(loop, want):
    d = hc.small_config()
    d.pop("loop")
    if loop:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    assert HybridConfig.from_dict(d).runs() == [(i, bool(a)) for i, a in want]
    assert orc.layer_runs(d) == [(i, bool(a)) for i, a in want]


@pytest.mark.parametrize("change", [
    lambda d: d["layers"][0].update(type="other"), lambda d: d["layers"][0]["mlp"].update(kind="routed"),
    lambda d: d["layers"][0]["mixer"]["decay"].pop(), lambda d: d["loop"].update(stop=9),
    lambda d: d["layers"][1]["mixer"]["rot"].update(dims=8), lambda d: d.update(width=0)])
def test_config_errors_are_refused(change):
    d = hc.small_config()
    change(d)
    with pytest.raises(ValueError):
        HybridConfig.from_dict(d)


def test_registry_knows_both_families(tmp_path):
    assert registry.architectures() == ["Berilix", "Qwen3", "Sabipel"]
    with pytest.raises(ValueError, match="unknown architecture"):
        registry.family_of({"architecture": "none"})
    fam = registry.family_of({"architecture": "Qwen3"})
    cfg = fam.config_from_dict(dict(num_layers=1, hidden_size=64, num_heads=2, num_kv_heads=1, head_dim=64, intermediate_size=64,
                                    vocab_size=32, architecture="Qwen3"))
    assert isinstance(cfg, ModelConfig) and cfg.rope_theta == 1e6
    hc.write_model(hc.plain_config(), {}, str(tmp_path))
    with pytest.raises(ValueError, match="runs in"):
        registry.load_model(str(tmp_path), torch.float16, "cpu")


# ---- weights ---------------------------------------------------------------------------------------------
def test_safetensors_round_trip_and_damaged_files(tmp_path):
    p = str(tmp_path / "m.safetensors")
    t = {"a": torch.randn(3, 5).bfloat16(), "b": torch.arange(7, dtype=torch.int32), "c": torch.randn(2, 2, 2), "e": torch.empty(0, 4)}
    safetensors.save_file(t, p)
    got = safetensors.load_file(p)
    assert set(got) == set(t) and all(torch.equal(got[k], t[k]) and got[k].dtype == t[k].dtype for k in t)
    raw = open(p, "rb").read()
    (n,) = struct.unpack("<Q", raw[:8])
    head = json.loads(raw[8:8 + n])
    for bad in (b"abc", struct.pack("<Q", 1 << 40) + raw[8:], raw[:-4]):
        open(p, "wb").write(bad)
        with pytest.raises(ValueError):
            safetensors.load_file(p)
    head["a"]["shape"] = [4, 5]
    blob = json.dumps(head).encode()
    open(p, "wb").write(struct.pack("<Q", len(blob)) + blob + raw[8 + n:])
    with pytest.raises(ValueError, match="a does not fit"):
        safetensors.load_file(p)


def test_stacked_projections_are_padded_and_checked():
    d = hc.odd_config()
    cfg, w = HybridConfig.from_dict(d), hc.weights(d)
    got = hybrid_weights(cfg, w, torch.float32, "cpu")
    lw = got["layers"][1]                                    # 3 heads of 9 / 13: 27, 27, 39, 39 rows padded to 32, 32, 40, 40
    assert lw["in_at"] == (0, 32, 64, 104) and lw["w_in"].shape == (144, 50)
    assert torch.equal(lw["w_in"][64:64 + 39], w["l1.mix.v"].float()) and not lw["w_in"][27:32].any()
    la = got["layers"][0]
    assert torch.equal(la["w_uk"].reshape(-1, 22), w["l0.mix.uk"].float())
    assert torch.equal(la["w_in"][la["in_at"][2]:la["in_at"][2] + 6], w["l0.mix.dkv"][22:].float())
    assert "norm2" not in got["layers"][2]
    for change in (lambda t: t.pop("l1.mix.q"), lambda t: t.update(extra=torch.zeros(1)), lambda t: t.update({"final.norm": torch.ones(3)})):
        t = dict(w)
        change(t)
        with pytest.raises(ValueError):
            hybrid_weights(cfg, t, torch.float32, "cpu")


def test_tensor_shapes_follow_the_configuration():
    shapes = hybrid_tensor_shapes(HybridConfig.from_dict(hc.small_config()))
    assert shapes["l1.mix.dkv"] == (64, 96) and shapes["l1.mix.uq"] == (3 * 56, 64) and shapes["side.embed"] == (160, 32)
    assert shapes["l2.mix.norm"] == (192,) and "l1.mlp.gate" not in shapes and "l1.norm2" not in shapes
    assert not any("side" in n for n in hybrid_tensor_shapes(HybridConfig.from_dict(hc.plain_config())))


# ---- cache -------------------------------------------------------------------------------------------------
def test_hybrid_cache_keeps_pages_and_state_slots_together():
    c = HybridCache([("state", 2, 4, 6), ("latent", 21)], num_blocks=5, max_batch=2, max_blocks_per_seq=4, device="cpu")
    assert c.stores[0].shape == (2, 2, 4, 6) and c.stores[0].dtype == torch.float32
    assert c.stores[1].shape == (5, 16, 24) and c.stores[1].dtype == torch.bfloat16      # rows rounded up to 16 bytes
    assert not c.enable_prefix_cache                                                     # pages alone do not bring a state back
    a, b = c.allocate("a", 40), c.allocate("b", 16)
    assert {a, b} == {0, 1} and c.get_num_free_blocks() == 1
    with pytest.raises(MemoryError):
        c.allocate("c", 1)
    first = c.get_block_table("a")
    c.release("a")
    assert c.get_num_free_blocks() == 4 and c.allocate("d", 33) == a and set(c.get_block_table("d")) == set(first)
    c.check_errors()
    c.status.fill_(2)
    with pytest.raises(RuntimeError, match="outside the cache"):
        c.check_errors()
    c.check_errors()                                                                     # reported once
    assert HybridCache([("latent", 8)], 2, 1, 2, "cpu", torch.float32).enable_prefix_cache
    with pytest.raises(ValueError):
        HybridCache([("ring", 8)], 2, 1, 2, "cpu")


class _FakeModel:
    """Records the passes a runner asks for; the logits of a token are its position."""

    class cfg:
        vocab_size = 50
    device, world, comm, group, supports_portions = torch.device("cpu"), 1, None, None, True

    def __init__(self):
        self.passes = []

    def make_cache(self, max_batch, max_seq_len, num_blocks=0):
        return HybridCache([("latent", 8)], num_blocks or 64, max_batch, (max_seq_len + 15) // 16, "cpu")

    def forward(self, token_ids, positions, **kw):
        self.passes.append((token_ids.tolist(), positions.tolist(), kw.get("lens"), kw.get("past"), kw["state_rows"].tolist()))
        return positions[kw["want"]].float()[:, None]

    def logits(self, hidden):
        return hidden.expand(-1, 50)


def _runner(monkeypatch):
    monkeypatch.setattr(torch.cuda, "Stream", lambda **kw: None)
    m = _FakeModel()
    return m, GenerationRunner(m, max_batch=4, max_seq_len=100)


def test_steps_group_decode_tokens_and_prompt_portions(monkeypatch):
    m, r = _runner(monkeypatch)
    for i in "abc":
        r.start(i)
    out = r.step([("a", [1, 2, 3], [0, 2])])
    assert out[0][:, 0].tolist() == [0, 2] and m.passes[-1] == ([1, 2, 3], [0, 1, 2], [3], [0], [0])
    out = r.step([("b", [4, 5], [1]), ("a", [6], [0]), ("c", [7], [])])
    assert [o[:, 0].tolist() for o in out] == [[1], [3], []]
    # a's single token is a decode pass; b's and c's first tokens are one prompt pass
    assert m.passes[-2] == ([6], [3], None, None, [0]) and m.passes[-1] == ([4, 5, 7], [0, 1, 0], [2, 1], [0, 0], [1, 2])
    r.step([("b", [8, 9, 10], [2])])
    assert m.passes[-1][:4] == ([8, 9, 10], [2, 3, 4], [3], [2])
    r.finish("b")
    r.start("d")
    r.step([("d", [1], [0])])
    assert m.passes[-1] == ([1], [0], [1], [0], [1])          # b's slot, from position 0


def test_step_refuses_bad_requests(monkeypatch):
    m, r = _runner(monkeypatch)
    r.start("a")
    for bad in ([("a", [], [])], [("a", [50], [])], [("a", [-1], [])], [("a", [1], [1])], [("a", [1] * 101, [])],
                [("a", [1], []), ("a", [2], [])]):
        with pytest.raises(ValueError):
            r.step(bad)
    assert m.passes == []


# ---- oracle --------------------------------------------------------------------------------------------------
def test_oracle_recurrence_equals_its_closed_form():
    g = torch.Generator().manual_seed(0)
    q, k, v = (torch.randn(9, 2, n, generator=g, dtype=torch.float64) for n in (3, 3, 5))
    d = torch.tensor([0.5, 0.9], dtype=torch.float64)
    o, s = orc.linear_attention_scan(q, k, v, d)
    for h in range(2):
        w = torch.tensor([[d[h] ** (i - j) if j <= i else 0.0 for j in range(9)] for i in range(9)], dtype=torch.float64)
        assert torch.allclose(o[:, h], ((q[:, h] @ k[:, h].T) * w) @ v[:, h])
    o1, s1 = orc.linear_attention_scan(q[:4], k[:4], v[:4], d)
    o2, s2 = orc.linear_attention_scan(q[4:], k[4:], v[4:], d, s1)
    assert torch.allclose(torch.cat([o1, o2]), o) and torch.allclose(s2, s)


def test_oracle_scores_depend_on_distances_only():
    g = torch.Generator().manual_seed(1)
    q, k = torch.randn(1, 12, generator=g, dtype=torch.float64), torch.randn(1, 12, generator=g, dtype=torch.float64)
    at = lambda x, p: orc.rotate(x, torch.tensor([p]), 100.0, 8)
    s = lambda p: (at(q, p) * at(k, p - 5)).sum()
    assert torch.allclose(s(5), s(400)) and torch.equal(at(q, 3)[:, 8:], q[:, 8:])


def test_oracle_is_causal():
    d = hc.small_config()
    w, t = hc.weights(d), hc.tokens(d, 12)
    a = orc.forward(d, w, t)
    assert torch.allclose(orc.forward(d, w, t[:7]), a[:7])


# ---- library ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("library, prefix", [("rows", "far"), ("hybrid", "fah"), ("mixers", "fam")])
def test_library_exports_every_declared_symbol(library, prefix):
    from flash_attn_v100_b200 import _lib
    from flash_attn_v100_b200.build import build
    build(library=library)
    lib = _lib.library(library)
    text = re.sub(r"/\*.*?\*/", "", open(os.path.join(ROOT, "include", f"fa_b200_{library}.h")).read(), flags=re.S)
    names = set(re.findall(rf"\b({prefix}_[a-z0-9_]+)\s*\(", text))
    assert names == set(_lib._ABIS[library][0]) and all(hasattr(lib, n) for n in names)


def test_calls_check_their_arguments_before_the_device():
    from flash_attn_v100_b200 import _lib
    lib = _lib.library("rows")
    p = ctypes.c_void_p(256)
    norm = lambda **kw: lib.far_residual_norm(ctypes.byref(_lib.ResidualNorm(**dict(dict(rows=1, cols=8, eps=1e-5, dtype=1, embed_scale=1.0), **kw))), None)
    assert norm() == -1
    assert b"x is null" in lib.far_last_error()
    assert norm(x=256, dtype=7) == -1
    assert norm(x=256, w=256, out=256, w2=256) == -1 and norm(x=256, embed_scale=2.0) == -1
    assert lib.far_gated_norm(p, p, 4, p, p, 8, 1, 8, 8, 0, 1e-5, 1, None) == -1
    assert lib.far_gated_norm(p, p, 8, p, p, 8, 1, 8, 3, 0, 1e-5, 1, None) == -1
    assert lib.far_side_gate(p, p, p, 10, 8, 4, p, 1, 8, 1, None) == -1
    assert lib.far_bigram_rows(p, None, p, p, p, 1, 2, 1, 7, 3, 5, p, p, None) == -1
    lib = _lib.library("hybrid")
    assert lib.fah_rotate_heads(p, p, p, 1, 2, 8, 4, 6, 1, None) == -1
    assert lib.fah_lightning(p, 10, 0, 4, 8, 2, 4, 4, p, p, 1, p, p, None, 1, 1, 1, p, None, 0, p, 1, None) == -1
    assert lib.fah_latent_prefill(p, p, p, None, 0, p, p, 1, 1, 1, 1, 2, 132, 64, 64, 0.1, p, p, None) == -2
    assert b"not built" in lib.fah_last_error()
    assert [lib.fah_latent_prefill_supported(*a) for a in ((128, 64, 128, 0.1, 1), (128, 64, 128, 0.1, 0), (20, 8, 8, 0.1, 1),
                                                           (64, 8, 8, -0.1, 1))] == [1, 0, 0, 0]
