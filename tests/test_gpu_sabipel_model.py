"""GPU: the Sabipel decoder through the engine's own runner, cache and entry points against the plain forward pass of
oracle/sabipel_oracle.py on the same weights.

In float32 logits must agree to rounding; in bfloat16 to a fraction of the logits' spread.  However a prompt is cut, whatever else
is in the batch and whichever pages and slots are used, the same logits must come out."""
import json
import os
import subprocess
import sys

import pytest
import torch

import sabipel_cases as sc
from oracle import sabipel_oracle as orc

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {torch.float32: 3e-4, torch.bfloat16: 8e-2}        # root mean square over the vocabulary, relative to the spread
TYPES = [torch.float32, torch.bfloat16]
CONFIGS = {"small": sc.small_config, "odd": sc.odd_config, "wide": sc.wide_config}


def runner(cfg, w, dtype, max_batch=4, max_seq=400, **kw):
    from flash_attn_v100_b200.engine import GenerationRunner
    return GenerationRunner(sc.model(cfg, w, dtype), max_batch, max_seq, **kw)


def play(r, toks, portions, rid="a"):
    """All logits of one request that arrives in the given portions; the request is finished again."""
    r.start(rid)
    out, at = [], 0
    for n in portions:
        out.append(r.step([(rid, toks[at:at + n], list(range(n)))])[0])
        at += n
    assert at == len(toks)
    r.finish(rid)
    r.check_errors()
    return torch.cat(out).cpu()


def agree(got, ref, dtype, factor=1.0):
    d = got.double() - ref.double()
    d = d - d.mean(-1, keepdim=True)
    err = d.pow(2).mean(-1).sqrt() / ref.double().std()
    assert float(err.max()) < TOL[dtype] * factor, (float(err.max()), int(err.argmax()))


@pytest.fixture(scope="module")
def case():
    made = {}

    def get(name, n=210):
        if (name, n) not in made:
            cfg = CONFIGS[name]()
            w, t = sc.weights(cfg, 3), sc.tokens(cfg, n)
            made[name, n] = cfg, w, t, orc.forward(cfg, w, t)
        return made[name, n]
    return get


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_logits_do_not_depend_on_how_a_prompt_is_cut(case, name, dtype):
    """The whole prompt, one token at a time, and portions down to two tokens (cut inside and at the edges of pages, key tiles
    and chunks, of the attention and of the recurrences) against the oracle."""
    cfg, w, t, ref = case(name)
    r = runner(cfg, w, dtype)
    n = len(t)
    for portions in ([n], [1] * 70, [2] * 10 + [3, 13, 64, 2, 1, 1, n - 104], [15, 1, 1, 47, 1, 63, 2, 33, n - 163], [100] + [1] * 60 + [50], [50, 50, 64, 46],
                     [128, 82], [129, 1, 80], [48, 2, 2, 49, n - 101]):
        got = play(r, t[:sum(portions)], portions)
        agree(got, ref[:sum(portions)], dtype)


@pytest.mark.parametrize("name", list(CONFIGS))
def test_residual_after_every_layer(case, name):
    cfg, w, t, _ = case(name)
    want, got = [], []
    orc.forward(cfg, w, t[:70], layers_out=want)
    r = runner(cfg, w, torch.float32)
    r.model.layer_hook = lambda x: got.append(x.cpu().clone())
    play(r, t[:70], [70])
    assert len(got) == len(want) == len(cfg["layers"])
    for a, b in zip(got, want):
        assert (a.double() - b).abs().max() < 1e-4 * b.abs().max()


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("name", ["small", "wide"])
def test_batches_of_unequal_requests_equal_each_alone(case, name, dtype):
    """Prompts, portions and decode tokens of different requests in one step; requests that come, go and are replaced."""
    cfg, w, t, ref = case(name)
    r = runner(cfg, w, dtype, max_batch=3)
    u = sc.tokens(cfg, 110, 7)
    ref_u = orc.forward(cfg, w, u)
    got = {k: [] for k in "abc"}

    def step(*entries):
        for (k, _, _), lg in zip(entries, r.step([(k, s[a:b], list(range(b - a))) for k, s, (a, b) in entries])):
            got[k].append(lg.cpu())
    for k in "abc":
        r.start(k)
    step(("a", t, (0, 33)), ("b", u, (0, 2)))
    step(("b", u, (2, 95)), ("c", t, (0, 1)), ("a", t, (33, 34)))
    for i in range(5):
        step(("a", t, (34 + i, 35 + i)), ("c", t, (1 + 2 * i, 3 + 2 * i)), ("b", u, (95 + i, 96 + i)))
    r.finish("a")
    agree(torch.cat(got["a"]), ref[:39], dtype)
    got["a"] = []
    r.start("a")                                            # a's pages and slot, another sequence
    step(("a", u, (0, 40)), ("c", t, (11, 200)))
    step(("c", t, (200, 201)), ("a", u, (40, 41)), ("b", u, (100, 101)))
    step(("c", t, (201, 210)), ("a", u, (41, 105)), ("b", u, (101, 110)))
    r.check_errors()
    agree(torch.cat(got["a"]), ref_u[:105], dtype)
    agree(torch.cat(got["b"]), ref_u[:110], dtype)
    agree(torch.cat(got["c"]), ref, dtype)


def test_pages_and_slots_that_are_used_again(case):
    """What a request left in its pages, state, convolution inputs and last token does not reach the next one, however that one
    starts."""
    cfg, w, t, ref = case("small")
    r = runner(cfg, w, torch.float32, max_batch=1, max_seq=224)
    noise = sc.tokens(cfg, 210, 9)
    for portions in ([1] * 8, [2, 70], [1, 1, 60], [210]):
        play(r, noise, [209, 1])
        for store in r.kv.stores:
            assert all(s.abs().sum() > 0 for s in store)
        agree(play(r, t[:sum(portions)], portions), ref[:sum(portions)], torch.float32)


def test_pages_of_past_chunks_are_given_up(case):
    """Every attention layer reads its current chunk only: a long request holds the pages of the chunks in use, others are free for
    the next request while it runs on."""
    cfg = sc.config([(sc.attention(2, 1, 16, 16, 64), 32), (sc.mlstm(2, 16, 16), 32), (sc.attention(4, 2, 16, 8, 32), None)])
    w, t = sc.weights(cfg, 1), sc.tokens(cfg, 300, 2)
    ref = orc.forward(cfg, w, t)
    for dtype in TYPES:
        r = runner(cfg, w, dtype, max_batch=2, max_seq=300, num_blocks=12)
        r.start("a")
        got, at = [], 0
        for n in [60, 64, 5, 40] + [1] * 30 + [64, 37]:
            got.append(r.step([("a", t[at:at + n], list(range(n)))])[0].cpu())
            at += n
            assert at // 64 * 4 <= sum(b < 0 for b in r.kv.get_block_table("a")) <= at // 64 * 4
            if at == 129:
                r.start("b")
                other = r.step([("b", t[:64], list(range(64)))])[0].cpu()
                r.finish("b")
        assert at == 300
        r.check_errors()
        agree(torch.cat(got), ref, dtype)
        agree(other, ref[:64], dtype)
        r.finish("a")
        assert r.kv.get_num_free_blocks() == 12


@pytest.mark.parametrize("dtype", TYPES)
def test_single_keys_decide(dtype):
    """Sharp attention with flat slopes: single keys hold most of the weight, so that one wrong, missing or extra key among hundreds
    shows, above all at the edges of a chunk; prompts, portions and decoding."""
    cfg = sc.config([(sc.attention(2, 1, 32, 32, 160, scale=1.0), 64), (sc.attention(1, 1, 24, 40, 97, v_mix=False, scale=1.0), None)], scale=1.0)
    w, t = sc.weights(cfg, 5), sc.tokens(cfg, 330, 5)
    for i in (0, 1):
        w[f"l{i}.mix.q.norm"] = w[f"l{i}.mix.q.norm"] * 1.2
    ref = orc.forward(cfg, w, t)
    spread = ref.std()
    for layer, size in ((0, 160), (1, 97)):                 # a chunk that is one token off does show
        for off in (-1, 1):
            other = json.loads(json.dumps(cfg))
            other["layers"][layer]["mixer"]["mask"]["size"] = size + off
            d = orc.forward(other, w, t) - ref
            assert float((d.std(-1) / spread).max()) > 3 * TOL[torch.bfloat16]
    moved = orc.forward(cfg, w, [(t[0] + 1) % cfg["vocab"]] + t[1:])
    assert float((moved - ref).std(-1)[90:160].max() / spread) > 0.1 and float((moved - ref)[194:].abs().max()) < 1e-9
    r = runner(cfg, w, dtype)
    for portions in ([330], [150] + [1] * 30 + [5, 10] + [1] * 10 + [125], [96, 2, 64, 30, 3, 2, 1, 132], [159, 1, 1, 169], [160, 170], [161, 169], [1] * 200 + [130]):
        agree(play(r, t, portions), ref, dtype, 1.0 if dtype == torch.float32 else 1.5)


@pytest.mark.parametrize("dtype", TYPES)
def test_first_tokens(case, dtype):
    """Sequences of one to four tokens, at once and one by one: the first bigram row, zeros ahead of the convolution, empty states."""
    for name in CONFIGS:
        cfg, w, t, _ = case(name)
        r = runner(cfg, w, dtype)
        for first in (0, 5, 9):
            for n in (1, 2, 3, 4):
                ref = orc.forward(cfg, w, t[first:first + n])
                for portions in ([n], [1] * n):
                    agree(play(r, t[first:first + n], portions), ref, dtype)


def test_long_decoding_keeps_the_state_exact():
    cfg = sc.config([(sc.mlstm(3, 32, 32), 48), (sc.mamba2(4, 16, 32, groups=2), None), (sc.attention(2, 2, 16, 16, 48), 32)])
    w, t = sc.weights(cfg, 6), sc.tokens(cfg, 390, 6)
    w["l0.mix.f.b"] = torch.tensor([9.0, 4.0, 0.0]).bfloat16()     # from a memory of thousands of tokens to one of two
    w["l1.mix.dt_bias"] = torch.tensor([-7.0, -4.0, -2.0, 1.0]).bfloat16()
    ref = orc.forward(cfg, w, t)
    for dtype in TYPES:
        agree(play(runner(cfg, w, dtype), t, [30] + [1] * 360), ref, dtype)


def test_a_lost_state_would_show(case):
    """The logits do depend on what hundreds of tokens ago went into the states."""
    cfg = sc.config([(sc.mlstm(3, 32, 32), 48), (sc.mamba2(4, 16, 32, groups=2), None)])
    w, t = sc.weights(cfg, 6), sc.tokens(cfg, 200, 6)
    w["l0.mix.f.b"] = torch.full((3,), 9.0).bfloat16()
    w["l1.mix.dt_bias"] = torch.full((4,), -6.0).bfloat16()
    ref = orc.forward(cfg, w, t)
    w0 = {k: v.clone() for k, v in w.items()}
    w0["pos"][:100] = w["pos"][100:200]
    late = orc.forward(cfg, w0, t[100:])
    assert float((ref[150:] - late[50:]).std(-1).median() / ref.std()) > 0.1
    for dtype in TYPES:
        agree(play(runner(cfg, w, dtype), t, [90, 2, 8, 60, 40]), ref, dtype)


@pytest.mark.parametrize("name", list(CONFIGS))
def test_greedy_generation_matches_the_oracle(case, name):
    """`generate`: prefill in chunks and portions, decode steps eagerly and from a CUDA graph, cached graph used twice."""
    cfg, w, _, _ = case(name)
    prompts = torch.tensor([sc.tokens(cfg, 37, s) for s in range(3)])
    want = [orc.greedy_generate(cfg, w, p.tolist(), 16)[0] for p in prompts]
    r = runner(cfg, w, torch.float32, max_batch=3, max_seq=64)
    for kw in (dict(), dict(prefill_chunk=2), dict(prefill_portion=5), dict(prefill_chunk=1, prefill_portion=36)):
        assert r.generate(prompts, 16, **kw).tolist() == want
    eager = runner(cfg, w, torch.float32, max_batch=3, max_seq=64, use_cuda_graph=False)
    assert eager.generate(prompts, 16).tolist() == want
    assert r.generate(prompts[:2], 16).tolist() == want[:2]


def test_bfloat16_graph_replay_reproduces_eager_tokens(case):
    for name in ("small", "wide"):
        cfg, w, _, _ = case(name)
        prompts = torch.tensor([sc.tokens(cfg, 50, s) for s in range(4)])
        a = runner(cfg, w, torch.bfloat16, use_cuda_graph=False).generate(prompts, 24)
        r = runner(cfg, w, torch.bfloat16)
        assert torch.equal(r.generate(prompts, 24), a) and torch.equal(r.generate(prompts, 24), a)


def test_the_table_of_positions_bounds_a_request(case):
    cfg = sc.config([(sc.mlstm(2, 16, 16), 32)], positions=40)
    w, t = sc.weights(cfg, 1), sc.tokens(cfg, 41)
    r = runner(cfg, w, torch.float32, max_seq=200)
    agree(play(r, t[:40], [39, 1]), orc.forward(cfg, w, t[:40]), torch.float32)
    r.start("a")
    with pytest.raises(ValueError, match="max_seq_len=40"):
        r.step([("a", t, [])])
    with pytest.raises(ValueError):
        r.generate(torch.tensor([t[:30]]), 11)


def test_trace_replay_and_command_line(case, tmp_path):
    import numpy as np
    cfg, w, t, ref = case("small")
    folder, out = tmp_path / "model", tmp_path / "out"
    folder.mkdir()
    out.mkdir()
    sc.write_model(cfg, w, str(folder))
    steps = [dict(step=0, entries=[dict(id="x", tokens=t[:60], want=[0, 59])], end=[]),
             dict(step=1, entries=[dict(id="x", tokens=t[60:62], want=[])], end=[]),
             dict(step=2, entries=[dict(id="x", tokens=t[62:63], want=[0])], end=["x"]),
             dict(step=3, entries=[dict(id="x", tokens=t[:5], want=[4])], end=["x"])]
    cmd = [os.path.join(ROOT, "bin", "trace_run"), "--model", str(folder), "--out", str(out), "--max-tokens", "64", "--dtype"]
    for dtype in TYPES:
        res = subprocess.run(cmd + [str(dtype)[6:]], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True,
                             timeout=240)
        assert res.returncode == 0, res.stderr[-2000:]
        assert res.stdout.split("\n")[:4] == [f"done {i}" for i in range(4)]
        assert sorted(os.listdir(out)) == ["0.f32", "2.f32", "3.f32"]
        for n, rows in ((0, [0, 59]), (2, [62]), (3, [4])):
            got = torch.from_numpy(np.fromfile(out / f"{n}.f32", dtype="<f4")).view(len(rows), -1)
            agree(got, ref[rows], dtype)
            os.unlink(out / f"{n}.f32")
    res = subprocess.run([sys.executable, "-m", "flash_attn_v100_b200.engine", "--model", str(folder), "--prompt",
                          ",".join(map(str, t[:20])), "--prompt", "3", "--max-new-tokens", "6", "--dtype", "float32"], cwd=ROOT,
                         capture_output=True, text=True, timeout=240)
    assert res.returncode == 0, res.stderr[-2000:]
    want = [orc.greedy_generate(cfg, w, p, 6)[0] for p in (t[:20], [3])]
    assert [list(map(int, line.split(","))) for line in res.stdout.strip().split("\n")] == want
