"""GPU: the hybrid decoder through the engine's own runner, cache and entry points against the plain forward pass of
oracle/berilix_oracle.py on the same weights.

In float32 logits must agree to rounding; in bfloat16 to a fraction of the logits' spread.  However a prompt is cut, whatever else
is in the batch and whichever pages and slots are used, the same logits must come out."""
import os
import subprocess
import sys

import pytest
import torch

import hybrid_cases as hc
from oracle import berilix_oracle as orc

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {torch.float32: 3e-4, torch.bfloat16: 6e-2}        # root mean square over the vocabulary, relative to the spread
CONFIGS = {"small": hc.small_config, "odd": hc.odd_config, "plain": hc.plain_config}


def runner(cfg, w, dtype, max_batch=4, max_seq=400, **kw):
    from flash_attn_v100_b200.engine import GenerationRunner
    return GenerationRunner(hc.model(cfg, w, dtype), max_batch, max_seq, **kw)


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

    def get(name, n=150):
        if (name, n) not in made:
            cfg = CONFIGS[name]()
            w, t = hc.weights(cfg, 3), hc.tokens(cfg, n)
            made[name, n] = cfg, w, t, orc.forward(cfg, w, t)
        return made[name, n]
    return get


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_logits_do_not_depend_on_how_a_prompt_is_cut(case, name, dtype):
    """The whole prompt, one token at a time, and portions down to two tokens (cut inside and at the edges of pages, key tiles
    and chunks) against the oracle."""
    cfg, w, t, ref = case(name)
    r = runner(cfg, w, dtype)
    n = len(t)
    for portions in ([n], [1] * 40, [2] * 10 + [3, 13, 64, 2, 1, 1, n - 104], [15, 1, 1, 47, 1, 63, 2, n - 130], [100] + [1] * (n - 100)):
        got = play(r, t[:sum(portions)], portions)
        agree(got, ref[:sum(portions)], dtype)


@pytest.mark.parametrize("name", ["small", "odd"])
def test_residual_after_every_layer_run(case, name):
    cfg, w, t, _ = case(name)
    want, got = [], []
    orc.forward(cfg, w, t[:40], layers_out=want)
    r = runner(cfg, w, torch.float32)
    r.model.layer_hook = lambda x: got.append(x.cpu().clone())
    play(r, t[:40], [40])
    assert len(got) == len(want) == len(orc.layer_runs(cfg))
    for a, b in zip(got, want):
        assert (a.double() - b).abs().max() < 1e-4 * b.abs().max()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_batches_of_unequal_requests_equal_each_alone(case, dtype):
    """Prompts, portions and decode tokens of different requests in one step; requests that come, go and are replaced."""
    cfg, w, t, ref = case("small")
    r = runner(cfg, w, dtype, max_batch=3)
    u = hc.tokens(cfg, 60, 7)
    ref_u = orc.forward(cfg, w, u)
    got = {k: [] for k in "abc"}

    def step(*entries):
        for (k, _, _), lg in zip(entries, r.step([(k, s[a:b], list(range(b - a))) for k, s, (a, b) in entries])):
            got[k].append(lg.cpu())
    for k in "abc":
        r.start(k)
    step(("a", t, (0, 33)), ("b", u, (0, 2)))
    step(("b", u, (2, 50)), ("c", t, (0, 1)), ("a", t, (33, 34)))
    for i in range(5):
        step(("a", t, (34 + i, 35 + i)), ("c", t, (1 + 2 * i, 3 + 2 * i)), ("b", u, (50 + i, 51 + i)))
    r.finish("a")
    agree(torch.cat(got["a"]), ref[:39], dtype)
    got["a"] = []
    r.start("a")                                            # a's pages and slot, another sequence
    step(("a", u, (0, 40)), ("c", t, (11, 90)))
    step(("c", t, (90, 91)), ("a", u, (40, 41)))
    r.check_errors()
    agree(torch.cat(got["a"]), ref_u[:41], dtype)
    agree(torch.cat(got["b"]), ref_u[:55], dtype)
    agree(torch.cat(got["c"]), ref[:91], dtype)


def test_pages_and_slots_that_are_used_again(case):
    """What a request left in its pages and state slot does not reach the next one, however that one starts."""
    cfg, w, t, ref = case("small")
    r = runner(cfg, w, torch.float32, max_batch=1, max_seq=160)
    noise = hc.tokens(cfg, 150, 9)
    for portions in ([1] * 8, [2, 70], [150]):
        play(r, noise, [150])
        for s in r.kv.stores:
            assert s.abs().sum() > 0
        agree(play(r, t[:sum(portions)], portions), ref[:sum(portions)], torch.float32)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_a_far_key_decides(dtype):
    """Sharp attention: the query and key projections are scaled until single keys hold most of the weight, so that one wrong, missing
    or extra key among hundreds shows; prompts, portions and decoding."""
    cfg = hc.config([hc.layer(hc.latent(2, 32, 16, 32, 64, 48, scale=0.5), 64), hc.layer(hc.latent(4, 16, 8, 24, 40, 32, scale=0.6), None)])
    w, t = hc.weights(cfg, 5), hc.tokens(cfg, 330, 5)
    for i in (0, 1):
        w[f"l{i}.mix.uq"] = w[f"l{i}.mix.uq"] * 1.5
    ref = orc.forward(cfg, w, t)
    moved = orc.forward(cfg, w, [(t[0] + 1) % cfg["vocab"]] + t[1:])
    far = (moved - ref).std(-1)[200:] / ref.std()
    assert float(far.max()) > 0.25               # a query hundreds of tokens on does depend on the first key
    r = runner(cfg, w, dtype)
    for portions in ([330], [300] + [1] * 30, [129, 2, 64, 5, 63, 16, 1, 50]):
        agree(play(r, t, portions), ref, dtype, 1.0 if dtype == torch.float32 else 1.5)


def test_long_decoding_keeps_the_state_exact():
    cfg = hc.config([hc.layer(hc.lightning(3, 32, 32, [0.5, 0.99, 0.9999]), 48), hc.layer(hc.latent(2, 16, 8, 16, 24, 24), None)])
    w, t = hc.weights(cfg, 6), hc.tokens(cfg, 390, 6)
    ref = orc.forward(cfg, w, t)
    for dtype in (torch.float32, torch.bfloat16):
        agree(play(runner(cfg, w, dtype), t, [30] + [1] * 360), ref, dtype)


@pytest.mark.parametrize("name", list(CONFIGS))
def test_greedy_generation_matches_the_oracle(case, name):
    """`generate`: prefill in chunks and portions, decode steps eagerly and from a CUDA graph, cached graph used twice."""
    cfg, w, _, _ = case(name)
    prompts = torch.tensor([hc.tokens(cfg, 37, s) for s in range(3)])
    want = [orc.greedy_generate(cfg, w, p.tolist(), 10)[0] for p in prompts]
    r = runner(cfg, w, torch.float32, max_batch=3, max_seq=64)
    for kw in (dict(), dict(prefill_chunk=2), dict(prefill_portion=5), dict(prefill_chunk=1, prefill_portion=36)):
        assert r.generate(prompts, 10, **kw).tolist() == want
    eager = runner(cfg, w, torch.float32, max_batch=3, max_seq=64, use_cuda_graph=False)
    assert eager.generate(prompts, 10).tolist() == want
    assert r.generate(prompts[:2], 10).tolist() == want[:2]
    logs = []
    runner(cfg, w, torch.float32, max_batch=3, max_seq=64, use_cuda_graph=False).generate(prompts, 3, logits_out=logs)
    agree(logs[0][2].cpu(), torch.stack([orc.forward(cfg, w, p.tolist())[-1] for p in prompts]), torch.float32)


def test_bfloat16_graph_replay_reproduces_eager_tokens(case):
    cfg, w, _, _ = case("small")
    prompts = torch.tensor([hc.tokens(cfg, 50, s) for s in range(4)])
    a = runner(cfg, w, torch.bfloat16, use_cuda_graph=False).generate(prompts, 24)
    r = runner(cfg, w, torch.bfloat16)
    assert torch.equal(r.generate(prompts, 24), a) and torch.equal(r.generate(prompts, 24), a)


def test_running_out_of_blocks_is_an_error_and_leaves_the_others_alone(case):
    cfg, w, t, ref = case("small")
    r = runner(cfg, w, torch.float32, max_batch=3, max_seq=128, num_blocks=6)
    r.start("a")
    r.start("b")
    first = r.step([("a", t[:60], [59])])[0]
    with pytest.raises(MemoryError):
        r.step([("b", t[:40], [0])])
    r.finish("b")
    nxt = r.step([("a", t[60:61], [0])])[0]
    agree(torch.cat([first, nxt]).cpu(), ref[59:61], torch.float32)


def test_qwen3_runs_through_the_same_steps():
    """The runner's step interface on the tensor-parallel decoder: one-pass prompts, then decode tokens, unequal requests."""
    from flash_attn_v100_b200.engine import GenerationRunner, TPDecoder, make_rank_weights, tiny_config
    from oracle import model_oracle as mo
    cfg = tiny_config()
    r = GenerationRunner(TPDecoder(cfg, make_rank_weights(cfg, 0, 1, 5, "cuda", gen_device="cpu")), 4, 64)
    g = torch.Generator().manual_seed(1)
    a, b = (torch.randint(0, cfg.vocab_size, (n,), generator=g).tolist() for n in (20, 9))
    ra, rb = (mo.forward_logits(cfg, 5, torch.tensor([s]))[0] for s in (a, b))
    r.start("a")
    r.start("b")
    out = r.step([("a", a[:12], [3, 11]), ("b", b[:7], [6])])
    assert (out[0].cpu() - ra[[3, 11]]).abs().max() < 3e-2 and (out[1].cpu() - rb[[6]]).abs().max() < 3e-2
    for i in range(2):
        out = r.step([("b", b[7 + i:8 + i], [0]), ("a", a[12 + i:13 + i], [0])])
        assert (out[0].cpu() - rb[[7 + i]]).abs().max() < 3e-2 and (out[1].cpu() - ra[[12 + i]]).abs().max() < 3e-2
    with pytest.raises(NotImplementedError):
        r.step([("a", a[14:17], [])])
    r.check_errors()


def test_trace_replay_and_command_line(case, tmp_path):
    import json
    import numpy as np
    cfg, w, t, ref = case("small")
    folder, out = tmp_path / "model", tmp_path / "out"
    folder.mkdir()
    out.mkdir()
    hc.write_model(cfg, w, str(folder))
    steps = [dict(step=0, entries=[dict(id="x", tokens=t[:30], want=[0, 29])], end=[]),
             dict(step=1, entries=[dict(id="x", tokens=t[30:32], want=[])], end=[]),
             dict(step=2, entries=[dict(id="x", tokens=t[32:33], want=[0])], end=["x"]),
             dict(step=3, entries=[dict(id="x", tokens=t[:5], want=[4])], end=["x"])]
    cmd = [os.path.join(ROOT, "bin", "trace_run"), "--model", str(folder), "--out", str(out), "--max-tokens", "48", "--dtype"]
    for dtype in (torch.float32, torch.bfloat16):
        res = subprocess.run(cmd + [str(dtype)[6:]], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True,
                             timeout=240)
        assert res.returncode == 0, res.stderr[-2000:]
        assert res.stdout.split("\n")[:4] == [f"done {i}" for i in range(4)]
        assert sorted(os.listdir(out)) == ["0.f32", "2.f32", "3.f32"]
        for n, rows in ((0, [0, 29]), (2, [32]), (3, [4])):
            got = torch.from_numpy(np.fromfile(out / f"{n}.f32", dtype="<f4")).view(len(rows), -1)
            agree(got, ref[rows], dtype)
            os.unlink(out / f"{n}.f32")
    res = subprocess.run([sys.executable, "-m", "flash_attn_v100_b200.engine", "--model", str(folder), "--prompt",
                          ",".join(map(str, t[:20])), "--prompt", "3", "--max-new-tokens", "6", "--dtype", "float32"], cwd=ROOT,
                         capture_output=True, text=True, timeout=240)
    assert res.returncode == 0, res.stderr[-2000:]
    want = [orc.greedy_generate(cfg, w, p, 6)[0] for p in (t[:20], [3])]
    assert [list(map(int, line.split(","))) for line in res.stdout.strip().split("\n")] == want
