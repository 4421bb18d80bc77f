"""Throughput of the hybrid decoder and its kernels beside the Qwen3-style decoder's at equal size (`bench.py --workload hybrid`).

Random weights and token ids.  Models: eight layers of width 4096, 32 heads, feed-forward 12288, vocabulary 32768; the hybrid
decoder has latent attention in every fourth layer, decayed linear attention in the others and a token side input of 256.
Kernels: every kernel of both at the sizes such layers give, one call per measurement with the L2 flushed before it, next to the
bytes or flops the operation needs.
"""
from __future__ import annotations

import torch

from .. import hybrid_ops as hops
from .. import ops
from .config import ClampedGluSpec, HybridConfig, HybridLayer, LatentAttentionSpec, LightningSpec, ModelConfig
from .hybrid import GLU_ALPHA, GLU_SHIFT, HybridDecoder
from .model import TPDecoder
from .runner import GenerationRunner
from .weights import hybrid_weights, make_rank_weights, random_hybrid_tensors

LAYERS, WIDTH, HEADS, DIM, ROT, FF, VOCAB, SIDE, Q_RANK, KV_RANK = 8, 4096, 32, 128, 64, 12288, 32768, 256, 1536, 512


def hybrid_config() -> HybridConfig:
    decay = tuple(1.0 - 2.0 ** (-2.0 - 6.0 * h / HEADS) for h in range(HEADS))
    lin = LightningSpec(HEADS, DIM, DIM, decay)
    lat = LatentAttentionSpec(HEADS, DIM, ROT, DIM, Q_RANK, KV_RANK, (DIM + ROT) ** -0.5, 1e6)
    glu = ClampedGluSpec(FF, 7.0)
    layers = tuple(HybridLayer(lat if i % 4 == 3 else lin, glu) for i in range(LAYERS))
    return HybridConfig(VOCAB, WIDTH, layers, 1e-6, SIDE)


def qwen_config() -> ModelConfig:
    return ModelConfig(LAYERS, WIDTH, HEADS, 8, DIM, FF, VOCAB)


class _Timer:
    """Median device time of a call, the L2 overwritten before every one."""

    def __init__(self, device, steps, warmup):
        self.flush = torch.empty(512 << 20, dtype=torch.uint8, device=device)
        self.steps, self.warmup = steps, max(warmup, 3)

    def __call__(self, fn) -> float:
        for _ in range(self.warmup):
            fn()
        ev = []
        for _ in range(self.steps):
            self.flush.fill_(1)
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            fn()
            b.record()
            ev.append((a, b))
        torch.cuda.synchronize()
        return sorted(a.elapsed_time(b) for a, b in ev)[self.steps // 2]


def _causal_flops(lens, heads, dqk, dv):
    return sum(2 * heads * (dqk + dv) * n * (n + 1) // 2 for n in lens)


def kernel_records(device, steps, warmup, peaks, which="all"):
    """[{kernel, model, case, ms, bytes | flops, frac}]: frac is of the measured copy bandwidth or bf16 burst peak."""
    time_of = _Timer(device, steps, warmup)
    g = torch.Generator(device=device).manual_seed(0)
    rnd = lambda *s: torch.randn(*s, generator=g, device=device).bfloat16()
    out = []

    def add(kernel, model, case, fn, nbytes=0, flops=0):
        if which not in ("all", kernel):
            return
        ms = time_of(fn)
        rec = {"kernel": kernel, "model": model, "case": case, "us": ms * 1e3}
        if flops:
            rec.update(bound="tensor", tflops=flops / ms / 1e9, frac=flops / ms / 1e9 / peaks["bf16_tflops"])
        else:
            rec.update(bound="hbm", gbs=nbytes / ms / 1e6, frac=nbytes / ms / 1e6 / peaks["hbm_gbs"])
        out.append(rec)

    st = torch.zeros(1, dtype=torch.int32, device=device)
    qcfg = ModelConfig(1, WIDTH, HEADS, 8, DIM, 2048, 2048)
    qwen = TPDecoder(qcfg, make_rank_weights(qcfg, 0, 1, 0, device), device=device)
    norm_w, vec_w = rnd(WIDTH), rnd(HEADS * DIM)
    decay = torch.tensor([1.0 - 2.0 ** (-2.0 - 6.0 * h / HEADS) for h in range(HEADS)], device=device)
    hd = HEADS * DIM
    for T, label in ((16384, "16384 tokens"), (256, "256 tokens")):
        x, xb, d = torch.randn(T, WIDTH, generator=g, device=device), rnd(T, WIDTH), rnd(T, WIDTH)
        add("residual_norm", "hybrid", label, lambda: hops.residual_norm(x, norm_w, 1e-6, delta=d), T * WIDTH * 12)
        add("add_rmsnorm", "qwen3", label, lambda: qwen._add_rmsnorm(xb, d, norm_w), T * WIDTH * 8)
        z = rnd(T, 4 * hd)
        add("gated_norm", "hybrid", label, lambda: hops.gated_norm(xb, z[:, 3 * hd:], vec_w, 1e-6), T * hd * 6)
        gu = rnd(T, 2 * FF)
        qwen.il = FF
        add("clamped_glu", "hybrid", label, lambda: hops.clamped_glu(gu, 7.0, GLU_ALPHA, GLU_SHIFT), T * FF * 6)
        add("silu_mul", "qwen3", label, lambda: qwen._silu_mul(gu), T * FF * 6)
        side, tok = rnd(VOCAB, LAYERS * SIDE), torch.randint(0, VOCAB, (T,), generator=g, device=device)
        zs = rnd(T, SIDE)
        add("side_gate", "hybrid", label, lambda: hops.side_gate(zs, side, tok, SIDE), T * SIDE * 6)
        del gu, z
        # latent rows, their projections and the two append kernels
        n_seq = T // 1024 if T >= 1024 else T
        per = T // n_seq
        blocks = (per + 15) // 16
        table = torch.arange(n_seq * blocks, dtype=torch.int32, device=device).view(n_seq, blocks)
        pos = torch.arange(per, dtype=torch.int32, device=device).repeat(n_seq)
        seq = torch.arange(n_seq, dtype=torch.int32, device=device).repeat_interleave(per).contiguous()
        cu = torch.arange(n_seq + 1, dtype=torch.int32, device=device) * per
        cos, sin = torch.rand(T, ROT // 2, generator=g, device=device), torch.rand(T, ROT // 2, generator=g, device=device)
        down, pool = rnd(T, Q_RANK + KV_RANK + ROT + HEADS), torch.zeros(n_seq * blocks, 16, KV_RANK + ROT, dtype=torch.bfloat16, device=device)
        wq, wkv = rnd(Q_RANK), rnd(KV_RANK)
        row = (Q_RANK + KV_RANK + ROT) * 2
        add("latent_prep", "hybrid", label, lambda: hops.latent_prep(
            down, 0, Q_RANK, Q_RANK, KV_RANK, Q_RANK + KV_RANK, ROT, wq, wkv, 1e-6, cos, sin, pool, table, seq, pos, st), T * 2 * row)
        add("latent_gather", "hybrid", label, lambda: hops.latent_gather(pool, table, cu, T, KV_RANK, ROT, st), T * (KV_RANK + ROT) * 4)
        q = rnd(T, HEADS * (DIM + ROT))
        add("rotate_heads", "hybrid", label, lambda: hops.rotate_heads_(q, cos, sin, HEADS, DIM + ROT, DIM, ROT), T * HEADS * ROT * 4)
        qkv = rnd(T, (HEADS + 16) * DIM)
        lw = {"qn": rnd(DIM), "kn": rnd(DIM)}
        kp, vp = (torch.zeros(n_seq * blocks, 8, 16, DIM, dtype=torch.float16, device=device) for _ in range(2))
        cosq, sinq = torch.rand(T, DIM, generator=g, device=device), torch.rand(T, DIM, generator=g, device=device)
        slots = torch.zeros(n_seq, dtype=torch.int32, device=device)
        cuq = cu if T > 256 else None
        add("qkv_rope_append", "qwen3", label, lambda: qwen._qkv_rope_append(qkv, lw, cosq, sinq, kp, vp, table, slots, blocks, cuq),
            T * ((HEADS + 16) * DIM * 4 + (16 * DIM * 2 if cuq is not None else 0) + DIM * 8))
        del qkv, q, down
    # prompt attention
    for lens in ((1024,) * 16, (4096,) * 4, (16384,)):
        T = sum(lens)
        label = f"{len(lens)} x {lens[0]} tokens"
        cu = torch.tensor([0] + torch.tensor(lens).cumsum(0).tolist(), dtype=torch.int32, device=device)
        n = len(lens)
        z = rnd(T, 4 * hd)
        state = torch.zeros(n, HEADS, DIM, DIM, device=device)
        rows, starts = torch.arange(n, dtype=torch.int32, device=device), torch.zeros(n, dtype=torch.int32, device=device)
        add("lightning (prompt)", "hybrid", label, lambda: hops.lightning(
            z, (0, hd, 2 * hd), HEADS, DIM, DIM, decay, state, rows, starts, st, cu_seqlens=cu, max_len=lens[0]), T * hd * 8)
        del z
        q, kv, kr, gate = rnd(T, HEADS * (DIM + ROT)), rnd(T, 2 * hd), rnd(T, ROT), rnd(T, HEADS)
        add("latent_prefill", "hybrid", label, lambda: hops.latent_prefill(q, kv, kr, gate, cu, cu, lens[0], HEADS, DIM, DIM, 0.07, st),
            flops=_causal_flops(lens, HEADS, DIM + ROT, DIM))
        q, k, v = rnd(T, HEADS, DIM).half(), rnd(T, 8, DIM).half(), rnd(T, 8, DIM).half()
        add("varlen_prefill", "qwen3", label, lambda: ops.forward_varlen_prefill_fp16(q, k, v, cu, lens[0], True, out_dtype=torch.bfloat16),
            flops=_causal_flops(lens, HEADS, DIM, DIM))
        del q, k, v, kv
    # decode steps
    for B, ctx in ((256, 2048), (64, 4096), (8, 8192)):
        label = f"{B} requests, {ctx} cached tokens"
        z = rnd(B, 4 * hd)
        state = torch.zeros(B, HEADS, DIM, DIM, device=device)
        rows, starts = torch.arange(B, dtype=torch.int32, device=device), torch.full((B,), ctx - 1, dtype=torch.int32, device=device)
        add("lightning (decode)", "hybrid", label, lambda: hops.lightning(z, (0, hd, 2 * hd), HEADS, DIM, DIM, decay, state, rows, starts, st),
            B * HEADS * DIM * DIM * 8 + B * hd * 8)
        del state
        blocks = ctx // 16
        table = torch.randperm(B * blocks, generator=torch.Generator().manual_seed(1)).to(torch.int32).view(B, blocks).to(device)
        pool = rnd(B * blocks, 16, KV_RANK + ROT)
        qa, q, gate = rnd(B, HEADS, KV_RANK), rnd(B, HEADS, DIM + ROT), rnd(B, HEADS)
        cos, sin = torch.rand(B, ROT // 2, generator=g, device=device), torch.rand(B, ROT // 2, generator=g, device=device)
        add("latent_attention (decode)", "hybrid", label, lambda: hops.latent_attention(
            qa, q, DIM, cos, sin, pool, table, rows, starts, gate, KV_RANK, ROT, 0.07, st),
            B * ctx * (KV_RANK + ROT) * 2 + B * HEADS * (2 * KV_RANK + ROT) * 2)
        del pool
        kp, vp = rnd(B * blocks, 8, 16, DIM).half(), rnd(B * blocks, 8, 16, DIM).half()
        qd, sl = rnd(B, HEADS, 1, DIM).half(), starts + 1
        add("paged_decode", "qwen3", label, lambda: ops.forward_paged_decode_gqa_fp16(qd, kp, vp, table, sl, blocks, out_dtype=torch.bfloat16),
            B * ctx * 8 * DIM * 4 + B * hd * 4)
        del kp, vp
    ops.check_async_errors(device)
    ops.check_prefill_errors(device)
    if int(st.item()):
        raise RuntimeError(f"a kernel recorded status {int(st.item())}")
    return out


def model_records(device, steps, warmup, hybrids=None):
    """Prefill and decode throughput of the hybrid decoders (name -> configuration) and of the Qwen3-style decoder through
    `GenerationRunner.generate`."""
    out = []
    shapes = ((256, 1024, 64, 16), (64, 4096, 64, 4), (8, 8192, 64, 2))
    hybrids = hybrids or {"hybrid": hybrid_config()}
    for name in (*hybrids, "qwen3"):
        if name in hybrids:
            cfg = hybrids[name]
            model = HybridDecoder(cfg, hybrid_weights(cfg, random_hybrid_tensors(cfg, 0, device), torch.bfloat16, device), device)
        else:
            cfg = qwen_config()
            model = TPDecoder(cfg, make_rank_weights(cfg, 0, 1, 0, device), device=device)
        for B, P, N, chunk in shapes:
            runner = GenerationRunner(model, max_batch=B, max_seq_len=P + N)
            prompts = torch.randint(0, VOCAB, (B, P), generator=torch.Generator().manual_seed(0)).to(device)
            times = []
            for it in range(max(warmup, 1) + steps):
                runner.generate(prompts, N, prefill_chunk=chunk)
                if it >= max(warmup, 1):
                    times.append(runner.last_timing_ms())
            pre, dec = (sorted(t[i] for t in times)[len(times) // 2] for i in (0, 1))
            out.append({"model": name, "requests": B, "prompt": P, "new_tokens": N, "prefill_tokens_per_s": B * P / pre * 1e3,
                        "decode_tokens_per_s": B * (N - 1) / dec * 1e3, "prefill_ms": pre, "decode_ms_per_step": dec / (N - 1)})
            del runner
            torch.cuda.empty_cache()
        del model
        torch.cuda.empty_cache()
    return out
