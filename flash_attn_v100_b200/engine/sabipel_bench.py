"""Throughput of the Sabipel decoder and its kernels beside the closest existing ones at equal size (`bench.py --workload sabipel`).

Random weights and token ids.  Models: eight layers of width 4096, feed-forward 12288, vocabulary 32768; Sabipel has exponential-gate
memories (32 heads of 128), state-space recurrences (64 heads of 64, 8 groups with a state of 128) and chunked attention (32 query
heads on 8, 128 columns, chunks of 2048); beside it the Berilix decoder (decayed linear attention, latent attention) and the Qwen3-style
decoder.  Kernels: at the sizes such layers give, one call per measurement with the L2 flushed before it, next to the bytes or
flops the operation needs.
"""
from __future__ import annotations

import torch

from .. import hybrid_ops as hops
from .. import mixer_ops as mops
from .. import ops
from .. import row_ops as rops
from . import hybrid_bench as hb
from .config import BigramSpec, ChunkedAttentionSpec, GeluSpec, HybridConfig, HybridLayer, Mamba2Spec, MlstmSpec, power_of_two_slopes
from .hybrid import GLU_ALPHA, GLU_SHIFT

WIDTH, HEADS, DIM, FF, VOCAB, KV_HEADS, CHUNK = hb.WIDTH, hb.HEADS, hb.DIM, hb.FF, hb.VOCAB, 8, 2048
SSD = Mamba2Spec(64, 64, 128, 8, 4, 8)
BUCKETS = 65521


def sabipel_config() -> HybridConfig:
    memory = MlstmSpec(HEADS, DIM, DIM, 15.0)
    attention = ChunkedAttentionSpec(HEADS, KV_HEADS, DIM, DIM, DIM ** -0.5, CHUNK, power_of_two_slopes(HEADS), True)
    order = (memory, SSD, SSD, attention) * (hb.LAYERS // 4)
    return HybridConfig(VOCAB, WIDTH, tuple(HybridLayer(m, GeluSpec(FF)) for m in order), 1e-6, parallel=True, embed_scale=4.0,
                        bigram=BigramSpec(BUCKETS, 8191, 131), max_positions=16384)


def kernel_records(device, steps, warmup, peaks, which="all"):
    """[{kernel, model, case, us, gbs | tflops, frac}]: frac is of the measured copy bandwidth or bf16 burst peak."""
    time_of = hb._Timer(device, steps, warmup)
    g = torch.Generator(device=device).manual_seed(0)
    rnd = lambda *s: torch.randn(*s, generator=g, device=device).bfloat16()
    f32 = lambda *s: torch.randn(*s, generator=g, device=device)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=device)
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
    hd, kd = HEADS * DIM, KV_HEADS * DIM
    inner, ch, GN = SSD.inner, SSD.channels, SSD.groups * SSD.state
    norm_w, norm_w2, vec_w = rnd(WIDTH), rnd(WIDTH), rnd(hd)
    slopes = torch.tensor(power_of_two_slopes(HEADS), device=device)
    conv_w, conv_b = rnd(SSD.conv, ch), rnd(ch)
    dt_bias, a_log, skip = f32(SSD.heads) - 3, torch.rand(SSD.heads, generator=g, device=device), f32(SSD.heads)
    bias_i, bias_f = rnd(HEADS), rnd(HEADS) + 3
    for T, label in ((16384, "16384 tokens"), (256, "256 tokens")):
        x, d = f32(T, WIDTH), rnd(T, WIDTH)
        add("residual_norm", "hybrid", label, lambda: rops.residual_norm(x, norm_w, 1e-6, delta=d), T * WIDTH * 12)
        add("residual_norm (two norms)", "sabipel", label, lambda: rops.residual_norm(x, norm_w, 1e-6, delta=d, w2=norm_w2), T * WIDTH * 14)
        embed, bigram, posn = rnd(VOCAB, WIDTH), rnd(BUCKETS + 1, WIDTH), rnd(8192, WIDTH)
        tok = torch.randint(0, VOCAB, (T,), generator=g, device=device)
        i2, i3 = tok.int() % BUCKETS, torch.arange(T, device=device).int() % 8192
        add("residual_norm (embeddings)", "sabipel", label, lambda: rops.residual_norm(x, norm_w, 1e-6, embed=embed, tokens=tok, init=True, embed_scale=4.0,
                                                                                       more=[(bigram, i2), (posn, i3)], w2=norm_w2), T * WIDTH * 14)
        del embed, bigram, posn
        o, z = rnd(T, hd), rnd(T, 4 * hd)
        wide = torch.empty(T, hd + FF, dtype=torch.bfloat16, device=device)
        add("gated_norm", "hybrid", label, lambda: rops.gated_norm(o, z[:, 3 * hd:], vec_w, 1e-6), T * hd * 6)
        add("gated_norm (per head)", "sabipel", label, lambda: rops.gated_norm(o, z[:, 3 * hd:], vec_w, 1e-6, group=DIM, out=wide[:, :hd]), T * hd * 6)
        add("gated_norm (silu first, parts)", "sabipel", label,
            lambda: rops.gated_norm(o, z[:, :hd], vec_w, 1e-6, group=inner // SSD.norm_groups, silu_first=True, out=wide[:, :hd]), T * hd * 6)
        gu = rnd(T, 2 * FF)
        add("clamped_glu", "hybrid", label, lambda: rops.clamped_glu(gu, 7.0, GLU_ALPHA, GLU_SHIFT), T * FF * 6)
        up = rnd(T, FF)
        add("gelu", "sabipel", label, lambda: rops.gelu(up, out=wide[:, hd:]), T * FF * 4)
        del gu, up, wide, z, o, x, d
        # per-token preparation of the mixers
        n_seq = T // 1024 if T >= 1024 else T
        per = T // n_seq
        prompt = per > 1
        cu = torch.arange(n_seq + 1, dtype=torch.int32, device=device) * per
        rows, starts = torch.arange(n_seq, dtype=torch.int32, device=device), torch.zeros(n_seq, dtype=torch.int32, device=device)
        seqs = mops.Sequences(rows, starts, cu if prompt else None, per)
        pos, seq = torch.arange(per, dtype=torch.int32, device=device).repeat(n_seq), rows.repeat_interleave(per).contiguous()
        tok = torch.randint(0, VOCAB, (T,), generator=g, device=device)
        last = torch.zeros(n_seq, dtype=torch.int32, device=device)
        add("bigram_rows", "sabipel", label, lambda: rops.bigram_rows(tok, starts, rows, last, BUCKETS, 8191, 131, st, cu_seqlens=seqs.cu_seqlens), T * 12)
        blocks = (per + 15) // 16
        table = torch.arange(n_seq * blocks, dtype=torch.int32, device=device).view(n_seq, blocks)
        kp, vp = (torch.zeros(n_seq * blocks, KV_HEADS, 16, DIM, dtype=torch.bfloat16, device=device) for _ in range(2))
        pages = mops.Pages(kp, vp, table, seq, pos, st)
        z, wq, wk, first = rnd(T, 2 * hd + 2 * kd), rnd(hd), rnd(kd), rnd(T, kd)
        add("kv_prep", "sabipel", label, lambda: mops.kv_prep(pages, z, (0, hd, hd + kd), HEADS, wq, wk, 1e-6, v_first=first, lam=0.5, contiguous_kv=prompt),
            T * (hd * 4 + kd * 4 + kd * 6 + (kd * 4 if prompt else 0)))
        if prompt:
            add("kv_gather", "sabipel", label, lambda: mops.kv_gather(pages, HEADS, rows, starts, cu, T), T * kd * 8)
        del z, first, kp, vp, pages
        if prompt:
            z = rnd(T, inner + ch + SSD.heads)
            ring = torch.zeros(n_seq, SSD.conv, ch, dtype=torch.bfloat16, device=device)
            add("conv_silu", "sabipel", label, lambda: mops.conv_silu(z, inner, conv_w, conv_b, ring, seqs, seq, pos, st), T * ch * 4)
            add("step_gates", "sabipel", label, lambda: mops.step_gates(z, inner + ch, dt_bias, a_log), T * SSD.heads * 10)
            z = rnd(T, 4 * hd + 2 * HEADS)
            m, nrm = torch.zeros(n_seq, 2, HEADS, device=device), torch.zeros(n_seq, 2, HEADS, DIM, device=device)
            add("max_gates", "sabipel", label, lambda: mops.max_gates(z, 4 * hd, 4 * hd + HEADS, bias_i, bias_f, 15.0, m, nrm, seqs, st), T * HEADS * 16)
            del z, ring
    # prompts
    for lens in ((1024,) * 16, (4096,) * 4, (16384,)):
        T, n = sum(lens), len(lens)
        label = f"{n} x {lens[0]} tokens"
        cu = i32([0] + torch.tensor(lens).cumsum(0).tolist())
        rows, starts = torch.arange(n, dtype=torch.int32, device=device), torch.zeros(n, dtype=torch.int32, device=device)
        seqs = mops.Sequences(rows, starts, cu, lens[0])
        z, state = rnd(T, 4 * hd), torch.zeros(n, HEADS, DIM, DIM, device=device)
        decay = torch.tensor([1.0 - 2.0 ** (-2.0 - 6.0 * h / HEADS) for h in range(HEADS)], device=device)
        add("lightning (prompt)", "hybrid", label, lambda: hops.lightning(z, (0, hd, 2 * hd), HEADS, DIM, DIM, decay, state, rows, starts, st, cu_seqlens=cu,
                                                                          max_len=lens[0]), T * hd * 8)
        la, b = -torch.rand(HEADS, T, generator=g, device=device) * 0.1, torch.rand(HEADS, T, generator=g, device=device)
        floor, n0, nrm = b + 0.5, torch.zeros(n, HEADS, DIM, device=device), torch.zeros(n, 2, HEADS, DIM, device=device)
        add("recurrence (normalised, prompt)", "sabipel", label, lambda: mops.recurrence(
            z, (0, hd, 2 * hd), HEADS, HEADS, DIM, DIM, la, b, state, seqs, st, floor=floor, n0=n0, norm=nrm, q_scale=DIM ** -0.5, norm_eps=1e-6), T * hd * 8)
        del z, state
        u, state = rnd(T, ch), torch.zeros(n, SSD.heads, SSD.state, SSD.vdim, device=device)
        la, b = -torch.rand(SSD.heads, T, generator=g, device=device) * 0.1, torch.rand(SSD.heads, T, generator=g, device=device)
        add("recurrence (state space, prompt)", "sabipel", label, lambda: mops.recurrence(
            u, (inner + GN, inner, 0), SSD.heads, SSD.groups, SSD.state, SSD.vdim, la, b, state, seqs, st, skip=skip), T * (2 * inner + 2 * GN) * 2)
        del u, state
        q, k, v, gate = rnd(T, hd), rnd(T, kd), rnd(T, kd), rnd(T, hd)
        for chunk in sorted({lens[0], min(lens[0], 1024)}):
            cc = i32(list(range(0, T + 1, chunk)))
            add("kv_prefill", "sabipel", f"{label}, chunks of {chunk}", lambda: mops.kv_prefill(q, k, v, cc, cc, chunk, HEADS, KV_HEADS, DIM ** -0.5, slopes, st, gate=gate),
                flops=hb._causal_flops((chunk,) * (T // chunk), HEADS, DIM, DIM))
        q, k, v = q.view(T, HEADS, DIM).half(), k.view(T, KV_HEADS, DIM).half(), v.view(T, KV_HEADS, DIM).half()
        add("varlen_prefill", "qwen3", label, lambda: ops.forward_varlen_prefill_fp16(q, k, v, cu, lens[0], True, out_dtype=torch.bfloat16),
            flops=hb._causal_flops(lens, HEADS, DIM, DIM))
        del q, k, v, gate
    # decode steps
    for B, ctx in ((256, 2048), (64, 4096), (8, 8192)):
        label = f"{B} requests, {ctx} cached tokens"
        rows, starts = torch.arange(B, dtype=torch.int32, device=device), torch.full((B,), ctx - 1, dtype=torch.int32, device=device)
        seqs = mops.Sequences(rows, starts)
        z, state = rnd(B, 4 * hd + 2 * HEADS), torch.zeros(B, HEADS, DIM, DIM, device=device)
        decay = torch.rand(HEADS, generator=g, device=device)
        add("lightning (decode)", "hybrid", label, lambda: hops.lightning(z, (0, hd, 2 * hd), HEADS, DIM, DIM, decay, state, rows, starts, st),
            B * HEADS * DIM * DIM * 8 + B * hd * 8)
        m, nrm = torch.zeros(B, 2, HEADS, device=device), torch.zeros(B, 2, HEADS, DIM, device=device)
        add("max_gate_step", "sabipel", label, lambda: mops.max_gate_step(z, (0, hd, 2 * hd), HEADS, DIM, DIM, 4 * hd, 4 * hd + HEADS, bias_i, bias_f, 15.0, state,
                                                                          nrm, m, seqs, st, q_scale=DIM ** -0.5, norm_eps=1e-6),
            B * HEADS * (DIM * DIM * 8 + DIM * 8) + B * hd * 8)
        del state
        z, state = rnd(B, inner + ch + SSD.heads), torch.zeros(B, SSD.heads, SSD.state, SSD.vdim, device=device)
        ring = torch.zeros(B, SSD.conv, ch, dtype=torch.bfloat16, device=device)
        add("ssd_step", "sabipel", label, lambda: mops.ssd_step(z, inner, SSD.heads, SSD.groups, SSD.state, SSD.vdim, inner + ch, dt_bias, a_log, skip, conv_w, conv_b,
                                                                ring, state, seqs, st),
            B * SSD.heads * SSD.state * SSD.vdim * 8 + B * (ch * 2 * (SSD.conv + 1) + inner * 2))
        del state, ring
        blocks = ctx // 16
        table = torch.randperm(B * blocks, generator=torch.Generator().manual_seed(1)).to(torch.int32).view(B, blocks).to(device)
        kp, vp = rnd(B * blocks, KV_HEADS, 16, DIM), rnd(B * blocks, KV_HEADS, 16, DIM)
        q, gate = rnd(B, hd), rnd(B, hd)
        pages = mops.Pages(kp, vp, table, rows, starts, st)
        add("kv_attention (decode)", "sabipel", label, lambda: mops.kv_attention(pages, q, HEADS, ctx, DIM ** -0.5, slopes=slopes, gate=gate),
            B * ctx * KV_HEADS * DIM * 4 + B * hd * 6)
        kh, vh, qd, sl = kp.half(), vp.half(), q.view(B, HEADS, 1, DIM).half(), starts + 1
        add("paged_decode", "qwen3", label, lambda: ops.forward_paged_decode_gqa_fp16(qd, kh, vh, table, sl, blocks, out_dtype=torch.bfloat16),
            B * ctx * KV_HEADS * DIM * 4 + B * hd * 4)
        del kp, vp, kh, vh, pages
    ops.check_async_errors(device)
    ops.check_prefill_errors(device)
    if int(st.item()):
        raise RuntimeError(f"a kernel recorded status {int(st.item())}")
    return out


def model_records(device, steps, warmup):
    return hb.model_records(device, steps, warmup, {"sabipel": sabipel_config(), "hybrid": hb.hybrid_config()})
