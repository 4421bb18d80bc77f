"""Run a handful of launches of one kernel on a small case, for `ncu`.

    python -m flash_attn_v100_b200.profile_runner --case paged_decode --batch 16 --iters 3

The case keeps a few hundred MB on the device (more than L2, so DRAM counters mean
something) and launches the kernel `iters` times after one warm-up call.
(The reference has the same kind of one-shot runner for its profiler: tp_profile_runner.py.)
"""
from __future__ import annotations

import argparse

import torch


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--case", default="paged_decode",
                    choices=["paged_decode", "int8_decode", "varlen_prefill", "contig_decode", "int8_kv_decode",
                             "sliding_window_decode", "latent_decode", "latent_prefill", "lightning_prefill",
                             "lightning_decode", "memory_prefill", "ssd_prefill", "memory_decode", "ssd_decode", "kv_prefill", "kv_decode"])
    ap.add_argument("--batch", type=int, default=16)
    ap.add_argument("--iters", type=int, default=3)
    ap.add_argument("--seed", type=int, default=0)
    args = ap.parse_args()
    if args.case.startswith(("latent", "lightning")):
        return hybrid(args)
    if args.case.startswith(("memory", "ssd", "kv")):
        return mixers(args)
    import flash_attn_v100 as fa
    import flash_attn_v100_b200
    from flash_attn_v100_b200.synthetic import make_paged_tables
    dev = torch.device("cuda", 0)
    g = torch.Generator(device=dev).manual_seed(args.seed)
    H_Q, H_KV, D = 32, 8, 128
    if args.case == "paged_decode":
        t = make_paged_tables(args.batch, 512, 8192, args.seed)
        kc = torch.randn(t["n_pages"], H_KV, 16, D, generator=g, device=dev, dtype=torch.float16)
        vc = torch.randn(t["n_pages"], H_KV, 16, D, generator=g, device=dev, dtype=torch.float16)
        q = torch.randn(args.batch, H_Q, 1, D, generator=g, device=dev, dtype=torch.float16)
        bt, sl = t["block_table"].to(dev), t["seq_lens"].to(dev)
        run = lambda: fa.forward_paged_decode_gqa_fp16(q, kc, vc, bt, sl, t["max_num_blocks"])
        tokens = int(t["seq_lens"].sum())
        print(f"case paged_decode: B={args.batch} tokens={tokens} kv_bytes={tokens * 4096}")
    elif args.case in ("int8_decode", "contig_decode"):
        N = 4096
        q = torch.randn(args.batch, H_Q, 1, D, generator=g, device=dev, dtype=torch.float16)
        k = torch.randn(args.batch, H_KV, N, D, generator=g, device=dev, dtype=torch.float16)
        v = torch.randn(args.batch, H_KV, N, D, generator=g, device=dev, dtype=torch.float16)
        if args.case == "int8_decode":
            qs = (q.abs().amax(-1).float().squeeze(-1) / 127).contiguous()
            ks = (k.abs().amax(-1).float() / 127).contiguous()
            run = lambda: fa.forward_decode_int8_gqa(q, k, v, qs, ks, N - 1)
        else:
            run = lambda: fa.forward_decode_gqa_fp16(q, k, v, True, N - 1)
        print(f"case {args.case}: B={args.batch} N={N} kv_bytes={args.batch * H_KV * N * D * 4}")
    elif args.case == "int8_kv_decode":
        N = 8192
        q = torch.randn(args.batch, H_Q, 1, D, generator=g, device=dev, dtype=torch.float16)
        k8 = torch.randint(-127, 128, (args.batch, H_KV, N, D), generator=g, device=dev, dtype=torch.int8)
        v8 = torch.randint(-127, 128, (args.batch, H_KV, N, D), generator=g, device=dev, dtype=torch.int8)
        ks = (torch.rand(args.batch, H_KV, N, generator=g, device=dev) * 0.01 + 0.02).half()
        vs = (torch.rand(args.batch, H_KV, N, generator=g, device=dev) * 0.01 + 0.02).half()
        run = lambda: fa.forward_decode_int8_kv_cache_gqa(q, k8, v8, ks, vs, N - 1)
        print(f"case int8_kv_decode: B={args.batch} N={N} kv_bytes={args.batch * H_KV * N * (D * 2 + 4)}")
    elif args.case == "sliding_window_decode":
        N, window, sink = 8192, 4096, 4
        q = torch.randn(args.batch, H_Q, 1, D, generator=g, device=dev, dtype=torch.float16)
        k = torch.randn(args.batch, H_KV, N, D, generator=g, device=dev, dtype=torch.float16)
        v = torch.randn(args.batch, H_KV, N, D, generator=g, device=dev, dtype=torch.float16)
        run = lambda: fa.forward_decode_sliding_window_gqa(q, k, v, True, N - 1, window, sink)
        print(f"case sliding_window_decode: B={args.batch} N={N} window={window} sink={sink} "
              f"kv_bytes={args.batch * H_KV * (window + 16) * D * 4}")
    else:
        gl = torch.Generator().manual_seed(args.seed)
        lens = torch.randint(128, 4097, (args.batch,), generator=gl).tolist()
        cu = [0]
        for n in lens:
            cu.append(cu[-1] + n)
        total = cu[-1]
        q = torch.randn(total, H_Q, D, generator=g, device=dev, dtype=torch.float16)
        k = torch.randn(total, H_KV, D, generator=g, device=dev, dtype=torch.float16)
        v = torch.randn(total, H_KV, D, generator=g, device=dev, dtype=torch.float16)
        cut = torch.tensor(cu, dtype=torch.int32, device=dev)
        run = lambda: fa.forward_varlen_prefill_fp16(q, k, v, cut, max(lens), True)
        flops = sum(4 * H_Q * D * n * (n + 1) // 2 for n in lens)
        print(f"case varlen_prefill: seqs={args.batch} total={total} flops={flops}")
    run()
    torch.cuda.synchronize()
    for _ in range(args.iters):
        run()
    torch.cuda.synchronize()
    flash_attn_v100_b200.check_async_errors()
    print("done")


def hybrid(args):
    """Kernels of the hybrid decoder: 32 heads of 128 (64 rotated), latent of 512, prompts of 1024 and 4096 cached tokens."""
    from flash_attn_v100_b200 import hybrid_ops as hops
    dev = torch.device("cuda", 0)
    g = torch.Generator(device=dev).manual_seed(args.seed)
    rnd = lambda *s: torch.randn(*s, generator=g, device=dev).bfloat16()
    st = torch.zeros(1, dtype=torch.int32, device=dev)
    H, D, R, L, B = 32, 128, 64, 512, args.batch
    rows = torch.arange(B, dtype=torch.int32, device=dev)
    if args.case == "latent_decode":
        ctx = 4096
        table = torch.randperm(B * ctx // 16).to(torch.int32).view(B, ctx // 16).to(dev)
        pool, qa, q, gate = rnd(B * ctx // 16, 16, L + R), rnd(B, H, L), rnd(B, H, D + R), rnd(B, H)
        cos, sin = (torch.rand(B, R // 2, generator=g, device=dev) for _ in range(2))
        pos = torch.full((B,), ctx - 1, dtype=torch.int32, device=dev)
        run = lambda: hops.latent_attention(qa, q, D, cos, sin, pool, table, rows, pos, gate, L, R, 0.07, st)
        print(f"case latent_decode: B={B} tokens={B * ctx} cache_bytes={B * ctx * (L + R) * 2}")
    elif args.case == "latent_prefill":
        n = 1024
        cu = torch.arange(B + 1, dtype=torch.int32, device=dev) * n
        q, kv, kr, gate = rnd(B * n, H * (D + R)), rnd(B * n, 2 * H * D), rnd(B * n, R), rnd(B * n, H)
        run = lambda: hops.latent_prefill(q, kv, kr, gate, cu, cu, n, H, D, D, 0.07, st)
        print(f"case latent_prefill: seqs={B} flops={B * 2 * H * (2 * D + R) * n * (n + 1) // 2}")
    else:
        prompt = args.case == "lightning_prefill"
        n = 1024 if prompt else 1
        cu = torch.arange(B + 1, dtype=torch.int32, device=dev) * n if prompt else None
        z, state = rnd(B * n, 3 * H * D), torch.zeros(B, H, D, D, device=dev)
        decay = 1.0 - torch.rand(H, generator=g, device=dev) * 0.2
        starts = torch.full((B,), 0 if prompt else 9, dtype=torch.int32, device=dev)
        run = lambda: hops.lightning(z, (0, H * D, 2 * H * D), H, D, D, decay, state, rows, starts, st, cu_seqlens=cu, max_len=n)
        print(f"case {args.case}: seqs={B} row_bytes={B * n * H * D * 8} state_bytes={B * H * D * D * 8}")
    for _ in range(args.iters + 1):
        run()
    torch.cuda.synchronize()
    if int(st.item()):
        raise RuntimeError(f"a kernel recorded status {int(st.item())}")
    print("done")


def mixers(args):
    """Kernels of the Sabipel decoder: 32 heads of 128 with a normaliser, 64 state-space heads of 64 in 8 groups with a state of 128, 32
    query heads on 8 of 128; prompts of 1024 and 4096 cached tokens."""
    from flash_attn_v100_b200 import mixer_ops as mops
    dev = torch.device("cuda", 0)
    g = torch.Generator(device=dev).manual_seed(args.seed)
    rnd = lambda *s: torch.randn(*s, generator=g, device=dev).bfloat16()
    f32 = lambda *s: torch.rand(*s, generator=g, device=dev)
    st = torch.zeros(1, dtype=torch.int32, device=dev)
    B, D = args.batch, 128
    rows = torch.arange(B, dtype=torch.int32, device=dev)
    kind, prompt = args.case.split("_")[0], args.case.endswith("prefill")
    n = 1024 if prompt else 1
    T, cu = B * n, torch.arange(B + 1, dtype=torch.int32, device=dev) * n
    seqs = mops.Sequences(rows, torch.full((B,), 0 if prompt else 9, dtype=torch.int32, device=dev), cu if prompt else None, n)
    if kind == "kv":
        H, G, ctx = 32, 8, 4096
        q, gate, slopes = rnd(T, H * D), rnd(T, H * D), f32(H)
        if prompt:
            k, v = rnd(T, G * D), rnd(T, G * D)
            run = lambda: mops.kv_prefill(q, k, v, cu, cu, n, H, G, D ** -0.5, slopes, st, gate=gate)
            print(f"case kv_prefill: seqs={B} flops={B * 4 * H * D * n * (n + 1) // 2}")
        else:
            table = torch.randperm(B * ctx // 16).to(torch.int32).view(B, ctx // 16).to(dev)
            pages = mops.Pages(rnd(B * ctx // 16, G, 16, D), rnd(B * ctx // 16, G, 16, D), table, rows, torch.full((B,), ctx - 1, dtype=torch.int32, device=dev), st)
            run = lambda: mops.kv_attention(pages, q, H, ctx, D ** -0.5, slopes=slopes, gate=gate)
            print(f"case kv_decode: B={B} tokens={B * ctx} cache_bytes={B * ctx * G * D * 4}")
    else:
        H, G, dv = (32, 32, D) if kind == "memory" else (64, 8, 64)
        hv, gk = H * dv, G * D
        state = torch.zeros(B, H, D, dv, device=dev)
        norm, m = torch.zeros(B, 2, H, D, device=dev), torch.zeros(B, 2, H, device=dev)
        la, b = -0.1 * f32(H, T), f32(H, T)
        extra = dict(floor=b + 0.5, n0=torch.zeros(B, H, D, device=dev), norm=norm, norm_eps=1e-6) if kind == "memory" else dict(skip=f32(H))
        if prompt:
            x = rnd(T, hv + 2 * gk)
            run = lambda: mops.recurrence(x, (hv + gk, hv, 0), H, G, D, dv, la, b, state, seqs, st, **extra)
        elif kind == "memory":
            x = rnd(T, hv + 2 * gk + 2 * H)
            run = lambda: mops.max_gate_step(x, (hv + gk, hv, 0), H, D, dv, hv + 2 * gk, hv + 2 * gk + H, rnd(H), rnd(H), 15.0, state, norm, m, seqs, st,
                                             q_scale=D ** -0.5, norm_eps=1e-6)
        else:
            x, ring, w, cb = rnd(T, hv + 2 * gk + H), rnd(B, 4, hv + 2 * gk), rnd(4, hv + 2 * gk), rnd(hv + 2 * gk)
            bias, a_log, skip = f32(H), f32(H), f32(H)
            run = lambda: mops.ssd_step(x, 0, H, G, D, dv, hv + 2 * gk, bias, a_log, skip, w, cb, ring, state, seqs, st)
        print(f"case {args.case}: seqs={B} row_bytes={T * (2 * hv + 2 * gk) * 2} state_bytes={B * H * D * dv * 8}")
    for _ in range(args.iters + 1):
        run()
    torch.cuda.synchronize()
    if int(st.item()):
        raise RuntimeError(f"a kernel recorded status {int(st.item())}")
    print("done")


if __name__ == "__main__":
    main()
