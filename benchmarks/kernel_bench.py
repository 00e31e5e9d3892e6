#!/usr/bin/env python
"""Per-kernel timings against the roofline (CUDA events, warm-up, L2 flushed between iterations).

    python benchmarks/kernel_bench.py [--what gemm,decode,prefill,small] [--json out.json]

Prints, for every kernel and shape of the Qwen3-8B serving step, the achieved TFLOP/s or GB/s, the
fraction of the measured peak (MEASURED_PEAKS.json when present) and the cuBLAS / PyTorch number for
the same shape where one exists.
"""
import argparse
import json
import math
import os
import sys

import torch

sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
from xllm_b200 import ops  # noqa: E402
from xllm_b200.ops import gemm_tcgen05  # noqa: E402


def peaks():
    p = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "MEASURED_PEAKS.json")
    if os.path.exists(p):
        d = json.load(open(p))
        return d["hbm_gbs"], d["bf16_tflops"], "measured"
    return 6650.0, 1590.0, "fallback"


_flush = None


def bench(fn, iters=10, warmup=3):
    global _flush
    if _flush is None:
        _flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")
    for _ in range(warmup):
        fn()
    ts = []
    for _ in range(iters):
        _flush.zero_()  # evict L2 (126 MB) between timed runs
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        e0.record()
        fn()
        e1.record()
        torch.cuda.synchronize()
        ts.append(e0.elapsed_time(e1))
    ts.sort()
    return ts[len(ts) // 2] * 1e-3 if ts else 0.0


def bench_pair(fa, fb, iters=10, warmup=3):
    """Two alternatives timed alternately (a, b, a, b, ...), L2 flushed before each: clock drift under the
    power cap hits both alike.  Returns the two medians in seconds."""
    bench(fa, iters=0, warmup=warmup)
    bench(fb, iters=0, warmup=warmup)
    ta, tb = [], []
    for _ in range(iters):
        for f, ts in ((fa, ta), (fb, tb)):
            _flush.zero_()
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            torch.cuda.synchronize()
            e0.record()
            f()
            e1.record()
            torch.cuda.synchronize()
            ts.append(e0.elapsed_time(e1))
    ta.sort()
    tb.sort()
    return ta[len(ta) // 2] * 1e-3, tb[len(tb) // 2] * 1e-3


def bench_rotating(fns, rounds=5, warmup=1):
    """Back-to-back launches of closures that work on different buffers (together larger than L2),
    one event pair around the whole train: per-launch time without host launch gaps."""
    for _ in range(warmup):
        for f in fns:
            f()
    ts = []
    for _ in range(rounds):
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        e0.record()
        for f in fns:
            f()
        e1.record()
        torch.cuda.synchronize()
        ts.append(e0.elapsed_time(e1) / len(fns))
    ts.sort()
    return ts[len(ts) // 2] * 1e-3


def gemm_rows(results, hbm, tf, tag):
    shapes = []
    for M in (8192, 2048, 256, 64, 8):
        shapes += [(M, 6144, 4096, "qkv"), (M, 4096, 4096, "o"), (M, 24576, 4096, "gate_up"), (M, 4096, 12288, "down")]
    shapes.append((256, 151936, 4096, "lm_head"))
    for M, N, K, name in shapes:
        wbytes = N * K * 2
        R = max(2, min(16, (300 << 20) // wbytes + 1)) if M <= 2048 and N < 100000 else 1
        xs = [torch.randn(M, K, device="cuda", dtype=torch.bfloat16) for _ in range(R)]
        ws = [torch.randn(N, K, device="cuda", dtype=torch.bfloat16) * 0.02 for _ in range(R)]
        out = torch.empty(M, N, device="cuda", dtype=torch.bfloat16)
        if R == 1:
            t_mine = bench(lambda: gemm_tcgen05.gemm_nt(xs[0], ws[0], out=out))
            t_lib = bench(lambda: torch.nn.functional.linear(xs[0], ws[0]))
        else:
            reps = max(1, 32 // R)
            t_mine = bench_rotating([(lambda i=i: gemm_tcgen05.gemm_nt(xs[i], ws[i], out=out)) for i in range(R)] * reps)
            t_lib = bench_rotating([(lambda i=i: torch.nn.functional.linear(xs[i], ws[i], )) for i in range(R)] * reps)
        flops = 2.0 * M * N * K
        bytes_ = 2.0 * (M * K + N * K + M * N)
        ideal = max(flops / (tf * 1e12), bytes_ / (hbm * 1e9))
        r = dict(kernel="gemm_bf16_tcgen05", shape=f"{name} M={M} N={N} K={K}", ms=t_mine * 1e3,
                 tflops=flops / t_mine / 1e12, gbs=bytes_ / t_mine / 1e9, frac_of_roofline=ideal / t_mine,
                 cublas_ms=t_lib * 1e3, vs_cublas=t_lib / t_mine, peaks=tag)
        results.append(r)
        print(f"gemm {r['shape']:<34} {r['ms']:8.3f} ms {r['tflops']:8.1f} TF/s  {r['gbs']:7.0f} GB/s  "
              f"roofline {r['frac_of_roofline']:.2f} ({tag})  cuBLAS {r['cublas_ms']:.3f} ms  x{r['vs_cublas']:.2f}")
        assert gemm_tcgen05.error_status() == 0
        del xs, ws


def decode_rows(results, hbm, tf, tag):
    nq, nkv, d, page = 32, 8, 128, 16
    for B, ctx in ((256, 1280), (256, 1536), (64, 4096), (16, 8192), (1, 32768)):
        nb = B * ((ctx + page - 1) // page) + 1
        kc = torch.randn(nb, nkv, page, d, device="cuda", dtype=torch.bfloat16)
        vc = torch.randn(nb, nkv, page, d, device="cuda", dtype=torch.bfloat16)
        bt = (torch.randperm(nb - 1, device="cuda")[: B * ((ctx + page - 1) // page)] + 1).view(B, -1).to(torch.int32)
        q = torch.randn(B, nq, d, device="cuda", dtype=torch.bfloat16)
        sl = torch.full((B,), ctx, device="cuda", dtype=torch.int32)
        out = torch.empty_like(q)
        splits = ops.decode_splits(B, nkv, nq // nkv)
        ws = ops.decode_workspace(B, nq, d, splits, "cuda")
        t = bench(lambda: ops.paged_decode_attention(q, kc, vc, bt, sl, 1 / math.sqrt(d), splits=splits, workspace=ws, out=out))
        bytes_ = 2.0 * B * ctx * nkv * d * 2
        r = dict(kernel="paged_decode_kernel", shape=f"B={B} ctx={ctx} nq={nq} nkv={nkv} splits={splits}", ms=t * 1e3,
                 gbs=bytes_ / t / 1e9, frac_of_roofline=bytes_ / t / 1e9 / hbm, peaks=tag)
        results.append(r)
        print(f"decode-attn {r['shape']:<44} {r['ms']:8.3f} ms {r['gbs']:7.0f} GB/s  {r['frac_of_roofline']:.2f} of {tag} HBM")


def prefill_rows(results, hbm, tf, tag):
    nq, nkv, d, page = 32, 8, 128, 16
    for B, L in ((8, 1024), (16, 1024), (2, 4096), (1, 8192)):
        nb = B * (L // page) + 1
        kc = torch.randn(nb, nkv, page, d, device="cuda", dtype=torch.bfloat16)
        vc = torch.randn(nb, nkv, page, d, device="cuda", dtype=torch.bfloat16)
        bt = (torch.arange(B * (L // page), device="cuda") + 1).view(B, -1).to(torch.int32)
        q = torch.randn(B * L, nq, d, device="cuda", dtype=torch.bfloat16)
        cu = (torch.arange(B + 1, device="cuda") * L).to(torch.int32)
        kl = torch.full((B,), L, device="cuda", dtype=torch.int32)
        out = torch.empty_like(q)
        t = bench(lambda: ops.paged_prefill_attention(q, kc, vc, bt, cu, kl, L, 1 / math.sqrt(d), out=out))
        flops = 4.0 * B * nq * d * L * L / 2
        r = dict(kernel="paged_prefill_kernel", shape=f"B={B} L={L}", ms=t * 1e3, tflops=flops / t / 1e12,
                 frac_of_roofline=flops / t / 1e12 / tf, peaks=tag)
        results.append(r)
        print(f"prefill-attn {r['shape']:<20} {r['ms']:8.3f} ms {r['tflops']:8.1f} TF/s  {r['frac_of_roofline']:.2f} of {tag} bf16 peak")


def small_rows(results, hbm, tf, tag):
    H = 4096
    for T in (256, 8192):
        x = torch.randn(T, H, device="cuda", dtype=torch.bfloat16)
        res = torch.randn(T, H, device="cuda", dtype=torch.bfloat16)
        w = torch.ones(H, device="cuda", dtype=torch.bfloat16)
        out = torch.empty_like(x)
        t = bench(lambda: ops.rmsnorm(x, w, 1e-6, residual=res, out=out))
        b = T * H * 2 * 4.0
        results.append(dict(kernel="add_rmsnorm", shape=f"T={T} H={H}", ms=t * 1e3, gbs=b / t / 1e9,
                            frac_of_roofline=b / t / 1e9 / hbm, peaks=tag))
        print(f"add_rmsnorm T={T:<6} {t*1e3:8.3f} ms {b/t/1e9:7.0f} GB/s")
        gu = torch.randn(T, 2 * 12288, device="cuda", dtype=torch.bfloat16)
        o2 = torch.empty(T, 12288, device="cuda", dtype=torch.bfloat16)
        t = bench(lambda: ops.silu_and_mul(gu, out=o2))
        b = T * 12288 * 2 * 3.0
        results.append(dict(kernel="silu_and_mul", shape=f"T={T} I=12288", ms=t * 1e3, gbs=b / t / 1e9,
                            frac_of_roofline=b / t / 1e9 / hbm, peaks=tag))
        print(f"silu_and_mul T={T:<6} {t*1e3:8.3f} ms {b/t/1e9:7.0f} GB/s")
    logits = torch.randn(256, 151936, device="cuda", dtype=torch.bfloat16)
    t = bench(lambda: ops.sample(logits))
    b = logits.numel() * 2.0
    results.append(dict(kernel="sample_greedy", shape="B=256 V=151936", ms=t * 1e3, gbs=b / t / 1e9,
                        frac_of_roofline=b / t / 1e9 / hbm, peaks=tag))
    print(f"sample greedy B=256 {t*1e3:8.3f} ms {b/t/1e9:7.0f} GB/s")


def gdn_rows(results, hbm, tf, tag):
    """Gated-delta-rule decode step (Qwen3-Next geometry: 32 value heads, 128 x 128 state per head).
    The state is read and written once: 2 x B x 32 x 64 KB per call, far larger than L2."""
    from xllm_b200.ops import gdn
    nv, dk, dv = 32, 128, 128
    for B in (64, 256):
        state = torch.randn(B, nv, dk, dv, device="cuda") * 0.1
        slots = torch.arange(B, device="cuda")
        q = torch.randn(B, nv, dk, device="cuda") * 0.1
        k = torch.nn.functional.normalize(torch.randn(B, nv, dk, device="cuda"), dim=-1)
        v = torch.randn(B, nv, dv, device="cuda")
        g = -torch.rand(B, nv, device="cuda")
        beta = torch.rand(B, nv, device="cuda")
        out = torch.empty(B, nv, dv, device="cuda")
        t = bench(lambda: gdn.decode_step(state, slots, q, k, v, g, beta, out=out))
        b = 2.0 * state.numel() * 4
        results.append(dict(kernel="gdn_decode_step", shape=f"B={B} nv={nv} dk={dk} dv={dv}", ms=t * 1e3, gbs=b / t / 1e9,
                            frac_of_roofline=b / t / 1e9 / hbm, peaks=tag))
        print(f"gdn_decode_step B={B:<4} {t*1e3:8.3f} ms {b/t/1e9:7.0f} GB/s  {b/t/1e9/hbm:5.2f} of {tag} copy bandwidth")


def mla_rows(results, hbm, tf, tag):
    """Absorbed MLA decode over the latent cache: every cached token is 1152 bytes, read once per
    group of 16 heads; 128 heads (TP 1) re-read it from L2."""
    from xllm_b200.ops import mla
    page = 16
    for N, nh, ctx in ((256, 16, 2048), (64, 16, 8192), (256, 128, 2048), (16, 128, 8192)):
        nb = N * (ctx // page) + 1
        cache = torch.randn(nb, 1, page, 576, device="cuda", dtype=torch.bfloat16)
        bt = (torch.randperm(nb - 1, device="cuda")[: N * (ctx // page)] + 1).view(N, -1).to(torch.int32)
        q = torch.randn(N, nh, 576, device="cuda", dtype=torch.bfloat16) * 0.3
        sl = torch.full((N,), ctx, device="cuda", dtype=torch.int32)
        out = torch.empty(N, nh, 512, device="cuda", dtype=torch.bfloat16)
        t = bench(lambda: mla.decode(q, cache, bt, 0.07, seq_lens=sl, out=out))
        b = N * ctx * 1152.0
        fl = 2.0 * N * nh * ctx * (576 + 512)
        results.append(dict(kernel="mla_decode_kernel", shape=f"rows={N} heads={nh} ctx={ctx}", ms=t * 1e3, gbs=b / t / 1e9,
                            tflops=fl / t / 1e12, frac_of_roofline=max(b / (hbm * 1e9), fl / (tf * 1e12)) / t, peaks=tag))
        print(f"mla_decode rows={N:<4} heads={nh:<4} ctx={ctx:<5} {t*1e3:8.3f} ms {b/t/1e9:7.0f} GB/s {fl/t/1e12:7.1f} TF/s")


def fp8_rows(results, hbm, tf, tag):
    """Block-scaled fp8 GEMM (1 x 128 activation scales, 128 x 128 weight scales) on DeepSeek-V3 shapes,
    with the bf16 tcgen05 GEMM, the per-tensor fp8 GEMM and cuBLAS bf16 on the same shapes."""
    from xllm_b200.ops import fp8
    for M, N, K, name in ((4096, 7168, 7168, "square"), (4096, 4096, 7168, "gate_up/8"), (4096, 7168, 2048, "down expert"),
                          (256, 7168, 7168, "decode"), (256, 24576, 1536, "q_b")):
        x = torch.randn(M, K, device="cuda", dtype=torch.bfloat16)
        w = torch.randn(N, K, device="cuda", dtype=torch.bfloat16) * 0.05
        a_q, a_s = fp8.quant_group128(x)
        w_q, w_s = fp8.quant_block128_ref(w)
        a_t, s_t = fp8.quant_per_token(x)
        ws1 = torch.ones(1, device="cuda")
        out = torch.empty(M, N, device="cuda", dtype=torch.bfloat16)
        t_blk = bench(lambda: fp8.block_scaled_mm(a_q, a_s, w_q, w_s, out=out))
        t_pt = bench(lambda: fp8.scaled_mm(a_t, w_q, s_t, ws1, out=out))
        t_bf = bench(lambda: gemm_tcgen05.gemm_nt(x, w, out=out))
        t_lib = bench(lambda: torch.nn.functional.linear(x, w))
        fl = 2.0 * M * N * K
        results.append(dict(kernel="gemm_fp8_block_kernel", shape=f"{name} M={M} N={N} K={K}", ms=t_blk * 1e3,
                            tflops=fl / t_blk / 1e12, per_tensor_fp8_ms=t_pt * 1e3, bf16_ms=t_bf * 1e3, cublas_bf16_ms=t_lib * 1e3,
                            peaks=tag))
        print(f"fp8 block {name:<12} M={M:<5} N={N:<6} K={K:<5} {t_blk*1e3:7.3f} ms {fl/t_blk/1e12:7.1f} TF/s | per-tensor fp8 "
              f"{t_pt*1e3:7.3f} ms | bf16 tcgen05 {t_bf*1e3:7.3f} ms | cuBLAS bf16 {t_lib*1e3:7.3f} ms")


def moe_rows(results, hbm, tf, tag):
    """The whole MoE layer (route, permute, grouped GEMM gate|up, SiLU-mul, grouped GEMM down, finalize) on
    Qwen3-30B-A3B and DeepSeek-V3-like expert shapes: the three-launch expert form against the grouped GEMM
    with the gated activation in its epilogue (interleaved expert weights)."""
    from xllm_b200.ops import moe
    for T, E, K, H, I, name in ((8192, 128, 8, 2048, 768, "qwen3-30b-a3b prefill"), (256, 128, 8, 2048, 768, "qwen3-30b-a3b decode"),
                                (8192, 32, 8, 7168, 2048, "deepseek-v3 experts of one EP-8 rank")):
        x = torch.randn(T, H, device="cuda", dtype=torch.bfloat16)
        logits = torch.randn(T, E, device="cuda")
        w1 = torch.randn(E, 2 * I, H, device="cuda", dtype=torch.bfloat16) * 0.05
        w2 = torch.randn(E, H, I, device="cuda", dtype=torch.bfloat16) * 0.05
        ws = moe.MoeWorkspace(T, K, E, E, H, I, "cuda")
        out = torch.empty_like(x)
        t_plain, t_fused = bench_pair(lambda: moe.fused_moe(x, logits, w1, w2, K, ws=ws, out=out),
                                      lambda: moe.fused_moe(x, logits, w1, w2, K, ws=ws, out=out, interleaved=True))
        fl = 2.0 * T * K * 3 * I * H
        results.append(dict(kernel="fused_moe", shape=f"{name} T={T} E={E} top{K} H={H} I={I}", ms=t_fused * 1e3,
                            tflops=fl / t_fused / 1e12, three_launch_ms=t_plain * 1e3, peaks=tag))
        print(f"moe {name:<38} T={T:<5} {t_fused*1e3:7.3f} ms {fl/t_fused/1e12:7.1f} TF/s ({fl/t_fused/1e12/tf*100:5.1f}% of {tag} cuBLAS bf16)"
              f" | GEMM, activation kernel, GEMM: {t_plain*1e3:7.3f} ms")


def bench_queued(fn, iters=10, warmup=3):
    """Like `bench`, but the timed launches are queued while the L2 flush still runs: device time without the host's
    launch latency, for kernels of a few microseconds."""
    bench(fn, iters=0, warmup=warmup)
    ts = []
    for _ in range(iters):
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        for _ in range(4):
            _flush.zero_()
        e0.record()
        fn()
        e1.record()
        torch.cuda.synchronize()
        ts.append(e0.elapsed_time(e1))
    ts.sort()
    return ts[len(ts) // 2] * 1e-3


def hybrid_rows(results, hbm, tf, tag):
    """The kernels of the hybrid decoders (Femirax) beside the like kernels of Qwen3-Next: decayed linear attention
    against the gated delta rule (decode, prompts), the fp32 residual update against add + RMSNorm, rotation + unit norm +
    cache write against norm + rotation + cache write, the side input's products and activation.  32 heads of 128, width
    4096."""
    from xllm_b200.ops import gdn
    from xllm_b200.ops.linear_attn import LinearAttention
    from xllm_b200.ops.residual import gelu_mul_rows, residual_update
    dev, bf, H, d, W = "cuda", torch.bfloat16, 32, 128, 4096
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    rows = lambda t, n: torch.randn(t, n, device=dev, dtype=bf)
    cs = torch.randn(8192, d, device=dev)

    def report(name, shape, t, nbytes, flops=0.0):
        ideal = max(nbytes / (hbm * 1e9), flops / (tf * 1e12))
        results.append(dict(kernel=name, shape=shape, ms=t * 1e3, gbs=nbytes / t / 1e9, tflops=flops / t / 1e12,
                            frac_of_roofline=ideal / t, peaks=tag))
        print(f"{name:<34} {shape:<26} {t*1e6:9.1f} us {nbytes/t/1e9:7.0f} GB/s {flops/t/1e12:7.1f} TF/s  {ideal/t:6.3f} of {tag}",
              flush=True)

    def op_of(kind):
        op = LinearAttention(H, d, d, k_scale=d ** -0.5)
        if kind == "retention":
            op.log_decay, op.cos_sin, op.rot = torch.full((H,), -0.01, device=dev), cs, d
        else:
            op.a2, op.a2_bias = rows(H * d, 16) * 0.1, torch.full((H * d,), 4.0, device=dev, dtype=bf)
            op.inv_tau, op.norm_w = 1 / 16, torch.ones(d, device=dev, dtype=bf)
        return op

    cut = lambda r: [r[:, i * H * d:(i + 1) * H * d] for i in range(4)] + [r[:, 4 * H * d:4 * H * d + 16]]
    for B in (16, 64, 256):
        st = torch.zeros(B + 1, H, d, d, device=dev)
        c, sl = cut(rows(B, 4 * H * d + 16)), i32(list(range(B)))
        kl, pos, out = torch.full_like(sl, 100), torch.full((B,), 99, device=dev), torch.empty(B, H * d, device=dev, dtype=bf)
        nb = 2 * B * H * d * d * 4 + B * H * d * 10
        for kind in ("retention", "channel decay"):
            op = op_of(kind)
            report(f"linattn_decode, {kind}", f"B={B}", bench_queued(
                lambda: op.decode(st, sl, kl, pos, c[0], c[1], c[2], g=c[3], r=c[4], out=out)), nb)
        q, k, v = (torch.randn(B, H, d, device=dev) for _ in range(3))
        g, be, o, s64 = -torch.rand(B, H, device=dev), torch.rand(B, H, device=dev), torch.empty(B, H, d, device=dev), sl.long()
        report("gdn_decode", f"B={B}", bench_queued(lambda: gdn.decode_step(st, s64, q, k, v, g, be, out=o)),
               2 * B * H * d * d * 4 + B * H * d * 16)
        del st
    for S, L in ((1, 2048), (1, 8192), (4, 2048)):
        T = S * L
        st = torch.zeros(S + 1, H, d, d, device=dev)
        c, sl = cut(rows(T, 4 * H * d + 16)), i32(list(range(S)))
        cu, kl, pos = i32([i * L for i in range(S + 1)]), i32([L] * S), torch.arange(L, device=dev).repeat(S)
        out = torch.empty(T, H * d, device=dev, dtype=bf)
        fl = 4.0 * T * H * d * d
        for kind in ("retention", "channel decay"):
            op = op_of(kind)
            report(f"linattn prompts, {kind}", f"{S} x {L}", bench_queued(
                lambda: op.prefill(st, sl, cu, kl, pos, c[0], c[1], c[2], g=c[3], r=c[4], out=out, max_q_len=L), iters=5),
                T * H * d * 10 + S * H * d * d * 8, fl)
        q, k, v = (torch.randn(L, H, d, device=dev) for _ in range(3))
        g, be, o = -torch.rand(L, H, device=dev), torch.rand(L, H, device=dev), torch.empty(L, H, d, device=dev)
        report("gdn_prefill", f"{S} x {L}", bench_queued(
            lambda: [gdn.prefill(st, s, True, q, k, v, g, be, out=o) for s in range(S)], iters=3), T * H * d * 16, 2 * fl)
    nq, nkv = 32, 8
    for T in (64, 8192):
        x, y, y2, w, res = torch.randn(T, W, device=dev), rows(T, W), rows(T, W), torch.ones(W, device=dev, dtype=bf), rows(T, W)
        report("residual_update", f"T={T}", bench_queued(lambda: residual_update(x, y, w_out=w)), T * W * 12)
        report("residual_update, normed branch", f"T={T}", bench_queued(lambda: residual_update(x, y, w=w, w_out=w)), T * W * 12)
        report("residual_update, two branches", f"T={T}", bench_queued(
            lambda: residual_update(x, y, w=w, y2=y2, w2=w, coef=0.5, w_out=w)), T * W * 14)
        report("rmsnorm (bf16 residual)", f"T={T}", bench_queued(lambda: ops.rmsnorm(y, w, 1e-6, residual=res)), T * W * 8)
        qkv, pos = rows(T, (nq + 2 * nkv) * d), torch.arange(T, device=dev) % 8192
        kc = torch.zeros(T // 16 + 2, nkv, 16, d, device=dev, dtype=bf)
        vc, sl, wn = torch.zeros_like(kc), torch.arange(16, 16 + T, dtype=torch.int32, device=dev), torch.ones(d, device=dev, dtype=bf)
        q, k = qkv[:, :nq * d], qkv[:, nq * d:(nq + nkv) * d]
        report("rope_norm_kv", f"T={T}", bench_queued(lambda: ops.rope_norm_kv_write(
            q, k, k, nq, nkv, d, pos, cs, d, sl, kc, vc, interleaved=True)), T * d * 2 * (2 * nq + 3 * nkv))
        report("rope_kv", f"T={T}", bench_queued(lambda: ops.rope_kv_write(
            qkv, nq, nkv, d, pos, cs, d, slots=sl, k_cache=kc, v_cache=vc, q_norm_w=wn, k_norm_w=wn)), T * d * 4 * (nq + 2 * nkv))
        for dim in (16, 64, 256):
            gate, table, ids = rows(T, dim), rows(32000, dim * 4), torch.randint(0, 32000, (T,), device=dev)
            xb, wg, wp = rows(T, W), rows(dim, W), rows(W, dim)
            nb, fl = 2.0 * (T * W + dim * W + T * dim), 2.0 * T * W * dim
            report("gelu_mul_rows", f"T={T} dim={dim}", bench_queued(lambda: gelu_mul_rows(gate, table, ids, dim, dim)), T * dim * 6)
            report("side gate GEMM", f"T={T} dim={dim}", bench_queued(lambda: ops.linear(xb, wg)), nb, fl)
            report("side gate, cuBLAS", f"T={T} dim={dim}", bench_queued(lambda: torch.nn.functional.linear(xb, wg)), nb, fl)
            report("side proj GEMM", f"T={T} dim={dim}", bench_queued(lambda: ops.linear(gate, wp)), nb, fl)
            report("side proj, cuBLAS", f"T={T} dim={dim}", bench_queued(lambda: torch.nn.functional.linear(gate, wp)), nb, fl)


def recurrent_rows(results, hbm, tf, tag):
    """The kernels of Sodedra beside their likes: gated delta rule with channel decays and matrix memory against the gated
    delta rule of Qwen3-Next and the decayed linear attention of Femirax (decode, prompts), windowed attention against the
    same kernels without a window, head norms and gates, fp32 projections, expert layers.  32 heads of 128, width 4096."""
    from xllm_b200.ops import gdn, moe
    from xllm_b200.ops.delta_rule import ChannelDelta
    from xllm_b200.ops.head_norm import head_gate, head_norm_gate
    from xllm_b200.ops.linear_attn import LinearAttention
    from xllm_b200.ops.mlstm import MatrixMemory
    from xllm_b200.ops.residual import residual_update
    dev, bf, H, d, W, R = "cuda", torch.bfloat16, 32, 128, 4096, 128
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    rows = lambda t, n: torch.randn(t, n, device=dev, dtype=bf)

    def report(name, shape, t, nbytes, flops=0.0):
        ideal = max(nbytes / (hbm * 1e9), flops / (tf * 1e12))
        results.append(dict(kernel=name, shape=shape, ms=t * 1e3, gbs=nbytes / t / 1e9, tflops=flops / t / 1e12,
                            frac_of_roofline=ideal / t, peaks=tag))
        print(f"{name:<34} {shape:<26} {t*1e6:9.1f} us {nbytes/t/1e9:7.0f} GB/s {flops/t/1e12:7.1f} TF/s  {ideal/t:6.3f} of {tag}",
              flush=True)

    delta = ChannelDelta(H, H, d, d, 4, q_scale=d ** -0.5, conv_w=rows(4, 3 * H * d) * 0.5, a2=rows(H * d, R) * 0.05,
                         dt_bias=torch.full((H * d,), -4.0, device=dev, dtype=bf), a_log=torch.zeros(H, device=dev, dtype=bf),
                         norm_w=torch.ones(d, device=dev, dtype=bf))
    mem = MatrixMemory(H, d, d, 15.0, q_scale=d ** -0.5, norm_w=torch.ones(H * d, device=dev, dtype=bf))
    lin = LinearAttention(H, d, d, k_scale=d ** -0.5)
    lin.log_decay = torch.full((H,), -0.01, device=dev)
    cut = lambda r: [r[:, i * H * d:(i + 1) * H * d] for i in range(4)] + [r[:, 4 * H * d:4 * H * d + R]]
    state = lambda n: torch.zeros(n, H, d, d, device=dev)
    for B in (16, 64, 256):
        st, ring = state(B + 1), torch.zeros(B + 1, 4, 3 * H * d, device=dev, dtype=bf)
        mst = {"S": st, "n": torch.zeros(B + 1, H, d, device=dev), "m": torch.zeros(B + 1, H, device=dev)}
        c, sl, z = cut(rows(B, 4 * H * d + R)), i32(list(range(B))), torch.randn(B, 2 * H, device=dev)
        kl, out, cu = torch.full_like(sl, 100), torch.empty(B, H * d, device=dev, dtype=bf), i32(list(range(B + 1)))
        pos = torch.full((B,), 99, device=dev)
        nb = 2 * B * H * d * d * 4 + B * H * d * 10
        report("delta_decode", f"B={B}", bench_queued(lambda: delta.decode(st, ring, sl, cu, kl, *c[:3], c[4], z, c[3], out)),
               nb + B * 3 * H * d * 2 * 4)
        report("mlstm_decode", f"B={B}", bench_queued(lambda: mem.decode(mst, sl, cu, kl, *c[:3], z[:, :H], z[:, H:], c[3], out)), nb)
        report("linattn_decode", f"B={B}", bench_queued(lambda: lin.decode(st, sl, kl, pos, *c[:3], g=c[3], out=out)), nb)
        q, k, v = (torch.randn(B, H, d, device=dev) for _ in range(3))
        g, be, o, s64 = -torch.rand(B, H, device=dev), torch.rand(B, H, device=dev), torch.empty(B, H, d, device=dev), sl.long()
        report("gdn_decode", f"B={B}", bench_queued(lambda: gdn.decode_step(st, s64, q, k, v, g, be, out=o)),
               2 * B * H * d * d * 4 + B * H * d * 16)
        del st, mst
    for S, L in ((1, 2048), (1, 8192), (4, 2048)):
        T = S * L
        st, ring = state(S + 1), torch.zeros(S + 1, 4, 3 * H * d, device=dev, dtype=bf)
        mst = {"S": st, "n": torch.zeros(S + 1, H, d, device=dev), "m": torch.zeros(S + 1, H, device=dev)}
        c, sl, z = cut(rows(T, 4 * H * d + R)), i32(list(range(S))), torch.randn(T, 2 * H, device=dev)
        cu, kl, pos = i32([i * L for i in range(S + 1)]), i32([L] * S), torch.arange(L, device=dev).repeat(S)
        out = torch.empty(T, H * d, device=dev, dtype=bf)
        fl, nb = 4.0 * T * H * d * d, T * H * d * 10 + S * H * d * d * 8
        report("delta rule prompts", f"{S} x {L}", bench_queued(
            lambda: delta.prefill(st, ring, sl, cu, kl, *c[:3], c[4], z, c[3], out), iters=5), nb, 2 * fl)
        report("mlstm prompts", f"{S} x {L}", bench_queued(
            lambda: mem.prefill(mst, sl, cu, kl, *c[:3], z[:, :H], z[:, H:], c[3], out), iters=5), nb, fl)
        report("linattn prompts", f"{S} x {L}", bench_queued(
            lambda: lin.prefill(st, sl, cu, kl, pos, *c[:3], g=c[3], out=out, max_q_len=L), iters=5), nb, fl)
        q, k, v = (torch.randn(L, H, d, device=dev) for _ in range(3))
        g, be, o = -torch.rand(L, H, device=dev), torch.rand(L, H, device=dev), torch.empty(L, H, d, device=dev)
        report("gdn_prefill", f"{S} x {L}", bench_queued(
            lambda: [gdn.prefill(st, s, True, q, k, v, g, be, out=o) for s in range(S)], iters=3), T * H * d * 16, 2 * fl)
    nq, nkv = 32, 8
    for S, L, win in ((4, 2048, 0), (4, 2048, 1024), (1, 8192, 0), (1, 8192, 1024)):
        T = S * L
        kc, vc = (rows(T // 16 * nkv * 16, d).view(T // 16, nkv, 16, d) for _ in range(2))
        bt = torch.arange(T // 16, device=dev, dtype=torch.int32).view(S, L // 16)
        cu, kl, q = i32([i * L for i in range(S + 1)]), i32([L] * S), rows(T, nq * d).view(T, nq, d)
        pairs = sum(min(i + 1, win or L) for i in range(L)) * S
        report("attention prompts", f"{S} x {L} window {win}", bench_queued(lambda: ops.paged_prefill_attention(
            q, kc, vc, bt, cu, kl, L, d ** -0.5, window=win), iters=5), T * d * 2 * (2 * nq + 2 * nkv), 4.0 * pairs * nq * d)
    for B, ctx, win in ((64, 4096, 0), (64, 4096, 1024), (256, 1024, 0), (256, 4096, 1024)):
        kc, vc = (rows(B * ctx // 16 * nkv * 16, d).view(B * ctx // 16, nkv, 16, d) for _ in range(2))
        bt = torch.arange(B * ctx // 16, device=dev, dtype=torch.int32).view(B, ctx // 16)
        kl, q = i32([ctx] * B), rows(B, nq * d).view(B, nq, d)
        splits = min(ops.decode_splits(B, nkv, nq // nkv), max(1, win // 256)) if win else None
        report("attention decode", f"B={B} ctx {ctx} window {win}", bench_queued(lambda: ops.paged_decode_attention(
            q, kc, vc, bt, kl, d ** -0.5, window=win, splits=splits)), 4.0 * B * min(ctx, win or ctx) * nkv * d)
        del kc, vc
    for T in (64, 8192):
        x, y, y2, w = torch.randn(T, W, device=dev), rows(T, W), rows(T, W), torch.ones(W, device=dev, dtype=bf)
        report("residual_update, two branches", f"T={T}", bench_queued(
            lambda: residual_update(x, y, y2=y2, w_out=w, w_out_offset=1.0)), T * W * 14)
        res = rows(T, W)
        report("rmsnorm (bf16 residual)", f"T={T}", bench_queued(lambda: ops.rmsnorm(y, w, 1e-6, residual=res)), T * W * 8)
        o, out, g, div = torch.randn(T, H, d, device=dev), torch.empty(T, H * d, device=dev, dtype=bf), rows(T, H * d), torch.ones(T, H, device=dev)
        wn = torch.ones(d, device=dev, dtype=bf)
        report("head_norm_gate", f"T={T}", bench_queued(lambda: head_norm_gate(o, out, div=div, g=g, w=wn, act="sigmoid")), T * H * d * 8)
        a = rows(T, H * d).view(T, H, d)
        report("head_gate", f"T={T}", bench_queued(lambda: head_gate(a, g, d)), T * H * d * 6)
        report("gate by tensor ops (Qwen3-Next)", f"T={T}", bench_queued(
            lambda: a.view(T, H * d) * torch.sigmoid(g.float()).to(bf)), T * H * d * 6)
        for N in (32, 64, 128):
            xb, wr = rows(T, W), rows(N, W)
            nb, fl = 2.0 * (T * W + N * W) + 4 * T * N, 2.0 * T * W * N
            report("fp32 projection", f"T={T} N={N}", bench_queued(lambda: ops.linear_f32(xb, wr)), nb, fl)
            report("router GEMM (bf16 result)", f"T={T} N={N}", bench_queued(lambda: ops.linear(xb, wr)), nb, fl)
        qkv, pos = rows(T, (nq + 2 * nkv) * d), torch.arange(T, device=dev) % 8192
        cs = torch.randn(8192, d, device=dev)
        kc = torch.zeros(T // 16 + 2, nkv, 16, d, device=dev, dtype=bf)
        vc, sl = torch.zeros_like(kc), torch.arange(16, 16 + T, dtype=torch.int32, device=dev)
        q, k, v = qkv[:, :nq * d], qkv[:, nq * d:(nq + nkv) * d], qkv[:, (nq + nkv) * d:]
        nb = T * d * 4 * (nq + 2 * nkv)
        report("rotation + cache write", f"T={T}", bench_queued(lambda: ops.rope_norm_kv_write(
            q, k, v, nq, nkv, d, pos, cs, d, sl, kc, vc, unit_norm=False)), nb)
        report("rope_kv", f"T={T}", bench_queued(lambda: ops.rope_kv_write(
            qkv, nq, nkv, d, pos, cs, d, slots=sl, k_cache=kc, v_cache=vc, q_norm_w=wn, k_norm_w=wn)), nb)
        E, K, I = 32, 4, W // 2
        w1, w2, xb = rows(E * 2 * I, W).view(E, 2 * I, W), rows(E * W, I).view(E, W, I), rows(T, W)
        lg, bias = torch.randn(T, E, device=dev), torch.randn(E, device=dev) * 0.1
        ws = moe.shared_workspace(T, K, E, E, W, I, torch.device(dev), bf, W)
        nb = 2.0 * (min(E, T * K) * 3 * I * W + 2 * T * W)
        report("experts (groups by best score)", f"T={T} E={E} top{K}", bench_queued(lambda: moe.fused_moe(
            xb, lg, w1, w2, K, bias=bias, n_group=8, topk_group=4, ws=ws, interleaved=True, group_score="max")), nb, 6.0 * T * K * W * I)
        report("experts (plain softmax)", f"T={T} E={E} top{K}", bench_queued(lambda: moe.fused_moe(
            xb, lg, w1, w2, K, ws=ws, interleaved=True)), nb, 6.0 * T * K * W * I)


def latent_rows(results, hbm, tf, tag):
    """The kernels of Lukinex beside their likes: windows with kept tokens and soft caps against plain windows, convolution and
    norm ahead of rotation and cache write against the write alone, lightning attention against retention, latent attention
    against MLA with a rotary part, clamped experts against SiLU, residual updates.  32 heads of 128, width 4096."""
    from xllm_b200.ops import mla, moe
    from xllm_b200.ops.glu import ClampedGLU
    from xllm_b200.ops.head_norm import head_norm_gate
    from xllm_b200.ops.linear_attn import LinearAttention
    from xllm_b200.ops.residual import residual_update
    dev, bf, H, d, W = "cuda", torch.bfloat16, 32, 128, 4096
    nq, nkv, R = 32, 8, 512
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    rows = lambda t, n: torch.randn(t, n, device=dev, dtype=bf)

    def report(name, shape, t, nbytes, flops=0.0):
        ideal = max(nbytes / (hbm * 1e9), flops / (tf * 1e12))
        results.append(dict(kernel=name, shape=shape, ms=t * 1e3, gbs=nbytes / t / 1e9, tflops=flops / t / 1e12,
                            frac_of_roofline=ideal / t, peaks=tag))
        print(f"{name:<38} {shape:<26} {t*1e6:9.1f} us {nbytes/t/1e9:7.0f} GB/s {flops/t/1e12:7.1f} TF/s  {ideal/t:6.3f} of {tag}",
              flush=True)

    kinds = (("plain", {}), ("kept", dict(keep=16)), ("capped", dict(softcap=30.0)), ("kept, capped", dict(keep=16, softcap=30.0)))
    for S, L, win in ((4, 2048, 1024), (1, 8192, 1024)):
        T = S * L
        kc, vc = (rows(T // 16 * nkv * 16, d).view(T // 16, nkv, 16, d) for _ in range(2))
        bt = torch.arange(T // 16, device=dev, dtype=torch.int32).view(S, L // 16)
        cu, kl, q = i32([i * L for i in range(S + 1)]), i32([L] * S), rows(T, nq * d).view(T, nq, d)
        for name, kw in kinds:
            keep = kw.get("keep", 0)
            pairs = sum(min(i + 1, win) + min(keep, max(0, i + 1 - win)) for i in range(L)) * S
            report(f"window prompts, {name}", f"{S} x {L} window {win}", bench_queued(lambda: ops.paged_prefill_attention(
                q, kc, vc, bt, cu, kl, L, d ** -0.5, window=win, **kw), iters=5), T * d * 2 * (2 * nq + 2 * nkv), 4.0 * pairs * nq * d)
    for B, ctx, win in ((64, 4096, 1024), (256, 4096, 1024)):
        kc, vc = (rows(B * ctx // 16 * nkv * 16, d).view(B * ctx // 16, nkv, 16, d) for _ in range(2))
        bt = torch.arange(B * ctx // 16, device=dev, dtype=torch.int32).view(B, ctx // 16)
        kl, q = i32([ctx] * B), rows(B, nq * d).view(B, nq, d)
        splits = min(ops.decode_splits(B, nkv, nq // nkv), max(1, win // 256))
        for name, kw in kinds:
            report(f"window decode, {name}", f"B={B} window {win}", bench_queued(lambda: ops.paged_decode_attention(
                q, kc, vc, bt, kl, d ** -0.5, window=win, splits=splits, **kw)), 4.0 * B * (win + kw.get("keep", 0)) * nkv * d)
        del kc, vc
    for B, ctx in ((16, 8192), (64, 4096), (256, 2048)):
        bt = (torch.randperm(B * (ctx // 16), device=dev) + 1).view(B, -1).to(torch.int32)
        sl, pos = i32([ctx] * B), torch.full((B,), ctx - 1, device=dev)
        for width, name in ((R, "latent decode"), (R + 64, "mla decode (rotary part)")):
            cache = rows((B * (ctx // 16) + 1) * 16, width).view(-1, 1, 16, width)
            q, out = rows(B, H * width).view(B, H, width) * 0.3, torch.empty(B, H, R, device=dev, dtype=bf)
            fn = (lambda: mla.latent_decode(q, cache, bt, 0.09, seq_lens=sl, out=out)) if width == R else \
                (lambda: mla.decode(q, cache, bt, 0.09, seq_lens=sl, out=out))
            report(name, f"B={B} ctx {ctx}", bench_queued(fn), 2.0 * B * ctx * width, 2.0 * B * H * ctx * (width + R))
            del cache
        uk, q = rows(H * d, R).view(H, d, R), rows(B, H * d).view(B, H, d)
        qa = torch.empty(B, H, R, device=dev, dtype=bf)
        report("query into latents (cuBLAS)", f"B={B}", bench_queued(lambda: torch.bmm(q.transpose(0, 1), uk, out=qa.transpose(0, 1))),
               2.0 * (H * d * R + B * H * (d + R)), 2.0 * B * H * d * R)
    for S, L in ((4, 512), (4, 2048), (1, 8192)):
        T, bt = S * L, torch.arange(1, S * L // 16 + 1, device=dev, dtype=torch.int32).view(S, L // 16)
        cu, kl, pos = i32([i * L for i in range(S + 1)]), i32([L] * S), torch.arange(L, device=dev).repeat(S)
        seq = torch.arange(S, device=dev, dtype=torch.int32).repeat_interleave(L)
        pairs = S * L * (L + 1) / 2
        cache, ukv, q = rows((T // 16 + 1) * 16, R).view(-1, 1, 16, R), rows(2 * H * d, R), rows(T, H * d).view(T, H, d)
        out, pages = torch.empty(T, H, d, device=dev, dtype=bf), torch.arange(T // 16, device=dev, dtype=torch.int32).view(S, -1)

        def expanded():
            kv = ops.linear(mla.latent_gather(cache, bt, kl, L), ukv)
            ops.ragged_prefill_attention(q, kv[:, :H * d], kv[:, H * d:], pages, 16, cu, kl, L, 0.09, out)

        fl = 4.0 * pairs * H * d
        report("latent prompts, expanded", f"{S} x {L}", bench_queued(expanded, iters=5), 0.0, fl + 4.0 * T * R * H * d)
        if T <= 2048:
            qa, oa = rows(T, H * R).view(T, H, R), torch.empty(T, H, R, device=dev, dtype=bf)
            report("latent prompts, row by row", f"{S} x {L}", bench_queued(lambda: mla.latent_decode(
                qa, cache, bt, 0.09, positions=pos, bt_rows=seq, out=oa), iters=5), 0.0, 4.0 * pairs * H * R)
            c2, q2 = rows((T // 16 + 1) * 16, R + 64).view(-1, 1, 16, R + 64), rows(T, H * (R + 64)).view(T, H, R + 64)
            report("mla prompts, row by row", f"{S} x {L}", bench_queued(lambda: mla.decode(
                q2, c2, bt, 0.09, positions=pos, bt_rows=seq, out=oa), iters=5), 0.0, 2.0 * pairs * H * (2 * R + 64))
        del cache
    decay = torch.linspace(0.9, 0.9995, H, device=dev).log()
    light = LinearAttention(H, d, d, in_silu=True, rows=True, log_decay=decay, norm_w=torch.ones(H * d, device=dev, dtype=bf))
    ret = LinearAttention(H, d, d, k_scale=d ** -0.5, log_decay=decay)
    cut = lambda r: [r[:, i * H * d:(i + 1) * H * d] for i in range(4)]
    for B in (64, 256):
        st, c, sl = torch.zeros(B + 1, H, d, d, device=dev), cut(rows(B, 4 * H * d)), i32(list(range(B)))
        kl, pos, out = i32([100] * B), torch.full((B,), 99, device=dev), torch.empty(B, H * d, device=dev, dtype=bf)
        for name, op in (("lightning decode", light), ("retention decode", ret)):
            report(name, f"B={B}", bench_queued(lambda: op.decode(st, sl, kl, pos, *c[:3], g=c[3], out=out)),
                   2 * B * H * d * d * 4 + B * H * d * 10)
        del st
    for S, L in ((4, 2048), (1, 8192)):
        T, st = S * L, torch.zeros(S + 1, H, d, d, device=dev)
        c, sl, cu, kl = cut(rows(T, 4 * H * d)), i32(list(range(S))), i32([i * L for i in range(S + 1)]), i32([L] * S)
        pos, out = torch.arange(L, device=dev).repeat(S), torch.empty(T, H * d, device=dev, dtype=bf)
        for name, op in (("lightning prompts", light), ("retention prompts", ret)):
            report(name, f"{S} x {L}", bench_queued(lambda: op.prefill(st, sl, cu, kl, pos, *c[:3], g=c[3], out=out, max_q_len=L), iters=5),
                   T * H * d * 10 + S * H * d * d * 8, 4.0 * T * H * d * d)
    C = (nq + 2 * nkv) * d
    for T in (64, 8192):
        qkv, cs, wn = rows(T, C), torch.randn(8192, d, device=dev), torch.ones(d, device=dev, dtype=bf)
        kc = torch.zeros(T // 16 + 2, nkv, 16, d, device=dev, dtype=bf)
        vc, sl = torch.zeros_like(kc), torch.arange(16, 16 + T, dtype=torch.int32, device=dev)
        q, k, v = qkv[:, :nq * d], qkv[:, nq * d:(nq + nkv) * d], qkv[:, (nq + nkv) * d:]
        n = T if T == 64 else 4                                       # decode rows, or four prompts
        ring, cw, L = torch.zeros(n + 1, 4, C, device=dev, dtype=bf), rows(4, C), T // n
        conv = (cw, ring, i32(list(range(n))), i32([i * L for i in range(n + 1)]), i32([L if n == 4 else 100] * n))
        pos, nb = torch.arange(T, device=dev) % 2048, T * d * 4 * (nq + 2 * nkv)
        write = lambda **kw: ops.rope_norm_kv_write(q, k, v, nq, nkv, d, pos, cs, d, sl, kc, vc, unit_norm=False, **kw)
        report("rotation + cache write", f"T={T}", bench_queued(lambda: write()), nb)
        report("norm + rotation + cache write", f"T={T}", bench_queued(lambda: write(q_w=wn, k_w=wn)), nb)
        report("convolution + rotation + cache write", f"T={T}", bench_queued(lambda: write(conv=conv, long_portions=n == 4)),
               nb + (T * C * 8 if T == 64 else 0))
        report("rope_kv (norm)", f"T={T}", bench_queued(lambda: ops.rope_kv_write(
            qkv, nq, nkv, d, pos, cs, d, slots=sl, k_cache=kc, v_cache=vc, q_norm_w=wn, k_norm_w=wn)), nb)
        x, y, y2, w = torch.randn(T, W, device=dev), rows(T, W), rows(T, W), torch.ones(W, device=dev, dtype=bf)
        report("residual, two normed, sum normed", f"T={T}", bench_queued(
            lambda: residual_update(x, y, w=w, y2=y2, w2=w, coef=0.5, w_sum=w, w_out=w)), T * W * 14)
        report("residual, two normed", f"T={T}", bench_queued(
            lambda: residual_update(x, y, w=w, y2=y2, w2=w, coef=0.5, w_out=w)), T * W * 14)
        o, g, out, wr = torch.randn(T, 1, W, device=dev), rows(T, W), rows(T, W), torch.ones(W, device=dev, dtype=bf)
        report("row norm + gate", f"T={T}", bench_queued(lambda: head_norm_gate(o, out, g=g, w=wr, act="sigmoid")), T * W * 8)
        report("head norm + gate", f"T={T}", bench_queued(lambda: head_norm_gate(o.view(T, H, d), out, g=g, w=wn, act="sigmoid")), T * W * 8)
        cw2, qr = torch.ones(R, device=dev, dtype=bf), 2048
        lat, cache = rows(T, qr + R), torch.zeros(T // 16 + 2, 1, 16, R, device=dev, dtype=bf)
        qw = torch.ones(qr, device=dev, dtype=bf)
        report("latent norms + cache write", f"T={T}", bench_queued(lambda: mla.latent_norm(
            lat[:, :qr], qw, qr, 1e-6, c=lat[:, qr:], c_w=cw2, slots=sl, cache=cache)), T * (qr + R) * 4)
        report("rmsnorm", f"T={T}", bench_queued(lambda: ops.rmsnorm(lat[:, :qr], qw, 1e-6)), T * qr * 4)
        E, K, I = 32, 4, W // 2
        w1, w2, xb, lg = rows(E * 2 * I, W).view(E, 2 * I, W), rows(E * W, I).view(E, W, I), rows(T, W), torch.randn(T, E, device=dev)
        ws = moe.shared_workspace(T, K, E, E, W, I, torch.device(dev), bf, W)
        nb = 2.0 * (min(E, T * K) * 3 * I * W + 2 * T * W)
        for name, act in (("clamped", ClampedGLU(7.0)), ("SiLU", "silu")):
            report(f"experts, {name}", f"T={T} E={E} top{K}", bench_queued(lambda: moe.fused_moe(
                xb, lg, w1, w2, K, ws=ws, interleaved=True, act=act)), nb, 6.0 * T * K * W * I)


def talking_rows(results, hbm, tf, tag):
    """The kernels of Vivazen beside their likes: attention with mixed heads against soft-capped attention without the mixture,
    windowed rotated latents with sinks against latents and MLA, convolution with row norms against convolution with rotation, the
    norm behind the sum against the other residual updates.  32 heads of 128, 8 key/value heads, width 4096."""
    from xllm_b200.models.layers import AttentionMetadata
    from xllm_b200.ops import mla, talking
    from xllm_b200.ops.head_norm import head_gate
    from xllm_b200.ops.residual import postnorm_update, residual_update
    dev, bf, d, W, nq, nkv, R, win = "cuda", torch.bfloat16, 128, 4096, 32, 8, 512, 1024
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    rows = lambda t, n: torch.randn(t, n, device=dev, dtype=bf)

    def report(name, shape, t, nbytes, flops=0.0):
        ideal = max(nbytes / (hbm * 1e9), flops / (tf * 1e12))
        results.append(dict(kernel=name, shape=shape, ms=t * 1e3, gbs=nbytes / t / 1e9, tflops=flops / t / 1e12,
                            frac_of_roofline=ideal / t, peaks=tag))
        print(f"{name:<38} {shape:<26} {t*1e6:9.1f} us {nbytes/t/1e9:7.0f} GB/s {flops/t/1e12:7.1f} TF/s  {ideal/t:6.3f} of {tag}",
              flush=True)

    talk = torch.eye(nq, device=dev, dtype=bf) + rows(nq, nq) * 0.1
    for S, L in ((4, 512), (4, 2048), (1, 8192)):
        T = S * L
        kc, vc = (rows(T // 16 * nkv * 16, d).view(T // 16, nkv, 16, d) for _ in range(2))
        bt = torch.arange(T // 16, device=dev, dtype=torch.int32).view(S, L // 16)
        cu, kl, q = i32([i * L for i in range(S + 1)]), i32([L] * S), rows(T, nq * d).view(T, nq, d)
        out, pairs = torch.empty_like(q), S * L * (L + 1) / 2
        nb = T * d * 2 * (2 * nq + 2 * nkv)
        report("prompts, capped", f"{S} x {L}", bench_queued(lambda: ops.paged_prefill_attention(
            q, kc, vc, bt, cu, kl, L, d ** -0.5, softcap=30.0, out=out), iters=5), nb, 4.0 * pairs * nq * d)
        report("prompts, capped, heads mixed", f"{S} x {L}", bench_queued(lambda: talking.prefill(
            q, kc, vc, bt, cu, kl, L, d ** -0.5, 30.0, talk, d, out, L, 0), iters=5), nb, pairs * nq * (4.0 * d + 2.0 * nq))
        lib, s = ops._lib.load(), ops.stream()
        lse = torch.empty(T, nq, device=dev)
        report("  row sums", f"{S} x {L}", bench_queued(lambda: lib.xllm_prefill_lse_tc(
            lse.data_ptr(), q.data_ptr(), q.stride(0), T, kc.data_ptr(), kc.shape[0], bt.data_ptr(), bt.stride(0), cu.data_ptr(),
            kl.data_ptr(), S, L, nq, nkv, 16, d ** -0.5, 30.0, ops.stream()), iters=5), 0.0, 2.0 * pairs * nq * d)
        n = min(T, max(128, talking.WORKSPACE_BYTES // (nq * L * 2) // 128 * 128))
        w = torch.empty(nq * n * L, device=dev, dtype=bf)
        r0 = T - n                                    # the last chunk of rows
        seen = sum(r % L + 1 for r in range(r0, T))
        for keys in (128, 512, 1024):
            report(f"  mixed weights of {n} rows, {keys} keys", f"{S} x {L}", bench_queued(lambda: lib.xllm_talk_weights(
                w.data_ptr(), n, L, q.data_ptr(), T, kc.data_ptr(), kc.shape[0], talk.data_ptr(), lse.data_ptr(), bt.data_ptr(), bt.stride(0), cu.data_ptr(),
                kl.data_ptr(), S, L, r0, n, nq, nkv, 16, d ** -0.5, 30.0, keys, ops.stream()), iters=5), 2.0 * seen * nq,
                seen * nq * (2.0 * d + 2.0 * nq))
        report(f"  values of {n} rows", f"{S} x {L}", bench_queued(lambda: lib.xllm_talk_values_tc(
            out.data_ptr(), d, w.data_ptr(), n, L, vc.data_ptr(), vc.shape[0], bt.data_ptr(), bt.stride(0), cu.data_ptr(), kl.data_ptr(), S, L,
            r0, n, nq, nkv, 16, ops.stream()), iters=5), 2.0 * seen * nq, 2.0 * seen * nq * d)
        del kc, vc, w
    for B, ctx in ((16, 8192), (64, 2048), (64, 8192), (256, 2048)):
        kc, vc = (rows(B * ctx // 16 * nkv * 16, d).view(B * ctx // 16, nkv, 16, d) for _ in range(2))
        bt = torch.randperm(B * ctx // 16, device=dev).to(torch.int32).view(B, ctx // 16)
        kl, q = i32([ctx] * B), rows(B, nq * d).view(B, nq, d)
        out, nb = torch.empty_like(q), 4.0 * B * ctx * nkv * d
        report("decode, capped", f"B={B} ctx {ctx}", bench_queued(lambda: ops.paged_decode_attention(
            q, kc, vc, bt, kl, d ** -0.5, softcap=30.0, out=out)), nb)
        report("decode, capped, heads mixed", f"B={B} ctx {ctx}", bench_queued(lambda: talking.decode(
            q, kc, vc, bt, kl, d ** -0.5, 30.0, talk, d, out, ctx)), nb)
        del kc, vc
    sink = torch.zeros(nq, device=dev)
    for B, ctx in ((16, 8192), (64, 4096), (256, 2048)):
        bt = (torch.randperm(B * (ctx // 16), device=dev) + 1).view(B, -1).to(torch.int32)
        sl, cache = i32([ctx] * B), rows((B * (ctx // 16) + 1) * 16, R + 64).view(-1, 1, 16, R + 64)
        q, out = rows(B, nq * (R + 64)).view(B, nq, R + 64) * 0.3, torch.empty(B, nq, R, device=dev, dtype=bf)
        for name, n, kw in (("latent decode, window, sinks", min(win, ctx), dict(window=win, sink=sink)), ("latent decode, sinks", ctx, dict(sink=sink)),
                            ("mla decode", ctx, {})):
            report(name, f"B={B} ctx {ctx}", bench_queued(lambda: mla.latent_decode(q, cache, bt, 0.09, seq_lens=sl, out=out, **kw)),
                   2.0 * B * n * (R + 64), 2.0 * B * nq * n * (2 * R + 64))
        del cache
    for S, L in ((4, 512), (4, 2048), (1, 8192)):
        T, bt = S * L, torch.arange(1, S * L // 16 + 1, device=dev, dtype=torch.int32).view(S, L // 16)
        cu, kl, pages = i32([i * L for i in range(S + 1)]), i32([L] * S), torch.arange(T // 128, device=dev, dtype=torch.int32).view(S, -1)
        cache, ukv, q = rows((T // 16 + 1) * 16, R + 64).view(-1, 1, 16, R + 64), rows(2 * nq * d, R + 64), rows(T, nq * d).view(T, nq, d)
        out = torch.empty(T, nq, d, device=dev, dtype=bf)
        for name, wn, kw in (("latent prompts, window, sinks", win, dict(window=win, sink=sink)), ("latent prompts", L, {})):
            def expanded():
                dense, n = mla.latent_gather(cache, bt, kl, L, cu, win) if kw else (mla.latent_gather(cache, bt, kl, L), kl)
                kv = ops.linear(dense, ukv)
                ops.ragged_prefill_attention(q, kv[:, :nq * d], kv[:, nq * d:], pages, 128, cu, n, L, 0.09, out, **kw)
            pairs = S * sum(min(i + 1, wn) for i in range(L))
            report(name, f"{S} x {L}", bench_queued(expanded, iters=5), 0.0, 4.0 * pairs * nq * d + 4.0 * T * (R + 64) * nq * d)
        del cache
    C = (nq + 2 * nkv) * d
    for T in (64, 8192):
        qkv, cs = rows(T, C), torch.randn(8192, d, device=dev)
        kc = torch.zeros(T // 16 + 2, nkv, 16, d, device=dev, dtype=bf)
        vc, sl = torch.zeros_like(kc), torch.arange(16, 16 + T, dtype=torch.int32, device=dev)
        q, k, v = qkv[:, :nq * d], qkv[:, nq * d:(nq + nkv) * d], qkv[:, (nq + nkv) * d:]
        n = T if T == 64 else 4                                       # decode rows, or four prompts
        ring, cw, L = torch.zeros(n + 1, 4, C, device=dev, dtype=bf), rows(4, C), T // n
        conv = (cw, ring, i32(list(range(n))), i32([i * L for i in range(n + 1)]), i32([L if n == 4 else 100] * n))
        pos, nb, one = torch.arange(T, device=dev) % 2048, T * d * 4 * (nq + 2 * nkv), torch.ones(nq * d, device=dev, dtype=bf)
        nb += T * C * 8 if T == 64 else 0
        report("convolution + rotation + cache write", f"T={T}", bench_queued(lambda: ops.rope_norm_kv_write(
            q, k, v, nq, nkv, d, pos, cs, d, sl, kc, vc, unit_norm=False, conv=conv, long_portions=n == 4)), nb)
        report("convolution + row norms + cache write", f"T={T}", bench_queued(lambda: talking.conv_row_norm_kv_write(
            q, k, v, nq, nkv, d, sl, kc, vc, one, one[:nkv * d], conv, long_portions=n == 4)), nb)
        x, y, w = torch.randn(T, W, device=dev), rows(T, W), torch.ones(W, device=dev, dtype=bf)
        report("residual, branch normed", f"T={T}", bench_queued(lambda: residual_update(x, y, w=w, w_out=w)), T * W * 12)
        for g in (1, 4):
            report(f"residual, sum normed, {g} parts", f"T={T}", bench_queued(lambda: postnorm_update(x, y, w, alpha=0.5, groups=g)), T * W * 12)
        ld = nq * d + R + 64 + nq
        lat, cache = rows(T, ld), torch.zeros(T // 16 + 2, 1, 16, R + 64, device=dev, dtype=bf)
        cw2, qa = torch.ones(R, device=dev, dtype=bf), torch.empty(T, nq, R + 64, device=dev, dtype=bf)
        ql, c, cos = lat[:, :nq * d], lat[:, nq * d:nq * d + R + 64], torch.randn(8192, 64, device=dev)
        nqa = T if T == 64 else 0
        report("latent rows + rotation", f"T={T}", bench_queued(lambda: mla.rope_write(
            ql, nq, 64, c, cw2, R, 64, R, cos, pos, sl, cache, 1e-6, qa=qa if nqa else None, qa_rows=nqa)),
            T * ((R + 64) * 4 + nq * 64 * 4) + nqa * nq * 64 * 2)
        c8 = rows(T, 2048 + R)
        report("latent norms + cache write", f"T={T}", bench_queued(lambda: mla.latent_norm(
            c8[:, :2048], torch.ones(2048, device=dev, dtype=bf), 2048, 1e-6, c=c8[:, 2048:], c_w=cw2, slots=sl,
            cache=cache.view(-1)[:(T // 16 + 2) * 16 * R].view(-1, 1, 16, R))), T * (2048 + R) * 4)
        a = rows(T, nq * d).view(T, nq, d)
        report("gate per head", f"T={T}", bench_queued(lambda: head_gate(a, lat[:, ld - nq:], d)), T * nq * d * 4)
        gu = rows(T, 6 * W)
        report("gelu gate", f"T={T}", bench_queued(lambda: gemm_tcgen05.act_and_mul_interleaved(gu, "gelu_tanh")), T * W * 18)
        report("silu gate", f"T={T}", bench_queued(lambda: gemm_tcgen05.act_and_mul_interleaved(gu, "silu")), T * W * 18)


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--what", default="gemm,decode,prefill,small")
    ap.add_argument("--json", default="")
    a = ap.parse_args()
    hbm, tf, tag = peaks()
    results = []
    for w in a.what.split(","):
        {"gemm": gemm_rows, "decode": decode_rows, "prefill": prefill_rows, "small": small_rows, "gdn": gdn_rows, "mla": mla_rows,
         "fp8": fp8_rows, "moe": moe_rows, "hybrid": hybrid_rows, "recurrent": recurrent_rows,
         "latent": latent_rows, "talking": talking_rows}[w](results, hbm, tf, tag)
    if a.json:
        with open(a.json, "w") as f:
            json.dump(results, f, indent=1)


if __name__ == "__main__":
    main()
