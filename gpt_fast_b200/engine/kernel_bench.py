"""Times single kernels of the library at given sizes (CUDA events around a
CUDA graph of repeated launches, so that host time is not measured), and is
the small, self-ending workload that profiler captures are taken on.

    python -m gpt_fast_b200.engine.kernel_bench linear --m 8 --n 28672 --k 4096 --mode swiglu
    python -m gpt_fast_b200.engine.kernel_bench linear --m 2048 --n 6144 --k 4096 --mode store
    python -m gpt_fast_b200.engine.kernel_bench attention --batch 8 --context 4000
    python -m gpt_fast_b200.engine.kernel_bench attention --batch 1 --context 0 --new 2048
    python -m gpt_fast_b200.engine.kernel_bench sample --batch 8 --vocab 128256
    python -m gpt_fast_b200.engine.kernel_bench experts --tokens 2048 --experts 16 --top 4 --ff 1792 --dim 2048
    python -m gpt_fast_b200.engine.kernel_bench streams --rows 2048 --dim 2048 --streams 4
    python -m gpt_fast_b200.engine.kernel_bench qkv --rows 2048 --heads 16 --kv_heads 4 --head_dim 128
    python -m gpt_fast_b200.engine.kernel_bench gla --tokens 2048 --heads 16 --head_dim 128 --v_dim 128

Weights are cycled through enough copies to exceed the L2 cache, so a memory-
bound kernel is timed against DRAM.  gpt-fast has no per-kernel timing; its
`--profile` exports a torch profiler trace of one sample (generate.py:380-407).
"""
import argparse
import math
import sys

import torch

from .. import ops
from ..ops.types import BatchMeta, PagedKV

L2_BYTES = 126e6


def graph_time_us(fn, reps, warm=2):
    for i in range(warm):
        fn(i)
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g):
        for i in range(reps):
            fn(i)
    g.replay()
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    g.replay()
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) / reps * 1e3


def bench_linear(a):
    M, N, K = a.m, a.n, a.k
    copies = max(2, int(3 * L2_BYTES // (N * K * 2)) + 1) if M <= 128 else 1
    ws = [torch.randn(N, K, device="cuda", dtype=torch.bfloat16) * 0.02 for _ in range(copies)]
    x = torch.randn(M, K, device="cuda", dtype=torch.bfloat16)
    out_dtype = torch.float32 if a.mode == "add" else torch.bfloat16
    out = torch.zeros(M, N // 2 if a.mode == "swiglu" else N, device="cuda", dtype=out_dtype)
    us = graph_time_us(lambda i: ops.linear(x, ws[i % copies], out, a.mode, defer=a.mode != "swiglu"), a.reps)
    gbs = N * K * 2 / us / 1e3
    tfs = 2.0 * M * N * K / us / 1e6
    print(f"linear M={M} N={N} K={K} mode={a.mode}: {us:.1f} us, weights at {gbs:.0f} GB/s, {tfs:.0f} TFLOP/s "
          f"(plan swap,bn,splits,stages = {ops.kernels().tc_plan(M, N, K, a.mode)})")


def paged_batch(batch, context, new, heads_kv, head_dim, device="cuda"):
    """`batch` sequences with `context` cached tokens each, bringing `new` tokens; pages in shuffled order."""
    total = context + new
    pages_each = -(-total // 64)
    n_pages = batch * pages_each
    perm = torch.randperm(n_pages).to(torch.int32).view(batch, pages_each)
    table = perm.to(device)
    cu = torch.arange(batch + 1, dtype=torch.int32) * new
    meta = BatchMeta(cu.to(device), torch.arange(batch, dtype=torch.int32).repeat_interleave(new).to(device),
                     torch.arange(batch, dtype=torch.int32).to(device),
                     torch.full((batch,), context, dtype=torch.int32, device=device), batch, batch * new, new, total,
                     ops.new_status(device))
    k = torch.randn(n_pages, heads_kv, 64, head_dim, device=device, dtype=torch.bfloat16)
    v = torch.randn(n_pages, heads_kv, 64, head_dim, device=device, dtype=torch.bfloat16)
    return meta, PagedKV(k, v, table, 64)


def bench_attention(a):
    H, G, d = a.heads, a.kv_heads, a.head_dim
    meta, kv = paged_batch(a.batch, a.context, a.new, G, d)
    q = torch.randn(meta.n_tokens, H, d, device="cuda", dtype=torch.bfloat16)
    out = torch.empty(meta.n_tokens, H * d, device="cuda", dtype=torch.bfloat16)
    kv_bytes = a.batch * (a.context + a.new) * G * d * 2 * 2
    if a.new == 1 and a.partials >= 0:
        # the decode step's kernel: rotary encoding and cache append from the q/k/v product (its partial sums), then attention
        W = (H + 2 * G) * d
        parts = torch.randn(a.partials, meta.n_tokens, W, device="cuda") if a.partials else None
        qkv = torch.randn(meta.n_tokens, W, device="cuda", dtype=torch.bfloat16)
        table = torch.empty(a.context + a.new + 64, d // 2, 2, device="cuda")
        ops.rope_table((1.0 / (10000 ** (torch.arange(d // 2).float() * 2 / d))).cuda(), table)
        us = graph_time_us(lambda i: ops.rope_append_attention(qkv, parts, kv, meta, table, out, H, G, d, "interleaved", True,
                                                               1 / math.sqrt(d)), a.reps)
        print(f"rotary + append + attention decode batch={a.batch} context={a.context} partial sums={a.partials}: {us:.1f} us, "
              f"K/V at {kv_bytes / us / 1e3:.0f} GB/s")
        ops.check_status(meta.status)
        return
    window = a.window or None
    extra = {}
    if a.bias == "table":                                   # a bias by head and distance: one row per distance up to the window
        extra["bias"] = torch.randn(window or a.context + a.new, H, device="cuda") * 0.5
    elif a.bias == "slopes":
        extra["slopes"] = torch.tensor([2.0 ** (-8.0 * (h + 1) / H) for h in range(H)], device="cuda")
    if a.new > 1 and a.tiles:
        run = lambda i: ops.kernels()._attention_bf16(q, kv, meta, out, H, G, d, 1 / math.sqrt(d), window, prefill=True, tiles=a.tiles,
                                                      max_blocks=a.max_blocks, **extra)
    else:
        run = lambda i: ops.attention(q, kv, meta, out, H, G, d, 1 / math.sqrt(d), window, **extra)
    us = graph_time_us(run, a.reps)
    what = f"window={a.window} bias={a.bias}"
    if a.new == 1:
        print(f"attention decode batch={a.batch} context={a.context} {what}: {us:.1f} us, K/V at {kv_bytes / us / 1e3:.0f} GB/s")
    else:
        T0, T1 = a.context, a.context + a.new
        seen = sum(min(p + 1, window or p + 1) for p in range(T0, T1))      # keys the queries see
        flops = a.batch * 4.0 * H * d * seen
        print(f"attention prefill batch={a.batch} context={a.context} new={a.new} {what}: {us:.1f} us, {flops / us / 1e6:.0f} TFLOP/s "
              f"(of the keys seen)")
    ops.check_status(meta.status)


def bench_sample(a):
    logits = torch.randn(a.batch, a.vocab, device="cuda")
    tok = torch.empty(a.batch, dtype=torch.int32, device="cuda")
    us = graph_time_us(lambda i: ops.sample(logits, tok, 0.8, a.top_k or None, 1), a.reps)
    print(f"sample batch={a.batch} vocab={a.vocab} top_k={a.top_k}: {us:.1f} us")
    us = graph_time_us(lambda i: ops.argmax(logits, tok), a.reps)
    print(f"argmax batch={a.batch} vocab={a.vocab}: {us:.1f} us")


def bench_norm(a):
    """RMSNorm of the residual stream, as a decode step runs it: the rows' pending partial sums are added on the way."""
    x = torch.randn(a.rows, a.dim, device="cuda")
    w = torch.ones(a.dim, device="cuda", dtype=torch.bfloat16)
    out = torch.empty(a.rows, a.dim, device="cuda", dtype=torch.bfloat16)
    pending = torch.randn(a.partials, a.rows, a.dim, device="cuda") if a.partials else None
    us = graph_time_us(lambda i: ops.rmsnorm(x, w, 1e-5, out, None, pending), a.reps)
    print(f"rmsnorm rows={a.rows} dim={a.dim} pending partial sums={a.partials}: {us:.1f} us")


def bench_experts(a):
    """The experts of a mixture (sort by expert, gather, gate/up with the activation, down, weighted sum), every kernel
    timed by events of its own (the weights of all experts exceed the L2 cache at the default sizes)."""
    T, E, top, F, D = a.tokens, a.experts, a.top, a.ff, a.dim
    g = torch.Generator(device="cuda").manual_seed(0)
    w13 = (torch.randn(E, 2 * F, D, device="cuda", generator=g) * D ** -0.5).bfloat16()
    w2 = (torch.randn(E, D, F, device="cuda", generator=g) * F ** -0.5).bfloat16()
    h = torch.randn(T, D, device="cuda", generator=g).bfloat16()
    idx = torch.stack([torch.randperm(E, device="cuda", generator=g)[:top] for _ in range(T)]).int()
    w = torch.rand(T, top, device="cuda", generator=g)
    x = torch.zeros(T, D, device="cuda")
    flush = torch.empty(int(2 * L2_BYTES), dtype=torch.uint8, device="cuda")
    best = {}
    for i in range(a.reps + 2):
        flush.zero_()
        torch.cuda.synchronize()
        with ops.trace() as rec:
            ops.moe_experts(h, idx, w, w13, w2, x, a.limit, 1.702, 1.0)
        for label, ms in ops.trace_times(rec):
            if i >= 2:
                label = label.split(" ")[0]
                best[label] = min(best.get(label, 1e9), ms * 1e3)
    total = sum(best.values())
    busy = len(torch.unique(idx))
    print(f"experts T={T} E={E} top={top} ff={F} dim={D}: " + ", ".join(f"{k} {v:.1f}" for k, v in best.items()) + f" us; total {total:.1f} us, "
          f"{2.0 * T * top * 3 * F * D / total / 1e6:.0f} TFLOP/s, the {busy} chosen experts' weights at {busy * 3 * F * D * 2 / total / 1e3:.0f} GB/s")


def bench_gla(a):
    """Gated linear attention over one prompt (--batch 1) or a decode step (--tokens 1) of `batch` sequences."""
    B, T, H, d, dv, rank = a.batch, a.tokens, a.heads, a.head_dim, a.v_dim, 16
    meta, _ = paged_batch(B, 0, T, 1, 8)
    W = 2 * H * d + 2 * H * dv + rank
    src = torch.randn(B * T, W, device="cuda").bfloat16()
    a2, bias = (torch.randn(H * d, rank, device="cuda") * 0.3).bfloat16(), torch.randn(H * d, device="cuda")
    norm, out = torch.ones(dv, device="cuda"), torch.empty(B * T, H * dv, device="cuda", dtype=torch.bfloat16)
    copies = max(1, int(2 * L2_BYTES // (B * H * d * dv * 4)) + 1) if T == 1 else 1
    states = [torch.zeros(B, H * d * dv, device="cuda") for _ in range(copies)]
    offs = (0, H * d, 2 * H * d, W - rank, 2 * H * d + H * dv)
    us = graph_time_us(lambda i: ops.gla(src, offs, rank, a2, bias, 16.0, states[i % copies], 0, norm, 1e-5, out, meta, H, d, dv, d ** -0.5), a.reps)
    if T == 1:
        print(f"gla decode batch={B} heads={H} {d} x {dv}: {us:.1f} us, states at {2 * B * H * d * dv * 4 / us / 1e3:.0f} GB/s")
    else:
        flops = B * T * H * 4.0 * d * dv                      # the recurrence itself: the state's update and its read-out
        print(f"gla prefill batch={B} tokens={T} heads={H} {d} x {dv}: {us:.1f} us, {flops / us / 1e6:.1f} TFLOP/s of the recurrence")
    ops.check_status(meta.status)


def bench_streams(a):
    """Several residual streams: a sublayer's output (a tensor, or partial sums) goes into them and the next input comes out normed.
    Enough copies of everything are cycled through to exceed the L2 cache."""
    T, D, n = a.rows, a.dim, a.streams
    nbytes = T * D * (4 * (2 * n + max(a.partials, 1)) + 2)
    copies = max(1, min(64, int(3 * L2_BYTES // nbytes) + 1))
    xs = [torch.randn(n, T, D, device="cuda") for _ in range(copies)]
    ys = [torch.randn(a.partials, T, D, device="cuda") if a.partials else torch.randn(T, D, device="cuda") for _ in range(copies)]
    mix, leave, enter = torch.eye(n, device="cuda"), torch.ones(n, device="cuda") * 1e-3, torch.full((n,), 1.0 / n, device="cuda")
    w, out = torch.ones(D, device="cuda", dtype=torch.bfloat16), [torch.empty(T, D, device="cuda", dtype=torch.bfloat16) for _ in range(copies)]
    us = graph_time_us(lambda i: ops.streams(xs[i % copies], n, False, xs[i % copies], mix, leave, [ys[i % copies]], enter, w, 1e-5, out[i % copies]), a.reps)
    print(f"streams rows={T} dim={D} streams={n} partial sums={a.partials}: {us:.1f} us, {nbytes / us / 1e3:.0f} GB/s")


def bench_qkv(a):
    """q, k and v of `rows` tokens with biases and a norm over the whole projection into queries and cache."""
    H, G, d, T = a.heads, a.kv_heads, a.head_dim, a.rows
    W = (H + 2 * G) * d
    new = T // a.batch
    meta, kv = paged_batch(a.batch, 512, new, G, d)
    nbytes = T * W * (2 + (4 * a.partials if a.partials else 2))
    copies = max(1, min(64, int(3 * L2_BYTES // nbytes) + 1))
    srcs = [torch.randn(T, W, device="cuda").bfloat16() for _ in range(copies)]
    parts = [torch.randn(a.partials, T, W, device="cuda") for _ in range(copies)] if a.partials else [None] * copies
    q = torch.empty(T, H, d, device="cuda", dtype=torch.bfloat16)
    table = torch.empty(512 + new + 64, a.rot // 2, 2, device="cuda")
    ops.rope_table((1.0 / (10000 ** (torch.arange(a.rot // 2).float() * 2 / a.rot))).cuda(), table)
    bias, qn, kn = torch.randn(W, device="cuda"), torch.ones(H * d, device="cuda").bfloat16(), torch.ones(G * d, device="cuda").bfloat16()
    us = graph_time_us(lambda i: ops.qkv_prepare(srcs[i % copies], parts[i % copies], (0, H * d, (H + G) * d), q, kv, meta, H, G, d, d, table=table,
                                                 rot_dims=a.rot, pairing=a.pairing, q_norm=qn, k_norm=kn, norm_eps=1e-5, norm_whole=True, bias=bias), a.reps)
    print(f"qkv rows={T} heads={H}/{G} of {d} pairs={a.pairing} partial sums={a.partials}: {us:.1f} us, {nbytes / us / 1e3:.0f} GB/s")
    ops.check_status(meta.status)


def main(argv=None):
    ap = argparse.ArgumentParser(prog="kernel_bench")
    sub = ap.add_subparsers(dest="what", required=True)
    p = sub.add_parser("linear")
    p.add_argument("--m", type=int, default=8); p.add_argument("--n", type=int, default=28672)
    p.add_argument("--k", type=int, default=4096); p.add_argument("--mode", default="swiglu", choices=["store", "add", "swiglu"])
    p.add_argument("--reps", type=int, default=10)
    p = sub.add_parser("attention")
    p.add_argument("--batch", type=int, default=8); p.add_argument("--context", type=int, default=4000)
    p.add_argument("--new", type=int, default=1); p.add_argument("--heads", type=int, default=32)
    p.add_argument("--kv_heads", type=int, default=8); p.add_argument("--head_dim", type=int, default=128)
    p.add_argument("--window", type=int, default=0, help="only the latest so many positions are seen (0: all)")
    p.add_argument("--bias", default="none", choices=["none", "table", "slopes"], help="a bias on the score by head and distance")
    p.add_argument("--tiles", type=int, default=0, help="prefill, head_dim 128: query tiles per block of the tcgen05 kernel (0: its own choice)")
    p.add_argument("--max_blocks", type=int, default=0, help="with --tiles 1: cap of the persistent kernel's grid (0: one block per SM)")
    p.add_argument("--partials", type=int, default=-1,
                   help="decode only: time the fused rotary + append + attention kernel fed by this many partial sums (0: bfloat16 qkv)")
    p.add_argument("--reps", type=int, default=10)
    p = sub.add_parser("sample")
    p.add_argument("--batch", type=int, default=8); p.add_argument("--vocab", type=int, default=128256)
    p.add_argument("--top_k", type=int, default=200); p.add_argument("--reps", type=int, default=10)
    p = sub.add_parser("norm")
    p.add_argument("--rows", type=int, default=8); p.add_argument("--dim", type=int, default=4096)
    p.add_argument("--partials", type=int, default=9); p.add_argument("--reps", type=int, default=10)
    p = sub.add_parser("experts")
    p.add_argument("--tokens", type=int, default=2048); p.add_argument("--experts", type=int, default=16)
    p.add_argument("--top", type=int, default=4); p.add_argument("--ff", type=int, default=1792)
    p.add_argument("--dim", type=int, default=2048); p.add_argument("--limit", type=float, default=7.0)
    p.add_argument("--reps", type=int, default=5)
    p = sub.add_parser("streams")
    p.add_argument("--rows", type=int, default=2048); p.add_argument("--dim", type=int, default=2048)
    p.add_argument("--streams", type=int, default=4); p.add_argument("--partials", type=int, default=0)
    p.add_argument("--reps", type=int, default=20)
    p = sub.add_parser("qkv")
    p.add_argument("--rows", type=int, default=2048); p.add_argument("--batch", type=int, default=1); p.add_argument("--heads", type=int, default=16)
    p.add_argument("--kv_heads", type=int, default=4); p.add_argument("--head_dim", type=int, default=128)
    p.add_argument("--rot", type=int, default=64); p.add_argument("--partials", type=int, default=0)
    p.add_argument("--pairing", default="interleaved", choices=["interleaved", "half"]); p.add_argument("--reps", type=int, default=20)
    p = sub.add_parser("gla")
    p.add_argument("--batch", type=int, default=1); p.add_argument("--tokens", type=int, default=2048)
    p.add_argument("--heads", type=int, default=16); p.add_argument("--head_dim", type=int, default=128)
    p.add_argument("--v_dim", type=int, default=128); p.add_argument("--reps", type=int, default=10)
    a = ap.parse_args(argv)
    {"gla": bench_gla, "streams": bench_streams, "qkv": bench_qkv, "experts": bench_experts, "linear": bench_linear, "attention": bench_attention, "sample": bench_sample, "norm": bench_norm}[a.what](a)
    ops.check_status(ops.new_status("cuda"))
    return 0


if __name__ == "__main__":
    sys.exit(main())
