"""Timing of single kernels at the sizes of a model, for profiling.

    python -m rllm_b200.kernels.microbench attention_decode --batch 8 --context 4096
    python -m rllm_b200.kernels.microbench attention_prefill --tokens 2048 [--impl tcgen05]
    python -m rllm_b200.kernels.microbench gemm_small_m --rows 8 [--variant residual|rstd]
    python -m rllm_b200.kernels.microbench gemm_tcgen05 --rows 2048
    python -m rllm_b200.kernels.microbench latent_attention --tokens 2048 --heads 16 --kv-rank 512 --rot-dim 64
    python -m rllm_b200.kernels.microbench latent_attention --batch 8 --context 4096 --tokens 1 ...
    python -m rllm_b200.kernels.microbench routed_experts --rows 2048 --experts 32 --top 4 --intermediate 1024
    python -m rllm_b200.kernels.microbench lightning_scan --tokens 2048 --heads 16 --head-dim 128 --v-dim 128
    python -m rllm_b200.kernels.microbench selective_scan --tokens 2048 --channels 4096 --state 16
    python -m rllm_b200.kernels.microbench mlstm_scan --tokens 2048 --heads 8 --head-dim 128 --v-dim 256
    python -m rllm_b200.kernels.microbench channel_delta --tokens 2048 --heads 16 --head-dim 128 --v-dim 128
    python -m rllm_b200.kernels.microbench ssd_scan --tokens 2048 --heads 64 --head-dim 64 --state 128 --groups 1
    python -m rllm_b200.kernels.microbench linear_state --variant retention --tokens 2048 --heads 16 --head-dim 128
    python -m rllm_b200.kernels.microbench shared_key_attention --tokens 8192 --heads 16 --kv-heads 4 --head-dim 128 --window 1024
    python -m rllm_b200.kernels.microbench streams --tokens 2048 --hidden 2048 --streams 4

Sizes default to the Llama-3.2-1B shape (32 heads, 8 kv heads, head 64, hidden
2048, intermediate 8192).  Times are CUDA-event times over ``--iters`` launches
after warm-up; inputs rotate over several buffers larger than L2 together, so
that weights and caches come from HBM as in a model step.  One line per case:
microseconds, and GB/s (memory-bound kernels) or TFLOP/s (products, attention
over prompts).
"""
from __future__ import annotations

import argparse
import math
import sys

import torch

from . import ops

DEV = "cuda:0"


def time_us(fn, iters: int, warmup: int = 3) -> float:
    for i in range(warmup):
        fn(i)
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    for i in range(iters):
        fn(i)
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) * 1e3 / iters


def time_graph_us(fn, iters: int) -> float:
    """Back-to-back launches inside one CUDA graph: no host gaps between kernels."""
    for i in range(3):
        fn(i)
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    s = torch.cuda.Stream()
    with torch.cuda.stream(s):
        with torch.cuda.graph(g):
            for i in range(iters):
                fn(i)
    torch.cuda.synchronize()
    g.replay()                      # the first replay also uploads the graph
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    g.replay()
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) * 1e3 / iters


def _mask_options(args, rows: int, nq: int, d: int):
    """The attention kernels' options from the command line: (keyword arguments, a word for the report)."""
    kw = {}
    if args.keep_first:
        kw["keep_first"] = args.keep_first
    if args.chunk:
        kw["chunk"] = args.chunk
    if args.softcap:
        kw["softcap"] = args.softcap
    if args.sinks:
        kw["sinks"] = torch.randn(nq, device=DEV)
    if args.slopes:
        kw["slopes"] = torch.tensor([2.0 ** (-args.slopes * (h + 1) / nq) for h in range(nq)], device=DEV)
    if args.gate:
        kw["gate"] = torch.randn(rows, nq if args.gate == "head" else nq * d, device=DEV).bfloat16()
        kw["gate_per_head"] = args.gate == "head"
    return kw, (" with " + ", ".join(sorted(k for k in kw if k != "gate_per_head")) if kw else "")


def _seen(p: int, window: int, keep: int, chunk: int) -> int:
    """Keys that the query at position p sees."""
    lo = max(0, p - window + 1) if window else 0
    if chunk:
        lo = max(lo, p // chunk * chunk)
    return p + 1 - lo + (min(keep, lo) if window else 0)


def attention_decode(args) -> None:
    nq, nkv, d, page = args.heads, args.kv_heads, args.head_dim, args.page
    B, ctx = args.batch, args.context
    pages = B * (ctx // page) + 8
    nc = max(2, min(8, int(300e6 // (pages * nkv * page * d * 4)) + 1))
    caches = [(torch.randn(pages, nkv, page, d, device=DEV).bfloat16(),
               torch.randn(pages, nkv, page, d, device=DEV).bfloat16()) for _ in range(nc)]
    table = torch.randperm(pages - 8, device=DEV).int().view(B, ctx // page).contiguous()
    err = torch.zeros(1, dtype=torch.int32, device=DEV)
    q = torch.randn(B, nq * d, device=DEV).bfloat16()
    out = torch.empty_like(q)
    seq_lens = torch.full((B,), ctx, dtype=torch.int32, device=DEV)
    ws = torch.empty(ops.attention_decode_workspace(B, nq, d, ctx), device=DEV)
    scale = 1 / math.sqrt(d)

    kw, word = _mask_options(args, B, nq, d)

    def run(i):
        k, v = caches[i % nc]
        ops.attention_decode_bf16(q, nq * d, out, k, v, table, seq_lens, B, ctx, nq, nkv, d, args.window, scale, err, ws,
                                  **kw)
    us = time_graph_us(run, args.iters)
    nbytes = B * _seen(ctx - 1, args.window, args.keep_first, args.chunk) * nkv * d * 2 * 2
    print(f"attention_decode batch {B} context {ctx} window {args.window}{word}: {us:.1f} us, "
          f"{nbytes / us / 1e3:.0f} GB/s of visible K and V")


def attention_prefill(args) -> None:
    nq, nkv, d, page = args.heads, args.kv_heads, args.head_dim, args.page
    T = args.tokens
    pages = T // page + 8
    k = torch.randn(pages, nkv, page, d, device=DEV).bfloat16()
    v = torch.randn(pages, nkv, page, d, device=DEV).bfloat16()
    table = torch.randperm(pages - 8, device=DEV).int().view(1, T // page).contiguous()
    err = torch.zeros(1, dtype=torch.int32, device=DEV)
    q = torch.randn(T, nq * d, device=DEV).bfloat16()
    out = torch.empty_like(q)
    seq_lens = torch.tensor([T], dtype=torch.int32, device=DEV)
    q_start = torch.tensor([0, T], dtype=torch.int32, device=DEV)
    scale = 1 / math.sqrt(d)

    fn = ops.attention_prefill_tcgen05 if args.impl == "tcgen05" else ops.attention_prefill_bf16
    kw, word = _mask_options(args, T, nq, d)

    def run(i):
        fn(q, nq * d, out, k, v, table, q_start, seq_lens, 0, 1, T, nq, nkv, d, args.window, scale, err, **kw)
    us = time_us(run, args.iters)
    flops = 4 * d * nq * sum(_seen(p, args.window, args.keep_first, args.chunk) for p in range(T))
    print(f"attention_prefill ({args.impl}) tokens {T} window {args.window}{word}: {us:.1f} us, "
          f"{flops / us / 1e6:.0f} TFLOP/s (visible pairs)")
    if int(err.item()):
        print(f"error word {int(err.item())}", file=sys.stderr)


def latent_attention(args) -> None:
    """--tokens > 1: one prompt of that many tokens; --tokens 1: --batch sequences of --context cached rows."""
    heads, dv, dk, page = args.heads, args.kv_rank, args.kv_rank + args.rot_dim, args.page
    if args.tokens > 1:
        S, nq, ctx = 1, args.tokens, args.tokens
    else:
        S, nq, ctx = args.batch, 1, args.context
    per = -(-ctx // page)
    cache = torch.randn(S * per + 4, 1, page, dk, device=DEV).bfloat16()
    table = torch.randperm(S * per, device=DEV).int().view(S, per).contiguous()
    T = S * nq
    q = torch.randn(T, heads * dk, device=DEV).bfloat16()
    out = torch.empty(T, heads * dv, device=DEV, dtype=torch.bfloat16)
    err = torch.zeros(1, dtype=torch.int32, device=DEV)
    q_start = torch.arange(0, T + 1, nq, dtype=torch.int32, device=DEV)
    seq_lens = torch.full((S,), ctx, dtype=torch.int32, device=DEV)
    scale = 1 / math.sqrt(dk)

    def run(i):
        ops.latent_attention_mma(q, out, cache, table, q_start, seq_lens, S, nq, heads, dk, dv, args.window, scale, None,
                                 err, max_seq_len=ctx)
    us = time_us(run, args.iters)
    vis = sum(min(p + 1, args.window or p + 1) for p in range(ctx - nq, ctx)) * S
    flops = 2 * (dk + dv) * heads * vis
    gb = 2 * S * min(ctx, (args.window or ctx) + nq) * dk / 1e9
    print(f"latent_attention tokens {T} context {ctx} heads {heads} rows of {dk} (values {dv}): {us:.1f} us, "
          f"{flops / us / 1e6:.1f} TFLOP/s, rows read once {gb / us * 1e6:.0f} GB/s")
    if int(err.item()):
        print(f"error word {int(err.item())}", file=sys.stderr)


def routed_experts(args) -> None:
    T, H, F, E, top = args.rows, args.hidden, args.intermediate, args.experts, args.top
    x = torch.randn(T, H, device=DEV).bfloat16()
    wgu = (torch.randn(E, 2 * F, H, device=DEV) * 0.02).bfloat16()
    wd = (torch.randn(E, H, F, device=DEV) * 0.02).bfloat16()
    ids = torch.stack([torch.randperm(E, device=DEV)[:top] for _ in range(T)]).int().contiguous()

    def run(i):
        ops.moe_experts(x, ids, wgu, wd, 7.0, 1.702)
    us = time_us(run, args.iters)
    used = min(E, T * top)
    print(f"routed_experts rows {T} x top {top} of {E} experts ({H} -> {F} -> {H}): {us:.1f} us, "
          f"{2 * 3 * H * F * T * top / us / 1e6:.1f} TFLOP/s, touched weights once {used * 3 * H * F * 2 / us / 1e3:.0f} GB/s")


def _shapes(args):
    H, I = args.hidden, args.intermediate
    qkv = (args.heads + 2 * args.kv_heads) * args.head_dim
    return [("qkv", qkv, H), ("o_proj", H, args.heads * args.head_dim), ("gate_up", 2 * I, H), ("down", H, I)]


def gemm_small_m(args) -> None:
    """--variant plain: the four projections.  residual: o and down adding into a float32 stream and
    preparing the next norm.  rstd: qkv and gate_up applying the norm's row factors."""
    M = args.rows
    for name, N, K in _shapes(args):
        silu = name == "gate_up"
        if args.only and name != args.only:
            continue
        if args.variant == "residual" and name not in ("o_proj", "down"):
            continue
        if args.variant == "rstd" and name not in ("qkv", "gate_up"):
            continue
        nw = max(2, int(300e6 // (N * K * 2)) + 1)
        ws = [(torch.randn(N, K, device=DEV) * 0.02).bfloat16() for _ in range(nw)]
        x = torch.randn(M, K, device=DEV).bfloat16()
        out = torch.empty(M, N // 2 if silu else N, device=DEV, dtype=torch.bfloat16)
        h = torch.randn(M, N, device=DEV)
        wn = torch.ones(N, device=DEV)
        parts = torch.ones(128, M, device=DEV)

        def run(i):
            if args.variant == "residual":
                ops.gemm_small_m_residual(x, ws[i % nw], h, wn)
            elif args.variant == "rstd":
                ops.gemm_small_m_rstd(x, parts, 1e-5, ws[i % nw], out, "silu_mul" if silu else "store")
            else:
                ops.gemm_small_m(x, ws[i % nw], out, "silu_mul" if silu else "store")
        us = time_graph_us(run, args.iters)
        print(f"gemm_small_m ({args.variant}) rows {M} {name}{' +silu' if silu else ''} [{N} x {K}]: {us:.1f} us, "
              f"{N * K * 2 / us / 1e3:.0f} GB/s of weight")


def gemm_tcgen05(args) -> None:
    M = args.rows
    for name, N, K in _shapes(args):
        if args.only and name != args.only:
            continue
        w = (torch.randn(N, K, device=DEV) * 0.02).bfloat16()
        x = torch.randn(M, K, device=DEV).bfloat16()
        silu = name == "gate_up"
        out = torch.empty(M, N // 2 if silu else N, device=DEV, dtype=torch.bfloat16)

        def run(i):
            ops.gemm_tcgen05(x, w, out, "silu_mul" if silu else "store")
        us = time_us(run, args.iters)
        print(f"gemm_tcgen05 rows {M} {name}{' +silu' if silu else ''} [{N} x {K}]: {us:.1f} us, "
              f"{2 * M * N * K / us / 1e6:.0f} TFLOP/s")
    ops.check_gemm_errors(torch.device(DEV))


def _one_sequence(T, batch):
    """(q_start, token_seq, slots, number of sequences, longest): one portion of T tokens, or ``batch``
    sequences of one token each when T == 1."""
    S = batch if T == 1 else 1
    per = 1 if T == 1 else T
    q_start = torch.arange(0, S * per + 1, per, dtype=torch.int32, device=DEV)
    token_seq = torch.arange(S, dtype=torch.int32, device=DEV).repeat_interleave(per)
    return q_start, token_seq, torch.arange(S, dtype=torch.int32, device=DEV), S, per


def lightning_scan(args) -> None:
    """The lightning-attention recurrence over one prompt portion, or one token of ``--batch`` sequences."""
    heads, d, dv = args.heads, args.head_dim, args.v_dim or args.head_dim
    q_start, _, slots, S, per = _one_sequence(args.tokens, args.batch)
    T, qk = S * per, heads * d
    bufs = [torch.randn(T, 2 * qk + 2 * heads * dv, device=DEV).bfloat16() for _ in range(4)]
    decay = torch.linspace(0.9, 0.999, heads, device=DEV)
    state = torch.zeros(S, heads, d, dv, device=DEV)
    err = torch.zeros(1, dtype=torch.int32, device=DEV)

    def run(i):
        a = bufs[i % 4]
        ops.lightning_scan(a[:, :qk], a[:, qk:2 * qk], a[:, 2 * qk:2 * qk + heads * dv], decay, state, q_start, slots,
                           S, err, max_q_len=per)
    us = time_us(run, args.iters)
    moved = T * heads * (4 * d + 6 * dv) + 8 * S * heads * d * dv
    print(f"lightning_scan tokens {T} ({S} sequences) heads {heads} x {d} x {dv}: {us:.1f} us, {moved / us / 1e3:.0f} GB/s "
          f"of rows and state, {4.0 * T * heads * d * dv / us / 1e6:.2f} TFLOP/s float32")


def linear_state(args) -> None:
    """The matrix-state recurrence with fixed decays (--variant retention) or decays per channel (--variant hgrn2), its
    norm and gate, over one prompt portion, or one token of ``--batch`` sequences."""
    heads, d, dv, gated = args.heads, args.head_dim, args.v_dim or args.head_dim, args.variant != "hgrn2"
    q_start, _, slots, S, per = _one_sequence(args.tokens, args.batch)
    T = S * per
    bufs = [torch.randn(T, heads * (2 * d + (2 if gated else 1) * dv), device=DEV).bfloat16() for _ in range(4)]
    state = torch.zeros(S, heads, d, dv, device=DEV)
    err = torch.zeros(1, dtype=torch.int32, device=DEV)
    pos = torch.arange(T, dtype=torch.int32, device=DEV)
    if gated:
        kind = dict(decay=torch.linspace(0.9, 0.999, heads, device=DEV), gated=True, rotary_dim=d, k_scale=d ** -0.5,
                    inv_freq=torch.tensor([1e4 ** (-2.0 * i / d) for i in range(d // 2)], dtype=torch.float64, device=DEV))
    else:
        kind = dict(f_bias=torch.randn(heads * d, device=DEV) + 2, lower=torch.rand(heads * d, device=DEV) * 0.9,
                    norm=torch.ones(dv, device=DEV))

    def run(i):
        ops.linear_state_scan(bufs[i % 4], state, q_start, slots, S, 1e-5, err, positions=pos, max_q_len=per,
                              num_decode=S if per == 1 else 0, **kind)
    us = time_graph_us(run, args.iters) if per == 1 else time_us(run, args.iters)
    moved = T * heads * (4 * d + (6 if gated else 4) * dv) + 8 * S * heads * d * dv
    print(f"linear_state ({'retention' if gated else 'hgrn2'}) tokens {T} ({S} sequences) heads {heads} x {d} x {dv}: "
          f"{us:.1f} us, {moved / us / 1e3:.0f} GB/s of rows and state, {4.0 * T * heads * d * dv / us / 1e6:.2f} TFLOP/s")


def shared_key_attention(args) -> None:
    """Attention over shared key rows (mixed heads): a prompt of ``--tokens``, or (--tokens 1) one token of ``--batch``
    sequences at ``--context``; a key row has all kv heads' keys.  TFLOP/s over the visible pairs: as issued (every head
    against the whole row), and as the unmixed heads and their mixture would count."""
    H, G, d, dv, page, W, keep = args.heads, args.kv_heads, args.head_dim, args.v_dim or args.head_dim, args.page, args.window, args.keep_first
    decode = args.tokens == 1
    S, n, ctx = (args.batch, 1, args.context) if decode else (1, args.tokens, args.tokens)
    dkp, dvp = -(-G * d // 64) * 64, 64 if dv <= 64 else 128
    pages = -(-ctx // page)
    nb = 2 if decode else 1
    kc = [torch.randn(S * pages, 1, page, dkp, device=DEV).bfloat16() for _ in range(nb)]
    vc = [torch.randn(S * pages, 1, page, G * dvp, device=DEV).bfloat16() for _ in range(nb)]
    table = torch.arange(S * pages, dtype=torch.int32, device=DEV).view(S, pages)
    q = torch.randn(S * n, H * dkp, device=DEV).bfloat16()
    out = torch.empty(S * n, H * dv, dtype=torch.bfloat16, device=DEV)
    q_start = torch.arange(0, S * n + 1, n, dtype=torch.int32, device=DEV)
    lens = torch.full((S,), ctx, dtype=torch.int32, device=DEV)
    err = torch.zeros(1, dtype=torch.int32, device=DEV)

    def run(i):
        if decode or args.impl == "mma":
            ops.shared_key_attention_mma(q, out, kc[i % nb], vc[i % nb], table, q_start, lens, S, n, H, G, dv, W, keep, d ** -0.5,
                                         err, ctx)
        else:
            ops.shared_key_attention_tcgen05(q, out, kc[0], vc[0], table, q_start, lens, 0, S, S * n, H, G, dv, W, keep,
                                             d ** -0.5, err)
    us = time_graph_us(run, args.iters) if decode else time_us(run, args.iters)
    assert int(err.item()) == 0
    pairs = sum(min(p + 1, W + min(keep, max(0, p + 1 - W))) if W else p + 1 for p in range(ctx - n, ctx)) * S
    head = f"shared_key_attention tokens {S * n} context {ctx} heads {H}/{G} x {d}/{dv} window {W}+{keep}: {us:.1f} us"
    if decode:
        print(f"{head}, {pairs * 2.0 * G * (d + dv) / us / 1e3:.0f} GB/s of visible keys and values")
    else:
        print(f"{head}, {2e-6 * pairs * H * (dkp + dv) / us:.0f} TFLOP/s issued, {2e-6 * pairs * H * (d + H + dv) / us:.0f} unmixed")


def talking_prep(args) -> None:
    """The mixed queries, key rows and values of ``--tokens`` tokens."""
    H, G, d, dv, page, T = args.heads, args.kv_heads, args.head_dim, args.v_dim or args.head_dim, args.page, args.tokens
    dkp, dvp = -(-G * d // 64) * 64, 64 if dv <= 64 else 128
    pages = -(-T // page)
    kc, vc = (torch.zeros(pages, 1, page, w, device=DEV, dtype=torch.bfloat16) for w in (dkp, G * dvp))
    width = H * d + G * (d + dv)
    bufs = [torch.randn(T, width, device=DEV).bfloat16() for _ in range(4)]
    inv = torch.tensor([1e4 ** (-2.0 * i / d) for i in range(d // 2)], dtype=torch.float64, device=DEV)
    pos, err = torch.arange(T, dtype=torch.int32, device=DEV), torch.zeros(1, dtype=torch.int32, device=DEV)
    seq, table = torch.zeros(T, dtype=torch.int32, device=DEV), torch.arange(pages, dtype=torch.int32, device=DEV).view(1, -1)
    bias, talk = torch.randn(width, device=DEV), torch.randn(H, H, device=DEV)
    us = time_us(lambda i: ops.talking_prep(bufs[i % 4], pos, seq, bias, talk, inv, d, table, kc, vc, H, G, d, dv, err), args.iters)
    print(f"talking_prep tokens {T} heads {H}/{G} x {d}/{dv}: {us:.1f} us, "
          f"{2.0 * T * (width + H * dkp + dkp + G * dvp) / us / 1e3:.0f} GB/s")


def mlstm_scan(args) -> None:
    """The matrix memory's recurrence over one prompt portion, or one token of ``--batch`` sequences."""
    heads, d, dv = args.heads, args.head_dim, args.v_dim or args.head_dim
    q_start, _, slots, S, per = _one_sequence(args.tokens, args.batch)
    T, qk = S * per, heads * d
    bufs = [torch.randn(T, 2 * qk + 2 * heads * dv, device=DEV).bfloat16() for _ in range(4)]
    pre = torch.randn(T, 2 * heads, device=DEV) * 2
    gates = torch.empty_like(pre)
    bias = torch.zeros(heads, device=DEV)
    state = torch.zeros(S, heads, ops.mlstm_state_size(d, dv), device=DEV)
    err = torch.zeros(1, dtype=torch.int32, device=DEV)

    def run(i):
        a = bufs[i % 4]
        gates.copy_(pre)                 # (the call turns the pre-activations into log gates in place)
        ops.mlstm_scan(a[:, :qk], a[:, qk:2 * qk], a[:, 2 * qk:2 * qk + heads * dv], gates, bias, bias, 10.0, d ** -0.5,
                       state, q_start, slots, S, heads, d, dv, err, q_lens=[per] * S)
    us = time_us(run, args.iters)
    moved = T * heads * (4 * d + 6 * dv) + 8 * S * heads * d * dv
    print(f"mlstm_scan tokens {T} ({S} sequences) heads {heads} x {d} x {dv}: {us:.1f} us (with a copy of the gates), "
          f"{moved / us / 1e3:.0f} GB/s of rows and state, {4.0 * T * heads * d * dv / us / 1e6:.2f} TFLOP/s float32")


def channel_delta(args) -> None:
    """The gated delta rule over one prompt portion, or one token of ``--batch`` sequences."""
    heads, d, dv = args.heads, args.head_dim, args.v_dim or args.head_dim
    q_start, _, slots, S, per = _one_sequence(args.tokens, args.batch)
    T = S * per
    bufs = [torch.randn(T, heads * (2 * d + dv), device=DEV).bfloat16() for _ in range(4)]
    step, b = torch.randn(T, heads * d, device=DEV), torch.randn(T, heads, device=DEV)
    dt_bias, a_log = torch.randn(heads * d, device=DEV) - 3, torch.randn(heads, device=DEV)
    state = torch.zeros(S, heads, d, dv, device=DEV)
    err = torch.zeros(1, dtype=torch.int32, device=DEV)

    def run(i):
        ops.channel_delta_scan(bufs[i % 4], step, b, dt_bias, a_log, 1e-6, state, q_start, slots, S, heads, heads, d, dv,
                               err, max_q_len=per)
    us = time_us(run, args.iters)
    moved = T * heads * (4 * d + 2 * dv + 4 * d + 4 * dv + 4) + 8 * S * heads * d * dv
    print(f"channel_delta tokens {T} ({S} sequences) heads {heads} x {d} x {dv}: {us:.1f} us, {moved / us / 1e3:.0f} GB/s "
          f"of rows and state, {6.0 * T * heads * d * dv / us / 1e6:.2f} TFLOP/s of the recurrence")


def channel_delta_step(args) -> None:
    """One token of ``--batch`` sequences through the delta-rule layer's kernel, between its two products."""
    heads, d, dv, H, r = args.heads, args.head_dim, args.v_dim or args.head_dim, args.hidden, 128
    S, ch = args.batch, heads * (2 * d + dv)
    bf = lambda *shape: (torch.randn(*shape, device=DEV) * 0.1).bfloat16()
    a, x = bf(S, ch + 2 * r), bf(S, H)
    w = {"b": bf(heads, H), "a2": bf(heads * d, r), "g2": bf(heads * dv, r), "conv": bf(ch, 4),
         "dt_bias": torch.randn(heads * d, device=DEV) - 3, "a_log": torch.randn(heads, device=DEV),
         "norm": torch.ones(heads * dv, device=DEV)}
    n = max(1, (256 << 20) // (S * heads * d * dv * 4))             # states that together exceed L2
    tails = torch.zeros(S, 3, ch, device=DEV)
    states = [torch.zeros(S, heads, d, dv, device=DEV) for _ in range(n + 1)]
    slots, err = torch.arange(S, dtype=torch.int32, device=DEV), torch.zeros(1, dtype=torch.int32, device=DEV)

    def run(i):
        ops.channel_delta_step(a, None, x, w, ch, ch + r, 4, 1e-6, 1e-6, tails, states[i % (n + 1)], slots, heads, heads,
                               d, dv, err)
    us = time_graph_us(run, args.iters)
    print(f"channel_delta_step {S} sequences heads {heads} x {d} x {dv}: {us:.1f} us, "
          f"{8 * S * heads * d * dv / us / 1e3:.0f} GB/s of state")


def ssd_scan(args) -> None:
    """The state-space recurrence over one prompt portion, or one token of ``--batch`` sequences."""
    heads, p, n, groups = args.heads, args.head_dim, args.state, args.groups
    q_start, _, slots, S, per = _one_sequence(args.tokens, args.batch)
    T = S * per
    bufs = [torch.randn(T, heads * p + 2 * groups * n, device=DEV).bfloat16() for _ in range(4)]
    dt, vec = torch.randn(T, heads, device=DEV), lambda: torch.randn(heads, device=DEV)
    dt_bias, a_log, skip = vec() - 3, vec(), vec()
    state = torch.zeros(S, heads, n, p, device=DEV)
    err = torch.zeros(1, dtype=torch.int32, device=DEV)

    def run(i):
        ops.ssd_scan(bufs[i % 4], dt, dt_bias, a_log, skip, state, q_start, slots, S, heads, groups, n, p, err, max_q_len=per)
    us = time_us(run, args.iters)
    moved = 2 * bufs[0].numel() + T * heads * (4 * p + 4) + 8 * S * heads * n * p
    print(f"ssd_scan tokens {T} ({S} sequences) heads {heads} x {n} x {p}: {us:.1f} us, {moved / us / 1e3:.0f} GB/s "
          f"of rows and state, {4.0 * T * heads * n * p / us / 1e6:.2f} TFLOP/s of the recurrence")


def selective_scan(args) -> None:
    """The convolution and the selective recurrence over one prompt portion, or one token of ``--batch`` sequences."""
    E, N, R = args.channels, args.state, max(1, args.channels // 32)
    q_start, token_seq, slots, S, per = _one_sequence(args.tokens, args.batch)
    T = S * per
    xz = [torch.randn(T, 2 * E, device=DEV).bfloat16() for _ in range(4)]
    proj = torch.randn(T, R + 2 * N, device=DEV).bfloat16()
    dt_raw = torch.randn(T, E, device=DEV)
    small = lambda *shape: torch.randn(*shape, device=DEV).bfloat16()
    w_conv, b_conv, dt_b, a_log, dskip = small(E, 4), small(E), small(E), small(E, N), small(E)
    state, tail = torch.zeros(S, N, E, device=DEV), torch.zeros(S, 3, E, device=DEV)
    err = torch.zeros(1, dtype=torch.int32, device=DEV)
    keep = {}

    def conv(i):
        keep["c"] = ops.causal_conv(xz[i % 4][:, :E], w_conv, b_conv, tail, q_start, token_seq, slots, S, per > 1, err)

    def scan(i):
        ops.selective_scan(keep["c"], dt_raw, dt_b, proj, R, R + N, a_log, dskip, xz[i % 4][:, E:], state, q_start, slots,
                           S, err, max_q_len=per)
    us = time_us(conv, args.iters)
    print(f"causal_conv tokens {T} channels {E} taps 4: {us:.1f} us, {4.0 * T * E / us / 1e3:.0f} GB/s")
    us = time_us(scan, args.iters)
    print(f"selective_scan tokens {T} ({S} sequences) channels {E} states {N}: {us:.1f} us, "
          f"{(10.0 * T * E + 8.0 * S * N * E) / us / 1e3:.0f} GB/s of rows and state")


def streams(args) -> None:
    """The write-back into all residual streams with the next read and its norm."""
    S, T, H = args.streams, args.tokens, args.hidden
    xs = [torch.randn(S, T, H, device=DEV) for _ in range(3)]
    y = torch.randn(T, H, device=DEV).bfloat16()
    vec = lambda n: torch.randn(n, device=DEV)
    mix, write, read, scale = torch.randn(S, S, device=DEV), vec(S), vec(S), vec(H).bfloat16()
    norm = (torch.tensor([0.5], device=DEV), vec(H).bfloat16(), vec(H).bfloat16())

    def run(i):
        ops.streams_write(xs[i % 3], y, scale, mix, write, next_read=read, norm=norm)
    us = time_us(run, args.iters)
    print(f"streams_write {S} streams x {T} x {H}: {us:.1f} us, {(8.0 * S + 4.0) * T * H / us / 1e3:.0f} GB/s")


def main(argv=None) -> int:
    p = argparse.ArgumentParser(prog="python -m rllm_b200.kernels.microbench", description=__doc__.split("\n\n")[0])
    p.add_argument("kernel", choices=["attention_decode", "attention_prefill", "gemm_small_m", "gemm_tcgen05",
                                      "latent_attention", "routed_experts", "lightning_scan", "selective_scan",
                                      "streams", "mlstm_scan", "channel_delta", "channel_delta_step", "ssd_scan",
                                      "linear_state", "shared_key_attention", "talking_prep"])
    p.add_argument("--batch", type=int, default=8)
    p.add_argument("--context", type=int, default=4096)
    p.add_argument("--tokens", type=int, default=2048)
    p.add_argument("--rows", type=int, default=8)
    p.add_argument("--iters", type=int, default=20)
    p.add_argument("--heads", type=int, default=32)
    p.add_argument("--kv-heads", type=int, default=8)
    p.add_argument("--head-dim", type=int, default=64)
    p.add_argument("--hidden", type=int, default=2048)
    p.add_argument("--intermediate", type=int, default=8192)
    p.add_argument("--page", type=int, default=16)
    p.add_argument("--kv-rank", type=int, default=512, help="latent_attention: values of a cached row")
    p.add_argument("--rot-dim", type=int, default=64, help="latent_attention: the rows' rotated key part")
    p.add_argument("--window", type=int, default=0, help="the attention kernels: keys a query sees (0: all)")
    p.add_argument("--keep-first", type=int, default=0, help="attention_*: with a window, first keys that stay visible")
    p.add_argument("--chunk", type=int, default=0, help="attention_*: a query sees the keys of its own chunk")
    p.add_argument("--softcap", type=float, default=0.0, help="attention_*: the tanh cap of the scaled scores")
    p.add_argument("--sinks", action="store_true", help="attention_*: one more term a head in the denominator")
    p.add_argument("--slopes", type=float, default=0.0,
                   help="attention_*: a distance bias with the slopes 2^(-x (h + 1) / heads) (0: none)")
    p.add_argument("--gate", choices=["head", "element"], default=None, help="attention_*: a sigmoid gate on the result")
    p.add_argument("--v-dim", type=int, default=0, help="lightning_scan: a value head's size (0: --head-dim)")
    p.add_argument("--channels", type=int, default=4096, help="selective_scan: inner channels")
    p.add_argument("--state", type=int, default=16, help="selective_scan: states a channel; ssd_scan: states a head's column")
    p.add_argument("--groups", type=int, default=1, help="ssd_scan: groups of heads that share B and C")
    p.add_argument("--streams", type=int, default=4, help="streams: residual streams")
    p.add_argument("--experts", type=int, default=32)
    p.add_argument("--top", type=int, default=4)
    p.add_argument("--variant", choices=["plain", "residual", "rstd", "retention", "hgrn2"], default="plain",
                   help="gemm_small_m: which epilogue / operand form; linear_state: which recurrence")
    p.add_argument("--only", choices=["qkv", "o_proj", "gate_up", "down"], default=None,
                   help="gemm_small_m, gemm_tcgen05: this projection alone")
    p.add_argument("--impl", choices=["mma", "tcgen05"], default="mma",
                   help="attention_prefill: the mma.sync kernel or the tcgen05 kernel")
    args = p.parse_args(argv)
    if not torch.cuda.is_available():
        print("microbench needs a CUDA device", file=sys.stderr)
        return 1
    {"attention_decode": attention_decode, "attention_prefill": attention_prefill,
     "gemm_small_m": gemm_small_m, "gemm_tcgen05": gemm_tcgen05, "latent_attention": latent_attention,
     "routed_experts": routed_experts, "lightning_scan": lightning_scan, "selective_scan": selective_scan,
     "streams": streams, "mlstm_scan": mlstm_scan, "channel_delta": channel_delta,
     "channel_delta_step": channel_delta_step, "linear_state": linear_state,
     "shared_key_attention": shared_key_attention, "talking_prep": talking_prep,
     "ssd_scan": ssd_scan}[args.kernel](args)
    return 0


if __name__ == "__main__":
    sys.exit(main())
