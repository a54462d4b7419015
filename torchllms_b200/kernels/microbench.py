"""Kernels timed alone, at the shapes of the Llama-3.1-8B layers by default.

    python -m torchllms_b200.kernels.microbench attention_decode
    python -m torchllms_b200.kernels.microbench attention_prefill --lengths 2048,8192 --impls mma,prefill
    python -m torchllms_b200.kernels.microbench gemm
    python -m torchllms_b200.kernels.microbench elementwise --tokens 2048
    python -m torchllms_b200.kernels.microbench peaks
    python -m torchllms_b200.kernels.microbench selective_scan --tokens 2048 --channels 4096 --state 16
    python -m torchllms_b200.kernels.microbench attention_options --length 2048 --span 1024
    python -m torchllms_b200.kernels.microbench rows --tokens 2048
    python -m torchllms_b200.kernels.microbench delta --tokens 2048 --heads 16

Every case is timed with CUDA events after warm-up.  Memory-bound kernels run inside a CUDA
graph over several copies of their operands (more than the 126 MB of L2 together), so that a
launch does not find its inputs in L2 from the one before.  Figures go to standard output; the
summaries under ``profiles/`` quote them.
"""

from __future__ import annotations

import argparse
from typing import Callable, List

import torch

from . import get_ops

HEADS, KV_HEADS, HEAD_DIM, WIDTH, HIDDEN, VOCAB = 32, 8, 128, 4096, 14336, 128256


def _time(fn: Callable[[], None], reps: int) -> float:
    """Microseconds per call of ``fn``."""
    for _ in range(3):
        fn()
    torch.cuda.synchronize()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record()
    for _ in range(reps):
        fn()
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) * 1e3 / reps


def _graphed(calls: List[Callable[[], None]]) -> Callable[[], None]:
    """One graph that makes every call once (they were warmed up before)."""
    for c in calls:
        c()
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g):
        for c in calls:
            c()
    return g.replay


def attention_decode(args) -> None:
    """Decode attention (kernel and merge) for B requests of one context length."""
    ops = get_ops()
    copies = 8
    for spec in args.shapes.split(","):
        B, ctx = (int(x) for x in spec.split("x"))
        for page in (int(x) for x in args.pages.split(",")):
            torch.manual_seed(0)
            blocks = -(-ctx // page)
            table = torch.zeros(B, args.max_len // page, dtype=torch.int32)
            table[:, :blocks] = torch.randperm(B * blocks).view(B, blocks).int()
            table = table.cuda()
            caches = [(torch.randn(B * blocks, KV_HEADS, page, HEAD_DIM, device="cuda", dtype=torch.bfloat16),
                       torch.randn(B * blocks, KV_HEADS, page, HEAD_DIM, device="cuda", dtype=torch.bfloat16))
                      for _ in range(copies)]
            q = torch.randn(B, HEADS, HEAD_DIM, device="cuda", dtype=torch.bfloat16)
            q_start = torch.arange(B + 1, dtype=torch.int32, device="cuda")
            kv_len = torch.full((B,), ctx, dtype=torch.int32, device="cuda")
            out = torch.empty_like(q)

            def layer(i):
                k, v = caches[i]
                return lambda: ops.paged_attention(q, k, v, table, q_start, kv_len, n_seqs=B, max_q_len=1,
                                                   max_kv_len=args.max_len, scale=HEAD_DIM ** -0.5, window=None,
                                                   page_size=page, impl="decode", out=out)
            us = _time(_graphed([layer(i) for i in range(copies)]), 10) / copies
            nbytes = B * ctx * KV_HEADS * HEAD_DIM * 2 * 2
            print(f"attention_decode {B:3d} x {ctx:6d} page {page:3d}: {us:7.1f} us  {nbytes / us / 1e6:5.2f} TB/s")


def attention_prefill(args) -> None:
    """Causal attention of one whole prompt of L tokens."""
    ops = get_ops()
    page = 16
    for L in (int(x) for x in args.lengths.split(",")):
        torch.manual_seed(0)
        blocks = -(-L // page)
        table = torch.randperm(blocks).int().view(1, blocks).cuda()
        k = torch.randn(blocks, KV_HEADS, page, HEAD_DIM, device="cuda", dtype=torch.bfloat16)
        v = torch.randn(blocks, KV_HEADS, page, HEAD_DIM, device="cuda", dtype=torch.bfloat16)
        q = torch.randn(L, HEADS, HEAD_DIM, device="cuda", dtype=torch.bfloat16)
        q_start = torch.tensor([0, L], dtype=torch.int32, device="cuda")
        kv_len = torch.tensor([L], dtype=torch.int32, device="cuda")
        out = torch.empty_like(q)
        flops = 4 * HEADS * HEAD_DIM * L * (L + 1) / 2
        for impl in args.impls.split(","):
            def call():
                ops.paged_attention(q, k, v, table, q_start, kv_len, n_seqs=1, max_q_len=L, max_kv_len=L,
                                    scale=HEAD_DIM ** -0.5, window=None, page_size=page, impl=impl, out=out)
            # ten launches in one graph: a short prompt's kernel takes less than the host needs to launch it
            us = _time(_graphed([call] * 10), 5) / 10
            ops.check_status()
            print(f"attention_prefill L {L:6d} {impl:8s}: {us:9.1f} us  {flops / us / 1e6:7.1f} TFLOP/s")


def gemm(args) -> None:
    """The projections of a decode step: x[M, K] . w[N, K]^T, the tcgen05 kernel beside torch.mm."""
    ops = get_ops()
    shapes = [("wo", WIDTH, WIDTH), ("w1;w3", 2 * HIDDEN, WIDTH), ("w2", WIDTH, HIDDEN),
              ("wq;wk;wv", (HEADS + 2 * KV_HEADS) * HEAD_DIM, WIDTH), ("head", VOCAB, WIDTH)]
    for M in (int(x) for x in args.rows.split(",")):
        for name, N, K in shapes:
            copies = max(2, int(300e6 // (N * K * 2)) + 1)
            ws = [torch.randn(N, K, device="cuda", dtype=torch.bfloat16) * 0.02 for _ in range(copies)]
            x = torch.randn(M, K, device="cuda", dtype=torch.bfloat16)
            ours = _time(_graphed([(lambda w=w: ops.gemm_tcgen05(x, w, torch.float32)) for w in ws]), 5) / copies
            lib = _time(_graphed([(lambda w=w: torch.mm(x, w.t())) for w in ws]), 5) / copies
            ops.check_status()
            print(f"gemm M {M:3d} {name:9s} {N:6d} x {K:5d}: tcgen05 {ours:7.1f} us ({N * K * 2 / ours / 1e6:4.2f} TB/s)   "
                  f"torch.mm {lib:7.1f} us")


def elementwise(args) -> None:
    """Residual add + RMSNorm and SwiGLU over T tokens (bfloat16 activations, float32 stream)."""
    ops = get_ops()
    T, copies = args.tokens, 6
    hs = [torch.randn(T, WIDTH, device="cuda") for _ in range(copies)]
    ds = [torch.randn(T, WIDTH, device="cuda", dtype=torch.bfloat16) for _ in range(copies)]
    w = torch.ones(WIDTH, device="cuda")
    us = _time(_graphed([(lambda i=i: ops.rmsnorm(hs[i], ds[i], w, 1e-5, torch.bfloat16)) for i in range(copies)]), 5) / copies
    print(f"rmsnorm T {T}: {us:7.1f} us  {T * WIDTH * 12 / us / 1e6:5.2f} TB/s")
    us = _time(_graphed([(lambda i=i: ops.rmsnorm(hs[i], ds[i], w, 1e-5, torch.bfloat16, deferred=True)) for i in range(copies)]), 5) / copies
    print(f"rmsnorm T {T}, scale deferred: {us:7.1f} us  {T * WIDTH * 12 / us / 1e6:5.2f} TB/s")
    # rotation of q and k and the write of k and v into pages, as a prompt portion of T tokens needs it
    row, page = (HEADS + 2 * KV_HEADS) * HEAD_DIM, 16
    qkvs = [torch.randn(T, row, device="cuda", dtype=torch.bfloat16) for _ in range(copies)]
    table = torch.randn(T, HEAD_DIM // 2, 2, device="cuda")
    positions = torch.arange(T, dtype=torch.int32, device="cuda")
    slots = torch.randperm(T, device="cuda").int()
    kp = torch.empty(-(-T // page), KV_HEADS, page, HEAD_DIM, device="cuda", dtype=torch.bfloat16)
    vp = torch.empty_like(kp)
    us = _time(_graphed([(lambda i=i: ops.rope_kv_write(qkvs[i], positions, table, n_heads=HEADS, n_kv_heads=KV_HEADS,
                                                        head_dim=HEAD_DIM, interleaved=True, k_pages=kp, v_pages=vp,
                                                        slot_mapping=slots, page_size=page)) for i in range(copies)]), 5) / copies
    print(f"rope + cache write T {T}: {us:7.1f} us  {T * row * 4 / us / 1e6:5.2f} TB/s")
    gus = [torch.randn(T, 2 * HIDDEN, device="cuda", dtype=torch.bfloat16) for _ in range(copies)]
    us = _time(_graphed([(lambda i=i: ops.swiglu(gus[i])) for i in range(copies)]), 5) / copies
    print(f"swiglu  T {T}: {us:7.1f} us  {T * HIDDEN * 6 / us / 1e6:5.2f} TB/s")


def peaks(args) -> None:
    """What this GPU gives a plain copy and a library bfloat16 product: the denominators of a roofline."""
    n = 1 << 30
    src = torch.empty(n, dtype=torch.int32, device="cuda")
    dst = torch.empty_like(src)
    us = _time(lambda: dst.copy_(src), 10)
    print(f"copy of {4 * n / 1e9:.1f} GB: {us:9.1f} us  {2 * 4 * n / us / 1e6:5.2f} TB/s (read + write)")
    m = 8192
    a = torch.randn(m, m, device="cuda", dtype=torch.bfloat16)
    b = torch.randn(m, m, device="cuda", dtype=torch.bfloat16)
    us = _time(lambda: torch.mm(a, b), 10)
    print(f"library product {m}^3 bfloat16, ten in a row: {us:9.1f} us  {2 * m ** 3 / us / 1e6:7.1f} TFLOP/s")
    us = _time(lambda: torch.mm(a, b), 400)
    print(f"library product {m}^3 bfloat16, four hundred in a row: {us:9.1f} us  {2 * m ** 3 / us / 1e6:7.1f} TFLOP/s")


def selective_scan(args) -> None:
    """The selective scan alone: one prompt portion of --tokens tokens, and a decode step of 8 requests."""
    ops = get_ops()
    T, C, N = args.tokens, args.channels, args.state
    torch.manual_seed(0)
    dev, bf = "cuda", torch.bfloat16
    for label, lens in ((f"portion of {T}", [T]), ("decode step of 8", [1] * 8)):
        n_tok = sum(lens)
        copies = max(1, min(8, (160 << 20) // max(1, n_tok * C * 8)))
        sets = []
        for _ in range(copies):
            xz = torch.randn(n_tok, 2 * C, device=dev).to(bf)
            dt = torch.randn(n_tok, C, device=dev).to(bf)
            bc = torch.randn(n_tok, 2 * N, device=dev).to(bf)
            sets.append((xz, dt, bc))
        A = -torch.exp(torch.randn(C, N, device=dev))
        D, bias = torch.randn(C, device=dev), torch.randn(C, device=dev)
        state = torch.zeros(len(lens), C, N, device=dev)
        q_start = torch.tensor([0] + list(torch.tensor(lens).cumsum(0)), dtype=torch.int32, device=dev)
        slot = torch.arange(len(lens), dtype=torch.int32, device=dev)
        fresh = torch.zeros(len(lens), dtype=torch.int32, device=dev)
        calls = [(lambda xz=xz, dt=dt, bc=bc: ops.selective_scan(xz[:, :C], dt, bc[:, :N], bc[:, N:], xz[:, C:], A, D, bias, state, q_start,
                                                                slot, fresh, n_seqs=len(lens), max_q_len=max(lens), out_dtype=bf))
                 for xz, dt, bc in sets]
        us = _time(_graphed(calls), 20) / copies
        moved = n_tok * C * 2 * 4 + n_tok * N * 4 + 2 * len(lens) * C * N * 4
        print(f"selective_scan {label}, {C} channels x {N}: {us:8.1f} us  {moved / us / 1e3:7.1f} GB/s of inputs, outputs and state")


def attention_options(args) -> None:
    """Attention with options (16 heads over 4, 128 wide): one prompt of --length tokens and a decode step of 8 requests of that
    length, over all keys, behind a window and inside chunks of --span, with softmax and with sigmoid weights."""
    ops = get_ops()
    H, G, d, page, dev, bf = 16, 4, 128, 16, "cuda", torch.bfloat16
    sinks, bias = torch.zeros(H, device=dev), torch.randn(H, device=dev) - 4.0
    kinds = (("softmax, cap, sinks", dict(softcap=30.0, sinks=sinks)), ("softmax, cap, sinks, window", dict(softcap=30.0, sinks=sinks, window=args.span)),
             ("softmax, sinks, chunks", dict(sinks=sinks, chunk=args.span)),
             ("sigmoid, cap, window", dict(softcap=30.0, weights="sigmoid", score_bias=bias, window=args.span)))
    for label, lens, past in ((f"prompt of {args.length}", [args.length], 0), (f"decode step of 8 x {args.length}", [1] * 8, args.length - 1)):
        T, B, kv = sum(lens), len(lens), past + max(lens)
        blocks = -(-kv // page)
        copies = max(1, min(16, (200 << 20) // (B * blocks * G * page * d * 4)))
        pages = [[torch.randn(B * blocks, G, page, d, device=dev).to(bf) for _ in range(copies)] for _ in "kv"]
        table = torch.arange(B * blocks, dtype=torch.int32, device=dev).view(B, blocks)
        q = torch.randn(T, H, d, device=dev).to(bf)
        q_start = torch.tensor([0] + list(torch.tensor(lens).cumsum(0)), dtype=torch.int32, device=dev)
        kv_len = torch.full((B,), kv, dtype=torch.int32, device=dev)
        for name, kw in kinds:
            kw = dict({"window": None}, **kw)
            us = _time(_graphed([(lambda i=i: ops.paged_attention(
                q, pages[0][i], pages[1][i], table, q_start, kv_len, n_seqs=B, max_q_len=max(lens), max_kv_len=kv, scale=d ** -0.5,
                page_size=page, **kw)) for i in range(copies)]), 5) / copies
            seen = sum(min(p + 1, kw["window"]) if kw["window"] else p % kw["chunk"] + 1 if kw.get("chunk") else p + 1
                       for n in lens for p in range(past, past + n))
            span = kw["window"] or kw.get("chunk") or kv
            print(f"{label}: {name}: {us:8.1f} us  {seen * H * d * 4 / us / 1e6:7.1f} TFLOP/s  "
                  f"{B * min(kv, span) * G * d * 4 / us / 1e3:7.1f} GB/s of keys and values")


def rows(args) -> None:
    """What stands between a layer's products, at width 2,048 (16 heads over 4, 128 wide, 64 rotated): norms, stores, sums
    and activations, over --tokens rows of bfloat16 and over 8 rows of four float32 partial sums."""
    ops = get_ops()
    H, G, d, D, page, dev, bf = 16, 4, 128, 2048, 16, "cuda", torch.bfloat16

    def line(name: str, calls, moved: float) -> None:
        us = _time(_graphed(calls), 5) / len(calls)
        print(f"{name}: {us:7.1f} us  {moved / us / 1e3:7.1f} GB/s")

    for T, splits, copies in ((args.tokens, 1, 4), (8, 4, 64)):
        def data(width):
            return [torch.randn(T, width, device=dev).to(bf) if splits == 1 else torch.randn(splits, T, width, device=dev) for _ in range(copies)]
        in_bytes = 2 if splits == 1 else 4 * splits
        positions = torch.arange(T, dtype=torch.int32, device=dev)
        table = torch.randn(max(T, 64), 32, 2, device=dev)
        kp = torch.zeros(-(-T // page), G, page, d, device=dev, dtype=bf)
        vp = torch.zeros_like(kp)
        store = dict(n_q_heads=H, n_k_heads=G, head_dim=d, v_head_dim=d, rot_dims=64, interleaved=False, n_extra=0, k_pages=kp, v_pages=vp,
                     slot_mapping=positions, page_size=page, out_dtype=bf)
        width = (H + 2 * G) * d
        bias, qn, kn = torch.randn(width, device=dev), torch.randn(H * d, device=dev), torch.randn(G * d, device=dev)
        qkv, qk = data(width), data((H + G) * d)
        moved = T * (width * in_bytes + width * 2)
        line(f"rope_store, {T} rows", [(lambda x=x: ops.rope_store(x, positions, table, n_v_heads=G, bias=bias, **store)) for x in qkv], moved)
        line(f"norm_rope_store, heads normed, {T} rows",
             [(lambda x=x: ops.norm_rope_store(x, positions, table, bias=bias, qk_head_norm=True, v_head_norm=True, eps=1e-6, **store)) for x in qkv], moved)
        line(f"norm_rope_store, rows normed, values are keys, {T} rows",
             [(lambda x=x: ops.norm_rope_store(x, positions, table, values_are_keys=True, q_norm=qn, k_norm=kn, eps=1e-6, **store)) for x in qk],
             T * ((H + G) * d * in_bytes + width * 2))
        hs, deltas = [torch.randn(T, D, device=dev) for _ in range(copies)], data(D)
        w, ls = torch.randn(D, device=dev), torch.randn(D, device=dev)
        moved = T * D * (10 + in_bytes)
        line(f"rmsnorm of a sum, {T} rows", [(lambda i=i: ops.rmsnorm(hs[i], deltas[i], w, 1e-6, bf)) for i in range(copies)], moved)
        line(f"rmsnorm of a scaled sum, 4 groups, {T} rows",
             [(lambda i=i: ops.rmsnorm(hs[i], deltas[i], w, 1e-6, bf, groups=4, delta_scale=ls)) for i in range(copies)], moved)
        line(f"norm_add and norm, {T} rows",
             [(lambda i=i: ops.norm_add(hs[i], deltas[i], w, 1e-6, bf, then_weight=w, then_eps=1e-6)) for i in range(copies)], moved)
        line(f"stream_join, {T} rows", [(lambda i=i: ops.stream_join(hs[i], deltas[i], ls, hs[(i + 1) % copies], w, out_dtype=bf)) for i in range(copies)],
             T * D * (16 + in_bytes))
        line(f"stream_inject, {T} rows", [(lambda i=i: ops.stream_inject(hs[i], hs[(i + 1) % copies], w)) for i in range(copies)], T * D * 12)
    n = 4 * args.tokens
    us = [torch.randn(n, D, device=dev).to(bf) for _ in range(4)]
    for act in ("gelu", "gelu_tanh", "silu", "relu2"):
        line(f"{act}, {n} rows", [(lambda u=u: ops.activation(u, act)) for u in us], n * D * 4)
    gu = [torch.randn(n, 2 * D, device=dev).to(bf) for _ in range(2)]
    line(f"clamped gate, {n} rows", [(lambda u=u: ops.glu(u, limit=7.0, alpha=1.702, up_offset=1.0)) for u in gu], n * D * 6)


def delta(args) -> None:
    """Mixers behind short convolutions (4 taps, heads of 128, a quarter as many shared heads): what follows the input
    projection, the matrix recurrences and the head norm, for one prompt of --tokens and for 8 decoded tokens (whose
    projections arrive as two float32 partial sums).  GB/s of the algorithmic bytes."""
    from ..parts.rope import precise_rotary_table
    ops = get_ops()
    H, d, page, taps, low, dev, bf = args.heads, 128, 16, 4, 256, "cuda", torch.bfloat16
    G, f32 = max(H // 4, 1), torch.float32
    i32 = lambda xs: torch.tensor(xs, dtype=torch.int32, device=dev)

    def line(name: str, calls, moved: float) -> None:
        us = _time(_graphed(calls), 5) / len(calls)
        print(f"{name}: {us:7.1f} us  {moved / us / 1e3:7.1f} GB/s")

    left, right = (2 * H + 2 * G) * d, 2 * G * d + H * d + H + low
    for T, B, splits, copies in ((args.tokens, 1, 1, 4), (8, 8, 2, 16)):
        rows = [torch.randn(splits, T, left + right, device=dev).to(bf if splits == 1 else f32) for _ in range(copies)]
        rows = [r if splits > 1 else r[0] for r in rows]
        each = 2 if splits == 1 else 4 * splits
        at = (i32([b * T // B for b in range(B + 1)]), i32(list(range(B))), i32([int(B == 1)] * B))
        how = dict(n_seqs=B, max_q_len=T // B)
        positions = torch.arange(T, dtype=torch.int32, device=dev)
        kp = torch.zeros(-(-T // page), G, page, d, device=dev, dtype=bf)
        vp, table = torch.zeros_like(kp), precise_rotary_table(d, 1e6, 1.0, max(T, 64), dev)
        n_left, n_right = (H + 2 * G) * d, (H + 2 * G) * d
        wl, wr = torch.randn(taps, n_left, device=dev), torch.randn(taps, n_right, device=dev)
        sl, sr = torch.zeros(B, taps - 1, n_left, device=dev), torch.zeros(B, taps - 1, n_right, device=dev)
        store = dict(n_q_heads=H, n_k_heads=G, head_dim=d, v_head_dim=d, rot_dims=d, n_extra=H * d, k_pages=kp, v_pages=vp,
                     slot_mapping=positions, page_size=page, out_dtype=bf)
        line(f"conv_rope_store, {T} rows", [(lambda r=r: ops.conv_rope_store(r[..., :left], wl, sl, positions, table, *at, **how, **store)) for r in rows],
             T * left * (each + 2))
        prep = dict(n_qk_heads=G, head_dim=d, n_v=H * d, n_small=H, n_low=low, low_pad=low, q_scale=d ** -0.5, unit_eps=1e-6, out_dtype=bf)
        line(f"delta_prep, {T} rows", [(lambda r=r: ops.delta_prep(r[..., left:], wr, sr, *at, **how, **prep)) for r in rows],
             T * (right * each + 2 * G * d * 4 + (H * d + H + low) * 2))
        if splits == 1:
            sc = torch.zeros(B, taps - 1, n_right, device=dev)
            line(f"short_conv of as many channels, {T} rows",
                 [(lambda r=r: ops.short_conv(r[:, left:left + n_right], wr.t().contiguous(), sc, *at, **how, activation="silu", residual=False, out_dtype=bf))
                  for r in rows], T * n_right * 4)
        q, k = torch.randn(T, G * d, device=dev) * d ** -0.5, torch.nn.functional.normalize(torch.randn(T, G, d, device=dev), dim=-1).flatten(1)
        v, beta, z = torch.randn(T, H * d, device=dev).to(bf), torch.randn(T, H, device=dev).to(bf), torch.randn(T, 2 * H * d, device=dev).to(bf)
        states = [torch.zeros(B, H, d, d, device=dev) for _ in range(copies)]
        rate, bias = torch.rand(H, device=dev), torch.randn(H * d, device=dev) - 3.0
        moved = T * (2 * G * d * 4 + H * d * 6) + B * H * d * d * (8 if B > 1 else 4)
        line(f"recurrence, a decay per channel, {T} tokens of {B}",
             [(lambda s=s: ops.linear_recurrence(q, k, v, s, *at, **how, beta_logits=beta, decay_logits=z[:, :H * d], decay_rate=rate, decay_bias=bias))
              for s in states], moved + T * H * d * 2)
        line(f"recurrence, a decay per head, {T} tokens of {B}",
             [(lambda s=s: ops.linear_recurrence(q, k, v, s, *at, **how, beta_logits=beta, decay_logits=z[:, :H], decay_rate=rate, decay_bias=bias[:H]))
              for s in states], moved)
        line(f"recurrence, fixed decays, {T} tokens of {B}",
             [(lambda s=s: ops.linear_recurrence(q, k, v, s, *at, **how, decay=rate)) for s in states], moved)
        os, outs = [torch.randn(T, H * d, device=dev) for _ in range(copies)], torch.empty(T, 2 * H * d, device=dev, dtype=bf)
        w = torch.randn(d, device=dev)
        line(f"head_norm_gate, {T} rows", [(lambda o=o: ops.head_norm_gate(o, z[:, H * d:], w, 1e-6, head_dim=d, out_dtype=bf, activation="sigmoid",
                                                                           out=outs[:, H * d:])) for o in os], T * H * d * 8)


def main(argv=None) -> None:
    parser = argparse.ArgumentParser(description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    sub = parser.add_subparsers(dest="case", required=True)
    p = sub.add_parser("attention_decode")
    p.add_argument("--shapes", default="8x2048,64x2048,8x8192,32x8192,1x2048,1x8192", help="requests x context, comma separated")
    p.add_argument("--pages", default="16,64")
    p.add_argument("--max-len", type=int, default=8192)
    p.set_defaults(run=attention_decode)
    p = sub.add_parser("attention_prefill")
    p.add_argument("--lengths", default="2048,8192")
    p.add_argument("--impls", default="mma,prefill")
    p.set_defaults(run=attention_prefill)
    p = sub.add_parser("gemm")
    p.add_argument("--rows", default="8,64")
    p.set_defaults(run=gemm)
    p = sub.add_parser("peaks")
    p.set_defaults(run=peaks)
    p = sub.add_parser("selective_scan")
    p.add_argument("--tokens", type=int, default=2048)
    p.add_argument("--channels", type=int, default=4096)
    p.add_argument("--state", type=int, default=16)
    p.set_defaults(run=selective_scan)
    p = sub.add_parser("attention_options")
    p.add_argument("--length", type=int, default=2048)
    p.add_argument("--span", type=int, default=1024)
    p.set_defaults(run=attention_options)
    p = sub.add_parser("rows")
    p.add_argument("--tokens", type=int, default=2048)
    p.set_defaults(run=rows)
    p = sub.add_parser("delta")
    p.add_argument("--tokens", type=int, default=2048)
    p.add_argument("--heads", type=int, default=16)
    p.set_defaults(run=delta)
    p = sub.add_parser("elementwise")
    p.add_argument("--tokens", type=int, default=2048)
    p.set_defaults(run=elementwise)
    args = parser.parse_args(argv)
    if not torch.cuda.is_available():
        raise SystemExit("the kernels need a CUDA device")
    args.run(args)


if __name__ == "__main__":
    main()
