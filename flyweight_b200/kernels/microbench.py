"""Run one kernel of the library alone on synthetic inputs, timed with CUDA events.

    python -m flyweight_b200.kernels.microbench gemm --tokens 8 --features 6144 --k 2048
    python -m flyweight_b200.kernels.microbench gemm --tokens 2048 --features 8192 --k 2048 --swiglu
    python -m flyweight_b200.kernels.microbench attention-decode --batch 8 --context 4096
    python -m flyweight_b200.kernels.microbench attention-prefill --tokens 2048
    python -m flyweight_b200.kernels.microbench shortconv --tokens 2048
    python -m flyweight_b200.kernels.microbench qk-norm-rope --tokens 2048
    python -m flyweight_b200.kernels.microbench causal-conv --tokens 16384
    python -m flyweight_b200.kernels.microbench gated-average --tokens 2048
    python -m flyweight_b200.kernels.microbench route --tokens 2048
    python -m flyweight_b200.kernels.microbench state-space --tokens 2048
    python -m flyweight_b200.kernels.microbench latent-decode --batch 64 --context 4096
    python -m flyweight_b200.kernels.microbench latent-prefill --tokens 2048
    python -m flyweight_b200.kernels.microbench sample --rows 8 --top-k 40

It is what the ncu summaries under ``profiles/`` were captured from (small cases of the same
kernels the engine runs), and a quick way to see what a shape costs.  Weight matrices are
rotated through enough copies to exceed the L2 cache, so the timed reads come from HBM.
"""
from __future__ import annotations

import argparse
import json
import math

import torch


def _time(fn, repeat: int, warmup: int = 3) -> float:
    for _ in range(warmup):
        fn()
    torch.cuda.synchronize()
    start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    start.record()
    for _ in range(repeat):
        fn()
    stop.record()
    torch.cuda.synchronize()
    return start.elapsed_time(stop) * 1e3 / repeat          # microseconds


def _time_graph(fn, repeat: int) -> float:
    """The same for kernels shorter than a Python call: ``repeat`` launches captured into one
    CUDA graph, the replay timed."""
    fn()
    torch.cuda.synchronize()
    stream = torch.cuda.Stream()
    graph = torch.cuda.CUDAGraph()
    with torch.cuda.stream(stream):
        with torch.cuda.graph(graph, stream=stream):
            for _ in range(repeat):
                fn()
    return _time(graph.replay, 5) / repeat


def run_gemm(args) -> dict:
    from . import tensorcore
    M, N, K = args.tokens, args.features, args.k
    rows = 2 * N if args.swiglu else N
    copies = max(2, min(16, int(160e6 // (rows * K * 2)) + 1))
    weights = [(torch.randn(rows, K, device="cuda") / math.sqrt(K)).to(torch.bfloat16)
               for _ in range(copies)]
    x = torch.randn(M, K, device="cuda").to(torch.bfloat16)
    turn = [0]

    def step():
        turn[0] = (turn[0] + 1) % copies
        w = weights[turn[0]]
        if args.swiglu:
            return tensorcore.swiglu_gate_up(x, w, args.splits or None, args.stages, args.tile_tokens)
        return tensorcore.gemm(x, w, torch.float32 if args.fp32_out else torch.bfloat16, None,
                               args.splits or None, args.stages, args.tile_tokens, args.wide)

    # a decode-sized product is shorter than a Python call: time it from a CUDA graph
    us = _time_graph(step, args.repeat) if M <= 128 else _time(step, args.repeat)
    flops = 2.0 * M * rows * K
    return {"kernel": "gemm_tcgen05", "tokens": M, "features": N, "k": K, "swiglu": args.swiglu,
            "us": us, "tflops": flops / us / 1e6, "weight_gb_s": rows * K * 2 / us / 1e3,
            "status": tensorcore.status()}


def _paged_inputs(batch, context, new, n_heads, n_kv, head_dim):
    pages_per = -(-context // 64)
    width = 16 * (-(-pages_per // 16))
    k_pool = torch.randn(batch * pages_per, n_kv, 64, head_dim, device="cuda").to(torch.bfloat16)
    v_pool = torch.randn(batch * pages_per, n_kv, 64, head_dim, device="cuda").to(torch.bfloat16)
    table = torch.full((batch, width), -1, dtype=torch.int32)
    for b in range(batch):
        table[b, :pages_per] = torch.arange(b * pages_per, (b + 1) * pages_per)
    q = torch.randn(batch * new, n_heads * head_dim, device="cuda").to(torch.bfloat16)
    return q, k_pool, v_pool, table.cuda(), width


def _shared_rows(args, k_pool):
    """``--shared-rows``: the form latent attention uses -- one pool head that every query head reads
    (in groups of at most 16), its rows keys and values at once, and a sink per head."""
    from . import attention
    groups = attention.head_groups(args.heads, 1)
    sink = torch.randn(args.heads, device="cuda", dtype=torch.float32)
    return k_pool, {"sink": sink, "groups": groups}, groups


def run_attention_decode(args) -> dict:
    from . import attention, ops
    B, ctx = args.batch, args.context
    if args.shared_rows:
        args.kv_heads = 1
    q, k_pool, v_pool, table, width = _paged_inputs(B, ctx, 1, args.heads, args.kv_heads, args.head_dim)
    positions = torch.full((B,), ctx - 1, dtype=torch.int32, device="cuda")
    tok_seg = torch.arange(B, dtype=torch.int32, device="cuda")
    extra, groups = {}, args.kv_heads
    if args.shared_rows:
        v_pool, extra, groups = _shared_rows(args, k_pool)
    splits, per, in_cluster = attention.decode_splits(B, groups, width, args.head_dim)
    if args.splits:
        splits, per, in_cluster = args.splits, -(-width // args.splits), args.cluster_merge
    scale = 1.0 / math.sqrt(args.head_dim)
    ops.set_decode_attention_tma(not args.cp_async, args.stages)
    call = lambda: ops.attention_decode_mma(q, k_pool, v_pool, positions, tok_seg, table,
                                           args.heads, 0, scale, splits, per, in_cluster, **extra)
    us = _time_graph(call, args.repeat) if args.graph else _time(call, args.repeat)
    ops.set_decode_attention_tma(True)
    kv_bytes = B * ctx * args.kv_heads * args.head_dim * 2 * (1 if args.shared_rows else 2)
    from . import tensorcore
    return {"kernel": "attention_decode_mma", "batch": B, "context": ctx, "splits": splits,
            "tiles_by": "cp.async" if args.cp_async or args.head_dim not in (64, 128) else "tma",
            "us": us, "kv_gb_s": kv_bytes / us / 1e3, "status": tensorcore.status()}


def run_attention_prefill(args) -> dict:
    from . import ops
    T = args.tokens
    if args.shared_rows:
        args.kv_heads = 1
    group = args.heads // args.kv_heads
    q, k_pool, v_pool, table, _ = _paged_inputs(1, T, T, args.heads, args.kv_heads, args.head_dim)
    extra = {}
    if args.shared_rows:
        v_pool, extra, groups = _shared_rows(args, k_pool)
        if args.mma_sync:
            group = args.heads // groups
        else:
            extra.pop("groups")
    positions = torch.arange(T, dtype=torch.int32, device="cuda")
    seg_start = torch.tensor([0, T], dtype=torch.int32, device="cuda")
    per_tile = max(1, (64 if args.mma_sync else 128) // group)
    n_tiles = -(-T // per_tile)
    tile_seg = torch.zeros(n_tiles, dtype=torch.int32, device="cuda")
    tile_tok0 = (torch.arange(n_tiles, dtype=torch.int32) * per_tile).cuda()
    scale = 1.0 / math.sqrt(args.head_dim)
    if args.softcap:
        extra["softcap"] = args.softcap
    if args.keep_first:
        extra["keep_first"] = args.keep_first
    kernel = ops.attention_prefill_mma if args.mma_sync else ops.attention_prefill_tcgen05
    us = _time(lambda: kernel(q, k_pool, v_pool, positions, seg_start, tile_seg, tile_tok0, n_tiles,
                              per_tile, table, args.heads, args.window, scale, **extra), args.repeat)
    flops = 2.0 * T * T * args.heads * args.head_dim        # causal: half of 4*T*T*h*d
    from . import tensorcore
    return {"kernel": "attention_prefill_mma" if args.mma_sync else "attention_prefill_tcgen05",
            "tokens": T, "us": us, "tflops": flops / us / 1e6, "status": tensorcore.status()}


def run_shortconv(args) -> dict:
    from . import ops
    T, H, L = args.tokens, args.hidden, args.taps
    p = torch.randn(T, 3 * H, device="cuda").to(torch.bfloat16)
    taps = torch.randn(H, L, device="cuda")
    state = torch.zeros(1, H, L - 1, device="cuda")
    seg_start = torch.tensor([0, T], dtype=torch.int32, device="cuda")
    seg_slot = torch.zeros(1, dtype=torch.int32, device="cuda")
    tok_seg = torch.zeros(T, dtype=torch.int32, device="cuda")
    us = _time_graph(lambda: ops.shortconv(p, taps, None, state, seg_start, seg_slot, tok_seg, 1,
                                           torch.bfloat16), args.repeat)
    return {"kernel": "shortconv", "tokens": T, "hidden": H, "taps": L, "us": us,
            "gb_s": T * H * 2 * 4 / us / 1e3}


def run_causal_conv(args) -> dict:
    """The convolution on q|k|v rows with the norm over q and over k in the same launch (``--no-norm``: the
    convolution alone), rows larger than L2 by default, a buffer larger than L2 written between launches."""
    from ..engine import Segment, StepBatch
    from . import mixing
    T, q, kv, taps = args.tokens, args.q_channels, args.kv_channels, args.taps
    C = q + 2 * kv
    dtype = torch.bfloat16 if args.bf16 else torch.float32
    rows = torch.randn(T, C + args.gate_columns, device="cuda").to(dtype)
    w = torch.randn(C, taps, device="cuda")
    state = torch.zeros(2, taps - 1, C, device="cuda") if taps > 1 else None
    batch = StepBatch([Segment("a", 0, 0, [0] * (T // 2), []), Segment("b", 1, 5, [0] * (T - T // 2), [])],
                      [[[0], [1]]], torch.device("cuda", 0))
    ranges = None if args.no_norm else [(0, torch.ones(q, device="cuda"), q, 1e-5), (q, torch.ones(kv, device="cuda"), kv, 1e-5)]
    flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")
    for _ in range(3):
        mixing.causal_conv(rows, w, state, batch, norm_ranges=ranges)
    times = []
    for _ in range(args.repeat):
        flush.zero_()
        start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        start.record()
        mixing.causal_conv(rows, w, state, batch, norm_ranges=ranges)
        stop.record()
        torch.cuda.synchronize()
        times.append(start.elapsed_time(stop) * 1e3)
    us = sorted(times)[len(times) // 2]
    return {"kernel": "causal_conv" + ("" if args.no_norm else "+norm"), "tokens": T, "channels": C, "taps": taps,
            "dtype": str(dtype).split(".")[-1], "us": us, "gb_s": 2 * T * C * rows.element_size() / us / 1e3}


def run_delta_rule(args) -> dict:
    """The gated delta rule's two kernels (prepare; scan) over ``batch`` segments of ``tokens`` tokens."""
    from ..engine.batch import Segment, StepBatch
    from . import recurrent
    H, G, d, e, L = args.heads, args.kv_heads, args.dim, args.vdim, args.taps
    dev = torch.device("cuda", 0)
    T = args.batch * args.tokens
    channels = 2 * G * d + H * e
    g = torch.Generator(device=dev).manual_seed(0)
    p = torch.randn((T, channels + H * e + 2 * H), generator=g, device=dev, dtype=torch.float32)
    taps = torch.randn((channels, L), generator=g, device=dev, dtype=torch.float32) * 0.5
    a_log = torch.zeros(H, device=dev, dtype=torch.float32)
    dt_bias = torch.zeros(H, device=dev, dtype=torch.float32)
    state = torch.zeros((args.batch, recurrent.delta_state_size(H, G, d, e, L)), device=dev, dtype=torch.float32)
    batch = StepBatch([Segment(f"r{i}", i, 0, [0] * args.tokens, []) for i in range(args.batch)],
                      [[[0]] * args.batch], dev)

    def step():
        recurrent.delta_rule(p, taps, a_log, dt_bias, state, batch, H, G, d, e)

    us = _time_graph(step, args.repeat) if args.graph else _time(step, args.repeat)
    state_bytes = 2 * args.batch * H * d * e * 4
    stream_bytes = T * (p.shape[1] + 2 * (channels + 2 * H) + H * e) * 4
    return {"kernel": "delta_rule", "batch": args.batch, "tokens": args.tokens, "heads": H, "kv_heads": G, "dim": d,
            "vdim": e, "taps": L, "us": us, "us_per_token": us / args.tokens,
            "gb_s": (state_bytes + stream_bytes) / us / 1e3, "gflops": 6.0 * T * H * d * e / us / 1e3}


def run_linear_attention(args) -> dict:
    """The decayed linear recurrence over ``batch`` segments of ``tokens`` tokens: token by token
    (``--scan``) or 64 tokens at a time on tensor cores."""
    from ..engine.batch import Segment, StepBatch
    from . import mixing
    H, d, e = args.heads, args.dim, args.vdim
    dev = torch.device("cuda", 0)
    T = args.batch * args.tokens
    g = torch.Generator(device=dev).manual_seed(0)
    p = torch.randn((T, 2 * H * d + 2 * H * e), generator=g, device=dev, dtype=torch.float32)
    decay = torch.linspace(0.9, 0.999, H, device=dev, dtype=torch.float32)
    state = torch.zeros((args.batch, H * d * e), device=dev, dtype=torch.float32)
    batch = StepBatch([Segment(f"r{i}", i, 0, [0] * args.tokens, []) for i in range(args.batch)],
                      [[[0]] * args.batch], dev)
    kernel = mixing.decay_scan if args.scan else mixing.decay_runs

    def step():
        kernel(p, 0, H * d, 2 * H * d, decay, state, batch, H, d, e, act_silu=True)

    us = _time(step, args.repeat)
    stream_bytes = T * (2 * H * d + 2 * H * e) * 4 + 2 * args.batch * H * d * e * 4
    return {"kernel": "decay_scan" if args.scan else "decay_runs", "batch": args.batch, "tokens": args.tokens,
            "heads": H, "dim": d, "vdim": e, "us": us, "gb_s": stream_bytes / us / 1e3,
            "gflops": 4.0 * T * H * d * e / us / 1e3}


def run_gated_average(args) -> dict:
    """The minGRU recurrence over ``batch`` segments of ``tokens`` tokens, ``width`` channels.  The projections
    are rotated through enough copies to exceed L2."""
    from ..engine.batch import Segment, StepBatch
    from . import mixing
    W, T = args.width, args.batch * args.tokens
    dev = torch.device("cuda", 0)
    dtype = torch.float32 if args.fp32 else torch.bfloat16
    row_bytes = T * 3 * W * 4
    copies = [torch.randn((T, 3 * W), device=dev) for _ in range(max(1, -(-(256 << 20) // row_bytes)))]
    bias = torch.zeros(W, device=dev)
    state = torch.zeros((args.batch, W), device=dev)
    batch = StepBatch([Segment(f"r{i}", i, 0, [0] * args.tokens, []) for i in range(args.batch)],
                      [[[0]] * args.batch], dev)

    def steps():
        for p in copies:
            mixing.gated_average(p, 0, W, 2 * W, bias, bias, state, batch, W, dtype)

    us = _time_graph(steps, args.repeat) / len(copies)
    moved = row_bytes + T * W * (4 if args.fp32 else 2) + 2 * args.batch * W * 4
    return {"kernel": "gated_average", "batch": args.batch, "tokens": args.tokens, "width": W, "us": us,
            "gb_s": moved / us / 1e3}


def run_state_space(args) -> dict:
    """The state-space recurrence over ``batch`` segments of ``tokens`` tokens (1: a decode step)."""
    from ..engine.batch import Segment, StepBatch
    from . import state_space
    H, G, n, e, T = args.heads, args.groups, args.state, args.vdim, args.batch * args.tokens
    dev = torch.device("cuda", 0)
    width = H * e + 2 * G * n
    state_bytes = args.batch * H * n * e * 4
    row_bytes = T * (width * 2 + H * 4 + H * e * 4)
    copies = max(1, min(16, -(-(256 << 20) // (row_bytes + state_bytes))))
    us_, ps, states = ([torch.randn(shape, device=dev).to(dtype) for _ in range(copies)]
                       for shape, dtype in (((T, width), torch.bfloat16), ((T, H), torch.float32),
                                            ((args.batch, H * n * e), torch.float32)))
    small = torch.zeros(H, device=dev)
    batch = StepBatch([Segment(f"r{i}", i, 0, [0] * args.tokens, []) for i in range(args.batch)],
                      [[[0]] * args.batch], dev)

    def steps():
        for u, p, state in zip(us_, ps, states):
            state_space.state_space(u, p, 0, small, small, small, state, batch, H, G, n, e,
                                    runs=False if args.scan else None)

    us = _time_graph(steps, args.repeat) / copies
    # the recurrence itself: two passes over the state a token (decay and write, read-out)
    return {"kernel": "state_space", "batch": args.batch, "tokens": args.tokens, "heads": H, "groups": G, "state": n,
            "vdim": e, "us": us, "gb_s": (row_bytes + 2 * state_bytes) / us / 1e3, "tflops": 4.0 * T * H * n * e / us / 1e6}


def _latent_case(args, contexts, tokens):
    """Pools (rotated through enough copies to exceed L2), a batch and its block table for latent rows."""
    from ..engine.batch import Segment, StepBatch
    dev = torch.device("cuda", 0)
    row = -(-(args.rank + args.rot) // 16) * 16
    pages = [-(-c // 64) for c in contexts]
    pool_bytes = sum(pages) * 64 * row * 2
    copies = max(1, min(16, -(-(256 << 20) // pool_bytes)))
    pools = [torch.randn((sum(pages), 1, 64, row), device=dev).to(torch.bfloat16) for _ in range(copies)]
    table, at = [], 0
    for n in pages:
        table.append(list(range(at, at + n)) + [-1] * (max(pages) - n))
        at += n
    batch = StepBatch([Segment(f"r{i}", i, c - tokens, [0] * tokens, []) for i, c in enumerate(contexts)], [table], dev)
    return row, pools, batch


def run_latent_decode(args) -> dict:
    """Single tokens of ``batch`` requests over ``context`` cached latent rows each."""
    from . import latent
    row, pools, batch = _latent_case(args, [args.context] * args.batch, 1)
    qa = torch.randn((args.batch, args.heads, row), device="cuda").to(torch.bfloat16)

    def steps():
        for pool in pools:
            latent.rows_attention(qa, pool, None, batch, batch.block_tables[0], args.rank, 0.1, args.batch)

    us = _time_graph(steps, args.repeat) / len(pools)
    moved = args.batch * args.context * row * 2
    return {"kernel": "latent_rows", "batch": args.batch, "context": args.context, "heads": args.heads, "row": row,
            "us": us, "gb_s": moved / us / 1e3,
            "tflops": 2.0 * args.batch * args.context * args.heads * (row + args.rank) / us / 1e6}


def run_latent_prefill(args) -> dict:
    """One prompt of ``tokens`` tokens over its own latent rows: expanded head keys and values, or the rows."""
    from . import latent
    row, pools, batch = _latent_case(args, [args.tokens], args.tokens)
    heads, dim, rot, vdim = args.heads, args.dim, args.rot, args.vdim
    hd = latent.expanded_head(dim, rot, vdim)
    w_kv = torch.randn((2 * heads * hd, row), device="cuda").to(torch.bfloat16)
    q = torch.randn((args.tokens, heads * (dim + rot)), device="cuda").to(torch.bfloat16)
    qa = torch.randn((args.tokens, heads, row), device="cuda").to(torch.bfloat16)
    table = torch.randn((args.tokens, rot // 2, 2), device="cuda")

    def steps():
        for pool in pools:
            if args.rows:
                latent.rows_attention(qa, pool, None, batch, batch.block_tables[0], args.rank, 0.1, 0)
            else:
                latent.expanded_prefill(q, pool, w_kv, table, batch, batch.block_tables[0], heads, dim, rot, rot,
                                        "interleaved", hd, 0.1, None, 0)

    steps()
    us = _time_graph(steps, args.repeat) / len(pools)
    per_pair = row + args.rank if args.rows else dim + rot + vdim
    return {"kernel": "latent_rows prompt" if args.rows else "latent expanded prompt", "tokens": args.tokens,
            "heads": heads, "us": us, "tflops": 1.0 * args.tokens ** 2 * heads * per_pair / us / 1e6}


def run_route(args) -> dict:
    """The router of routed experts: scores of ``outputs`` outputs and the choice of ``top``."""
    from . import experts
    h = torch.randn((args.tokens, args.hidden), device="cuda").to(torch.bfloat16)
    router = torch.randn((args.outputs, args.hidden), device="cuda") / math.sqrt(args.hidden)
    router16 = router.to(torch.bfloat16)
    router = router16.float()
    us = _time_graph(lambda: experts.route(h, router, None, 1, 1, args.top, args.scores,
                                           None if args.simt else router16), args.repeat)
    return {"kernel": "moe_route", "tokens": args.tokens, "outputs": args.outputs, "top": args.top, "us": us,
            "gflops": 2.0 * args.tokens * args.outputs * args.hidden / us / 1e3}


def run_qk_norm_rope(args) -> dict:
    from . import ops
    T, nh, nkv, hd = args.tokens, args.heads, args.kv_heads, args.head_dim
    pages = -(-T // 64)
    qkv = torch.randn(T, (nh + 2 * nkv) * hd, device="cuda").to(torch.bfloat16)
    w = torch.ones(hd, device="cuda")
    angles = torch.arange(T, dtype=torch.float64)[:, None] * (1e6 ** (-torch.arange(hd // 2, dtype=torch.float64) * 2 / hd))
    table = torch.stack([angles.cos(), angles.sin()], -1).float().cuda()
    positions = torch.arange(T, dtype=torch.int32, device="cuda")
    tok_seg = torch.zeros(T, dtype=torch.int32, device="cuda")
    block_table = torch.arange(pages, dtype=torch.int32, device="cuda")[None]
    k_pool = torch.zeros(pages, nkv, 64, hd, device="cuda", dtype=torch.bfloat16)
    v_pool = torch.zeros_like(k_pool)
    us = _time_graph(lambda: ops.qk_norm_rope(qkv, w, w, table, positions, tok_seg, block_table,
                                              k_pool, v_pool, nh, nkv, hd, hd, 1e-5, torch.bfloat16),
                     args.repeat)
    return {"kernel": "qk_norm_rope", "tokens": T, "us": us,
            "gb_s": T * (nh + 2 * nkv) * hd * 2 * 2 / us / 1e3}


def run_sample(args) -> dict:
    from ..sampling import sampler
    from ..sampling.config import SamplingConfig
    rows, vocab = args.rows, args.vocab
    # enough copies of the logits that the timed reads come from HBM
    copies = max(2, min(16, int(160e6 // (rows * vocab * 4)) + 1))
    # Gaussian logits of the given spread: at temperature 0.8 and top-p 0.95 a spread of 3 keeps about
    # 1,200 candidates of 65,536 (a flat row), a spread of 4 about 200 (a peaked one, like a model's)
    logits = [torch.randn(rows, vocab, device="cuda") * args.logit_scale for _ in range(copies)]
    config = SamplingConfig(temperature=args.temperature, top_k=args.top_k, top_p=args.top_p, min_p=0.0, seed=1)
    uniforms = [((i * 37) % 97) / 97.0 for i in range(rows)]
    turn = [0]

    def step():
        turn[0] = (turn[0] + 1) % copies
        if args.temperature <= 0.0:
            return sampler.argmax(logits[turn[0]])
        return sampler.sample(logits[turn[0]], [config] * rows, uniforms)

    if args.kernel_only and args.temperature > 0.0:
        # the launches alone: the rows' settings are staged once, not by every call's Python
        import struct
        from . import lib
        from .lib import ptr, stream
        k = min(args.top_k, vocab) if args.top_k > 0 else vocab
        large = k > sampler.SMALL_K
        record = struct.pack("<fifffffi", args.temperature, args.top_k, args.top_p, 0.0, 1.0, 0.0, 0.0, 0)
        params = torch.frombuffer(bytearray(record * rows), dtype=torch.uint8).cuda()
        uni = torch.tensor(uniforms, dtype=torch.float64, device="cuda")
        out = torch.empty(rows, dtype=torch.int32, device="cuda")
        vpad = 1
        while vpad < vocab:
            vpad <<= 1
        keys = torch.empty((rows, vpad), dtype=torch.int64, device="cuda") if large else None

        def step():
            turn[0] = (turn[0] + 1) % copies
            lib.call("fwb_sample", ptr(logits[turn[0]]), rows, vocab, ptr(params), ptr(uni), None, 0, ptr(out),
                     ptr(keys), None, vpad if large else 0, 1 if large else 0, stream())

    us = _time(step, args.repeat)
    return {"kernel": "argmax" if args.temperature <= 0.0 else "sample_kernel", "rows": rows, "vocab": vocab,
            "top_k": args.top_k, "top_p": args.top_p, "logit_scale": args.logit_scale,
            "kernel_only": bool(args.kernel_only), "us": us, "gb_s": rows * vocab * 4 / us / 1e3}


def main(argv=None) -> int:
    parser = argparse.ArgumentParser(prog="python -m flyweight_b200.kernels.microbench",
                                     description=__doc__,
                                     formatter_class=argparse.RawDescriptionHelpFormatter)
    sub = parser.add_subparsers(dest="kernel", required=True)
    gemm = sub.add_parser("gemm")
    gemm.add_argument("--tokens", type=int, default=8)
    gemm.add_argument("--features", type=int, default=2048)
    gemm.add_argument("--k", type=int, default=2048)
    gemm.add_argument("--swiglu", action="store_true", help="features = F; the weight is [2F][K]")
    gemm.add_argument("--fp32-out", action="store_true")
    gemm.add_argument("--splits", type=int, default=0)
    gemm.add_argument("--stages", type=int, default=0)
    gemm.add_argument("--tile-tokens", type=int, default=0, help="128 or 256 (0: by token count)")
    gemm.add_argument("--wide", type=int, default=-1, help="two feature tiles per CTA: 1/0 (-1: auto)")
    for name in ("attention-decode", "attention-prefill"):
        p = sub.add_parser(name)
        p.add_argument("--batch", type=int, default=8)
        p.add_argument("--context", type=int, default=4096)
        p.add_argument("--tokens", type=int, default=2048)
        p.add_argument("--heads", type=int, default=32)
        p.add_argument("--kv-heads", type=int, default=8)
        p.add_argument("--head-dim", type=int, default=64)
        p.add_argument("--splits", type=int, default=0)
        p.add_argument("--shared-rows", action="store_true",
                       help="one pool head for all query heads, rows as keys and values, a sink per head")
        p.add_argument("--graph", action="store_true",
                       help="decode: the launches captured in a CUDA graph (kernels shorter than a Python call)")
        p.add_argument("--window", type=int, default=0, help="prefill: a sliding window")
        p.add_argument("--keep-first", type=int, default=0, help="prefill: positions kept beside the window")
        p.add_argument("--softcap", type=float, default=0.0)
        p.add_argument("--mma-sync", action="store_true", help="the mma.sync prompt kernel")
        p.add_argument("--cluster-merge", action="store_true", help="with --splits <= 8: merge inside the kernel")
        p.add_argument("--cp-async", action="store_true", help="decode: key and value tiles by cp.async, not TMA")
        p.add_argument("--stages", type=int, default=0, help="decode by TMA: ring depth, 2 to 8 (0: the launcher's choice)")
    conv = sub.add_parser("shortconv")
    conv.add_argument("--tokens", type=int, default=2048)
    conv.add_argument("--hidden", type=int, default=2048)
    conv.add_argument("--taps", type=int, default=3)
    cconv = sub.add_parser("causal-conv")
    cconv.add_argument("--tokens", type=int, default=16384)
    cconv.add_argument("--q-channels", type=int, default=2048)
    cconv.add_argument("--kv-channels", type=int, default=512)
    cconv.add_argument("--taps", type=int, default=3)
    cconv.add_argument("--gate-columns", type=int, default=32, help="columns behind q|k|v that the rows carry along")
    cconv.add_argument("--bf16", action="store_true")
    cconv.add_argument("--no-norm", action="store_true")
    rope = sub.add_parser("qk-norm-rope")
    rope.add_argument("--tokens", type=int, default=2048)
    rope.add_argument("--heads", type=int, default=32)
    rope.add_argument("--kv-heads", type=int, default=8)
    rope.add_argument("--head-dim", type=int, default=64)
    delta = sub.add_parser("delta-rule")
    delta.add_argument("--batch", type=int, default=1)
    delta.add_argument("--tokens", type=int, default=2048)
    delta.add_argument("--heads", type=int, default=16)
    delta.add_argument("--kv-heads", type=int, default=8)
    delta.add_argument("--dim", type=int, default=128)
    delta.add_argument("--vdim", type=int, default=128)
    delta.add_argument("--taps", type=int, default=4)
    delta.add_argument("--graph", action="store_true")
    lin = sub.add_parser("linear-attention")
    lin.add_argument("--batch", type=int, default=1)
    lin.add_argument("--tokens", type=int, default=2048)
    lin.add_argument("--heads", type=int, default=16)
    lin.add_argument("--dim", type=int, default=128)
    lin.add_argument("--vdim", type=int, default=128)
    lin.add_argument("--scan", action="store_true", help="the token-by-token kernel")
    avg = sub.add_parser("gated-average")
    avg.add_argument("--batch", type=int, default=1)
    avg.add_argument("--tokens", type=int, default=2048)
    avg.add_argument("--width", type=int, default=2048)
    avg.add_argument("--fp32", action="store_true")
    rt = sub.add_parser("route")
    rt.add_argument("--tokens", type=int, default=2048)
    rt.add_argument("--hidden", type=int, default=2048)
    rt.add_argument("--outputs", type=int, default=32)
    rt.add_argument("--top", type=int, default=8)
    rt.add_argument("--simt", action="store_true", help="the fp32-FMA kernel at every size")
    rt.add_argument("--scores", default="sigmoid")
    ssm = sub.add_parser("state-space")
    ssm.add_argument("--batch", type=int, default=1)
    ssm.add_argument("--tokens", type=int, default=2048)
    ssm.add_argument("--heads", type=int, default=64)
    ssm.add_argument("--groups", type=int, default=1)
    ssm.add_argument("--state", type=int, default=128)
    ssm.add_argument("--vdim", type=int, default=64)
    ssm.add_argument("--scan", action="store_true", help="the token-by-token kernel")
    for name in ("latent-decode", "latent-prefill"):
        lat = sub.add_parser(name)
        lat.add_argument("--batch", type=int, default=64)
        lat.add_argument("--context", type=int, default=4096)
        lat.add_argument("--tokens", type=int, default=2048)
        lat.add_argument("--heads", type=int, default=32)
        lat.add_argument("--rank", type=int, default=256)
        lat.add_argument("--rot", type=int, default=32)
        lat.add_argument("--dim", type=int, default=64)
        lat.add_argument("--vdim", type=int, default=64)
        lat.add_argument("--rows", action="store_true", help="prompt: over the rows themselves")
    smp = sub.add_parser("sample")
    smp.add_argument("--rows", type=int, default=8)
    smp.add_argument("--vocab", type=int, default=65536)
    smp.add_argument("--temperature", type=float, default=0.8, help="0: arg-max")
    smp.add_argument("--top-k", type=int, default=40, help="0: the whole vocabulary")
    smp.add_argument("--top-p", type=float, default=0.95)
    smp.add_argument("--logit-scale", type=float, default=3.0, help="spread of the Gaussian logits")
    smp.add_argument("--kernel-only", action="store_true", help="time the launches without the Python call around them")
    for p in sub.choices.values():
        p.add_argument("--repeat", type=int, default=20)
    args = parser.parse_args(argv)
    runner = {"gemm": run_gemm, "attention-decode": run_attention_decode,
              "attention-prefill": run_attention_prefill, "shortconv": run_shortconv,
              "causal-conv": run_causal_conv,
              "qk-norm-rope": run_qk_norm_rope, "sample": run_sample, "delta-rule": run_delta_rule,
              "linear-attention": run_linear_attention, "gated-average": run_gated_average, "route": run_route,
              "state-space": run_state_space, "latent-decode": run_latent_decode, "latent-prefill": run_latent_prefill}[args.kernel]
    print(json.dumps(runner(args)))
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
