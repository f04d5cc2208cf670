"""Times one kernel of the library alone, at a given shape, with CUDA events.

    python -m llm_inference_b200.cli.microbench gemm --m 8 --n 17920 --k 1536 [--swiglu] [--library]
    python -m llm_inference_b200.cli.microbench decode_attention --batch 64 --context 2048
    python -m llm_inference_b200.cli.microbench prefill_attention --tokens 2048

Between timed launches a buffer larger than the L2 cache is overwritten, so every launch
reads its operands from HBM. Prints one JSON line with the median time and the bytes or flops
per second it corresponds to. Used for roofline numbers and as the small case for profiler
captures.
"""

from __future__ import annotations

import argparse
import json
import statistics
import sys
from ctypes import c_void_p
from types import SimpleNamespace

import numpy as np
import torch


class _Ctx(SimpleNamespace):
    @property
    def stream(self):
        return c_void_p(torch.cuda.current_stream().cuda_stream)


def make_ctx(positions=None, token_seq=None, starts=None, runs=None, options=None):
    from ..csrc.library import kernels
    from ..parts.context import Workspace

    dev = torch.device("cuda:0")
    ws = Workspace(dev)
    as_dev = lambda v: torch.tensor(v, dtype=torch.int32, device=dev) if v is not None else None
    ctx = _Ctx(
        lib=kernels(), device=dev, err=torch.zeros(1, dtype=torch.int32, device=dev), workspace=ws,
        options=dict(options or {}), positions=as_dev(positions), token_seq=as_dev(token_seq),
        num_tokens=len(positions) if positions is not None else 0,
        buffer=lambda name, shape, dtype=None, per_token=True: ws.get(name, shape, dtype, per_token=per_token),
    )
    if runs is not None:
        ctx.num_seqs = len(runs)
        ctx.seq_q_start = as_dev(np.concatenate([[0], np.cumsum(runs)[:-1]]).tolist())
        ctx.seq_q_len = as_dev(list(runs))
        ctx.seq_kv_len = as_dev([s + r for s, r in zip(starts, runs)])
        ctx.max_q_len = max(runs)
        ctx.max_kv_len = max(s + r for s, r in zip(starts, runs))
        ctx.num_decode_seqs = len(runs) if max(runs) == 1 else 0
    return ctx


def time_launches(fn, iters: int, warmup: int = 3) -> float:
    flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")
    for _ in range(warmup):
        fn()
    times = []
    for _ in range(iters):
        flush.fill_(1)
        torch.cuda.synchronize()
        start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        start.record()
        fn()
        end.record()
        torch.cuda.synchronize()
        times.append(start.elapsed_time(end) * 1e3)
    return statistics.median(times)


def time_back_to_back(fns, launches: int) -> float:
    """Microseconds per launch when ``fns`` run round-robin back to back on the device. The
    launches are captured in a CUDA graph, so host launch cost does not enter; the operands
    of all of them together must exceed the L2 cache."""
    for fn in fns:
        fn()
    torch.cuda.synchronize()
    graph = torch.cuda.CUDAGraph()
    with torch.cuda.graph(graph):
        for i in range(launches):
            fns[i % len(fns)]()
    graph.replay()
    torch.cuda.synchronize()
    start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    start.record()
    graph.replay()
    end.record()
    torch.cuda.synchronize()
    return start.elapsed_time(end) * 1e3 / launches


TRACE_POINTS = ("resident", "predecessor done", "first stage landed", "last stage landed", "accumulator complete",
                "partial tiles met", "slice stored", "leaving")


def trace_back_to_back(lib, fns, launches: int) -> dict:
    """The tcgen05 product's own timeline (b200_stream_gemm_trace) of ``launches`` launches that run
    back to back in a CUDA graph: for every point of a block's life, when the first, the median
    and the last block of a launch passed it, in microseconds after the last block of the launch
    in front left; averaged over the later half of the launches."""
    from ..csrc.library import ptr

    for fn in fns:
        fn()
    torch.cuda.synchronize()
    stamps = lib.b200_stream_gemm_trace_stamps()
    stride = 4096 * stamps
    buffer = torch.zeros(launches, stride, dtype=torch.int64, device="cuda")
    lib.b200_stream_gemm_trace(ptr(buffer), launches, stride)
    graph = torch.cuda.CUDAGraph()
    try:
        with torch.cuda.graph(graph):
            for i in range(launches):
                fns[i % len(fns)]()
    finally:
        lib.b200_stream_gemm_trace(None, 0, 0)
    for _ in range(3):
        graph.replay()
    torch.cuda.synchronize()
    data = buffer.cpu().numpy().reshape(launches, -1, stamps)
    blocks = int((data[1, :, 0] != 0).sum())
    data = data[:, :blocks, :].astype(np.float64) / 1e3  # microseconds
    rows = {name: [] for name in TRACE_POINTS}
    spans = []
    for j in range(launches // 2, launches):
        origin = data[j - 1, :, stamps - 1].max()
        spans.append(data[j, :, stamps - 1].max() - origin)
        for i, name in enumerate(TRACE_POINTS):
            column = data[j, :, i]
            column = column[column != 0]
            if column.size:
                rows[name].append((column.min() - origin, float(np.median(column)) - origin, column.max() - origin))
    table = {name: [round(float(v), 2) for v in np.mean(np.array(values), axis=0)] for name, values in rows.items() if values}
    return {"blocks": blocks, "us_per_launch": round(float(np.mean(spans)), 2), "first_median_last_us": table}


def bench_gemm(args) -> dict:
    from ..parts import ops

    m, n, k = args.m, args.n, args.k
    x = torch.randn(m, k, device="cuda").to(torch.bfloat16)
    w = (torch.randn(n, k, device="cuda") / k**0.5).to(torch.bfloat16)
    ctx = make_ctx(positions=[0] * m, options={"gemm": args.gemm})
    if args.plan is not None:
        ctx.lib.lib.b200_stream_gemm_plan_override(*args.plan)
    if args.rotate:
        # Enough copies of the weights that one round exceeds the L2 cache several times.
        copies = max(2, -(-(512 << 20) // (w.numel() * 2)))
        weights = [w] + [w.clone() for _ in range(copies - 1)]
        out = torch.empty(m, n // 2 if args.swiglu else n, device="cuda", dtype=torch.float32 if args.f32_out else torch.bfloat16)
        if args.swiglu and args.gemm == "library":
            mid = torch.empty(m, n, device="cuda", dtype=torch.bfloat16)
            fns = [lambda wi=wi: (ops.linear(ctx, x, wi, mid), ops.gated_mul(ctx, mid, out)) for wi in weights]
        elif args.swiglu:
            fns = [lambda wi=wi: ops.linear_gated(ctx, x, wi, out) for wi in weights]
        else:
            fns = [lambda wi=wi: ops.linear(ctx, x, wi, out) for wi in weights]
        if args.trace:
            if args.gemm != "tcgen05":
                raise SystemExit("--trace records the tcgen05 product's own timestamps: give --gemm tcgen05")
            return {"kernel": "gemm", "m": m, "n": n, "k": k, "swiglu": args.swiglu, "mode": "back-to-back, traced",
                    **trace_back_to_back(ctx.lib.lib, fns, 4 * copies)}
        us = time_back_to_back(fns, 4 * copies)
        nbytes = w.numel() * 2 + x.numel() * 2 + out.numel() * out.element_size()
        return {"kernel": "gemm", "m": m, "n": n, "k": k, "gemm": args.gemm, "swiglu": args.swiglu, "mode": "back-to-back",
                "us": us, "GBps": nbytes / us / 1e3}
    if args.swiglu:
        out = torch.empty(m, n // 2, device="cuda", dtype=torch.bfloat16)
        if args.gemm == "library":
            mid = torch.empty(m, n, device="cuda", dtype=torch.bfloat16)

            def fn():
                ops.linear(ctx, x, w, mid)
                ops.gated_mul(ctx, mid, out)
        else:
            fn = lambda: ops.linear_gated(ctx, x, w, out)
    else:
        out = torch.empty(m, n, device="cuda", dtype=torch.float32 if args.f32_out else torch.bfloat16)
        fn = lambda: ops.linear(ctx, x, w, out)
    us = time_launches(fn, args.iters)
    nbytes = w.numel() * 2 + x.numel() * 2 + out.numel() * out.element_size()
    return {"kernel": "gemm", "m": m, "n": n, "k": k, "gemm": args.gemm, "swiglu": args.swiglu, "us": us,
            "GBps": nbytes / us / 1e3, "TFLOPs": 2.0 * m * n * k / us / 1e6}


def bench_attention(args, decode: bool, mixed: bool = False) -> dict:
    """``mixed``: attention whose softmax weights are mixed over heads (parts/mixed_attention.py): one pass per kv
    head, every query head's weights applied to that head's values, then the kernel that mixes and gates. Its
    flops count what the passes execute (``kv_heads`` times the scores and the weighted sums of all query heads).
    ``--softcap``, ``--bias-reach`` and ``--chunk`` shape the scores (``ops.ScoreShape``); flops then count the visible keys."""
    from ..parts import attention_dispatch, ops
    from ..parts.context import CacheView

    q_heads, kv_heads, dim, page = args.q_heads, args.kv_heads, args.head_dim, args.page
    if decode:
        starts, runs = [args.context - 1] * args.batch, [1] * args.batch
    else:
        starts, runs = [args.context - args.tokens], [args.tokens]
    lens = [s + r for s, r in zip(starts, runs)]
    need = [-(-n // page) for n in lens]
    num_pages = sum(need) + 1
    order = np.random.default_rng(0).permutation(num_pages - 1)
    tables = np.zeros((len(lens), max(need)), dtype=np.int32)
    at = 0
    for s, c in enumerate(need):
        tables[s, :c] = order[at : at + c]
        at += c
    positions = [p for s, r in zip(starts, runs) for p in range(s, s + r)]
    token_seq = [i for i, r in enumerate(runs) for _ in range(r)]
    options = {"attention": "plain" if args.plain else args.attention, "decode_loader": args.loader}
    if args.splits:
        options["decode_splits"] = args.splits
    if args.stages:
        options["decode_stages"] = args.stages
    ctx = make_ctx(positions, token_seq, starts, runs, options)
    q = torch.randn(len(positions), q_heads * dim, device="cuda").to(torch.bfloat16)
    out = torch.empty_like(q)
    table = torch.from_numpy(tables).cuda()
    # --layers N: N arenas of the same geometry, as the layers of a model have; back to back
    # they exceed the L2 cache when one of them does not.
    fns = []
    for _ in range(max(1, args.layers)):
        keys = torch.randn(num_pages, kv_heads, page, dim, device="cuda").to(torch.bfloat16)
        values = torch.randn_like(keys)
        view = CacheView(0, True, keys, values, table, num_pages, tables.shape[1], page, args.window, args.keep_first)
        if mixed:
            planes = torch.empty(kv_heads, len(positions), q_heads * dim, device="cuda", dtype=torch.bfloat16)
            talk = torch.randn(q_heads, q_heads, device="cuda")
            gate = torch.randn_like(q)

            def passes(view=view, planes=planes):
                attention_dispatch.attend_value_planes(ctx, view, q, planes, q_heads, kv_heads, dim, dim**-0.5)
                ops.mix_heads_gate(ctx, planes, talk, gate, q_heads, kv_heads, dim, dim, out)

            fns.append(passes)
            continue
        bias = torch.randn(q_heads, args.bias_reach + 1, device="cuda") if args.bias_reach else None
        shape = ops.ScoreShape(args.softcap, bias, args.chunk, bias.max(dim=1).values.contiguous() if bias is not None else None,
                               torch.zeros(q_heads, device="cuda") if args.sigmoid else None, torch.zeros(q_heads, device="cuda") if args.sink else None)
        fns.append(lambda view=view, shape=shape: attention_dispatch.attend(ctx, view, q, out, q_heads, kv_heads, dim, dim**-0.5, shape=shape))
    # --rotate: back to back inside a CUDA graph, so that neither the host's launch cost nor
    # the idle gap before a lone launch enters (with one arena the cache stays in L2, as it
    # does in a small model's step, where the layer's keys were written just before).
    us = time_back_to_back(fns, 16 * len(fns)) if args.rotate else time_launches(fns[0], args.iters)
    kv_bytes = sum(lens) * kv_heads * dim * 2 * 2
    flops = sum(4.0 * q_heads * dim * r * (s + (r + 1) / 2) for s, r in zip(starts, runs)) * (kv_heads if mixed else 1)
    if args.window and not mixed:  # keys a row sees: its window, and the kept ones in front of it
        seen = [min(p + 1, args.window) + min(args.keep_first, max(0, p + 1 - args.window)) for p in positions]
        flops = sum(4.0 * q_heads * dim * n for n in seen)
        kv_bytes = sum(min(n, args.window + args.keep_first) for n in lens) * kv_heads * dim * 2 * 2 if decode else kv_bytes
    if args.chunk and not mixed:
        flops = sum(4.0 * q_heads * dim * (p % args.chunk + 1) for p in positions)
    return {"kernel": ("mixed_" if mixed else "") + ("decode_attention" if decode else "prefill_attention"), "batch": len(lens), "context": args.context,
            "tokens": len(positions), "softcap": args.softcap, "bias_reach": args.bias_reach, "chunk": args.chunk, "window": args.window, "keep_first": args.keep_first, "sigmoid": args.sigmoid, "sink": args.sink, "loader": args.loader, "splits": args.splits, "stages": args.stages,
            "layers": args.layers, "us": us, "GBps": kv_bytes / us / 1e3, "TFLOPs": flops / us / 1e6}


def bench_latent_attention(args, decode: bool) -> dict:
    """Attention over cached latents (parts/latent_attention.py): ``--q-heads`` heads over rows of
    ``--rank`` + ``--rot-dim`` numbers; bytes are the cached rows read once per request, flops the
    scores and the weighted sums over those rows (2 * (2 rank + rot_dim) per head, query and key)."""
    from ..parts import attention_dispatch
    from ..parts.context import CacheView

    heads, rank, rot, page = args.q_heads, args.rank, args.rot_dim, args.page
    if decode:
        starts, runs = [args.context - 1] * args.batch, [1] * args.batch
    else:
        starts, runs = [args.context - args.tokens], [args.tokens]
    lens = [s + r for s, r in zip(starts, runs)]
    need = [-(-n // page) for n in lens]
    num_pages = sum(need) + 1
    order = np.random.default_rng(0).permutation(num_pages - 1)
    tables = np.zeros((len(lens), max(need)), dtype=np.int32)
    at = 0
    for s, c in enumerate(need):
        tables[s, :c] = order[at : at + c]
        at += c
    positions = [p for s, r in zip(starts, runs) for p in range(s, s + r)]
    token_seq = [i for i, r in enumerate(runs) for _ in range(r)]
    options = {"attention": "plain" if args.plain else "auto"}
    if args.splits:
        options["latent_pieces"] = args.splits
    ctx = make_ctx(positions, token_seq, starts, runs, options)
    tokens = len(positions)
    q_lat = (torch.randn(heads, tokens, rank, device="cuda") / rank**0.5).to(torch.bfloat16)
    q_rot = torch.randn(tokens, heads * rot, device="cuda").to(torch.bfloat16)
    gate = torch.randn(tokens, heads, device="cuda").to(torch.bfloat16)
    sink = torch.zeros(heads, device="cuda")
    out = torch.empty_like(q_lat)
    table = torch.from_numpy(tables).cuda()
    fns = []
    for _ in range(max(1, args.layers)):
        rows = torch.randn(num_pages, 1, page, rank + rot, device="cuda").to(torch.bfloat16)
        view = CacheView(0, True, rows, None, table, num_pages, tables.shape[1], page, 0)
        fns.append(lambda view=view: attention_dispatch.attend_latent(ctx, view, q_lat, q_rot, sink, gate, out, heads, rank, rot, (rank + rot) ** -0.5))
    us = time_back_to_back(fns, 16 * len(fns)) if args.rotate else time_launches(fns[0], args.iters)
    row_bytes = sum(lens) * (rank + rot) * 2
    flops = sum(2.0 * heads * (2 * rank + rot) * r * (s + (r + 1) / 2) for s, r in zip(starts, runs))
    return {"kernel": "latent_decode_attention" if decode else "latent_prefill_attention", "batch": len(lens), "context": args.context,
            "tokens": tokens, "heads": heads, "rank": rank, "rot_dim": rot, "pieces": args.splits, "layers": args.layers,
            "us": us, "GBps": row_bytes / us / 1e3, "TFLOPs": flops / us / 1e6}


def bench_delta_recurrence(args) -> dict:
    """The gated delta rule's recurrence (parts/delta_rule.py) over ``--batch`` requests of
    ``--tokens`` tokens each: ``--q-heads`` heads with states of ``--head-dim`` x ``--vdim``. Flops:
    per token and head three products over the state (decay, k-dot and update, q-dot). ``--per-head``: the form with one
    decay per head; ``--kv-heads`` q/k heads are shared by its heads; ``--portions``: chunk by chunk or token by token."""
    from ..parts import ops

    heads, dk, dv, batch, tokens = args.q_heads, args.head_dim, args.vdim, args.batch, args.tokens
    runs, starts = [tokens] * batch, [0] * batch
    positions = [p for r in runs for p in range(r)]
    token_seq = [i for i, r in enumerate(runs) for _ in range(r)]
    ctx = make_ctx(positions, token_seq, starts, runs, {"delta_portions": args.portions})
    ctx.seq_slot = torch.arange(batch, dtype=torch.int32, device="cuda")
    total = batch * tokens
    unit = lambda x: x / x.norm(dim=-1, keepdim=True)
    q = unit(torch.randn(total, heads, dk, device="cuda")).reshape(total, heads * dk).contiguous()
    k = unit(torch.randn(total, heads, dk, device="cuda")).reshape(total, heads * dk).contiguous()
    v = torch.randn(total, heads * dv, device="cuda")
    beta = torch.rand(total, heads, device="cuda")
    decay = torch.rand(total, heads * dk, device="cuda") * 0.2 + 0.8
    state = torch.zeros(batch, heads, dk, dv, device="cuda")
    out = torch.empty(total, heads * dv, device="cuda")
    moved = 4.0 * (total * (3 * heads * dk + 2 * heads * dv + heads) + 2 * batch * heads * dk * dv)
    run = lambda: ops.delta_recurrence(ctx, q, k, v, beta, decay, state, out, heads, heads, dk, dv)
    if args.per_head:
        kvh = args.kv_heads
        q, k = (x.view(total, heads, dk)[:, :kvh].reshape(total, kvh * dk).contiguous() for x in (q, k))
        kq = (q.view(total, kvh, dk) * k.view(total, kvh, dk)).sum(-1).contiguous()
        decay = decay.view(total, heads, dk)[:, :, 0].log().contiguous()
        moved = 4.0 * (total * (2 * kvh * dk + kvh + 2 * heads * dv + 2 * heads) + 2 * batch * heads * dk * dv)
        run = lambda: ops.delta_head_recurrence(ctx, q, k, v, beta, decay, kq, state, out, heads, kvh, dk, dv)
    us = time_launches(run, args.iters)
    return {"kernel": "delta_head_recurrence" if args.per_head else "delta_recurrence", "batch": batch, "tokens": tokens, "heads": heads, "dim": dk, "vdim": dv, "us": us,
            "us_per_token": us / tokens, "GBps": moved / us / 1e3, "TFLOPs": 7.0 * total * heads * dk * dv / us / 1e6}


def bench_delta_step(args) -> dict:
    """Everything between the two products of the delta rule with one decay per head (parts/delta_rule.py, ``head_delta``) for one
    token of each of ``--batch`` requests: the fused kernel, or with ``--plain`` the chain of kernels of prompt portions. Bytes: the
    states and the convolution's history once each way, and the projections."""
    from ..parts import PartSpec, build_part, ops

    heads, kvh, dk, dv, batch, taps = args.q_heads, args.kv_heads, args.head_dim, args.vdim, args.batch, 4
    ctx = make_ctx([5] * batch, list(range(batch)), [5] * batch, [1] * batch, {"delta_step": "chain" if args.plain else "auto"})
    ctx.seq_slot = torch.arange(batch, dtype=torch.int32, device="cuda")
    ctx.buffer = lambda name, shape, dtype=None, per_token=True: ctx.workspace.get(name, shape, dtype or torch.bfloat16, per_token=per_token)
    part = build_part("mixer", PartSpec("head_delta", dict(prefix="", hidden_size=64, heads=heads, kv_heads=kvh, dim=dk, vdim=dv, taps=taps, eps=1e-5)))
    part.load({s.name: torch.randn(s.shape) * 0.1 for s in part.tensor_specs()}, torch.bfloat16, torch.device("cuda"))
    proj = torch.randn(batch, part.w_in.shape[0], device="cuda").to(torch.bfloat16)
    state = torch.zeros(batch, heads, dk, dv, device="cuda")
    history = torch.zeros(batch, taps - 1, part.channels, device="cuda", dtype=torch.bfloat16)
    out = torch.empty(batch, heads * dv, device="cuda", dtype=torch.bfloat16)
    us = time_launches(lambda: part.mix(ctx, proj, state, history, out), args.iters)
    moved = 8.0 * batch * heads * dk * dv + 2.0 * (proj.numel() + out.numel() + 2 * history.numel())
    return {"kernel": "delta_step", "batch": batch, "heads": heads, "kv_heads": kvh, "dim": dk, "vdim": dv, "chain": args.plain, "us": us, "GBps": moved / us / 1e3}


def bench_wkv_recurrence(args) -> dict:
    """The recurrence of the mixer with a decay per channel and a bonus for the current token
    (parts/wkv.py) over ``--batch`` requests of ``--tokens`` tokens each: ``--q-heads`` heads with states of
    ``--head-dim`` x ``--head-dim``. Flops: per token and head two products over the state (read-out; decay
    and update)."""
    from ..parts import ops

    heads, dim, batch, tokens = args.q_heads, args.head_dim, args.batch, args.tokens
    runs, starts = [tokens] * batch, [0] * batch
    ctx = make_ctx([p for r in runs for p in range(r)], [i for i, r in enumerate(runs) for _ in range(r)], starts, runs)
    ctx.seq_slot = torch.arange(batch, dtype=torch.int32, device="cuda")
    total = batch * tokens
    r, k, v = (torch.randn(total, heads * dim, device="cuda") for _ in range(3))
    bonus = torch.randn(total, heads, device="cuda")
    decay = torch.rand(total, heads * dim, device="cuda") * 0.2 + 0.8
    state = torch.zeros(batch, heads, dim, dim, device="cuda")
    out = torch.empty(total, heads * dim, device="cuda")
    us = time_launches(lambda: ops.wkv_recurrence(ctx, r, k, v, bonus, decay, state, out, heads, dim, dim), args.iters)
    moved = 4.0 * (total * (5 * heads * dim + heads) + 2 * batch * heads * dim * dim)
    return {"kernel": "wkv_recurrence", "batch": batch, "tokens": tokens, "heads": heads, "dim": dim, "us": us,
            "us_per_token": us / tokens, "GBps": moved / us / 1e3, "TFLOPs": 5.0 * total * heads * dim * dim / us / 1e6}


def bench_mlstm(args) -> dict:
    """The matrix memory between its products (parts/mlstm.py: gates, recurrence, norm and gate) over ``--batch`` requests of
    ``--tokens`` tokens each: ``--q-heads`` heads with states of ``--head-dim`` x ``--vdim``. Flops: per token and head two
    products over the state (decay and update; read-out)."""
    from ..parts import ops

    heads, dk, dv, batch, tokens = args.q_heads, args.head_dim, args.vdim, args.batch, args.tokens
    runs, starts = [tokens] * batch, [0] * batch
    ctx = make_ctx([p for r in runs for p in range(r)], [i for i, r in enumerate(runs) for _ in range(r)], starts, runs)
    ctx.seq_slot = torch.arange(batch, dtype=torch.int32, device="cuda")
    total = batch * tokens
    widths = [heads * dk, heads * dk, heads * dv, heads * dv, heads, heads]
    columns = tuple(sum(widths[:i]) for i in range(6))
    proj = torch.randn(total, sum(widths), device="cuda")
    state = [torch.zeros(batch, heads, dk, dv, device="cuda"), torch.zeros(batch, heads, dk, device="cuda"), torch.zeros(batch, heads, device="cuda")]
    bias, norm = torch.zeros(heads, device="cuda"), torch.ones(heads * dv, device="cuda")
    out = torch.empty(total, heads * dv, device="cuda", dtype=torch.bfloat16)
    us = time_launches(lambda: ops.mlstm(ctx, proj, columns, bias, bias, 10.0, state, heads, dk, dv, norm, 1e-5, out), args.iters)
    moved = 4.0 * (total * (sum(widths) + 2 * heads * dv) + 2 * batch * heads * dk * (dv + 1)) + 2.0 * total * heads * dv
    return {"kernel": "mlstm (gates + recurrence + output)", "batch": batch, "tokens": tokens, "heads": heads, "dim": dk, "vdim": dv, "us": us,
            "us_per_token": us / tokens, "GBps": moved / us / 1e3, "TFLOPs": 5.0 * total * heads * dk * (dv + 1) / us / 1e6}


def bench_delta_general_recurrence(args) -> dict:
    """The generalized delta rule's recurrence (parts/delta_rule.py, ``general_delta``) over ``--batch`` requests of
    ``--tokens`` tokens each: ``--q-heads`` heads with states of ``--head-dim`` x ``--head-dim``. Flops: per token and head
    three products over the state (the unit key's dot; decay, removal and update; read-out)."""
    from ..parts import ops

    heads, dim, batch, tokens = args.q_heads, args.head_dim, args.batch, args.tokens
    runs, starts = [tokens] * batch, [0] * batch
    ctx = make_ctx([p for r in runs for p in range(r)], [i for i, r in enumerate(runs) for _ in range(r)], starts, runs)
    ctx.seq_slot = torch.arange(batch, dtype=torch.int32, device="cuda")
    total = batch * tokens
    r, k, v = (torch.randn(total, heads * dim, device="cuda") for _ in range(3))
    u = (k.view(total, heads, dim) / k.view(total, heads, dim).norm(dim=-1, keepdim=True)).reshape(total, heads * dim).contiguous()
    au = u * torch.rand_like(u)
    decay = torch.rand(total, heads * dim, device="cuda") * 0.2 + 0.8
    state = torch.zeros(batch, heads, dim, dim, device="cuda")
    out = torch.empty(total, heads * dim, device="cuda")
    us = time_launches(lambda: ops.delta_general_recurrence(ctx, r, k, v, decay, au, u, state, out, heads, dim, dim), args.iters)
    moved = 4.0 * (total * 7 * heads * dim + 2 * batch * heads * dim * dim)
    return {"kernel": "delta_general_recurrence", "batch": batch, "tokens": tokens, "heads": heads, "dim": dim, "us": us,
            "us_per_token": us / tokens, "GBps": moved / us / 1e3, "TFLOPs": 7.0 * total * heads * dim * dim / us / 1e6}


def bench_moe_experts(args) -> dict:
    """The routed experts' two products (parts/feed_forward.py, ``routed_experts``) for ``--tokens`` tokens of width
    ``--k``: ``--experts`` experts of inner width ``--n``, ``--top`` per token chosen at random; bfloat16 on tensor
    cores unless ``--plain``. Flops: 6 x slots x inner x width. Bytes: every chosen expert's weights once plus the
    slots' rows in and out."""
    from ..parts import ops

    tokens, width, ff, experts, top = args.tokens, args.k, args.n, args.experts, args.top
    options = {"moe": "plain"} if args.plain else ({"moe_stages": args.stages} if args.stages else {})  # --stages: ring depth of the tcgen05 form
    ctx = make_ctx(list(range(tokens)), [0] * tokens, options=options)
    ctx.dtype = torch.bfloat16
    h = torch.randn(tokens, width, device="cuda", dtype=torch.bfloat16)
    w_gate_up = torch.randn(experts, 2 * ff, width, device="cuda", dtype=torch.bfloat16) * width**-0.5
    w_down = torch.randn(experts, width, ff, device="cuda", dtype=torch.bfloat16) * ff**-0.5
    ids = torch.stack([torch.randperm(experts, device="cuda")[:top] for _ in range(tokens)]).to(torch.int32).contiguous()
    out = torch.empty(tokens * top, width, device="cuda")
    ctx.buffer = lambda name, shape, dtype=None, per_token=True: ctx.workspace.get(name, shape, dtype or torch.bfloat16, per_token=per_token)
    us = time_launches(lambda: ops.moe_experts(ctx, h, ids, w_gate_up, w_down, 7.0, out), args.iters)
    used = int(torch.unique(ids).numel())
    slots = tokens * top
    moved = 2.0 * used * 3 * ff * width + 2.0 * slots * (width + 2 * ff) + 4.0 * slots * width
    return {"kernel": "moe_experts (sort + gate/up + down)", "tokens": tokens, "width": width, "inner": ff, "experts": experts, "top": top,
            "experts_used": used, "us": us, "TFLOPs": 6.0 * slots * ff * width / us / 1e6, "GBps": moved / us / 1e3}


def bench_resident(args) -> dict:
    """One decode step as the resident kernel at a named shape: time per step, and for each kind of
    phase how long the slowest block takes to ask for its operand, to finish, and how long block 0
    then waits at the barrier (timestamps the kernel records when handed a trace buffer)."""
    import numpy as np

    from .. import models  # noqa: F401
    from ..config import parse_config
    from ..engine.engine import Engine
    from ..engine.loading import random_model
    from ..engine.runner import StepEntry
    from .presets import PRESETS

    _, config = parse_config(dict(PRESETS[args.shape]))
    model = random_model(config, seed=0, dtype="bfloat16", device="cuda:0")
    engine = Engine(model=model, max_num_sequences=16, max_model_length=2 * args.context, kv_cache_bytes=8 << 30,
                    prefill_chunk_size=2048, prefill_burst_size=2048, max_batch_tokens=2048 + 16, cuda_graphs=False,
                    decode_kernel="resident")
    runner = engine.runner
    if runner.options["resident"] is None:
        raise SystemExit("the resident kernel does not take this shape")
    rng = np.random.default_rng(0)
    ids = list(range(1, args.batch + 1))
    for rid in ids:
        engine.cache.open(rid)
        for begin in range(0, args.context, 2048):
            runner.step([StepEntry(rid, [int(t) for t in rng.integers(0, config.vocab_size, min(2048, args.context - begin))], ())])
    phases = 2 + 5 * len(model.schedule)
    trace = torch.zeros(phases * 4, dtype=torch.int64, device="cuda")
    runner.options["resident_trace"] = trace
    step = lambda: runner.step([StepEntry(rid, (int(rng.integers(0, config.vocab_size)),), (0,)) for rid in ids])
    for _ in range(3):
        step()
    trace.zero_()
    us = time_launches(step, args.iters)
    trace.zero_()
    step()
    torch.cuda.synchronize()
    runner.check()
    stamps = trace.cpu().numpy().reshape(phases, 4).astype(np.float64) / 1e3
    names = ["embedding"] + ["q/k/v", "attention", "output", "gate/up", "down"] * len(model.schedule) + ["head"]
    kinds: dict[str, list] = {}
    for name, (enter, asked, finished, left) in zip(names, stamps):
        asked = asked if asked > 0 else enter
        kinds.setdefault(name, []).append((asked - enter, finished - asked, max(left - finished, 0.0) if left > 0 else 0.0))
    summary = {
        name: dict(zip(("operand_asked_us", "work_us", "barrier_us"), (round(float(v), 2) for v in np.mean(rows, axis=0))))
        for name, rows in kinds.items()
    }
    engine.close()
    return {"kernel": "resident_decode", "shape": args.shape, "batch": args.batch, "context": args.context, "us_per_step": us,
            "kernel_us": float(stamps[-1, 2] - stamps[0, 0]), "phases": summary}


def bench_timeline(args) -> dict:
    """One layer of a replayed decode step on the timeline: for every kernel of the step's second
    layer, when its first block started, when it ended and how long after its predecessor's end
    (Kineto timestamps through torch.profiler; no kernel is replayed or serialised)."""
    import numpy as np
    from torch.profiler import ProfilerActivity, profile

    from .. import models  # noqa: F401
    from ..config import parse_config
    from ..engine.engine import Engine
    from ..engine.loading import random_model
    from ..engine.runner import StepEntry
    from .presets import PRESETS

    _, config = parse_config(dict(PRESETS[args.shape]))
    model = random_model(config, seed=0, dtype="bfloat16", device="cuda:0")
    kv_bytes = 2 * config.num_hidden_layers * config.num_key_value_heads * config.head_dim * 2 * args.batch * (args.context + 256)
    engine = Engine(model=model, max_num_sequences=max(16, args.batch), max_model_length=2 * args.context,
                    kv_cache_bytes=kv_bytes + (1 << 30), prefill_chunk_size=2048, prefill_burst_size=2048,
                    max_batch_tokens=2048 + max(16, args.batch))
    runner = engine.runner
    rng = np.random.default_rng(0)
    ids = list(range(1, args.batch + 1))
    for rid in ids:
        engine.cache.open(rid)
        for begin in range(0, args.context, 2048):
            runner.step([StepEntry(rid, [int(t) for t in rng.integers(0, config.vocab_size, min(2048, args.context - begin))], ())])
    step = lambda: runner.step([StepEntry(rid, (int(rng.integers(0, config.vocab_size)),), (0,)) for rid in ids])
    for _ in range(6):
        step()
    torch.cuda.synchronize()
    with profile(activities=[ProfilerActivity.CUDA]) as prof:
        for _ in range(3):
            step()
        torch.cuda.synchronize()
    events = sorted((e for e in prof.events() if e.device_type == torch.autograd.DeviceType.CUDA), key=lambda e: e.time_range.start)
    firsts = [i for i, e in enumerate(events) if "embedding" in e.name]
    if len(firsts) < 3:
        raise SystemExit("the profiler did not see three steps")
    per_step = firsts[2] - firsts[1]
    # The second layer of the middle step: from its first norm to the next layer's first norm
    # (two norm kernels per layer in the stock arrangement).
    norms = [i for i in range(firsts[1], firsts[2]) if "rmsnorm" in events[i].name]
    if len(norms) < 5:
        raise SystemExit("the step does not show two norm kernels per layer")
    start, per_layer = norms[2], norms[4] - norms[2]
    origin = events[firsts[1]].time_range.start
    rows, previous_end = [], events[start - 1].time_range.end
    for e in events[start : start + per_layer]:
        rows.append({"kernel": e.name[:60], "start_us": round(e.time_range.start - origin, 1),
                     "end_us": round(e.time_range.end - origin, 1), "after_us": round(e.time_range.end - previous_end, 1)})
        previous_end = e.time_range.end
    engine.close()
    return {"kernel": "decode step timeline", "shape": args.shape, "batch": args.batch, "context": args.context,
            "kernels_per_step": per_step, "layer_us": round(sum(r["after_us"] for r in rows), 1), "layer": rows}


def main(argv=None) -> int:
    parser = argparse.ArgumentParser(description=__doc__.split("\n\n")[0])
    parser.add_argument("kernel", choices=["gemm", "decode_attention", "prefill_attention", "resident", "timeline",
                                           "latent_decode_attention", "latent_prefill_attention", "delta_recurrence", "delta_step", "wkv_recurrence",
                                           "moe_experts", "mlstm", "delta_general_recurrence", "mixed_decode_attention",
                                           "mixed_prefill_attention"])
    parser.add_argument("--experts", type=int, default=32, help="moe_experts: number of experts")
    parser.add_argument("--top", type=int, default=4, help="moe_experts: experts per token")
    parser.add_argument("--rank", type=int, default=512, help="latent attention: size of the cached latent")
    parser.add_argument("--rot-dim", type=int, default=64, help="latent attention: size of the shared rotated key part")
    parser.add_argument("--vdim", type=int, default=128, help="delta_recurrence: value size per head")
    parser.add_argument("--shape", default="qwen2.5-1.5b", help="resident, timeline: a named model shape")
    parser.add_argument("--m", type=int, default=8)
    parser.add_argument("--n", type=int, default=17920)
    parser.add_argument("--k", type=int, default=1536)
    parser.add_argument("--swiglu", action="store_true")
    parser.add_argument("--f32-out", action="store_true")
    parser.add_argument("--library", action="store_true", help="time the vendor library's product instead")
    parser.add_argument("--gemm", default="auto", choices=["auto", "tcgen05", "skinny", "library"])
    parser.add_argument("--rotate", action="store_true", help="launch back to back over rotating copies of the weights")
    parser.add_argument("--trace", action="store_true",
                        help="with --rotate --gemm tcgen05: the blocks' own timestamps instead of the launch time")
    parser.add_argument("--plan", type=int, nargs=3, metavar=("STAGES", "BLOCKS", "CLUSTER"), default=None,
                        help="tcgen05 product: force ring depth, blocks aimed at and cluster width (0 = the planner's choice)")
    parser.add_argument("--batch", type=int, default=8)
    parser.add_argument("--context", type=int, default=2048)
    parser.add_argument("--tokens", type=int, default=2048)
    parser.add_argument("--q-heads", type=int, default=12)
    parser.add_argument("--kv-heads", type=int, default=2)
    parser.add_argument("--head-dim", type=int, default=128)
    parser.add_argument("--page", type=int, default=64)
    parser.add_argument("--window", type=int, default=0)
    parser.add_argument("--keep-first", type=int, default=0, help="attention: first keys that stay visible in front of the window")
    parser.add_argument("--sigmoid", action="store_true", help="attention: sigmoid weights instead of a softmax")
    parser.add_argument("--sink", action="store_true", help="attention: a sink per head in the softmax")
    parser.add_argument("--per-head", action="store_true", help="delta_recurrence: the form with one decay per head")
    parser.add_argument("--portions", default="auto", choices=["auto", "chunks", "tokens"], help="delta_recurrence --per-head: how portions are walked")
    parser.add_argument("--plain", action="store_true")
    parser.add_argument("--softcap", type=float, default=0.0, help="attention: cap of the scores (0: none)")
    parser.add_argument("--bias-reach", type=int, default=0, help="attention: a random bias by distance up to this many positions (0: none)")
    parser.add_argument("--chunk", type=int, default=0, help="attention: keys visible inside the query's chunk of this many positions (0: all)")
    parser.add_argument("--attention", default="auto", choices=["auto", "flash", "tcgen05"])
    parser.add_argument("--loader", default="auto", choices=["auto", "tma", "cp_async"], help="how decode attention loads keys and values")
    parser.add_argument("--splits", type=int, default=0, help="blocks per (request, kv head) in decode attention (0: the engine's rule)")
    parser.add_argument("--stages", type=int, default=0, help="ring depth of the TMA decode kernel (0: the engine's default)")
    parser.add_argument("--layers", type=int, default=1, help="attention: rotate over this many arenas")
    parser.add_argument("--iters", type=int, default=20)
    args = parser.parse_args(argv)
    if args.library:
        args.gemm = "library"
    if args.kernel == "gemm":
        result = bench_gemm(args)
    elif args.kernel == "resident":
        result = bench_resident(args)
    elif args.kernel == "timeline":
        result = bench_timeline(args)
    elif args.kernel.startswith("latent_"):
        result = bench_latent_attention(args, args.kernel == "latent_decode_attention")
    elif args.kernel == "delta_recurrence":
        result = bench_delta_recurrence(args)
    elif args.kernel == "delta_step":
        result = bench_delta_step(args)
    elif args.kernel == "wkv_recurrence":
        result = bench_wkv_recurrence(args)
    elif args.kernel == "moe_experts":
        result = bench_moe_experts(args)
    elif args.kernel == "mlstm":
        result = bench_mlstm(args)
    elif args.kernel == "delta_general_recurrence":
        result = bench_delta_general_recurrence(args)
    elif args.kernel.startswith("mixed_"):
        result = bench_attention(args, args.kernel == "mixed_decode_attention", mixed=True)
    else:
        result = bench_attention(args, args.kernel == "decode_attention")
    print(json.dumps(result))
    return 0


if __name__ == "__main__":
    sys.exit(main())
