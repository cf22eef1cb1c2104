"""Times one kernel of the library at a given size with CUDA events.

    python -m questwend_b200.kernels.microbench gemm --m 8 --n 24576 --k 4096 [--impl stream|small|library]
    python -m questwend_b200.kernels.microbench attn_decode --batch 8 --ctx 1152 [--heads 32 --kv-heads 8 --head-dim 128]
    python -m questwend_b200.kernels.microbench attn_prefill --tokens 2048
    python -m questwend_b200.kernels.microbench rmsnorm --m 8 --k 4096
    python -m questwend_b200.kernels.microbench sample --batch 8 --vocab 151936 --temp 0.8 --top-k 40 --top-p 0.95
    python -m questwend_b200.kernels.microbench moe --m 8 --k 2048 --n 1408 --experts 64 --top-k 6 --shared 2816
    python -m questwend_b200.kernels.microbench decode_shapes --m 8        (every product of a Qwen3-8B decode step)

Inputs rotate through enough copies to exceed the 126 MB L2, so every timed launch reads from HBM.
Prints one JSON line per case: microseconds (median of the timed launches), the bytes the kernel has to
move, and GB/s.  Also the program to put under ncu for a capture of one kernel on a small case.
"""
from __future__ import annotations

import argparse
import sys
import json
import math
import statistics

import torch

from . import ops

DEV = torch.device("cuda:0")

L2_BYTES = 126 * 1024 * 1024


def _time(fn, n_variants: int, iters: int, warmup: int = 3, burst: int = 10) -> float:
    """Median microseconds per launch; each timed region holds `burst` launches back to back, so that
    the host's launch overhead does not hide a kernel of a few microseconds."""
    for i in range(warmup):
        fn(i % n_variants)
    torch.cuda.synchronize()
    burst = max(burst, n_variants)
    graph = torch.cuda.CUDAGraph()          # the burst is replayed from a graph: no host time between launches
    with torch.cuda.graph(graph):
        for k in range(burst):
            fn(k % n_variants)
    graph.replay()
    torch.cuda.synchronize()
    times = []
    for _ in range(iters):
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        graph.replay()
        b.record()
        torch.cuda.synchronize()
        times.append(a.elapsed_time(b) * 1e3 / burst)
    return statistics.median(times)


def bench_gemm(M: int, N: int, K: int, impl: str, iters: int, dtype=torch.bfloat16, tile_n=None) -> dict:
    elem = 2 if dtype == torch.bfloat16 else 4
    copies = max(2, math.ceil(2 * L2_BYTES / (N * K * elem)))
    ws = [torch.randn(N, K, device="cuda", dtype=torch.float32).mul_(0.02).to(dtype) for _ in range(copies)]
    x = torch.randn(M, K, device="cuda").to(dtype)
    if impl == "stream":
        fn = lambda i: ops.gemm_stream(x, ws[i])
    elif impl == "ring":
        fn = lambda i: ops.gemm_ring(x, ws[i])
    elif impl == "ring_swiglu":
        fn = lambda i: ops.gemm_ring_swiglu(x, ws[i])
    elif impl == "ring_add":                # added onto a 32-bit matrix (the residual stream) in the epilogue
        acc = torch.zeros(M, N, device="cuda")
        fn = lambda i: ops.gemm_ring(x, ws[i], residual=acc)
    elif impl == "ring_split":              # equal shares per block, the pieces left as planes (where whole tiles are as
        plan = ops.ring_split_plan(N, K, x.device)          # good there is no split form: the plain one is timed)
        fn = (lambda i: ops.gemm_ring_split(x, ws[i], plan)) if plan else (lambda i: ops.gemm_ring(x, ws[i]))
    elif impl == "stream_swiglu":
        fn = lambda i: ops.gemm_stream_swiglu(x, ws[i])
    elif impl == "small":
        fn = lambda i: ops.gemm_small(x, ws[i])
    elif impl == "tc":
        fn = lambda i: ops.gemm_tc(x, ws[i], tile_n=tile_n)
    elif impl == "tc_add":
        acc = torch.zeros(M, N, device="cuda")
        fn = lambda i: ops.gemm_tc(x, ws[i], epilogue="add", out=acc, tile_n=tile_n)
    elif impl == "tc_swiglu":
        fn = lambda i: ops.gemm_tc(x, ws[i], epilogue="swiglu", tile_n=tile_n)
    elif impl == "library_add":
        acc = torch.zeros(M, N, device="cuda")
        fn = lambda i: torch.addmm(acc, x, ws[i].t(), out_dtype=torch.float32, out=acc)
    elif impl == "library_swiglu":
        fn = lambda i: ops.silu_mul(torch.mm(x, ws[i].t(), out_dtype=torch.float32), torch.bfloat16, ops.GATE_UP_GROUP)
    else:
        fn = (lambda i: torch.mm(x, ws[i].t(), out_dtype=torch.float32)) if dtype == torch.bfloat16 else \
             (lambda i: torch.mm(x, ws[i].t()))
    us = _time(fn, copies, iters)
    nbytes = N * K * elem + M * K * elem + M * N * 4
    return {"kernel": f"gemm_{impl}", "M": M, "N": N, "K": K, "us": us, "bytes": nbytes,
            "GBps": nbytes / us / 1e3, "TFLOPs": 2.0 * M * N * K / us / 1e6}


def bench_attn_decode(B, ctx, Hq, Hkv, hd, iters, dtype=torch.bfloat16, split=0, runs_target=0, run_pages_max=0, max_len=0,
                      fused=False) -> dict:
    page = ops.PAGE_SIZE
    pages_per = math.ceil(ctx / page)
    per_copy = B * pages_per
    elem = 2 if dtype == torch.bfloat16 else 4
    copy_bytes = 2 * per_copy * Hkv * page * hd * elem
    copies = max(2, math.ceil(2 * L2_BYTES / copy_bytes))
    n_pages = per_copy * copies
    k_pool = torch.randn(n_pages, Hkv, page, hd, device="cuda").to(dtype)
    v_pool = torch.randn(n_pages, Hkv, page, hd, device="cuda").to(dtype)
    tables = [(torch.arange(per_copy, dtype=torch.int32, device="cuda") + c * per_copy).reshape(B, pages_per).contiguous()
              for c in range(copies)]
    q = torch.randn(B, Hq, hd, device="cuda").to(dtype)
    seq_len = torch.full((B,), ctx, dtype=torch.int32, device="cuda")
    if split:       # runs of exactly this many keys instead of the kernels' own choice
        how = dict(split_tokens=split, runs_target=1, run_pages_max=max(1, split // page))
    else:
        how = {}
        if runs_target:
            how["runs_target"] = runs_target
        if run_pages_max:
            how["run_pages_max"] = run_pages_max
    max_len = max_len or ctx            # the bound a graph is captured for may be larger than the sequences
    fn = lambda i: ops.attn_decode(q, k_pool, v_pool, tables[i], seq_len, 1 / math.sqrt(hd), max_len, **how)
    if fused:       # the kernel that also norms and rotates q and k and writes the new key and value (what a step of few sequences runs)
        how.pop("split_tokens", None)
        qkv = torch.randn(B, (Hq + 2 * Hkv) * hd, device="cuda")
        w = torch.ones(hd, device="cuda")
        inv = torch.tensor([1e6 ** (-2.0 * i / hd) for i in range(hd // 2)], dtype=torch.float64, device="cuda")
        cos, sin = ops.rope_table(seq_len - 1, inv)
        fn = lambda i: ops.attn_decode_fused(qkv, w, w, cos, sin, 1e-6, k_pool, v_pool, tables[i], seq_len, 1 / math.sqrt(hd), max_len,
                                             Hq, Hkv, hd, **how)
    us = _time(fn, copies, iters)
    nbytes = 2 * B * ctx * Hkv * hd * elem
    return {"kernel": "attn_decode_fused" if fused else "attn_decode", "B": B, "ctx": ctx, "Hq": Hq, "Hkv": Hkv, "hd": hd, "us": us, "bytes": nbytes,
            "GBps": nbytes / us / 1e3}


def bench_attn_prefill(T, Hq, Hkv, hd, iters, dtype=torch.bfloat16) -> dict:
    page = ops.PAGE_SIZE
    n_pages = math.ceil(T / page)
    k_pool = torch.randn(n_pages, Hkv, page, hd, device="cuda").to(dtype)
    v_pool = torch.randn(n_pages, Hkv, page, hd, device="cuda").to(dtype)
    table = torch.arange(n_pages, dtype=torch.int32, device="cuda").reshape(1, n_pages)
    q = torch.randn(T, Hq, hd, device="cuda").to(dtype)
    cu = torch.tensor([0, T], dtype=torch.int32, device="cuda")
    pos0 = torch.zeros(1, dtype=torch.int32, device="cuda")
    fn = lambda i: ops.attn_prefill(q, k_pool, v_pool, table, cu, pos0, T, 1 / math.sqrt(hd))
    us = _time(fn, 1, iters)
    flops = 4.0 * Hq * hd * T * (T + 1) / 2
    return {"kernel": "attn_prefill", "T": T, "Hq": Hq, "Hkv": Hkv, "hd": hd, "us": us, "TFLOPs": flops / us / 1e6}


def bench_rmsnorm(M, K, iters) -> dict:
    copies = max(2, math.ceil(2 * L2_BYTES / (M * K * 4)))
    copies = min(copies, 64)
    xs = [torch.randn(M, K, device="cuda") for _ in range(copies)]
    d = torch.randn(M, K, device="cuda")
    w = torch.ones(K, device="cuda")
    fn = lambda i: ops.rmsnorm(xs[i], w, 1e-6, torch.bfloat16, delta=d, write_sum=True)
    us = _time(fn, copies, iters)
    return {"kernel": "rmsnorm", "M": M, "K": K, "us": us}


def bench_rope(T, Hq, Hkv, hd, iters, store_kv=True) -> dict:
    """q/k norm + rotation + cache write of one prompt of T tokens (``rope``)."""
    page = ops.PAGE_SIZE
    n_pages = math.ceil(T / page)
    copies = max(2, min(8, math.ceil(2 * L2_BYTES / (T * (Hq + 2 * Hkv) * hd * 4))))
    qkvs = [torch.randn(T, (Hq + 2 * Hkv) * hd, device="cuda") for _ in range(copies)]
    k_pool = torch.zeros(n_pages * copies, Hkv, page, hd, device="cuda", dtype=torch.bfloat16)
    v_pool = torch.zeros_like(k_pool)
    tables = [(torch.arange(n_pages, dtype=torch.int32, device="cuda") + c * n_pages).reshape(1, n_pages) for c in range(copies)]
    w = torch.ones(hd, device="cuda")
    pos = torch.arange(T, dtype=torch.int32, device="cuda")
    seq = torch.zeros(T, dtype=torch.int32, device="cuda")
    inv_freq = torch.tensor([1e6 ** (-2.0 * i / hd) for i in range(hd // 2)], dtype=torch.float64, device="cuda")
    cos, sin = ops.rope_table(pos, inv_freq)
    fn = lambda i: ops.qk_norm_rope_store(qkvs[i], w, w, cos, sin, seq, pos, tables[i], k_pool, v_pool, Hq, Hkv, hd, hd, 1e-6,
                                          store_kv=store_kv)
    us = _time(fn, copies, iters)
    nbytes = T * (Hq + 2 * Hkv) * hd * 4 + T * (Hq + 2 * Hkv) * hd * 2
    return {"kernel": "qk_norm_rope_store", "T": T, "Hq": Hq, "Hkv": Hkv, "hd": hd, "us": us, "bytes": nbytes, "GBps": nbytes / us / 1e3}


def bench_sample(B, V, temperature, top_k, top_p, iters, spread=3.0) -> dict:
    copies = max(2, math.ceil(2 * L2_BYTES / (B * V * 4)))
    copies = min(copies, 64)
    rows = [torch.randn(B, V, device="cuda") * spread for _ in range(copies)]
    seq = torch.arange(B, dtype=torch.int32, device="cuda")
    out = torch.empty(B, dtype=torch.int32, device="cuda")
    fn = lambda i: ops.sample(rows[i], temperature, top_k=top_k, top_p=top_p, seed=1, sequence_index=seq, step=i, out=out)
    us = _time(fn, copies, iters)
    return {"kernel": "sample", "B": B, "V": V, "temperature": temperature, "top_k": top_k, "top_p": top_p, "us": us,
            "bytes": B * V * 4, "GBps": B * V * 4 / us / 1e3}


def bench_pool_attention(B, tokens, ctx, Hq, Hkv, dim, vdim, window, pool, iters, dtype=torch.bfloat16) -> dict:
    """Attention over a window and pooled blocks: ``B`` sequences that bring ``tokens`` new tokens each after ``ctx``
    cached ones (tokens = 1: the decode kernels; more: the prompt kernel).  Random keys, values and block rows."""
    from ..cache.manager import CacheManager
    from ..engine.engine import StepEntry, build_step_context
    from ..parts.base import KVSpec
    kinds = (KVSpec(Hkv, dim, window, value_dim=vdim), KVSpec(Hkv, dim, window, value_dim=vdim, stride=max(1, pool)))
    n = ctx + tokens
    cache = CacheManager([(kinds, None, None)], B * n + 64 * B, B, n + 64, dtype, DEV)
    slots = cache.open(B)
    if ctx:
        build_step_context(cache, [StepEntry(s, [0] * ctx, []) for s in slots], 10, DEV)
        for s in slots:
            cache.advance(s, ctx)
    rows, blocks = cache.unit_cache(0), cache.unit_cache(0).more[0]
    for u in (rows, blocks):
        u.k_pool.normal_()
        u.v_pool.normal_()
    step = build_step_context(cache, [StepEntry(s, [0] * tokens, []) for s in slots], 10, DEV)[0]
    q = torch.randn(B * tokens, Hq, dim, device=DEV).to(dtype)
    cs = torch.ones(B * tokens, vdim // 2, device=DEV)
    t0, t1 = step.page_tables[rows.group_id], step.page_tables[blocks.group_id]
    us = _time(lambda i: ops.pool_attention(q, rows.k_pool, rows.v_pool, blocks.k_pool, blocks.v_pool, t0, t1, step, cs, cs,
                                            dim ** -0.5, window, pool, False), 1, iters, burst=3)
    seen = sum(min(p + 1, window or p + 1) + (max(0, (p - window + 1) // pool) if window and pool else 0) for p in range(ctx, n))
    return {"what": "pool_attention", "batch": B, "tokens": tokens, "ctx": ctx, "heads": Hq, "kv_heads": Hkv, "dim": dim,
            "vdim": vdim, "window": window, "pool": pool, "us": us,
            "tflops_of_visible_keys": 2 * B * Hq * (dim + vdim) * seen / us / 1e6,
            "gb_s_of_visible_rows": (B * Hkv * (seen / tokens) * (dim + vdim) * q.element_size() / us / 1e3) if tokens == 1 else None}


def bench_maps_attention(B, tokens, ctx, Hq, Hkv, maps, dim, vdim, softcap, chunk, iters, dtype=torch.bfloat16, impl="auto") -> dict:
    """Attention with ``maps`` score maps per head (two: differential) over the same values: ``B`` sequences that bring
    ``tokens`` new tokens each after ``ctx`` cached ones (tokens = 1: the decode kernels; more: a prompt kernel).  Random
    queries, keys and values."""
    from ..cache.manager import CacheManager
    from ..engine.engine import StepEntry, build_step_context
    from ..parts.base import KVSpec
    n = ctx + tokens
    cache = CacheManager([(KVSpec(Hkv, maps * dim, 0, value_dim=vdim), None, None)], B * n + 64 * B, B, n + 64, dtype, DEV)
    slots = cache.open(B)
    if ctx:
        build_step_context(cache, [StepEntry(s, [0] * ctx, []) for s in slots], 10, DEV)
        for s in slots:
            cache.advance(s, ctx)
    unit = cache.unit_cache(0)
    unit.k_pool.normal_()
    unit.v_pool.normal_()
    step = build_step_context(cache, [StepEntry(s, [0] * tokens, []) for s in slots], 10, DEV)[0]
    q = torch.randn(B * tokens, Hq, maps * dim, device=DEV).to(dtype)
    table = step.page_tables[unit.group_id]
    us = _time(lambda i: ops.maps_attention(q, unit.k_pool, unit.v_pool, table, step, maps, dim ** -0.5, softcap=softcap, chunk=chunk,
                                            lam=0.5, norm_out=maps == 2, eps=1e-5, out_scale=0.5, impl=impl), 1, iters, burst=3)
    seen = sum(p + 1 - ((p // chunk) * chunk if chunk else 0) for p in range(ctx, n))
    return {"what": "maps_attention", "batch": B, "tokens": tokens, "ctx": ctx, "heads": Hq, "kv_heads": Hkv, "maps": maps,
            "dim": dim, "vdim": vdim, "softcap": softcap, "chunk": chunk, "impl": impl, "us": us,
            "tflops_of_visible_keys": 2 * B * Hq * maps * (dim + vdim) * seen / us / 1e6,
            "gb_s_of_visible_rows": (B * Hkv * (seen / tokens) * (maps * dim + vdim) * q.element_size() / us / 1e3) if tokens == 1 else None}


def bench_shaped_attention(B, tokens, ctx, Hq, Hkv, dim, softcap, window, extras, iters, dtype=torch.bfloat16, impl="auto") -> dict:
    """Attention with shaped scores: ``B`` sequences that bring ``tokens`` new tokens each after ``ctx`` cached ones (tokens = 1:
    the decode kernels; more: a prompt kernel).  ``extras``: words out of "slopes sink temp mix gate".  Random queries, keys and
    values; keys and values of one size."""
    from ..cache.manager import CacheManager
    from ..engine.engine import StepEntry, build_step_context
    from ..parts.base import KVSpec
    n = ctx + tokens
    cache = CacheManager([(KVSpec(Hkv, dim, window, value_dim=dim), None, None)], B * n + 64 * B, B, n + 64, dtype, DEV)
    slots = cache.open(B)
    if ctx:
        build_step_context(cache, [StepEntry(s, [0] * ctx, []) for s in slots], 10, DEV)
        for s in slots:
            cache.advance(s, ctx)
    unit = cache.unit_cache(0)
    unit.k_pool.normal_()
    unit.v_pool.normal_()
    step = build_step_context(cache, [StepEntry(s, [0] * tokens, []) for s in slots], 10, DEV)[0]
    q = torch.randn(B * tokens, Hq, dim, device=DEV).to(dtype)
    table = step.page_tables[unit.group_id]
    kw = {"softcap": softcap, "window": window, "impl": impl}
    if "slopes" in extras:
        kw["slopes"] = torch.tensor([2.0 ** (-8.0 * (h + 1) / Hq) for h in range(Hq)], device=DEV)
    if "sink" in extras:
        kw["sinks"] = torch.zeros(Hq, device=DEV)
    if "temp" in extras:
        kw["head_scale"] = torch.ones(Hq, device=DEV)
    if "mix" in extras:
        kw["head_mix"] = (torch.eye(Hq, device=DEV) + 0.1 * torch.randn(Hq, Hq, device=DEV)).contiguous()
    if "gate" in extras:
        kw["gate"] = torch.randn(B * tokens, Hq, device=DEV)
    us = _time(lambda i: ops.bias_attention(q, unit.k_pool, unit.v_pool, table, step, dim ** -0.5, **kw), 1, iters, burst=3)
    seen = sum(min(p + 1, window) if window else p + 1 for p in range(ctx, n))
    value_heads = Hkv if "mix" in extras else 1
    return {"what": "shaped_attention", "batch": B, "tokens": tokens, "ctx": ctx, "heads": Hq, "kv_heads": Hkv, "dim": dim,
            "softcap": softcap, "window": window, "extras": extras, "impl": impl, "us": us,
            "tflops_of_visible_keys": 2 * B * Hq * dim * (1 + value_heads) * seen / us / 1e6,
            "gb_s_of_visible_rows": (B * Hkv * (seen / tokens) * 2 * dim * q.element_size() / us / 1e3) if tokens == 1 else None}


def bench_moe(T, D, F, E, top, shared, activation, iters, dtype=torch.bfloat16) -> dict:
    """Routed experts of width ``F`` for ``T`` tokens of ``D`` values, each with ``top`` random experts out of ``E``, and a
    shared expert of width ``shared`` (0: none): the expert-streaming kernels, or the sorted form where that fits."""
    gated = activation == "gated_silu"
    up = (0.02 * torch.randn(E, (2 if gated else 1) * F, D, device=DEV)).to(dtype)
    down = (0.02 * torch.randn(E, D, F, device=DEV)).to(dtype)
    s_up, s_down = ((0.02 * torch.randn(shared, D, device=DEV)).to(dtype), (0.02 * torch.randn(D, shared, device=DEV)).to(dtype)) if shared else (None, None)
    x = torch.randn(T, D, device=DEV).to(dtype)
    gate = torch.rand(T, device=DEV) if shared else None
    # one choice for every copy of the inputs, so that the chosen experts do not stay in L2
    routes = [ops.moe_route(torch.randn(T, E, device=DEV), top, True, scores="sigmoid") for _ in range(8)]
    grouped = ops.moe_grouped_fits(x, up, down)
    if grouped:
        out = torch.zeros(T, D, device=DEV)
        fn = lambda i: ops.moe_experts_grouped(x, up, down, *routes[i % 8], activation, shared=out if shared else None, gate=gate)
    else:
        fn = lambda i: ops.moe_experts(x, up, down, *routes[i % 8], activation, s_up, s_down, gate)
    us = _time(fn, 8, iters)
    used = statistics.mean(len(torch.unique(c)) for c, _ in routes)
    per = (3 if gated else 2) * D * F
    n_bytes = (used * per + 2 * D * shared) * x.element_size()
    return {"what": "moe", "tokens": T, "width": D, "expert": F, "experts": E, "top": top, "shared": shared, "activation": activation,
            "form": "grouped" if grouped else "streamed", "us": us, "experts_used": used, "bytes": n_bytes, "gb_s": n_bytes / us / 1e3,
            "tflops": 2 * T * top * per / us / 1e6}


def bench_mlstm(B, tokens, H, K, P, iters) -> dict:
    """The mLSTM's matrix memory (``H`` heads of ``K`` x ``P``, 32-bit): ``B`` sequences that bring ``tokens`` new tokens each
    (1: the kernel for single tokens; 64 and more: the chunked form; else the scan)."""
    from types import SimpleNamespace
    T, at = B * tokens, H * (2 * K + 2 * P)
    proj = torch.randn(T, at + -(-2 * H // 8) * 8, device=DEV)
    bias = torch.zeros(H, device=DEV)
    state, m = torch.zeros(B, H, P + 1, K, device=DEV), torch.zeros(B, H, P + 1, device=DEV)
    step = SimpleNamespace(cu_seqlens=torch.arange(0, T + 1, tokens, device=DEV).int(), slots=torch.arange(B, device=DEV).int(), n_seqs=B,
                           max_new=tokens, single_token=tokens == 1)
    us = _time(lambda i: ops.mlstm_scan(proj, at, at + H, bias, bias, 15.0, state, m, step, H, K, P, K ** -0.5, 1e-6), 1, iters, burst=3)
    n_bytes = 4 * (T * H * (2 * K + 2 * P + 3) + 2 * B * H * (P + 1) * K)
    return {"what": "mlstm", "batch": B, "tokens": tokens, "heads": H, "key": K, "value": P, "us": us, "bytes": n_bytes,
            "gb_s": n_bytes / us / 1e3, "tflops": T * H * 4 * K * (P + 1) / us / 1e6}


def main() -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("what", choices=["gemm", "attn_decode", "attn_prefill", "rmsnorm", "rope", "decode_shapes", "sample", "pool_attn", "maps_attn", "shaped_attn", "moe", "mlstm"])
    ap.add_argument("--m", type=int, default=8)
    ap.add_argument("--n", type=int, default=24576)
    ap.add_argument("--k", type=int, default=4096)
    ap.add_argument("--impl", default="stream", choices=["stream", "stream_swiglu", "ring", "ring_swiglu", "ring_add", "ring_split", "small", "library", "tc", "tc_add", "tc_swiglu", "library_add", "library_swiglu"])
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--ctx", type=int, default=1152)
    ap.add_argument("--tokens", type=int, default=2048)
    ap.add_argument("--heads", type=int, default=32)
    ap.add_argument("--kv-heads", type=int, default=8)
    ap.add_argument("--head-dim", type=int, default=128)
    ap.add_argument("--vocab", type=int, default=151936)
    ap.add_argument("--temp", type=float, default=0.8)
    ap.add_argument("--top-k", type=int, default=40)
    ap.add_argument("--top-p", type=float, default=0.95)
    ap.add_argument("--iters", type=int, default=20)
    ap.add_argument("--tile-n", type=int, default=None)
    ap.add_argument("--max-len", type=int, default=0, help="decode attention: the bound on the lengths (default: the context)")
    ap.add_argument("--split", type=int, default=0, help="keys per run of the decode attention kernel (0: its own choice)")
    ap.add_argument("--runs-target", type=int, default=0, help="tensor-core decode attention: about this many runs a sequence")
    ap.add_argument("--run-pages-max", type=int, default=0, help="tensor-core decode attention: at most this many pages a run")
    ap.add_argument("--fused", action="store_true", help="decode attention with the q/k norm, rotation and cache write inside")
    ap.add_argument("--value-dim", type=int, default=0, help="pool_attn, mlstm: size of a value (default: the head size)")
    ap.add_argument("--window", type=int, default=1024, help="pool_attn: the window")
    ap.add_argument("--maps", type=int, default=2, help="maps_attn: score maps per head")
    ap.add_argument("--softcap", type=float, default=0.0, help="maps_attn: the cap on the scores (0: none)")
    ap.add_argument("--chunk", type=int, default=0, help="maps_attn: positions per chunk (0: plain causal)")
    ap.add_argument("--attn-impl", default="auto", choices=["auto", "tc", "mma", "plain"], help="maps_attn: the prompt kernel")
    ap.add_argument("--pool", type=int, default=16, help="pool_attn: tokens per pooled block")
    ap.add_argument("--experts", type=int, default=64, help="moe: experts (--m tokens, --k their width, --n an expert's width, --top-k choices)")
    ap.add_argument("--shared", type=int, default=0, help="moe: width of the shared expert (0: none)")
    ap.add_argument("--activation", default="gelu", help="moe: the experts' activation ('gated_silu': gated experts)")
    ap.add_argument("--extras", default="", help="shaped_attn: words out of 'slopes sink temp mix gate'")
    args = ap.parse_args()
    dtype = torch.bfloat16 if args.dtype == "bfloat16" else torch.float32
    if args.what == "gemm":
        print(json.dumps(bench_gemm(args.m, args.n, args.k, args.impl, args.iters, dtype, args.tile_n)))
    elif args.what == "decode_shapes":
        for name, n, k in (("qkv", 6144, 4096), ("o", 4096, 4096), ("gate_up", 24576, 4096), ("down", 4096, 12288),
                           ("lm_head", 151936, 4096)):
            r = bench_gemm(args.m, n, k, args.impl, args.iters, dtype, args.tile_n)
            r["name"] = name
            print(json.dumps(r))
    elif args.what == "attn_decode":
        print(json.dumps(bench_attn_decode(args.batch, args.ctx, args.heads, args.kv_heads, args.head_dim, args.iters, dtype, args.split,
                                           args.runs_target, args.run_pages_max, fused=args.fused, max_len=args.max_len)))
    elif args.what == "pool_attn":
        print(json.dumps(bench_pool_attention(args.batch, args.tokens, args.ctx if args.tokens == 1 else 0, args.heads, args.kv_heads,
                                              args.head_dim, args.value_dim or args.head_dim, args.window, args.pool, args.iters, dtype)))
    elif args.what == "maps_attn":
        print(json.dumps(bench_maps_attention(args.batch, args.tokens, args.ctx if args.tokens == 1 else 0, args.heads, args.kv_heads,
                                              args.maps, args.head_dim, args.value_dim or args.head_dim, args.softcap, args.chunk,
                                              args.iters, dtype, args.attn_impl)))
    elif args.what == "shaped_attn":
        print(json.dumps(bench_shaped_attention(args.batch, args.tokens, args.ctx if args.tokens == 1 else 0, args.heads, args.kv_heads,
                                                args.head_dim, args.softcap, args.window if "--window" in sys.argv else 0, args.extras,
                                                args.iters, dtype, args.attn_impl)))
    elif args.what == "moe":
        print(json.dumps(bench_moe(args.m, args.k, args.n, args.experts, args.top_k, args.shared, args.activation, args.iters, dtype)))
    elif args.what == "mlstm":
        print(json.dumps(bench_mlstm(args.batch, args.tokens, args.heads, args.head_dim, args.value_dim or args.head_dim, args.iters)))
    elif args.what == "sample":
        print(json.dumps(bench_sample(args.batch, args.vocab, args.temp, args.top_k, args.top_p, args.iters)))
    elif args.what == "attn_prefill":
        print(json.dumps(bench_attn_prefill(args.tokens, args.heads, args.kv_heads, args.head_dim, args.iters, dtype)))
    elif args.what == "rope":
        print(json.dumps(bench_rope(args.tokens, args.heads, args.kv_heads, args.head_dim, args.iters)))
    else:
        print(json.dumps(bench_rmsnorm(args.m, args.k, args.iters)))
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
