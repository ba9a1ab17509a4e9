"""Per-kernel timings at the Llama-8B shapes: ``python -m mfq_b200.ops.bench_kernels [--json out.json]``.

Each kernel is timed in isolation with CUDA events over ``reps`` launches after a warm-up, rotating through
enough independent weight copies that every launch reads its weights from HBM (more than 4x the 126 MB L2),
and reported against the measured roofline denominators (copy bandwidth / cuBLAS bf16 rate) when
``MEASURED_PEAKS.json`` is present in the working directory.
"""

from __future__ import annotations

import argparse
import json
import math
import os

import torch

from . import kernels as K
from . import reference as ref
from ..engine.kv_cache import PagedKVCache

L2_BYTES = 126 << 20


def time_ms(fn, reps: int, warmup: int = 3) -> float:
    """Device time per launch: ``reps`` launches captured in one CUDA graph, best of three replays (graph
    replay removes the host launch cost, which would otherwise hide kernels of a few microseconds)."""
    for i in range(warmup):
        fn(i)
    torch.cuda.synchronize()
    side = torch.cuda.Stream()
    side.wait_stream(torch.cuda.current_stream())
    graph = torch.cuda.CUDAGraph()
    with torch.cuda.stream(side):
        fn(0)
    torch.cuda.current_stream().wait_stream(side)
    with torch.cuda.graph(graph):
        for i in range(reps):
            fn(i)
    best = float("inf")
    for _ in range(3):
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        a.record()
        graph.replay()
        b.record()
        torch.cuda.synchronize()
        best = min(best, a.elapsed_time(b) / reps)
    return best


def peaks() -> dict:
    if os.path.exists("MEASURED_PEAKS.json"):
        p = json.load(open("MEASURED_PEAKS.json"))
        return {"hbm_gbs": p["hbm_gbs"], "tflops": p["bf16_tflops"], "kind": "measured"}
    return {"hbm_gbs": 6650.0, "tflops": 1590.0, "kind": "fallback"}


def bench_gemm(m: int, n: int, k: int, reps: int, splits=None, tile=None) -> dict:
    copies = max(1, min(16, math.ceil(4 * L2_BYTES / (n * k))))
    w = [torch.randint(-100, 100, (n, k), device="cuda", dtype=torch.int8).view(torch.float8_e4m3fn) for _ in range(copies)]
    ws = torch.rand((math.ceil(n / 128), k // 128), device="cuda") * 0.01 + 0.001
    x = torch.randint(-100, 100, (m, k), device="cuda", dtype=torch.int8).view(torch.float8_e4m3fn)
    xs = torch.rand(m, device="cuda") * 0.01 + 0.001
    out = torch.empty((m, n), device="cuda", dtype=torch.bfloat16)
    ms = time_ms(lambda i: K.fp8_gemm(x, xs, w[i % copies], ws, out=out, splits=splits, token_tile=tile), reps)
    byt = n * k + m * k + 2 * m * n
    gemv = splits is None and tile is None and K.use_gemv(m, n, k)
    return {"kernel": "fp8_gemv" if gemv else "fp8_gemm", "m": m, "n": n, "k": k, "us": ms * 1e3, "gbs": byt / ms / 1e6,
            "tflops": 2 * m * n * k / ms / 1e9, "splits": splits if splits else K.pick_splits(m, n, k)}


def bench_w4_gemm(m: int, n: int, k: int, reps: int, splits=None) -> dict:
    """4-bit in-pipeline-decode GEMM: same shapes as the FP8 GEMM, 5 bits per weight of HBM traffic."""
    from . import w4
    copies = max(1, min(16, math.ceil(4 * L2_BYTES / (n * k * 5 // 8))))
    base = w4.quantize_torch(torch.randn((n, k), device="cuda") * 0.02)
    ws = [base] + [w4.W4Weight(base.packed.clone(), base.group.clone(), n, k, base.group_size) for _ in range(copies - 1)]
    x = torch.randn((m, k), device="cuda").to(torch.bfloat16)
    out = torch.empty((m, n), device="cuda", dtype=torch.bfloat16)
    ms = time_ms(lambda i: w4.w4_gemm(x, ws[i % copies], out=out, splits=splits), reps)
    byt = n * k * 5 // 8 + 2 * m * k + 2 * m * n
    return {"kernel": "w4_gemm", "m": m, "n": n, "k": k, "us": ms * 1e3, "gbs": byt / ms / 1e6, "tflops": 2 * m * n * k / ms / 1e9}


def bench_attn(batch: int, ctx: int, hq: int, hk: int, d: int, splits: int, reps: int) -> dict:
    pages_per = math.ceil(ctx / 16)
    layers = max(1, math.ceil(4 * L2_BYTES / (batch * ctx * hk * d * 2)))
    cache = PagedKVCache(layers=layers, kv_heads=hk, head_dim=d, num_pages=batch * pages_per + 1, max_seqs=batch,
                         max_pages_per_seq=pages_per, device="cuda")
    cache.k.view(torch.int8).random_(-100, 100)
    cache.v.view(torch.int8).random_(-100, 100)
    cache.k_scale.fill_(0.01)
    cache.v_scale.fill_(0.01)
    for b in range(batch):
        cache.assign(b, b, ctx)
    q = torch.randn((batch, hq, d), device="cuda").to(torch.bfloat16)
    sl = torch.full((batch,), ctx, dtype=torch.int32, device="cuda")
    out = torch.empty_like(q)
    kvs = [cache.layer(i) for i in range(layers)]
    ms = time_ms(lambda i: K.paged_attn_decode(q, kvs[i % layers], cache.block_table, sl, sm_scale=0.088, splits=splits, out=out), reps)
    byt = batch * ctx * hk * (2 * d + 8)
    return {"kernel": "paged_attn_decode", "batch": batch, "ctx": ctx, "hq": hq, "hk": hk, "d": d, "splits": splits, "us": ms * 1e3, "gbs": byt / ms / 1e6}


def bench_mla_decode(batch: int, ctx: int, heads: int, splits: int, reps: int) -> dict:
    """Shared-row latent attention: 576-wide key rows and their 512-wide latent as values, one row per token."""
    from . import mla as mla_ops
    pages_per = math.ceil(ctx / 16)
    layers = max(1, math.ceil(4 * L2_BYTES / (batch * ctx * 2 * 576)))
    cache = PagedKVCache(layers=layers, kv_heads=1, head_dim=576, num_pages=batch * pages_per + 1, max_seqs=batch,
                         max_pages_per_seq=pages_per, device="cuda")
    cache.k.view(torch.int8).random_(-100, 100)
    cache.v.view(torch.int8).random_(-100, 100)
    cache.k_scale.fill_(0.01)
    cache.v_scale.fill_(0.01)
    for b in range(batch):
        cache.assign(b, b, ctx)
    q = torch.randn((batch, heads, 576), device="cuda").to(torch.bfloat16)
    sl = torch.full((batch,), ctx, dtype=torch.int32, device="cuda")
    out = torch.empty((batch, heads, 512), dtype=torch.bfloat16, device="cuda")
    kvs = [cache.layer(i) for i in range(layers)]
    ms = time_ms(lambda i: mla_ops.decode(q, kvs[i % layers], cache.block_table, sl, sm_scale=0.07, splits=splits, out=out), reps)
    byt = batch * ctx * (576 + 512 + 8) * math.ceil(heads / 16)  # every 16-head tile streams the rows once
    return {"kernel": "mla_decode", "batch": batch, "ctx": ctx, "heads": heads, "splits": splits, "us": ms * 1e3,
            "gbs": byt / ms / 1e6, "unique_gbs": batch * ctx * (576 + 512 + 8) / ms / 1e6}


def bench_prefill(t: int, hq: int, hk: int, reps: int, d: int = 128) -> list[dict]:
    q = torch.randn((t, hq, d), device="cuda").to(torch.bfloat16)
    k = torch.randn((t, hk, d), device="cuda").to(torch.bfloat16)
    v = torch.randn((t, hk, d), device="cuda").to(torch.bfloat16)
    out = torch.empty_like(q)
    ms = time_ms(lambda _: K.attn_prefill_bf16(q, k, v, 0.088, out=out), reps)
    rows = [{"kernel": "attn_prefill_bf16", "t": t, "hq": hq, "hk": hk, "d": d, "us": ms * 1e3,
             "tflops": 4 * t * t * hq * d / 2 / ms / 1e9}]
    pages = math.ceil(t / 16)
    cache = PagedKVCache(layers=1, kv_heads=hk, head_dim=d, num_pages=pages + 1, max_seqs=1, max_pages_per_seq=pages, device="cuda")
    cache.assign(0, 0, t)
    qkv = torch.randn((t, (hq + 2 * hk) * d), device="cuda").to(torch.bfloat16)
    pos = torch.arange(t, dtype=torch.int32, device="cuda")
    slots = cache.slots(0, 0, t).cuda()
    kd, vd = torch.empty_like(k), torch.empty_like(v)
    ms = time_ms(lambda _: K.rope_kv_write(qkv, pos, slots, cache.layer(0), n_q=hq, n_kv=hk, head_dim=d, theta=5e5, q_out=out,
                                           kd_out=kd, vd_out=vd), reps)
    rows.append({"kernel": "rope_kv_write", "t": t, "us": ms * 1e3, "gbs": t * (hq + 2 * hk) * d * 5 / ms / 1e6})
    return rows


def bench_small(m: int, h: int, i: int, reps: int) -> list[dict]:
    x = torch.randn((m, h), device="cuda").to(torch.bfloat16)
    w = torch.ones(h, device="cuda", dtype=torch.bfloat16)
    gu = torch.randn((m, 2 * i), device="cuda").to(torch.bfloat16)
    out = []
    ms = time_ms(lambda _: K.rmsnorm_quant(x, w, 1e-5), reps)
    out.append({"kernel": "rmsnorm_quant", "m": m, "h": h, "us": ms * 1e3, "gbs": m * h * 3 / ms / 1e6})
    ms = time_ms(lambda _: K.quant_rows(x), reps)
    out.append({"kernel": "quant_rows", "m": m, "h": h, "us": ms * 1e3, "gbs": m * h * 3 / ms / 1e6})
    ms = time_ms(lambda _: K.silu_mul_quant(gu), reps)
    out.append({"kernel": "silu_mul_quant", "m": m, "i": i, "us": ms * 1e3, "gbs": m * i * 5 / ms / 1e6})
    return out


def bench_dense(m: int, n: int, k: int, reps: int, stage: str = "", tile=None, splits=None) -> dict:
    """Unquantized (bf16) product with an output stage: "" (bias), "clipped" / "gelu" (gated unit), "add" (to the fp32 stream)."""
    from . import dense
    copies = max(1, min(16, math.ceil(4 * L2_BYTES / (2 * n * k))))
    lin = [dense.DenseLinear((torch.randn((n, k), device="cuda") * k ** -0.5).to(torch.bfloat16),
                             torch.zeros(n, device="cuda"), {"clipped": (1.702, 7.0), "gelu": "gelu"}.get(stage)) for _ in range(copies)]
    x = torch.randn((m, k), device="cuda").to(torch.bfloat16)
    add = stage == "add"
    out = torch.zeros((m, lin[0].out_width), device="cuda", dtype=torch.float32 if add else torch.bfloat16)
    ms = time_ms(lambda i: lin[i % copies](x, tile=tile, splits=splits, **{"add_to" if add else "out": out}), reps)
    t, sp = dense.plan(m, n, k)
    return {"kernel": "dense_gemv" if (t if tile is None else tile) == 0 else "dense_gemm", "m": m, "n": n, "k": k, "stage": stage, "us": ms * 1e3,
            "gbs": (2 * (n * k + m * k) + out.numel() * (8 if add else 2)) / ms / 1e6, "tflops": 2 * m * n * k / ms / 1e9,
            "tile": t if tile is None else tile, "splits": sp if splits is None else splits}


def _plain_cache(batch: int, ctx: int, hk: int, d: int, e: int, layers: int):
    from ..engine.kv_cache import PlainPagedKVCache
    pages_per = math.ceil(ctx / 16)
    cache = PlainPagedKVCache([(hk, d, e)] * layers, torch.bfloat16, num_pages=batch * pages_per + 1, max_seqs=batch,
                              max_pages_per_seq=pages_per, device="cuda")
    for pool in cache.pools:
        pool.k.normal_()
        pool.v.normal_()
    for b in range(batch):
        cache.assign(b, b, ctx)
    return cache


def bench_window_decode(batch: int, ctx: int, hq: int, hk: int, d: int, window: int, cap: float, reps: int, splits=None) -> dict:
    """One token per sequence over unquantized pages; every key inside the window is read once."""
    from . import window_attn
    seen = min(ctx, window)
    layers = max(1, min(32, math.ceil(4 * L2_BYTES / (batch * seen * hk * d * 4))))
    cache = _plain_cache(batch, ctx, hk, d, d, layers)
    q = torch.randn((batch, hq, d), device="cuda").to(torch.bfloat16)
    sl = torch.full((batch,), ctx, dtype=torch.int32, device="cuda")
    out = torch.empty_like(q)
    splits = window_attn.decode_splits(batch, hk, seen) if splits is None else splits
    ms = time_ms(lambda i: window_attn.decode(q, cache.layer(i % layers), cache.block_table, sl, window=window, scale=0.088, cap=cap,
                                              splits=splits, out=out), reps)
    return {"kernel": "window_attn_decode", "batch": batch, "ctx": ctx, "hq": hq, "hk": hk, "d": d, "window": window, "cap": cap,
            "splits": splits, "us": ms * 1e3, "gbs": batch * seen * hk * d * 4 / ms / 1e6}


def bench_window_prefill(t: int, hq: int, hk: int, d: int, window: int, cap: float, reps: int) -> dict:
    from . import window_attn
    cache = _plain_cache(1, t, hk, d, d, 1)
    q = torch.randn((t, hq, d), device="cuda").to(torch.bfloat16)
    out = torch.empty_like(q)
    starts, lens = (torch.tensor(v, dtype=torch.int32, device="cuda") for v in ([0, t], [t]))
    ms = time_ms(lambda _: window_attn.prefill(q, cache.layer(0), cache.block_table, starts, lens, t, window=window, scale=0.088, cap=cap,
                                               out=out), reps)
    w = min(window, t)
    pairs = w * (w + 1) // 2 + (t - w) * w  # visible (query, key) pairs
    return {"kernel": "window_attn_prefill", "t": t, "hq": hq, "hk": hk, "d": d, "window": window, "cap": cap, "us": ms * 1e3,
            "tflops": 4 * pairs * hq * d / ms / 1e9}


def bench_dense_small(m: int, h: int, reps: int) -> list[dict]:
    """The fp32 stream and the per-head stage (32 / 8 heads of 128)."""
    from . import dense, window_attn
    y = torch.randn((m, h), device="cuda").to(torch.bfloat16)
    x, act, w = torch.randn((m, h), device="cuda"), torch.empty_like(y), torch.ones(h, device="cuda")
    ms = time_ms(lambda _: dense.norm_add(y, w, x, act, h, 1e-5), reps)
    rows = [{"kernel": "norm_add", "m": m, "h": h, "us": ms * 1e3, "gbs": m * h * 12 / ms / 1e6}]
    hq, hk, d = 32, 8, 128
    cache = _plain_cache(1, m, hk, d, d, 1)
    qkv = torch.randn((m, (hq + 2 * hk) * d), device="cuda").to(torch.bfloat16)
    first = torch.randn((m, hk * d), device="cuda").to(torch.bfloat16)
    pos, slots, one = torch.arange(m, dtype=torch.int32, device="cuda"), cache.slots(0, 0, m).cuda(), torch.ones(d, device="cuda")
    rope = window_attn.rope_table(5e5, d, m, "cuda")
    ms = time_ms(lambda _: window_attn.qkv_finish(qkv, cache.layer(0), pos, slots, heads=hq, kv_heads=hk, dim=d, q_norm=one, k_norm=one,
                                                  rope=rope, rot=d, eps=1e-5, v_first=first, mix=0.5), reps)
    rows.append({"kernel": "qkv_finish", "t": m, "us": ms * 1e3, "gbs": m * ((hq + 2 * hk) * d * 4 + hk * d * 2) / ms / 1e6})
    return rows


def bench_two_maps(batch: int, ctx: int, h: int, hk: int, d: int, e: int, window: int, keep: int, reps: int) -> list[dict]:
    """Differential attention (two maps of ``d`` channels, values of ``e``): one token per sequence, or for batch 0 one prompt of
    ``ctx`` tokens and the difference of the maps."""
    from . import window_attn
    seen, diff = window_attn.visible_keys(ctx, window, keep), window_attn.Difference(0.5, 0.5, 1e-6, e)
    how = dict(window=window, keep=keep, scale=d ** -0.5, cap=0.0)
    shape = {"heads": h, "hk": hk, "d": d, "e": e, "window": window, "keep": keep}
    if batch:
        layers = max(1, min(32, math.ceil(4 * L2_BYTES / (batch * seen * hk * (2 * d + e) * 2))))
        cache = _plain_cache(batch, ctx, hk, 2 * d, e, layers)
        q = torch.randn((batch, 2 * h, d), device="cuda").to(torch.bfloat16)
        sl = torch.full((batch,), ctx, dtype=torch.int32, device="cuda")
        splits = window_attn.decode_splits(batch, hk, seen)
        ms = time_ms(lambda i: window_attn.decode(q, cache.layer(i % layers), cache.block_table, sl, diff=diff, splits=splits, **how), reps)
        return [{"kernel": "window_attn_decode (two maps, difference)", "batch": batch, "ctx": ctx, **shape, "splits": splits, "us": ms * 1e3,
                 "gbs": batch * seen * hk * (2 * d + e) * 2 / ms / 1e6}]
    cache = _plain_cache(1, ctx, hk, 2 * d, e, 1)
    q = torch.randn((ctx, 2 * h, d), device="cuda").to(torch.bfloat16)
    starts, lens = (torch.tensor(v, dtype=torch.int32, device="cuda") for v in ([0, ctx], [ctx]))
    maps = torch.empty((ctx, 2 * h, e), device="cuda", dtype=torch.bfloat16)
    ms = time_ms(lambda _: window_attn.prefill(q, cache.layer(0), cache.block_table, starts, lens, ctx, maps=2, out=maps, **how), reps)
    pairs = sum(min(i + 1, window + min(keep, max(0, i + 1 - window))) for i in range(ctx))
    out = window_attn.difference(maps, hk, diff)
    md = time_ms(lambda _: window_attn.difference(maps, hk, diff, out=out), reps)
    return [{"kernel": "window_attn_prefill (two maps)", "t": ctx, **shape, "us": ms * 1e3, "tflops": 2 * pairs * 2 * h * (d + e) / ms / 1e9},
            {"kernel": "map_difference", "t": ctx, **shape, "us": md * 1e3, "gbs": ctx * h * e * 6 / md / 1e6}]


def bench_gla(batch: int, tokens: int, h: int, dk: int, dv: int, reps: int) -> dict:
    """Gated linear attention: ``tokens`` 1: a decode step of ``batch`` sequences, else one prompt in chunks."""
    from . import gla
    geo = gla.Geometry(h, dk, dv, dk, dv, 16, 16.0, 1e-6)
    w2, bias = (torch.randn((h * dk, 16), device="cuda") * 0.25).to(torch.bfloat16), torch.randn(h * dk, device="cuda") + 2
    norm, slots = torch.ones(dv, device="cuda"), torch.arange(batch, dtype=torch.int32, device="cuda")
    proj = torch.randn((batch * tokens, geo.width), device="cuda").to(torch.bfloat16)
    row = batch * tokens * (geo.width + h * dv) * 2
    if tokens == 1:
        layers = max(1, min(32, math.ceil(4 * L2_BYTES / (batch * h * dk * dv * 4))))
        states = [torch.zeros((batch, h, dk, dv), device="cuda") for _ in range(layers)]
        ms = time_ms(lambda i: gla.recurrent(proj, w2, bias, norm, states[i % layers], slots, geo), reps)
        return {"kernel": "gla_recurrent", "batch": batch, "h": h, "dk": dk, "dv": dv, "us": ms * 1e3,
                "gbs": (batch * h * dk * dv * 8 + row) / ms / 1e6}
    state, starts = torch.zeros((1, h, dk, dv), device="cuda"), torch.tensor([0, tokens], dtype=torch.int32, device="cuda")
    ms = time_ms(lambda _: gla.chunked(proj, w2, bias, norm, state, slots, geo, starts, tokens), reps)
    return {"kernel": "gla_chunk (three kernels)", "t": tokens, "h": h, "dk": dk, "dv": dv, "us": ms * 1e3, "gbs": row / ms / 1e6}


def bench_gdn(batch: int, tokens: int, reps: int) -> dict:
    """Gated DeltaNet at 16 key / 32 value heads of 128, the same way (without its convolution)."""
    from . import gdn
    hk, hv, d = 16, 32, 128
    n = batch * tokens
    qkv, z = torch.randn((n, (2 * hk + hv) * d), device="cuda"), torch.randn((n, hv * d), device="cuda").to(torch.bfloat16)
    a, zero, one = torch.randn((n, hv), device="cuda").to(torch.bfloat16), torch.zeros(hv, device="cuda"), torch.ones(d, device="cuda")
    layers = max(1, min(32, math.ceil(4 * L2_BYTES / (batch * hv * d * d * 4)))) if tokens == 1 else 1
    states = [torch.zeros((batch, hv, d, d), device="cuda") for _ in range(layers)]
    slots = torch.arange(batch, dtype=torch.int32, device="cuda")
    ms = time_ms(lambda i: gdn.recurrent(qkv, z, a, a, zero, zero, one, states[i % layers], slots, tokens, hk, hv), reps)
    bytes_ = n * ((2 * hk + hv) * d * 4 + hv * d * 4) + (batch * hv * d * d * 8 if tokens == 1 else 0)
    return {"kernel": "gdn_recurrent" if tokens == 1 else "gdn_chunk (three kernels)", "batch": batch, "t": tokens, "us": ms * 1e3, "gbs": bytes_ / ms / 1e6}


def bench_bias(batch: int, ctx: int, hq: int, hk: int, d: int, most: int, reps: int) -> dict:
    """Attention with a score cap, a distance bias up to ``most`` and a sink: one token per sequence, or for batch 0 one prompt."""
    from . import window_attn
    table = torch.randn((hq, len(window_attn.log_buckets(32, most))), device="cuda")
    how = dict(window=1 << 30, scale=0.088, cap=50.0, bias=window_attn.DistanceBias.from_table(table), sink=torch.zeros(hq, device="cuda"))
    layers = max(1, min(32, math.ceil(4 * L2_BYTES / (batch * ctx * hk * d * 4)))) if batch else 1
    cache = _plain_cache(max(1, batch), ctx, hk, d, d, layers)
    shape = {"batch": batch, "ctx": ctx, "hq": hq, "hk": hk, "d": d, "bias_max": most}
    q = torch.randn((batch or ctx, hq, d), device="cuda").to(torch.bfloat16)
    out = torch.empty_like(q)
    if batch:
        sl, splits = torch.full((batch,), ctx, dtype=torch.int32, device="cuda"), window_attn.decode_splits(batch, hk, ctx)
        ms = time_ms(lambda i: window_attn.decode(q, cache.layer(i % layers), cache.block_table, sl, splits=splits, out=out, **how), reps)
        return {"kernel": "window_attn_decode (bias, sink)", **shape, "splits": splits, "us": ms * 1e3, "gbs": batch * ctx * hk * d * 4 / ms / 1e6}
    starts, lens = (torch.tensor(v, dtype=torch.int32, device="cuda") for v in ([0, ctx], [ctx]))
    ms = time_ms(lambda _: window_attn.prefill(q, cache.layer(0), cache.block_table, starts, lens, ctx, out=out, **how), reps)
    return {"kernel": "window_attn_prefill (bias, sink)", **shape, "us": ms * 1e3, "tflops": 2 * ctx * (ctx + 1) * hq * d / ms / 1e9}


def bench_latent(batch: int, ctx: int, heads: int, window: int, reps: int, splits=None, sink: bool = False) -> list[dict]:
    """Latent attention at rank 512, 128 + 64 query channels, values of 128: a decode step (attention and the products into and out of
    latent space), or for batch 0 one prompt (copy of the rows, expansion, attention)."""
    from . import dense, latent_attn
    d, rot, e, rank, seen = 128, 64, 128, 512, min(ctx, window)
    r, layers = rank + rot, max(1, min(32, math.ceil(4 * L2_BYTES / (max(1, batch) * seen * 576 * 2))))
    cache = _plain_cache(max(1, batch), ctx, 1, r, 0, layers)
    shape = {"batch": batch, "ctx": ctx, "heads": heads, "window": window} | ({"sink": True} if sink else {})
    sinks = torch.zeros(heads, device="cuda") if sink else None
    if batch:
        q = torch.randn((batch, heads, r), device="cuda").to(torch.bfloat16)
        sl = torch.full((batch,), ctx, dtype=torch.int32, device="cuda")
        splits = latent_attn.decode_splits(batch, heads, seen) if splits is None else splits
        ms = time_ms(lambda i: latent_attn.decode(q, cache.layer(i % layers).k, cache.block_table, sl, rank=rank, window=window, scale=0.07, splits=splits, sink=sinks), reps)
        rows = [{"kernel": "latent_decode", **shape, "splits": splits, "us": ms * 1e3, "gbs": batch * seen * r * 2 / ms / 1e6,
                 "tile_gbs": batch * seen * r * 2 * math.ceil(heads / 16) / ms / 1e6}]
        copies = 16
        for name, n, k in (("into latent space", rank, d), ("out of it", e, rank)):
            lin = [dense.DenseLinear(torch.randn((heads * n, k), device="cuda").to(torch.bfloat16), groups=heads) for _ in range(copies)]
            x, out = torch.randn((batch, heads * k), device="cuda").to(torch.bfloat16), torch.empty((batch, heads * n), device="cuda", dtype=torch.bfloat16)
            ms = time_ms(lambda i: lin[i % copies](x, out=out), reps)
            rows.append({"kernel": f"product per head, {name}", "batch": batch, "heads": heads, "us": ms * 1e3,
                         "gbs": 2 * (heads * n * k + batch * heads * (n + k)) / ms / 1e6})
        return rows
    seq, shift = (torch.tensor(v, dtype=torch.int32, device="cuda") for v in latent_attn.visible_pages([(0, ctx)], window))
    rows_ = latent_attn.visible_rows(cache.layer(0).k, cache.block_table, seq, shift)
    ms = time_ms(lambda _: latent_attn.visible_rows(cache.layer(0).k, cache.block_table, seq, shift), reps)
    rows = [{"kernel": "latent_pages", **shape, "us": ms * 1e3, "gbs": ctx * r * 4 / ms / 1e6}]
    lin = dense.DenseLinear(torch.randn((heads * (d + rot + e), r), device="cuda").to(torch.bfloat16))
    kv = lin(rows_)
    ms = time_ms(lambda _: lin(rows_), reps)
    rows.append({"kernel": "dense_gemm (expansion)", **shape, "us": ms * 1e3, "tflops": 2 * ctx * heads * (d + e) * rank / ms / 1e9})
    q = torch.randn((ctx, heads, d + rot), device="cuda").to(torch.bfloat16)
    out = torch.empty((ctx, heads, e), device="cuda", dtype=torch.bfloat16)
    starts, lens = (torch.tensor(v, dtype=torch.int32, device="cuda") for v in ([0, ctx], [ctx]))
    ms = time_ms(lambda _: latent_attn.prefill_rows(q, kv, shift, starts, lens, ctx, head0=0, heads=heads, dk=d + rot, dv=e, window=window, scale=0.07,
                                                    sink=sinks, out=out), reps)
    w = min(window, ctx)
    pairs = w * (w + 1) // 2 + (ctx - w) * w
    return rows + [{"kernel": "window_attn_prefill (expanded rows)", **shape, "us": ms * 1e3, "tflops": 2 * pairs * heads * (d + rot + e) / ms / 1e9}]


def bench_time_mixing(batch: int, tokens: int, h: int, d: int, reps: int) -> dict:
    """Time mixing, as :func:`bench_gla`."""
    from . import gla
    geo = gla.Geometry(h, d, d, d, d, 64, 1.0, 1e-6, decay="exp", scaled=False)
    w2, bias = (torch.randn((h * d, 64), device="cuda") * 0.1).to(torch.bfloat16), torch.randn(h * d, device="cuda") - 2
    norm, bonus, slots = torch.ones((h, d), device="cuda"), torch.ones(h * d, device="cuda"), torch.arange(batch, dtype=torch.int32, device="cuda")
    proj = torch.randn((batch * tokens, geo.width), device="cuda").to(torch.bfloat16)
    row = batch * tokens * (geo.width + h * d) * 2
    if tokens == 1:
        layers = max(1, min(64, math.ceil(4 * L2_BYTES / (batch * h * d * d * 4))))
        states = [torch.zeros((batch, h, d, d), device="cuda") for _ in range(layers)]
        ms = time_ms(lambda i: gla.recurrent(proj, w2, bias, norm, states[i % layers], slots, geo, bonus=bonus), reps)
        return {"kernel": "gla_recurrent (time mixing)", "batch": batch, "h": h, "d": d, "us": ms * 1e3, "gbs": (batch * h * d * d * 8 + row) / ms / 1e6}
    state, starts = torch.zeros((1, h, d, d), device="cuda"), torch.tensor([0, tokens], dtype=torch.int32, device="cuda")
    ms = time_ms(lambda _: gla.chunked(proj, w2, bias, norm, state, slots, geo, starts, tokens, bonus=bonus), reps)
    return {"kernel": "gla_chunk (time mixing, three kernels)", "t": tokens, "h": h, "d": d, "us": ms * 1e3, "gbs": row / ms / 1e6}


def bench_delta(batch: int, tokens: int, h: int, hk: int, d: int, reps: int) -> list[dict]:
    """Delta rule with a decay per channel (and its convolution), as :func:`bench_gla`."""
    from . import delta, dense
    geo = delta.Geometry(h, hk, d, d, d, d, 64, 64, 4, 1e-6)
    bf = lambda *s: (torch.randn(s, device="cuda") * 0.1).to(torch.bfloat16)
    w = delta.Weights(torch.randn((4, geo.channels), device="cuda"), bf(h * d, 64), torch.randn(h * d, device="cuda") - 2, torch.ones(h, device="cuda"),
                      dense.DenseLinear(bf(h * d, 64)), torch.ones(d, device="cuda"))
    slots, n = torch.arange(batch, dtype=torch.int32, device="cuda"), batch * tokens
    proj, x = torch.randn((n, geo.width), device="cuda").to(torch.bfloat16), torch.randn((n, geo.channels), device="cuda").to(torch.bfloat16)
    hist, out = torch.zeros((batch, 3, geo.channels), device="cuda"), torch.empty((n, geo.channels), device="cuda", dtype=torch.bfloat16)
    row = n * (geo.width + h * d) * 2
    if tokens == 1:
        layers = max(1, min(32, math.ceil(4 * L2_BYTES / (batch * h * d * d * 4))))
        states = [torch.zeros((batch, h, d, d), device="cuda") for _ in range(layers)]
        ms = time_ms(lambda i: delta.recurrent(x, proj, w, states[i % layers], slots, geo), reps)
        mc = time_ms(lambda _: delta.conv(proj, w.conv, hist, slots, geo.channels, out=out), reps)
        return [{"kernel": "delta_recurrent", "batch": batch, "h": h, "d": d, "us": ms * 1e3, "gbs": (batch * h * d * d * 8 + row) / ms / 1e6},
                {"kernel": "short_conv", "batch": batch, "c": geo.channels, "us": mc * 1e3, "gbs": batch * geo.channels * 28 / mc / 1e6}]
    state, starts = torch.zeros((1, h, d, d), device="cuda"), torch.tensor([0, tokens], dtype=torch.int32, device="cuda")
    ms = time_ms(lambda _: delta.chunked(x, proj, w, state, slots, geo, starts, tokens), reps)
    mc = time_ms(lambda _: delta.conv(proj, w.conv, hist, slots, geo.channels, starts=starts, max_q=tokens, out=out), reps)
    return [{"kernel": "delta_chunk (four kernels)", "t": tokens, "h": h, "hk": hk, "d": d, "us": ms * 1e3, "gbs": row / ms / 1e6},
            {"kernel": "short_conv (two kernels)", "t": tokens, "c": geo.channels, "us": mc * 1e3, "gbs": n * geo.channels * 4 / mc / 1e6}]


def bench_experts(tokens: int, width: int, ff: int, experts: int, top: int, reps: int) -> list[dict]:
    """Routed experts of one layer in bf16 (routing, products, addition to the stream), and the same in block-scaled FP8."""
    from . import dense, dense_moe, moe
    h, x = torch.randn((tokens, width), device="cuda").to(torch.bfloat16), torch.zeros((tokens, width), device="cuda")
    logits = torch.randn((tokens, experts), device="cuda")
    copies = max(1, min(4, math.ceil(4 * L2_BYTES / (experts * 3 * width * ff * 2))))
    bf = lambda *s: torch.randn(s, device="cuda", dtype=torch.bfloat16) * 0.02
    banks = [dense_moe.ExpertBank(experts, bf(experts * 2 * ff, width), bf(experts * width, ff)) for _ in range(copies)]
    bias = torch.zeros(experts, device="cuda")
    used = len(torch.unique(dense_moe.topk(logits, top, bias, 1.0)[0]))

    def layer(i):
        ids, wt = dense_moe.topk(logits, top, bias, 2.5)
        dense_moe.add_experts(h, ids, wt, banks[i % copies], x, 1.0)
    ms = time_ms(layer, reps)
    shape = {"tokens": tokens, "width": width, "ff": ff, "experts": experts, "top": top, "used": used}
    flops = 6 * tokens * top * width * ff
    rows = [{"kernel": "experts, bf16", **shape, "us": ms * 1e3, "gbs": used * 3 * width * ff * 2 / ms / 1e6, "tflops": flops / ms / 1e9}]
    del banks
    f8 = lambda *s: torch.randint(-100, 100, s, device="cuda", dtype=torch.int8).view(torch.float8_e4m3fn)
    sc = lambda e, n, k: torch.rand((e, math.ceil(n / 128), k // 128), device="cuda") * 0.01
    gu, dn = [f8(experts, 2 * ff, width) for _ in range(copies)], [f8(experts, width, ff) for _ in range(copies)]
    gus, dns, xq, xs = sc(experts, 2 * ff, width), sc(experts, width, ff), f8(tokens, width), torch.rand(tokens, device="cuda")
    ids, wt = dense_moe.topk(logits, top, bias, 2.5)
    ms = time_ms(lambda i: moe.moe_ffn_fp8(xq, xs, ids, wt, gu[i % copies], gus, dn[i % copies], dns), reps)
    return rows + [{"kernel": "experts, FP8", **shape, "us": ms * 1e3, "gbs": used * 3 * width * ff / ms / 1e6, "tflops": flops / ms / 1e9}]


def bench_ssd(batch: int, tokens: int, h: int, groups: int, n: int, p: int, reps: int, chunk=None, heads=None) -> list[dict]:
    """State-space recurrence with its convolution and gated norm, as :func:`bench_gla`."""
    from . import ssd
    geo, t = ssd.Geometry(h, groups, n, p, p, 4, groups, 1e-5), batch * tokens
    w = ssd.Weights(torch.randn((4, geo.channels), device="cuda"), torch.randn(geo.channels, device="cuda"), torch.randn(h, device="cuda") - 2,
                    torch.ones(h, device="cuda"), torch.ones(h, device="cuda"), torch.ones(h * p, device="cuda"))
    proj, x = torch.randn((t, geo.row), device="cuda").to(torch.bfloat16), torch.randn((t, geo.channels), device="cuda").to(torch.bfloat16)
    slots, hist, out = torch.arange(batch, dtype=torch.int32, device="cuda"), torch.zeros((batch, 3, geo.channels), device="cuda"), torch.empty_like(x)
    y, row = torch.empty((t, geo.inner), device="cuda", dtype=torch.bfloat16), t * (geo.channels + geo.inner + h) * 2
    shape = {"batch": batch, "t": tokens, "h": h, "groups": groups, "n": n, "p": p}
    mn = time_ms(lambda _: ssd.gate_norm(y, proj, w, geo), reps)
    rows = [{"kernel": "ssd_gate_norm", **shape, "us": mn * 1e3, "gbs": t * geo.inner * 6 / mn / 1e6}]
    if tokens == 1:
        layers = max(1, min(32, math.ceil(4 * L2_BYTES / (batch * h * n * p * 4))))
        states = [torch.zeros((batch, h, n, p), device="cuda") for _ in range(layers)]
        ms = time_ms(lambda i: ssd.recurrent(x, proj, w, states[i % layers], slots, geo, out=y), reps)
        mc = time_ms(lambda _: ssd.conv(proj, w.conv, hist, slots, geo.channels, bias=w.conv_bias, out=out), reps)
        return rows + [{"kernel": "ssd_recurrent", **shape, "us": ms * 1e3, "gbs": (batch * h * n * p * 8 + row) / ms / 1e6},
                       {"kernel": "short_conv (bias)", "batch": batch, "c": geo.channels, "us": mc * 1e3, "gbs": batch * geo.channels * 28 / mc / 1e6}]
    state, starts = torch.zeros((1, h, n, p), device="cuda"), torch.tensor([0, tokens], dtype=torch.int32, device="cuda")
    ms = time_ms(lambda _: ssd.chunked(x, proj, w, state, slots, geo, starts, tokens, out=y, chunk=chunk, heads=heads), reps)
    mc = time_ms(lambda _: ssd.conv(proj, w.conv, hist, slots, geo.channels, starts=starts, max_q=tokens, bias=w.conv_bias, out=out), reps)
    plan = ssd.chunk_plan(geo, tokens, tokens)
    return rows + [{"kernel": "ssd_chunk (three kernels)", **shape, "chunk": chunk or plan[0], "heads": heads or plan[1], "us": ms * 1e3, "gbs": row / ms / 1e6},
                   {"kernel": "short_conv (bias, two kernels)", "t": tokens, "c": geo.channels, "us": mc * 1e3, "gbs": t * geo.channels * 4 / mc / 1e6}]


def bench_sublayer_input(m: int, h: int, reps: int) -> list[dict]:
    """Norm and convolution of the stream in one kernel, and the norm alone: one row each of ``m`` sequences, and a prompt of ``m``."""
    from . import dense
    x, w, k = torch.randn((m, h), device="cuda"), torch.ones(h, device="cuda"), torch.randn((4, h), device="cuda")
    rows, state, slots = [], torch.zeros((min(m, 64), 3, h), device="cuda"), torch.arange(min(m, 64), dtype=torch.int32, device="cuda")
    if m <= 64:
        ms = time_ms(lambda _: dense.norm_conv_out(x, w, k, state, slots, h, 1e-5, torch.bfloat16), reps)
        rows.append({"kernel": "norm_conv (decode)", "m": m, "h": h, "us": ms * 1e3, "gbs": m * h * 30 / ms / 1e6})
    else:
        starts = torch.tensor([0, m], dtype=torch.int32, device="cuda")
        ms = time_ms(lambda _: dense.norm_conv_out(x, w, k, state, slots[:1], h, 1e-5, torch.bfloat16, starts=starts, max_q=m), reps)
        rows.append({"kernel": "norm_conv (prompt)", "m": m, "h": h, "us": ms * 1e3, "gbs": m * h * 6 / ms / 1e6})
    ms = time_ms(lambda _: dense.norm_out(x, w, h, 1e-5, torch.bfloat16), reps)
    return rows + [{"kernel": "norm_out", "m": m, "h": h, "us": ms * 1e3, "gbs": m * h * 6 / ms / 1e6}]


def bench_chunks(batch: int, ctx: int, hq: int, hk: int, d: int, size: int, reps: int) -> list[dict]:
    """Attention in chunks of ``size`` with rotated values: one token at the end of a chunk per sequence, or for batch 0 one prompt; and
    the per-head stage in front of it."""
    from . import window_attn
    seen, n = min(ctx, size), batch or ctx
    layers = max(1, min(32, math.ceil(4 * L2_BYTES / (batch * seen * hk * d * 4)))) if batch else 1
    cache = _plain_cache(max(1, batch), ctx, hk, d, d, layers)
    shape = {"batch": batch, "ctx": ctx, "hq": hq, "hk": hk, "d": d, "size": size}
    q, out = torch.randn((n, hq, d), device="cuda").to(torch.bfloat16), torch.empty((n, hq, d), device="cuda", dtype=torch.bfloat16)
    turn = window_attn.ValueTurn(window_attn.rope_table(5e5, d, ctx, "cuda"), d)
    how = dict(window=1 << 30, chunk=size, scale=0.088, cap=0.0)
    pos = torch.arange(n, dtype=torch.int32, device="cuda")
    qkv, one = torch.randn((n, (hq + 2 * hk) * d), device="cuda").to(torch.bfloat16), torch.ones(d, device="cuda")
    slots = (cache.slots(0, 0, n) if not batch else torch.cat([cache.slots(b, 0, 1) for b in range(batch)])).cuda()
    stage = lambda turned: time_ms(lambda _: window_attn.qkv_finish(qkv, cache.layer(0), pos, slots, heads=hq, kv_heads=hk, dim=d, q_norm=one, k_norm=one,
                                                                    rope=turn.rope, rot=d, eps=1e-5, turn=turn if turned else None), reps)
    rows = [{"kernel": f"qkv_finish ({name})", **shape, "us": ms * 1e3, "gbs": n * (hq + 2 * hk) * d * 4 / ms / 1e6}
            for name, ms in (("values normed and rotated", stage(True)), ("plain values", stage(False)))]
    if batch:
        sl, splits = torch.full((batch,), ctx, dtype=torch.int32, device="cuda"), window_attn.decode_splits(batch, hk, seen)
        ms = time_ms(lambda i: window_attn.decode(q, cache.layer(i % layers), cache.block_table, sl, splits=splits, turn=turn, out=out, **how), reps)
        return rows + [{"kernel": "window_attn_decode (chunks, turned)", **shape, "splits": splits, "us": ms * 1e3, "gbs": batch * seen * hk * d * 4 / ms / 1e6}]
    starts, lens = (torch.tensor(v, dtype=torch.int32, device="cuda") for v in ([0, ctx], [ctx]))
    ms = time_ms(lambda _: window_attn.prefill(q, cache.layer(0), cache.block_table, starts, lens, ctx, out=out, **how), reps)
    mt = time_ms(lambda _: window_attn.turn_back(out, turn, pos), reps)
    pairs = ctx // seen * (seen * (seen + 1) // 2)
    return rows + [{"kernel": "window_attn_prefill (chunks)", **shape, "us": ms * 1e3, "tflops": 4 * pairs * hq * d / ms / 1e9},
                   {"kernel": "turn_back", **shape, "us": mt * 1e3, "gbs": n * hq * d * 4 / mt / 1e6}]


def bench_low_queries(m: int, q_rank: int, rank: int, rot: int, reps: int) -> dict:
    """Norms of the query latent and of the shared latent row, and its page write."""
    from . import latent_attn, window_attn
    cache = _plain_cache(1, m, 1, rank + rot, 0, 1)
    proj, pos = torch.randn((m, q_rank + rank + rot), device="cuda").to(torch.bfloat16), torch.arange(m, dtype=torch.int32, device="cuda")
    slots, rope = cache.slots(0, 0, m).cuda(), window_attn.rope_table(5e5, rot, m, "cuda")
    a, b = torch.ones(q_rank, device="cuda"), torch.ones(rank, device="cuda")
    ms = time_ms(lambda _: latent_attn.down(proj, cache.layer(0).k, pos, slots, q_rank=q_rank, real_q_rank=q_rank, rank=rank, rot=rot, real_rank=rank,
                                            real_rot=rot, q_norm=a, norm_w=b, rope=rope, eps=1e-5), reps)
    return {"kernel": "latent_down", "m": m, "q_rank": q_rank, "rank": rank, "us": ms * 1e3, "gbs": m * (q_rank + rank + rot) * 4 / ms / 1e6}


def main() -> None:
    ap = argparse.ArgumentParser()
    ap.add_argument("--json", default="")
    ap.add_argument("--reps", type=int, default=20)
    ap.add_argument("--quick", action="store_true")
    ap.add_argument("--only", default="", help="comma separated kernel families: gemm,w4,attn,mla,small,prefill,dense,maps,gla,bias,latent,mixing,delta,experts,input,chunks,sink,ssd")
    ap.add_argument("--tp", type=int, default=1, help="time one rank's shard of a tensor-parallel group of this size")
    args = ap.parse_args()
    pk = peaks()
    rows = []
    only = set(filter(None, args.only.split(",")))
    want = lambda family: not only or family in only
    tp = args.tp
    shapes = [("qkv", 6144 // tp, 4096), ("o_proj", 4096, 4096 // tp), ("gate_up", 28672 // tp, 4096), ("down", 4096, 14336 // tp),
              ("lm_head", 128256 // tp, 4096)]
    for m in ((1, 64) if args.quick else (1, 16, 64, 512, 4096)) if want("gemm") else ():
        for name, n, k in shapes:
            if name == "lm_head" and m > 64:
                continue
            r = bench_gemm(m, n, k, args.reps)
            r["name"] = name
            rows.append(r)
            if r["kernel"] == "fp8_gemv":  # the tcgen05 GEMM on the same shape, for comparison
                r = bench_gemm(m, n, k, args.reps, splits=K.pick_splits(m, n, k), tile=K._token_tile(m))
                r["name"] = name
                rows.append(r)
    for m in ((1, 64) if args.quick else (1, 16, 64, 512, 4096)) if want("w4") else ():
        for name, n, k in shapes[:4]:
            r = bench_w4_gemm(m, n, k, args.reps)
            r["name"] = name
            rows.append(r)
    for batch, ctx in ((1, 4096), (64, 4096)) if want("attn") else ():
        for splits in sorted({1, 4, K.attn_splits_for(batch, max(1, 8 // tp), ctx)}):
            rows.append(bench_attn(batch, ctx, 32 // tp, max(1, 8 // tp), 128, splits, args.reps))
        # 256-wide heads of the hybrid model: 16 query heads on 2 KV heads
        rows.append(bench_attn(batch, ctx, 16, 2, 256, K.attn_splits_for(batch, 2, ctx), args.reps))
    for batch, ctx in ((1, 4096), (64, 4096)) if want("mla") else ():
        for splits in ((1, 8, 16) if batch == 1 else (1, 2, 4)):
            rows.append(bench_mla_decode(batch, ctx, max(16, 128 // tp), splits, args.reps))
    for m in (1, 64, 4096) if want("small") else ():
        rows += bench_small(m, 4096, 14336, args.reps)
    for t in (1024, 4096) if want("prefill") else ():
        rows += bench_prefill(t, 32, 8, args.reps)
        rows += bench_prefill(t, 16, 2, args.reps, d=256)[:1]
    for m in ((1, 64) if args.quick else (1, 16, 64, 512, 4096)) if want("dense") else ():
        for name, n, k in shapes:
            if name == "lm_head" and m > 64:
                continue
            rows.append({**bench_dense(m, n, k, args.reps, "clipped" if name == "gate_up" else ""), "name": name})
    if want("dense"):
        for batch in (1, 64):
            for window, cap in ((4096, 0.0), (4096, 50.0), (1024, 50.0)):
                rows.append(bench_window_decode(batch, 4096, 32, 8, 128, window, cap, args.reps))
        for t in (1024, 4096):
            for window, cap in ((1 << 30, 0.0), (1 << 30, 50.0), (1024, 50.0)):
                rows.append(bench_window_prefill(t, 32, 8, 128, window, cap, args.reps))
        for m in (1, 64, 4096):
            rows += bench_dense_small(m, 4096, args.reps)
    if want("maps"):
        for d, e, h in ((64, 128, 32), (128, 256, 16)):
            for window, keep in ((4096, 0), (1024, 64)):
                for batch in (1, 64, 0):
                    rows += bench_two_maps(batch, 4096, h, 8, d, e, window, keep, args.reps)
        for m in (1, 64, 4096):
            for name, n, k, stage in (("o_proj", 4096, 4096, "add"), ("gate_up", 28672, 4096, "gelu"), ("down", 4096, 14336, "add")):
                rows.append({**bench_dense(m, n, k, args.reps, stage), "name": name})
        from . import dense
        for m in (1, 64, 4096):
            x, w = torch.randn((m, 4096), device="cuda"), torch.ones(4096, device="cuda")
            ms = time_ms(lambda _: dense.norm_out(x, w, 4096, 1e-5, torch.bfloat16), args.reps)
            rows.append({"kernel": "norm_out", "m": m, "h": 4096, "us": ms * 1e3, "gbs": m * 4096 * 6 / ms / 1e6})
    if want("gla"):
        for batch, tokens in ((1, 1), (64, 1), (1, 2048), (1, 4096)):
            for h, dk, dv in ((32, 128, 128), (16, 128, 256)):
                rows.append(bench_gla(batch, tokens, h, dk, dv, args.reps))
            rows.append(bench_gdn(batch, tokens, args.reps))
    if want("bias"):
        for batch in (1, 64, 0):
            for most in (256, 2048):
                rows.append(bench_bias(batch, 4096, 32, 8, 128, most, args.reps))
            rows.append(bench_window_decode(batch, 4096, 32, 8, 128, 4096, 50.0, args.reps) if batch else bench_window_prefill(4096, 32, 8, 128, 1 << 30, 50.0, args.reps))
    if want("latent"):
        for heads in (16, 32):
            for batch, window in ((1, 4096), (64, 4096), (64, 1024), (0, 4096), (0, 1024)):
                rows += bench_latent(batch, 4096, heads, window, args.reps)
        for batch, splits in ((1, 16), (64, 2)):
            rows.append(bench_mla_decode(batch, 4096, 16, splits, args.reps))
        rows += bench_prefill(4096, 32, 32, args.reps, d=256)[:1]  # how the FP8 latent models prefill: heads padded to 256 channels
    if want("mixing"):
        from . import dense, gla
        for batch, tokens in ((1, 1), (64, 1), (1, 2048), (1, 4096)):
            rows.append(bench_time_mixing(batch, tokens, 64, 64, args.reps))
            rows.append(bench_gla(batch, tokens, 64, 64, 64, args.reps))
        for m in (1, 64, 4096):
            x, w = torch.randn((m, 4096), device="cuda"), torch.ones(4096, device="cuda")
            ms = time_ms(lambda _: dense.layer_norm_out(x, w, w, 4096, 1e-5, torch.bfloat16), args.reps)
            rows.append({"kernel": "layer_norm_out", "m": m, "h": 4096, "us": ms * 1e3, "gbs": m * 4096 * 6 / ms / 1e6})
            h, mu, last = x.to(torch.bfloat16), torch.rand((5, 4096), device="cuda"), torch.zeros((64, 4096), device="cuda")
            slots = torch.arange(64 if m == 64 else 1, dtype=torch.int32, device="cuda")
            ragged = (torch.tensor([0, m], dtype=torch.int32, device="cuda"), torch.zeros(m, dtype=torch.int32, device="cuda")) if m > 64 else ()
            ms = time_ms(lambda _: gla.token_shift(h, mu, last, slots, *ragged), args.reps)
            rows.append({"kernel": "token_shift", "m": m, "h": 4096, "us": ms * 1e3, "gbs": m * 4096 * 12 / ms / 1e6})
    if want("delta"):
        for batch, tokens in ((1, 1), (64, 1), (1, 2048), (1, 4096)):
            rows += bench_delta(batch, tokens, 32, 16, 128, args.reps)
            rows.append(bench_gdn(batch, tokens, args.reps))
    if want("experts"):
        for tokens in (1, 16, 64, 512, 4096):
            rows += bench_experts(tokens, 4096, 2048, 32, 4, args.reps)
    if want("input"):
        for m in (1, 64, 4096):
            rows += bench_sublayer_input(m, 4096, args.reps)
            rows.append(bench_low_queries(m, 1536, 512, 64, args.reps))
    if want("chunks"):
        for batch in (1, 64, 0):
            for size in (4096, 1024):
                rows += bench_chunks(batch, 4096, 32, 8, 128, size, args.reps)
                rows.append(bench_window_decode(batch, 4096, 32, 8, 128, size, 0.0, args.reps) if batch
                            else bench_window_prefill(4096, 32, 8, 128, size, 0.0, args.reps))
    if want("sink"):
        for batch, window in ((1, 4096), (64, 4096), (64, 1024), (0, 4096), (0, 1024)):
            for sink in (True, False):
                rows += bench_latent(batch, 4096, 32, window, args.reps, sink=sink)
    if want("ssd"):
        for batch, tokens in ((1, 1), (64, 1), (1, 2048), (1, 4096)):
            for h, groups in ((64, 1), (64, 8)):
                rows += bench_ssd(batch, tokens, h, groups, 128, 64, args.reps)
            rows.append(bench_gla(batch, tokens, 32, 128, 128, args.reps))
            rows.append(bench_gla(batch, tokens, 64, 128, 64, args.reps))
    for r in rows:
        if "gbs" in r:
            r["hbm_frac"] = r["gbs"] / pk["hbm_gbs"]
        if "tflops" in r:
            r["tensor_frac_of_bf16"] = r["tflops"] / pk["tflops"]
        print(json.dumps({k: (round(v, 3) if isinstance(v, float) else v) for k, v in r.items()}))
    if args.json:
        json.dump({"peaks": pk, "rows": rows}, open(args.json, "w"), indent=1)


if __name__ == "__main__":
    main()
