#!/usr/bin/env python
"""Micro-benchmarks of the sm_100a kernels, one op per run, device-timed with CUDA events.

    python examples/benchmark/kernels.py --op=gemm --m=32 --n=28672 --k=4096
    python examples/benchmark/kernels.py --op=decode_attention --batch=32 --seqlen=1344
    python examples/benchmark/kernels.py --op=prefill_attention --batch=4 --seqlen=2048
    python examples/benchmark/kernels.py --op=moe --tokens=128 --experts=128 --topk=8 --n=768 --k=2048
    python examples/benchmark/kernels.py --op=gated_delta_scan --batch=32 --seqlen=1024
    python examples/benchmark/kernels.py --op=latent_prefill --batch=2 --seqlen=2048 --hq=16 --window=4096
    python examples/benchmark/kernels.py --op=latent_decode --batch=32 --seqlen=4096 --hq=32 --window=4096
    python examples/benchmark/kernels.py --op=wkv_scan --batch=8 --seqlen=512 --hq=32 --hd=128
    python examples/benchmark/kernels.py --op=stream --tokens=4096 --k=4096
    python examples/benchmark/kernels.py --op=gqa_prefill --batch=2 --seqlen=2048 --window=4096
    python examples/benchmark/kernels.py --op=gqa_decode --batch=32 --seqlen=1344 --window=4096
    python examples/benchmark/kernels.py --op=pool_prefill --batch=2 --seqlen=8192 --window=1024 --pool=16
    python examples/benchmark/kernels.py --op=pool_decode --batch=32 --seqlen=8192 --window=1024 --pool=16
    python examples/benchmark/kernels.py --op=gated_scan --batch=8 --seqlen=512 --k=4096
    python examples/benchmark/kernels.py --op=add_norm --tokens=4096 --k=4096
    python examples/benchmark/kernels.py --op=relu_mixture --tokens=32 --experts=32 --topk=4 --n=1536 --k=2048
    python examples/benchmark/kernels.py --op=channel_delta --batch=8 --seqlen=512 --hq=32 --hd=128
    python examples/benchmark/kernels.py --op=mixture --tokens=32 --experts=32 --topk=4 --n=1024 --k=2048
    python examples/benchmark/kernels.py --op=decode_layers --model=llama-3.1-8b --batch=32 --seqlen=1344
    python examples/benchmark/kernels.py --op=gemm_chain_timeline --model=llama-3.1-8b --batch=32
    python examples/benchmark/kernels.py --op=moe_w4_timeline --tokens=128 --experts=128 --topk=8 --n=768 --k=2048

Every op works on inputs larger than the L2 (or rotates through several copies of its operands
so that each launch reads cold data); `--iters` timed launches follow `--warmup` untimed ones.
The JSON line gives the time per launch, the algorithmic bytes and FLOPs, and the fractions of
the measured copy bandwidth and bf16 GEMM rate (`MEASURED_PEAKS.json` at the repository root
when present).  `--iters=1 --warmup=1` is the form to put under a profiler.
"""
from __future__ import annotations

import contextlib
import json
import math
import os
import sys
from dataclasses import dataclass

ROOT = os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
sys.path.insert(0, ROOT)

import torch  # noqa: E402

from zml_b200 import flags, ops  # noqa: E402


@dataclass
class Args:
    op: str = "gemm"
    m: int = 32
    n: int = 4096
    k: int = 4096
    batch: int = 32
    seqlen: int = 1344
    hq: int = 32
    hkv: int = 8
    hd: int = 128
    tokens: int = 128
    experts: int = 128
    topk: int = 8
    model: str = "llama-3.1-8b"
    iters: int = 20
    warmup: int = 3
    splits: int = 0          # decode_attention: KV chunks per sequence (0: the planner's choice)
    w4: int = 0              # moe: 1 = NVFP4 expert weights de-quantised inside the grouped GEMM
    window: int = 4096       # latent and gated attention: keys a position sees; differential attention: its chunk
    pool: int = 16           # windowed attention with pooled blocks: tokens per block
    sink: int = 0            # latent attention: 1 = a sink per head and no output gate
    copies: int = 0          # operand copies to rotate through (0: enough to exceed the L2)
    help = __doc__


def peaks() -> dict:
    try:
        with open(os.path.join(ROOT, "MEASURED_PEAKS.json")) as f:
            p = json.load(f)
        return {"hbm_gbs": float(p.get("hbm_gbs", 6650.0)), "bf16_tflops": float(p.get("bf16_tflops", 1590.0)), "source": "measured"}
    except (OSError, ValueError):
        return {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "source": "fallback"}


def timed(fns, iters: int, warmup: int) -> float:
    """Milliseconds per launch; fns are rotated so that consecutive launches use different operands."""
    for i in range(warmup):
        fns[i % len(fns)]()
    torch.cuda.synchronize()
    s, e = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    s.record()
    for i in range(iters):
        fns[(warmup + i) % len(fns)]()
    e.record()
    torch.cuda.synchronize()
    return s.elapsed_time(e) / iters


def timed_graph(fns, iters: int, warmup: int) -> float:
    """As `timed`, for launches shorter than their submission: the iterations are captured in one CUDA graph."""
    for i in range(warmup):
        fns[i % len(fns)]()
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g):
        for i in range(iters):
            fns[i % len(fns)]()
    return timed([g.replay], 5, 2) / iters


def n_copies(args: Args, bytes_per_copy: int) -> int:
    if args.copies:
        return args.copies
    return max(2, min(16, math.ceil(256e6 / max(bytes_per_copy, 1)) + 1))


def report(args: Args, ms: float, nbytes: float, flops: float, extra=None) -> None:
    pk = peaks()
    out = {"op": args.op, "ms": round(ms, 5), "us": round(ms * 1e3, 2), "bytes": int(nbytes), "flops": int(flops),
           "gbs": round(nbytes / ms / 1e6, 1), "tflops": round(flops / ms / 1e9, 1),
           "frac_hbm": round(nbytes / ms / 1e6 / pk["hbm_gbs"], 3), "frac_bf16": round(flops / ms / 1e9 / pk["bf16_tflops"], 3),
           "peaks": pk["source"], "iters": args.iters}
    out.update(extra or {})
    print(json.dumps(out))


def bench_gemm(a: Args) -> None:
    dev = "cuda"
    wb = a.n * a.k * 2
    c = n_copies(a, wb)
    ws = [torch.randn(a.n, a.k, device=dev).bfloat16() * 0.02 for _ in range(c)]
    x = torch.randn(a.m, a.k, device=dev).bfloat16()
    out = torch.empty(a.m, a.n, device=dev, dtype=torch.bfloat16)
    fns = [(lambda w=w: ops.gemm(x, w, out=out, static_w=True)) for w in ws]
    ms = timed(fns, a.iters, a.warmup)
    import ctypes
    from zml_b200.ops import _lib
    plan = (ctypes.c_int * 6)()
    _lib.lib().zb_gemm_describe_plan(a.m, a.n, a.k, plan)
    bn = plan[1]
    extra = {"m": a.m, "n": a.n, "k": a.k, "copies": c,
             "plan": {"swap_ab": plan[0], "tile_tokens": bn, "grid": plan[2], "k_blocks_per_cta": plan[3], "cluster": plan[4]},
             "cluster_capacity": {s: _lib.lib().zb_gemm_cluster_capacity(bn, s) for s in (2, 3, 4, 6, 8)} if plan[0] else {}}
    report(a, ms, wb + (a.m * a.k + a.m * a.n) * 2, 2.0 * a.m * a.n * a.k, extra)


def _kv(a: Args, copies: int, page: int = 64):
    pages_per = (a.seqlen + page - 1) // page
    total = a.batch * pages_per + 1
    caches = [(torch.randn(total, page, a.hkv, a.hd, device="cuda").bfloat16(), torch.randn(total, page, a.hkv, a.hd, device="cuda").bfloat16())
              for _ in range(copies)]
    bt = (torch.arange(a.batch * pages_per, dtype=torch.int32, device="cuda") + 1).view(a.batch, pages_per)
    return caches, bt


def bench_decode_attention(a: Args) -> None:
    kvb = a.batch * a.seqlen * a.hkv * a.hd * 2 * 2
    c = n_copies(a, kvb)
    caches, bt = _kv(a, c)
    q = torch.randn(a.batch, a.hq, a.hd, device="cuda").bfloat16()
    sl = torch.full((a.batch,), a.seqlen, dtype=torch.int32, device="cuda")
    splits = a.splits or ops.decode_plan_splits(a.batch, a.hkv, a.seqlen)
    fns = [(lambda kc=kc, vc=vc: ops.paged_decode(q, kc, vc, bt, sl, num_splits=splits, max_seq_len=a.seqlen)) for kc, vc in caches]
    ms = timed(fns, a.iters, a.warmup)
    report(a, ms, kvb, 4.0 * a.batch * a.hq * a.seqlen * a.hd, {"batch": a.batch, "seqlen": a.seqlen, "splits": splits, "copies": c})


def bench_prefill_attention(a: Args) -> None:
    caches, bt = _kv(a, 2)
    t = a.batch * a.seqlen
    q = torch.randn(t, a.hq, a.hd, device="cuda").bfloat16()
    sl = torch.full((a.batch,), a.seqlen, dtype=torch.int32, device="cuda")
    qs = (torch.arange(a.batch + 1, dtype=torch.int32, device="cuda") * a.seqlen).int()
    fns = [(lambda kc=kc, vc=vc: ops.paged_prefill(q, kc, vc, bt, sl, qs)) for kc, vc in caches]
    ms = timed(fns, a.iters, a.warmup)
    flops = 4.0 * a.batch * a.hq * a.hd * a.seqlen * (a.seqlen + 1) / 2
    report(a, ms, (2 * t * a.hq * a.hd + 2 * t * a.hkv * a.hd) * 2, flops, {"batch": a.batch, "seqlen": a.seqlen})


def bench_moe(a: Args) -> None:
    from zml_b200 import moe
    d, f, e, k = a.k, a.n, a.experts, a.topk
    wb = e * 3 * d * f * 2
    c = n_copies(a, wb)
    sets = []
    for _ in range(c):
        g = torch.randn(e, f, d, device="cuda").bfloat16() * 0.02
        u = torch.randn(e, f, d, device="cuda").bfloat16() * 0.02
        gu, dn = moe.interleave_gate_up(g, u), torch.randn(e, d, f, device="cuda").bfloat16() * 0.02
        del g, u
        if a.w4:
            q = (moe.Nvfp4Experts.quantize(gu), moe.Nvfp4Experts.quantize(dn))
            sets.append((q[0].dequantize(), q[1].dequantize(), q))
        else:
            sets.append((gu, dn, None))
        del gu, dn
    x = torch.randn(a.tokens, d, device="cuda").bfloat16()
    logits = torch.randn(a.tokens, e, device="cuda")
    ids, w = moe.router_topk(logits, k, True)
    fns = [(lambda gu=gu, dn=dn, q=q: moe.fused_experts(x, ids, w, gu, dn, 0, e, q)) for gu, dn, q in sets]
    ms = timed(fns, a.iters, a.warmup)
    active = min(e, a.tokens * k)
    wbytes = active * 3 * d * f * (0.5 + 1.0 / 16 if a.w4 else 2)
    report(a, ms, wbytes, 6.0 * a.tokens * k * d * f, {"tokens": a.tokens, "experts": e, "topk": k, "copies": c, "w4": a.w4})


def bench_gated_delta_scan(a: Args) -> None:
    from zml_b200.ops import linear_attn as la
    hk, hv, dk, dv = 16, 32, 128, 128
    t = a.batch * a.seqlen
    cols = 2 * hk * dk + 2 * hv * dv + 2 * hv
    proj = torch.randn(t, cols, device="cuda").bfloat16()
    state = torch.zeros(a.batch, hv, dk, dv, device="cuda")
    a_log = torch.log(torch.empty(hv, device="cuda").uniform_(1, 8))
    dtb = torch.zeros(hv, device="cuda")
    nw = torch.ones(dv, device="cuda").bfloat16()
    qs = (torch.arange(a.batch + 1, dtype=torch.int32, device="cuda") * a.seqlen).int()
    # one token per sequence: a decode step, with a past; else whole sequences
    sl = torch.full((a.batch,), a.seqlen + (a.seqlen == 1), dtype=torch.int32, device="cuda")
    slots = torch.arange(a.batch, dtype=torch.int32, device="cuda")
    oz, ob = 2 * hk * dk + hv * dv, 2 * hk * dk + 2 * hv * dv
    fn = lambda: la.gated_delta_scan(proj[:, :oz], proj[:, oz:ob], proj[:, ob + hv:ob + 2 * hv], proj[:, ob:ob + hv], a_log, dtb,
                                     nw, 1e-6, state, qs, sl, slots, hk, hv, dk, dv)
    ms = (timed_graph if a.seqlen == 1 else timed)([fn], a.iters, a.warmup)
    report(a, ms, t * cols * 2 + t * hv * dv * 2 + 2 * state.numel() * 4, 6.0 * t * hv * dk * dv, {"batch": a.batch, "seqlen": a.seqlen})


def _latent(a: Args):
    """Layer sizes of the latent-attention benchmarks and a filled cache with one block table per copy."""
    from zml_b200.ops import latent as lat
    d = lat.LatentDims(a.hq, 128, 64, 128, 512, 1536, a.window, 192 ** -0.5, 500000.0)
    pages_per = (a.seqlen + 63) // 64
    bt = (torch.arange(a.batch * pages_per, dtype=torch.int32, device="cuda") + 1).view(a.batch, pages_per)
    c = n_copies(a, a.batch * min(a.seqlen, a.window) * d.row * 2)
    caches = [torch.randn(a.batch * pages_per + 1, 64, d.row, device="cuda").bfloat16() for _ in range(c)]
    return lat, d, bt, caches


def bench_latent_prefill(a: Args) -> None:
    """The prefill kernel alone, and the whole attention of a layer behind the query projection (gather, key / value
    projection, query packing, attention with the gate)."""
    from types import SimpleNamespace
    lat, d, bt, caches = _latent(a)
    t = a.batch * a.seqlen
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device="cuda")
    qs, sl = [i * a.seqlen for i in range(a.batch + 1)], [a.seqlen] * a.batch
    meta = SimpleNamespace(is_prefill=True, q_start_host=qs, seq_lens_host=sl, q_start=i32(qs), seq_lens=i32(sl), plans={}, block_table=bt,
                           positions=torch.arange(a.seqlen, dtype=torch.int32, device="cuda").repeat(a.batch))
    q = torch.randn(t, d.heads * 192, device="cuda").bfloat16()
    gate = None if a.sink else torch.randn(t, d.heads * 128, device="cuda").bfloat16()
    sink = torch.randn(d.heads, device="cuda") if a.sink else None
    w = torch.randn(d.heads * 256, 512, device="cuda").bfloat16() * 0.05
    inv = d.inv_freq("cuda")
    pairs = sum(min(i + 1, a.window) for i in range(a.seqlen)) * a.batch
    flops = 2.0 * pairs * d.heads * (192 + 128)
    ms = timed([lambda c=c: lat.prefill(q, gate, w, inv, c, meta, d, sink) for c in caches], a.iters, a.warmup)
    report(a, ms, t * d.heads * (192 + 256) * 2, flops + 2.0 * t * 512 * d.heads * 256, {"part": "whole", "batch": a.batch, "seqlen": a.seqlen, "heads": a.hq, "window": a.window})
    shape = {"batch": a.batch, "seqlen": a.seqlen, "heads": a.hq, "window": a.window}
    x, kv, rot_out, plan = lat.expand(caches[0], w, meta, d)
    qp = lat.pack_q(q, inv, meta.positions, d)
    ms = timed([lambda: lat.attend_expanded(qp, gate, x, kv, rot_out, plan, meta, d, sink)], a.iters, a.warmup)
    report(a, ms, t * d.heads * (192 + 192 + 128 + 128) * 2, flops, dict(shape, part="attention kernel"))
    ms = timed([lambda: lat.pack_q(q, inv, meta.positions, d)], a.iters, a.warmup)
    report(a, ms, t * d.heads * 192 * 4, 0, dict(shape, part="query packing"))
    ms = timed([lambda c=c: lat.expand(c, w, meta, d) for c in caches], a.iters, a.warmup)
    report(a, ms, t * (576 * 4 + 512 * 2 + d.heads * 512), 2.0 * t * 512 * d.heads * 256, dict(shape, part="gather and key / value projection"))


def bench_latent_decode(a: Args) -> None:
    lat, d, bt, caches = _latent(a)
    q = torch.randn(a.batch, d.heads * 192, device="cuda").bfloat16()
    gate = None if a.sink else torch.randn(a.batch, d.heads * 128, device="cuda").bfloat16()
    sink = torch.randn(d.heads, device="cuda") if a.sink else None
    uk = [torch.randn(d.heads, 512, 128, device="cuda").bfloat16() for _ in range(8)]
    uv = [torch.randn(d.heads, 128, 512, device="cuda").bfloat16() for _ in range(8)]
    inv, pos = d.inv_freq("cuda"), torch.full((a.batch,), a.seqlen - 1, dtype=torch.int32, device="cuda")
    qs, sl = torch.arange(a.batch + 1, dtype=torch.int32, device="cuda"), torch.full((a.batch,), a.seqlen, dtype=torch.int32, device="cuda")
    ql = lat.absorb_q(q, uk[0], inv, pos, d)
    splits = a.splits or lat.decode_plan_splits(a.batch, d, a.seqlen)
    keys = a.batch * min(a.seqlen, a.window)
    shape = {"batch": a.batch, "seqlen": a.seqlen, "heads": a.hq, "window": a.window, "splits": splits}
    ms = timed_graph([lambda c=c: lat.attend(ql, c, bt, qs, sl, d, decode=True, num_splits=splits, sink=sink) for c in caches], a.iters, a.warmup)
    report(a, ms, keys * d.row * 2, 2.0 * keys * d.heads * (576 + 512), dict(shape, part="attention kernel"))
    o = lat.attend(ql, caches[0], bt, qs, sl, d, decode=True, num_splits=splits, sink=sink)
    wb = d.heads * 512 * 128 * 2
    ms = timed_graph([lambda w=w: lat.absorb_q(q, w, inv, pos, d) for w in uk], a.iters, a.warmup)
    report(a, ms, wb, 2.0 * a.batch * d.heads * 512 * 128, dict(shape, part="queries into the latent space"))
    ms = timed_graph([lambda w=w: lat.absorb_out(o, w, gate, d) for w in uv], a.iters, a.warmup)
    report(a, ms, wb, 2.0 * a.batch * d.heads * 512 * 128, dict(shape, part="results out of it"))


def bench_wkv_scan(a: Args) -> None:
    from zml_b200.ops import linear_attn as la
    H, D, t = a.hq, a.hd, a.batch * a.seqlen
    x = [torch.randn(t, H * D, device="cuda").bfloat16() for _ in range(4)]
    z = torch.randn(t, H * D, device="cuda")
    v = [torch.randn(H * D, device="cuda") for _ in range(3)]
    qs = (torch.arange(a.batch + 1, dtype=torch.int32, device="cuda") * a.seqlen).int()
    sl = torch.full((a.batch,), a.seqlen + 1, dtype=torch.int32, device="cuda")
    slots = torch.arange(a.batch, dtype=torch.int32, device="cuda")
    states = [torch.zeros(a.batch, H, D, D, device="cuda") for _ in range(n_copies(a, a.batch * H * D * D * 8) if a.seqlen == 1 else 1)]
    ms = (timed_graph if a.seqlen == 1 else timed)([lambda s=s: la.wkv_scan(*x, z, *v, 1e-5, s, qs, sl, slots, H, D, decode=a.seqlen == 1) for s in states], a.iters, a.warmup)
    report(a, ms, t * H * D * (5 * 2 + 4) + 2 * states[0].numel() * 4, 6.0 * t * H * D * D, {"batch": a.batch, "seqlen": a.seqlen, "heads": H, "dim": D})


def _gqa(a: Args):
    """A capped, sunk, windowed and gated attention at the sizes of the plain paged benchmarks, with filled caches."""
    from types import SimpleNamespace
    from zml_b200.ops import gqa
    s = gqa.GqaSpec(a.hq, a.hkv, a.hd, a.hd, a.hd // 2, scale=a.hd ** -0.5, cap=50.0, window=a.window, keep=16, sink=True)
    c = n_copies(a, a.batch * a.seqlen * a.hkv * a.hd * 4) if a.op == "gqa_decode" else 2
    caches, bt = _kv(a, c)
    n = a.seqlen if a.op == "gqa_prefill" else 1
    t = a.batch * n
    qs = (torch.arange(a.batch + 1, dtype=torch.int32, device="cuda") * n).int()
    sl = torch.full((a.batch,), a.seqlen, dtype=torch.int32, device="cuda")
    splits = a.splits or ops.decode_plan_splits(a.batch, a.hkv, s.visible(a.seqlen))
    meta = SimpleNamespace(is_prefill=n > 1, q_start=qs, seq_lens=sl, block_table=bt, total_q_blocks=a.batch * ((n + 63) // 64), num_splits=splits,
                           max_seq_len=a.seqlen)
    nq = (a.hq + 2 * a.hkv) * a.hd
    proj = torch.randn(t, nq + a.hq * a.hd, device="cuda").bfloat16()
    return gqa, s, caches, meta, proj, nq, t


def bench_gqa_prefill(a: Args) -> None:
    gqa, s, caches, meta, proj, nq, t = _gqa(a)
    q = torch.randn(t, a.hq, a.hd, device="cuda").bfloat16()
    ms = timed([lambda c=c: gqa.attention(q, proj[:, nq:], c, meta, s) for c in caches], a.iters, a.warmup)
    pairs = a.seqlen * (a.seqlen + 1) / 2 if a.window >= a.seqlen else a.window * (a.seqlen - (a.window - 1) / 2)
    shape = {"batch": a.batch, "seqlen": a.seqlen, "hq": a.hq, "hkv": a.hkv, "hd": a.hd, "window": a.window}
    report(a, ms, (3 * t * a.hq * a.hd + 2 * t * a.hkv * a.hd) * 2, 4.0 * a.batch * a.hq * a.hd * pairs, dict(shape, part="attention"))
    slots = (torch.arange(t, dtype=torch.int32, device="cuda") + 64).int()
    pos = (torch.arange(t, device="cuda") % a.seqlen).int()
    w, f = torch.ones(a.hd, device="cuda"), s.inv_freq("cuda")
    ms = timed([lambda c=c: gqa.prep(proj, w, w, f, pos, slots, c, 1e-6, s) for c in caches], a.iters, a.warmup)
    report(a, ms, 2 * t * nq * 2, 0, dict(shape, part="norms, rotation, cache write"))
    pos_full, lay = pos, dict(q_norm_w=w.bfloat16(), k_norm_w=w.bfloat16())
    ms = timed([lambda c=c: ops.rope_kvwrite(proj[:, :nq], pos_full, slots, f, c[0], c[1], a.hq, a.hkv, a.hd, 0, a.hd // 2, **lay) for c in caches], a.iters,
               a.warmup)
    report(a, ms, 2 * t * nq * 2, 0, dict(shape, part="the same in the other families"))


def bench_gqa_decode(a: Args) -> None:
    gqa, s, caches, meta, proj, nq, t = _gqa(a)
    q = torch.randn(t, a.hq, a.hd, device="cuda").bfloat16()
    ms = timed_graph([lambda c=c: gqa.attention(q, proj[:, nq:], c, meta, s) for c in caches], a.iters, a.warmup)
    kvb = a.batch * min(a.seqlen, a.window + 16) * a.hkv * a.hd * 4
    report(a, ms, kvb, 4.0 * a.batch * a.hq * min(a.seqlen, a.window) * a.hd, {"batch": a.batch, "seqlen": a.seqlen, "window": a.window, "splits": meta.num_splits})
    sl = meta.seq_lens
    ms = timed_graph([lambda c=c: ops.paged_decode(q, *c, meta.block_table, sl, num_splits=meta.num_splits, max_seq_len=a.seqlen) for c in caches], a.iters, a.warmup)
    kvb = a.batch * a.seqlen * a.hkv * a.hd * 4
    report(a, ms, kvb, 4.0 * a.batch * a.hq * a.seqlen * a.hd, {"batch": a.batch, "seqlen": a.seqlen, "part": "the plain kernel"})


def _pool(a: Args, n: int):
    """A capped attention over a window and the pooled blocks in front of it, and the same without blocks, with filled caches."""
    from types import SimpleNamespace
    from zml_b200.ops import gqa
    s = gqa.GqaSpec(a.hq, a.hkv, a.hd, a.hd, a.hd // 2, scale=a.hd ** -0.5, cap=50.0, window=a.window, pool=a.pool, whole_norm=True,
                    yarn=gqa.Yarn(4.0, 4096, 32.0, 1.0))
    plain = gqa.GqaSpec(a.hq, a.hkv, a.hd, a.hd, a.hd // 2, scale=a.hd ** -0.5, cap=50.0, window=a.window)
    caches, bt = _kv(a, n_copies(a, a.batch * min(a.seqlen, a.window) * a.hkv * a.hd * 4) if n == 1 else 2)
    rows = gqa.pool_rows(a.pool, 64)
    caches = [(k, v, *(torch.randn(k.shape[0], rows, a.hkv, a.hd, device="cuda").bfloat16() for _ in range(2))) for k, v in caches]
    t = a.batch * n
    qs = (torch.arange(a.batch + 1, dtype=torch.int32, device="cuda") * n).int()
    sl = torch.full((a.batch,), a.seqlen, dtype=torch.int32, device="cuda")
    pos = (a.seqlen - n + torch.arange(t, device="cuda") % n).int()
    metas = [SimpleNamespace(is_prefill=n > 1, q_start=qs, seq_lens=sl, block_table=bt, positions=pos, total_q_blocks=a.batch * ((n + 63) // 64),
                             num_splits=a.splits or ops.decode_plan_splits(a.batch, a.hkv, x.visible(a.seqlen)), max_seq_len=a.seqlen) for x in (s, plain)]
    proj = torch.randn(t, s.columns(), device="cuda").bfloat16()
    shape = {"batch": a.batch, "seqlen": a.seqlen, "hq": a.hq, "hkv": a.hkv, "hd": a.hd, "window": a.window, "pool": a.pool}
    return gqa, (s, plain), caches, metas, proj, bt, shape, t


def bench_pool_prefill(a: Args) -> None:
    gqa, specs, caches, metas, proj, bt, shape, t = _pool(a, a.seqlen)
    q = torch.randn(t, a.hq, a.hd, device="cuda").bfloat16()
    w = min(a.window, a.seqlen)
    pairs = w * (a.seqlen - (w - 1) / 2)
    blocks = sum((i - w + 1) // a.pool for i in range(w, a.seqlen))
    nbytes = (2 * t * a.hq * a.hd + 2 * t * a.hkv * a.hd) * 2
    for s, meta, n, part in ((specs[0], metas[0], pairs + blocks, "window and pooled blocks"), (specs[1], metas[1], pairs, "window alone")):
        ms = timed([lambda c=c: gqa.attention(q, None, c if s.pool else c[:2], meta, s) for c in caches], a.iters, a.warmup)
        report(a, ms, nbytes, 4.0 * a.batch * a.hq * a.hd * n, dict(shape, part=part))
    slots = (bt[:, :, None] * 64 + torch.arange(64, dtype=torch.int32, device="cuda")).reshape(a.batch, -1)[:, :a.seqlen].reshape(-1).int().contiguous()
    qn, kn = torch.ones(a.hq * a.hd, device="cuda"), torch.ones(a.hkv * a.hd, device="cuda")
    freq, pos = specs[0].inv_freq("cuda"), metas[0].positions
    kept = specs[1]
    for part, fn in (("norms over the projections, rotation, cache write", lambda c: gqa.prep(proj, qn, kn, freq, pos, slots, c, 1e-6, specs[0])),
                     ("norms per head, rotation, cache write", lambda c: gqa.prep(proj, qn[:a.hd], kn[:a.hd], freq, pos, slots, c[:2], 1e-6, kept))):
        ms = timed([lambda c=c: fn(c) for c in caches], a.iters, a.warmup)
        report(a, ms, 2 * t * proj.shape[1] * 2, 0, dict(shape, part=part))
    ms = timed([lambda c=c: gqa.pool_new(c, metas[0], specs[0]) for c in caches], a.iters, a.warmup)
    report(a, ms, t * a.hkv * a.hd * 4 * (1 + 1 / a.pool), 0, dict(shape, part="pooled blocks"))


def bench_pool_decode(a: Args) -> None:
    gqa, specs, caches, metas, proj, bt, shape, t = _pool(a, 1)
    q = torch.randn(t, a.hq, a.hd, device="cuda").bfloat16()
    w = min(a.window, a.seqlen)
    for s, meta, n, part in ((specs[0], metas[0], w + (a.seqlen - w) // a.pool, "window and pooled blocks"), (specs[1], metas[1], w, "window alone")):
        ms = timed_graph([lambda c=c: gqa.attention(q, None, c if s.pool else c[:2], meta, s) for c in caches], a.iters, a.warmup)
        report(a, ms, a.batch * n * a.hkv * a.hd * 4, 4.0 * a.batch * a.hq * n * a.hd, dict(shape, part=part, splits=meta.num_splits))
    slots = (bt[:, (a.seqlen - 1) // 64] * 64 + (a.seqlen - 1) % 64).int()
    qn, kn = torch.ones(a.hq * a.hd, device="cuda"), torch.ones(a.hkv * a.hd, device="cuda")
    freq, pos = specs[0].inv_freq("cuda"), metas[0].positions
    for part, fn in (("norms over the projections, rotation, cache write, a block per sequence", lambda c: gqa.prep(proj, qn, kn, freq, pos, slots, c, 1e-6, specs[0], step_table=bt)),
                     ("norms per head, rotation, cache write", lambda c: gqa.prep(proj, qn[:a.hd], kn[:a.hd], freq, pos, slots, c[:2], 1e-6, specs[1]))):
        ms = timed_graph([lambda c=c: fn(c) for c in caches], a.iters, a.warmup)
        report(a, ms, 2 * t * proj.shape[1] * 2, 0, dict(shape, part=part))


def bench_gated_scan(a: Args) -> None:
    from zml_b200.ops import _lib
    from zml_b200.ops import linear_attn as la
    n, t, decode = a.k, a.batch * a.seqlen, a.seqlen == 1
    qs = (torch.arange(a.batch + 1, dtype=torch.int32, device="cuda") * a.seqlen).int()
    sl = torch.full((a.batch,), a.seqlen + decode, dtype=torch.int32, device="cuda")
    slots, zb, xb = torch.arange(a.batch, dtype=torch.int32, device="cuda"), torch.randn(n, device="cuda") - 2, torch.randn(n, device="cuda")
    projs = [torch.randn(t, 3 * n, device="cuda").bfloat16() for _ in range(n_copies(a, t * n * 6))]
    state = torch.zeros(a.batch, n, device="cuda")
    nb = a.batch * ((a.seqlen + la.GATED_ROWS - 1) // la.GATED_ROWS)
    fns = [lambda p=p: la.gated_scan(p[:, :n], p[:, n:2 * n], p[:, 2 * n:], zb, xb, state, qs, sl, slots, 0.7, decode=decode, num_blocks=nb) for p in projs]
    with contextlib.nullcontext() if decode else _lib.serial_launches():          # as the engine launches them
        ms = timed_graph(fns, a.iters, a.warmup)
    report(a, ms, t * n * 8 + a.batch * n * 8, 0, {"batch": a.batch, "seqlen": a.seqlen, "width": n})


def bench_add_norm(a: Args) -> None:
    """The residual sum with the norm in front of the next sublayer and its convolution: two launches for prompts, one for a step."""
    from zml_b200.ops import stream
    t, d = a.tokens, a.k
    c = max(2, min(64, math.ceil(256e6 / (t * d * 8)) + 1))
    xs = [torch.randn(t, d, device="cuda") for _ in range(c)]
    y, w, b = torch.randn(t, d, device="cuda"), torch.ones(d, device="cuda"), torch.zeros(d, device="cuda")
    conv = stream.InputConv(torch.randn(4, d, device="cuda"), torch.zeros(t, 3, d, device="cuda"))
    qs, sl, slots = torch.tensor([0, t], dtype=torch.int32, device="cuda"), torch.tensor([t], dtype=torch.int32, device="cuda"), torch.arange(t, dtype=torch.int32, device="cuda")
    kw = dict(w=w, b=b, eps=1e-5)
    ms = timed_graph([lambda x=x: stream.add_norm(x, y, act_dtype=torch.float32, **kw) for x in xs], a.iters, a.warmup)
    report(a, ms, t * d * 16, 0, {"part": "residual sum and norm", "tokens": t, "d": d})
    ms = timed_graph([lambda x=x: stream.stream_conv(x, conv, qs, sl, slots, torch.bfloat16) for x in xs], a.iters, a.warmup)
    report(a, ms, t * d * 6, 0, {"part": "convolution", "tokens": t, "d": d})
    lens = torch.full((t,), 9, dtype=torch.int32, device="cuda")
    ms = timed_graph([lambda x=x: stream.add_norm(x, y, act_dtype=torch.bfloat16, conv=conv, seq_lens=lens, slots=slots, **kw) for x in xs], a.iters, a.warmup)
    report(a, ms, t * d * (14 + 24), 0, {"part": "step: residual sum, norm, convolution", "tokens": t, "d": d})
    ms = timed_graph([lambda x=x: stream.post_norm(x, w, 1e-5, y, 2.0, act_dtype=torch.bfloat16, conv=conv, seq_lens=lens, slots=slots) for x in xs], a.iters, a.warmup)
    report(a, ms, t * d * (14 + 24), 0, {"part": "step: norm behind a sublayer, convolution", "tokens": t, "d": d})
    ms = timed_graph([lambda x=x: stream.sandwich_norm(x, y, w, 0.5, w, 1e-5, act_dtype=torch.bfloat16) for x in xs], a.iters, a.warmup)
    report(a, ms, t * d * 14, 0, {"part": "norms on both sides of a sublayer", "tokens": t, "d": d})


def bench_relu_mixture(a: Args) -> None:
    """Router by sigmoid scores, routed and shared experts with squared units, and the residual sum with the norm that follows; beside
    it a gated mixture with the same active parameters and its norms."""
    from zml_b200.moe import ops as mops
    from zml_b200.ops import stream
    e, k, f, d, t = a.experts, a.topk, a.n, a.k, a.tokens
    c = max(2, min(8, math.ceil(300e6 / (e * f * d * 4)) + 1))
    rand = lambda *s: torch.randn(*s, device="cuda").bfloat16() * 0.02
    ws = [mops.pad_plain_experts(rand(e + 1, f, d), rand(e + 1, d, f)) for _ in range(c)]
    fg = f * 2 // 3
    gated = [mops.pad_experts(rand(e + 1, fg, d), rand(e + 1, fg, d), rand(e + 1, d, fg)) for _ in range(c)]
    router, bias = rand(e + 1, d), torch.zeros(e + 1, device="cuda").bfloat16()
    corr, w, b = torch.zeros(e, device="cuda"), torch.ones(d, device="cuda"), torch.zeros(d, device="cuda")
    h, x = torch.randn(t, d, device="cuda").bfloat16(), torch.randn(t, d, device="cuda")

    def mine(i):
        z = ops.gemm(h, router[:e], out_dtype=torch.float32, static_w=True)
        ids, wt = mops.route(z, k, e, corr, 1, 0, "sigmoid", False, 1.0, False)
        rows, pos = mops.expert_rows(h, ids, *ws[i], 0, e + 1, "relu2")
        return stream.add_norm(x, stream.ExpertRows(rows, pos, wt), w, b, 1e-6, torch.float32)

    def theirs(i):
        z = ops.gemm(h, router, bias=bias, out_dtype=torch.float32, static_w=True)
        ids, wt = mops.router_topk(z, k + 1)
        rows, pos = mops.expert_rows(h, ids, *gated[i], 0, e + 1)
        return stream.sandwich_norm(x, stream.ExpertRows(rows, pos, wt), w, 0.5, w, 1e-6, act_dtype=torch.bfloat16)

    active = min(e, t * k) + 1
    for part, fn in (("squared units, shared expert", mine), ("gated units, one more choice", theirs)):
        ms = timed_graph([lambda i=i, fn=fn: fn(i) for i in range(c)], a.iters, a.warmup)
        report(a, ms, active * 2 * f * d * 2, 4.0 * t * (k + 1) * f * d, {"part": part, "tokens": t, "experts": e, "top": k, "ff": f, "d": d})


def _diff(a: Args, n: int):
    """Differential heads (two maps of hd / 2 over values of hd) that see their chunk of `window` tokens, with filled caches: a
    key / value head takes the bytes of a plain one of size hd."""
    from types import SimpleNamespace
    from zml_b200.ops import gqa
    s = gqa.GqaSpec(a.hq, a.hkv, a.hd // 2, a.hd, a.hd // 4, scale=(a.hd // 2) ** -0.5, chunk=a.window, maps=2)
    caches, bt = _kv(a, n_copies(a, a.batch * a.seqlen * a.hkv * a.hd * 4) if n == 1 else 2)
    t = a.batch * n
    qs = (torch.arange(a.batch + 1, dtype=torch.int32, device="cuda") * n).int()
    sl = torch.full((a.batch,), a.seqlen, dtype=torch.int32, device="cuda")
    meta = SimpleNamespace(is_prefill=n > 1, q_start=qs, seq_lens=sl, block_table=bt, total_q_blocks=a.batch * ((n + 63) // 64),
                           num_splits=a.splits or ops.decode_plan_splits(a.batch, a.hkv, s.visible(a.seqlen)), max_seq_len=a.seqlen)
    proj = torch.randn(t, s.columns(), device="cuda").bfloat16()
    slots = (torch.arange(t, dtype=torch.int32, device="cuda") + 64).int()
    pos = (torch.arange(t, device="cuda") % a.seqlen).int()
    freq = s.inv_freq("cuda")
    prep = lambda c: gqa.prep(proj, None, None, freq, pos, slots, c, 1e-6, s)
    return gqa, s, caches, meta, prep, gqa.DiffMix(0.3, 0.5, 1e-6), t


def bench_diff_prefill(a: Args) -> None:
    gqa, s, caches, meta, prep, mix, t = _diff(a, a.seqlen)
    q = prep(caches[0])
    shape = {"batch": a.batch, "seqlen": a.seqlen, "hq": a.hq, "hkv": a.hkv, "map": s.dim, "vdim": s.vdim, "chunk": s.chunk}
    pairs = a.batch * sum(i % s.chunk + 1 for i in range(a.seqlen))
    ms = timed([lambda c=c: gqa.attention(q, None, c, meta, s, mix) for c in caches], a.iters, a.warmup)
    report(a, ms, (t * a.hq * 2 * a.hd + 2 * t * a.hkv * a.hd) * 2, 2.0 * pairs * s.rows_q * (s.dim + s.vdim), dict(shape, part="attention"))
    ms = timed([lambda c=c: prep(c) for c in caches], a.iters, a.warmup)
    report(a, ms, t * 2 * s.columns() * 2, 0, dict(shape, part="rotation, cache write"))


def bench_diff_decode(a: Args) -> None:
    gqa, s, caches, meta, prep, mix, t = _diff(a, 1)
    q = prep(caches[0])
    seen = (a.seqlen - 1) % s.chunk + 1
    ms = timed_graph([lambda c=c: gqa.attention(q, None, c, meta, s, mix) for c in caches], a.iters, a.warmup)
    report(a, ms, a.batch * seen * a.hkv * a.hd * 4, 2.0 * a.batch * seen * s.rows_q * (s.dim + s.vdim),
           {"batch": a.batch, "seqlen": a.seqlen, "seen": seen, "splits": meta.num_splits, "hq": a.hq, "hkv": a.hkv, "map": s.dim, "vdim": s.vdim})


def bench_channel_delta(a: Args) -> None:
    from zml_b200.ops import linear_attn as la
    H, D, t = a.hq, a.hd, a.batch * a.seqlen
    decode = a.seqlen == 1
    qs = (torch.arange(a.batch + 1, dtype=torch.int32, device="cuda") * a.seqlen).int()
    sl = torch.full((a.batch,), a.seqlen + decode, dtype=torch.int32, device="cuda")
    slots = torch.arange(a.batch, dtype=torch.int32, device="cuda")
    layers = []
    for _ in range(n_copies(a, a.batch * H * D * D * 4) if decode else 1):
        m = la.ChannelDelta(H, H, D, D, torch.randn(4, 3 * H * D, device="cuda"), torch.rand(H, device="cuda"), torch.rand(H * D, device="cuda") * 4 - 5,
                            torch.ones(D, device="cuda"), 1e-6)
        m.alloc(a.batch, torch.bfloat16, "cuda")
        layers.append(m)
    proj = torch.randn(t, 3 * H * D + (H + 7) // 8 * 8, device="cuda").bfloat16()
    low = torch.randn(t, 2 * H * D, device="cuda")
    fns = [lambda m=m: la.channel_delta(proj, m.channels, low, m, qs, sl, slots, decode, a.batch * ((a.seqlen + 7) // 8)) for m in layers]
    from zml_b200.ops import _lib
    with contextlib.nullcontext() if decode else _lib.serial_launches():          # as the engine launches them
        ms = (timed_graph if decode else timed)(fns, a.iters, a.warmup)
    nbytes = t * H * D * (3 * 2 + 2 * 4 + 2) + a.batch * H * D * D * 8
    report(a, ms, nbytes, 6.0 * t * H * D * D, {"batch": a.batch, "seqlen": a.seqlen, "heads": H, "dim": D})


def bench_mixture(a: Args) -> None:
    """Router, experts and the norm that sums their rows; the same with the other families' mixture and norm kernels."""
    from zml_b200.moe import ops as mops
    from zml_b200.ops import stream
    e, k, f, d, t = a.experts, a.topk, a.n, a.k, a.tokens
    c = max(2, min(8, math.ceil(300e6 / (e * f * d * 6)) + 1))
    ws = [mops.pad_experts(*(torch.randn(e, *s, device="cuda").bfloat16() * 0.02 for s in ((f, d), (f, d), (d, f)))) for _ in range(c)]
    router, bias = torch.randn(e, d, device="cuda").bfloat16() * 0.05, torch.zeros(e, device="cuda").bfloat16()
    h, x, res = torch.randn(t, d, device="cuda").bfloat16(), torch.randn(t, d, device="cuda"), torch.randn(t, d, device="cuda").bfloat16()
    nw, nb = torch.ones(d, device="cuda"), torch.ones(d, device="cuda").bfloat16()

    def mine(w):
        z = ops.gemm(h, router, bias=bias, out_dtype=torch.float32, static_w=True)
        ids, wt = mops.router_topk(z, k)
        rows, pos = mops.expert_rows(h, ids, *w, 0, e)
        return stream.sandwich_norm(x, stream.ExpertRows(rows, pos, wt), nw, 0.5, nw, 1e-6, act_dtype=torch.bfloat16)

    def theirs(w):
        z = ops.gemm(h, router, out_dtype=torch.float32, static_w=True)
        ids, wt = mops.router_topk(z, k)
        return ops.rmsnorm(mops.fused_experts(h, ids, wt, *w, 0, e, residual=res), nb)

    active = min(e, t * k)
    for part, fn in (("mixture", mine), ("other families", theirs)):
        ms = timed_graph([lambda w=w, fn=fn: fn(w) for w in ws], a.iters, a.warmup)
        report(a, ms, active * 3 * f * d * 2, 6.0 * t * k * f * d, {"part": part, "tokens": t, "experts": e, "top": k, "ff": f, "d": d})


def bench_shared_mixture(a: Args) -> None:
    """Router, routed and shared experts with clipped units, and the streams' update that sums their rows; the same sizes with the
    routed mixture alone, and with the mixture, shared expert and norm of the Qwen3.5-MoE family."""
    from zml_b200 import moe
    from zml_b200.moe import ops as mops
    from zml_b200.ops import stream
    e, k, f, d, t = a.experts, a.topk, a.n, a.k, a.tokens
    c = max(2, min(8, math.ceil(300e6 / (e * f * d * 6)) + 1))
    rand = lambda *s: torch.randn(*s, device="cuda").bfloat16() * 0.02
    ws = [mops.pad_experts(rand(e + 1, f, d), rand(e + 1, f, d), rand(e + 1, d, f)) for _ in range(c)]
    router, sg = rand(e + 1, d), rand(8, d)
    corr, limits = torch.zeros(e, device="cuda"), torch.full((e + 1,), 7.0, device="cuda")
    h, res = torch.randn(t, d, device="cuda").bfloat16(), torch.randn(t, d, device="cuda").bfloat16()
    x = torch.randn(t, 4, d, device="cuda")
    nw, nb = torch.ones(d, device="cuda"), torch.ones(d, device="cuda").bfloat16()
    hm = stream.HyperMix(torch.full((4,), 0.25, device="cuda"), torch.eye(4, device="cuda"), torch.ones(4, device="cuda"))
    dense = [(torch.cat([rand(f, d), rand(f, d)], 0), rand(d, f)) for _ in range(c)]

    def mine(i, shared, update=True):
        w1, w2 = ws[i]
        z = ops.gemm(h, router, out_dtype=torch.float32, static_w=True)
        ids, wt = mops.route(z, k, e, corr, shared, 0)
        s = 1 - shared
        rows, pos = mops.expert_rows(h, ids, w1[s:], w2[s:], 0, e + shared, "clipped_glu", limits[s:])
        return stream.hyper_norm(x, stream.ExpertRows(rows, pos, wt), hm, hm.inp, nw, 1e-6, torch.bfloat16) if update else rows

    def theirs(i):
        w1, w2 = ws[i]
        z = ops.gemm(h, router[:e], out_dtype=torch.float32, static_w=True)
        ids, wt = mops.router_topk(z, k)
        y = ops.gemm(ops.swiglu(ops.gemm(h, dense[i][0], static_w=True)), dense[i][1], static_w=True)
        gate = torch.sigmoid(ops.gemm(h, sg, out_dtype=torch.float32, static_w=True)[:, :1])
        y = (y.float() * gate).to(y.dtype)
        return ops.rmsnorm(moe.forward_moe(h, ids, wt, w1[1:], w2[1:], None, e, residual=res, extra_partial=y), nb)

    active = min(e, t * k) + 1
    for part, fn in (("mixture with shared expert, streams", lambda i: mine(i, 1)), ("the same without the streams", lambda i: mine(i, 1, False)),
                     ("without the shared expert", lambda i: mine(i, 0)), ("other family, one stream", theirs)):
        ms = timed_graph([lambda i=i, fn=fn: fn(i) for i in range(c)], a.iters, a.warmup)
        report(a, ms, active * 3 * f * d * 2, 6.0 * t * (k + 1) * f * d, {"part": part, "tokens": t, "experts": e, "top": k, "ff": f, "d": d})


def bench_hyper(a: Args) -> None:
    """The streams' update behind a sublayer with the norm in front of the next one, beside the norms of a single stream."""
    from zml_b200.ops import stream
    t, d = a.tokens, a.k
    y, w = torch.randn(t, d, device="cuda"), torch.ones(d, device="cuda")
    for s in (1, 2, 4, 8):
        hm = stream.HyperMix(torch.full((s,), 1.0 / s, device="cuda"), torch.eye(s, device="cuda"), torch.ones(s, device="cuda"))
        xs = [torch.randn(t, s, d, device="cuda") for _ in range(max(2, min(64, math.ceil(256e6 / (t * d * s * 8)) + 1)))]
        ms = timed_graph([lambda x=x: stream.hyper_norm(x, y, hm, hm.inp, w, 1e-6, torch.bfloat16) for x in xs], a.iters, a.warmup)
        report(a, ms, t * d * (8 * s + 6), 0, {"part": "hyper_norm", "streams": s, "tokens": t, "d": d})
        del xs


def bench_stream(a: Args) -> None:
    """The norm behind a sublayer, the input convolution (with and without interpolations) and the decode step's fusion."""
    from zml_b200.ops import stream
    t, d = a.tokens, a.k
    c = max(2, math.ceil(256e6 / (t * d * 8)) + 1)
    xs = [torch.randn(t, d, device="cuda") for _ in range(c)]
    y, w = torch.randn(t, d, device="cuda"), torch.ones(d, device="cuda")
    mu = torch.rand(5, d, device="cuda")
    qs, sl, slots = torch.tensor([0, t], dtype=torch.int32, device="cuda"), torch.tensor([t], dtype=torch.int32, device="cuda"), torch.zeros(t, dtype=torch.int32, device="cuda")
    ms = timed_graph([lambda x=x: stream.post_norm(x, w, 1e-5, y, 2.0, act_dtype=torch.bfloat16) for x in xs], a.iters, a.warmup)
    report(a, ms, t * d * 14, 0, {"part": "post_norm", "tokens": t, "d": d})
    ms = timed_graph([lambda x=x: stream.sandwich_norm(x, y, w, 0.5, w, 1e-5, act_dtype=torch.bfloat16) for x in xs], a.iters, a.warmup)
    report(a, ms, t * d * 14, 0, {"part": "sandwich_norm", "tokens": t, "d": d})
    for mixes in (False, True):
        conv = stream.InputConv(torch.randn(4, d, device="cuda"), torch.zeros(1, 4 if mixes else 3, d, device="cuda"), mu if mixes else None)
        ms = timed_graph([lambda x=x: stream.stream_conv(x, conv, qs, sl, slots, torch.bfloat16) for x in xs], a.iters, a.warmup)
        report(a, ms, t * d * (4 + (10 if mixes else 2)), 0, {"part": "stream_conv", "mixes": mixes, "tokens": t, "d": d})


def bench_decode_layers(a: Args) -> None:
    """CUDA-graph time per decoder layer of a whole decode step, and of its parts."""
    from zml_b200.models.llama import AttnMeta
    from zml_b200.models.registry import build_model
    model = build_model(a.model, device="cuda")
    c, B, L, page = model.config, a.batch, a.seqlen, 64
    pages_per = (L + 64) // page + 1
    kv = torch.zeros(model.kv_cache_shape(B * pages_per + 1, page), dtype=torch.bfloat16, device="cuda")
    bt = (torch.arange(B * pages_per, dtype=torch.int32, device="cuda") + 1).view(B, pages_per)
    pos = torch.full((B,), L, dtype=torch.int32, device="cuda")
    slot = (bt[:, L // page] * page + L % page).int()
    splits = ops.decode_plan_splits(B, model.hkv, L + 64)
    meta = AttnMeta(False, pos, slot, bt, pos + 1, num_splits=splits, max_seq_len=L + 64)
    x0 = torch.randn(B, c.hidden_size, device="cuda").bfloat16()
    nl = c.num_hidden_layers
    qd = torch.randn(B, model.hq, c.hd, device="cuda").bfloat16()

    fused = hasattr(model, "wants_fused_layout") and model.wants_fused_layout()
    if fused:
        model.prepare_fused()

    def full():
        x = x0.clone()
        if fused:      # norms and SwiGLU inside the GEMM epilogues, row statistics handed from GEMM to GEMM
            st = ops.row_sumsq(x)
            for l in range(nl):
                x, st = model._layer_fused(l, x, st, meta, kv)
            return
        for l in range(nl):
            x = model.layer(l, x, meta, kv)

    def gemms():
        x = x0.clone()
        if fused:
            st = ops.row_sumsq(x)
            for l in range(nl):
                lw = model.layers[l]
                qkv = ops.gemm(x, lw.qkv, static_w=True, row_stats=st, eps=1e-5)
                x, st = ops.gemm(qkv[:, :model.hq * c.hd], lw.o, residual=x, out=x, static_w=True, emit_stats=True)
                act = ops.gemm(x, lw.gate_up, static_w=True, row_stats=st, eps=1e-5, swiglu=True)
                x, st = ops.gemm(act, lw.down, residual=x, out=x, static_w=True, emit_stats=True)
            return
        for l in range(nl):
            lw = model.layers[l]
            qkv = ops.gemm(x, lw.qkv, static_w=True)
            x = ops.gemm(qkv[:, :model.hq * c.hd], lw.o, residual=x, static_w=True)
            gu = ops.gemm(x, lw.gate_up, static_w=True)
            x = ops.gemm(gu[:, :model.f_local], lw.down, residual=x, static_w=True)

    def attn():
        for l in range(nl):
            ops.paged_decode(qd, kv[l, 0], kv[l, 1], bt, pos + 1, num_splits=splits, max_seq_len=L + 64)

    def graph_us(fn) -> float:
        s = torch.cuda.Stream()
        s.wait_stream(torch.cuda.current_stream())
        with torch.cuda.stream(s):
            fn()
        torch.cuda.current_stream().wait_stream(s)
        torch.cuda.synchronize()
        g = torch.cuda.CUDAGraph()
        with torch.cuda.graph(g):
            fn()
        return timed([g.replay], a.iters, a.warmup) / nl * 1e3
    row = {"full_us_per_layer": round(graph_us(full), 1), "gemms_us_per_layer": round(graph_us(gemms), 1),
           "attention_us_per_layer": round(graph_us(attn), 1)}
    wbytes = sum(t.numel() * 2 for lw in model.layers[:1] for t in (lw.qkv, lw.o, lw.gate_up, lw.down))
    kvb = B * (L + 1) * model.hkv * c.hd * 2 * 2
    ms = row["full_us_per_layer"] / 1e3
    report(a, ms, wbytes + kvb, 2.0 * B * wbytes / 2, dict(row, model=a.model, batch=B, seqlen=L, weight_bytes_per_layer=wbytes, kv_bytes_per_layer=kvb))


def bench_gemm_chain_timeline(a: Args) -> None:
    """Phase stamps (globaltimer, microseconds since the first CTA's entry) of the four GEMMs of a
    decoder layer launched back to back in a CUDA graph: do consecutive kernels overlap, and where
    does each one spend its time?  Uses the library's GEMM timeline hook."""
    import ctypes
    from zml_b200.models.llama import PRESETS, LlamaConfig
    from zml_b200.ops import _lib
    lib = _lib.lib()
    lib.zb_gemm_set_timeline.argtypes = [ctypes.c_void_p, ctypes.c_int]
    c = LlamaConfig.from_hf(PRESETS[a.model])
    h, f, qkv_n = c.hidden_size, c.intermediate_size, (c.num_attention_heads + 2 * c.num_key_value_heads) * c.hd
    sets = [[torch.randn(n, k, device="cuda").bfloat16() * 0.02 for (n, k) in ((qkv_n, h), (h, c.num_attention_heads * c.hd), (2 * f, h), (h, f))]
            for _ in range(3)]
    x = torch.randn(a.batch, h, device="cuda").bfloat16()

    def chain(ws):
        xx = x
        qkv = ops.gemm(xx, ws[0], static_w=True)
        xx = ops.gemm(qkv[:, :c.num_attention_heads * c.hd], ws[1], residual=xx, static_w=True)
        gu = ops.gemm(xx, ws[2], static_w=True)
        return ops.gemm(gu[:, :f], ws[3], residual=xx, static_w=True)
    for ws in sets:
        chain(ws)
    torch.cuda.synchronize()
    slots, stride = 8, 160 * 12
    tl = torch.zeros(slots * stride, dtype=torch.int64, device="cuda")
    s = torch.cuda.Stream()
    s.wait_stream(torch.cuda.current_stream())
    with torch.cuda.stream(s):
        chain(sets[0])
    torch.cuda.current_stream().wait_stream(s)
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    lib.zb_gemm_set_timeline(tl.data_ptr(), slots)
    with torch.cuda.graph(g):
        chain(sets[1])
        chain(sets[2])
    lib.zb_gemm_set_timeline(None, 0)
    for _ in range(2):
        tl.zero_()
        torch.cuda.synchronize()
        g.replay()
        torch.cuda.synchronize()
    t = tl.view(slots, 160, 12).cpu()
    base = t[0, :, 0][t[0, :, 0] > 0].min()
    names = ["qkv", "o_proj", "gate_up", "down"] * 2
    rows = []
    for k in range(slots):
        r = t[k]
        live = r[:, 0] > 0
        rel = (r[live] - base).double() / 1000.0
        med = lambda i: round(float(rel[:, i][r[live][:, i] > 0].median()), 2)
        rows.append({"gemm": names[k], "ctas": int(live.sum()), "entry_min": round(float(rel[:, 0].min()), 2),
                     "entry_max": round(float(rel[:, 0].max()), 2), "dep_wait_done": med(2), "first_tile": med(3),
                     "last_commit": med(4), "epilogue_done": med(6), "exit_max": round(float(rel[:, 7].max()), 2)})
    print(json.dumps({"op": a.op, "model": a.model, "batch": a.batch, "unit": "us since first entry", "launches": rows}))


def bench_moe_w4_timeline(a: Args) -> None:
    """Phase stamps of CTA 0 of the NVFP4 grouped GEMM (gate|up of the --op=moe shapes): per load stage of 4 k-blocks
    the nanoseconds, from the first copy request, at which the producer requested the copies, a de-quantising warp
    saw them, it obtained an operand stage, the two groups finished their tensor-memory stores, the MMA thread had
    both operands, and it had issued its MMAs."""
    from zml_b200 import moe
    from zml_b200.moe import ops as mops
    from zml_b200.ops import _lib
    d, f, e, k = a.k, a.n, a.experts, a.topk
    g = torch.randn(e, f, d, device="cuda").bfloat16() * 0.02
    u = torch.randn(e, f, d, device="cuda").bfloat16() * 0.02
    qs = [moe.Nvfp4Experts.quantize(moe.interleave_gate_up(g, u)) for _ in range(2)]
    x = torch.randn(a.tokens, d, device="cuda").bfloat16()
    ids, _ = moe.router_topk(torch.randn(a.tokens, e, device="cuda"), k, True)
    meta, sorted_pair, _ = mops.moe_align(ids, 0, e)
    xs = mops.gather(x, sorted_pair, meta, e, k, a.tokens * k)
    avg = max(1, a.tokens * k // e)
    for i in range(3):
        mops.grouped_gemm_w4(xs, qs[i % 2], meta, swiglu=True, avg_tokens=avg)
    torch.cuda.synchronize()
    buf = torch.zeros(64 * 8, dtype=torch.int64, device="cuda")
    _lib.lib().zb_moe_w4_set_timeline(buf.data_ptr())
    mops.grouped_gemm_w4(xs, qs[1], meta, swiglu=True, avg_tokens=avg)
    torch.cuda.synchronize()
    _lib.lib().zb_moe_w4_set_timeline(None)
    t = buf.cpu().view(64, 8)
    t0 = int(t[0, 0])
    names = ["copies_requested", "copies_seen", "operand_stage_free", "stores_done_group0", "stores_done_group1", "mma_operands_ready",
             "mmas_issued"]
    stages = [{n: (int(v) - t0 if int(v) else None) for n, v in zip(names, t[q, :7])} for q in range(40) if int(t[q, 0])]
    print(json.dumps({"op": a.op, "tokens": a.tokens, "experts": e, "stages": stages}))


OPS = {"moe_w4_timeline": bench_moe_w4_timeline, "gemm_chain_timeline": bench_gemm_chain_timeline, "gemm": bench_gemm, "decode_attention": bench_decode_attention, "prefill_attention": bench_prefill_attention,
       "moe": bench_moe, "gated_delta_scan": bench_gated_delta_scan, "decode_layers": bench_decode_layers,
       "latent_prefill": bench_latent_prefill, "latent_decode": bench_latent_decode, "wkv_scan": bench_wkv_scan, "stream": bench_stream,
       "diff_prefill": bench_diff_prefill, "diff_decode": bench_diff_decode, "hyper": bench_hyper, "shared_mixture": bench_shared_mixture,
       "gqa_prefill": bench_gqa_prefill, "gqa_decode": bench_gqa_decode, "channel_delta": bench_channel_delta, "mixture": bench_mixture,
       "pool_prefill": bench_pool_prefill, "pool_decode": bench_pool_decode, "gated_scan": bench_gated_scan, "add_norm": bench_add_norm,
       "relu_mixture": bench_relu_mixture}


def main(argv=None) -> int:
    args = flags.parse(argv, Args)
    if args.op not in OPS:
        print(f"unknown --op={args.op}; one of {sorted(OPS)}", file=sys.stderr)
        return 2
    if not torch.cuda.is_available():
        print(json.dumps({"op": args.op, "skipped": "no CUDA device"}))
        return 0
    OPS[args.op](args)
    ops.raise_on_status()
    return 0


if __name__ == "__main__":
    sys.exit(main())
