"""Grouped-query attention with the options of `GqaSpec`: norms on queries and keys (per head or over a whole projection), partial
rotation, stretched positions, a score cap, a sliding window with kept first tokens, pooled blocks or chunks, a sink, an output
gate, differential heads, key and value sizes of their own
(libzb_cuda.so: gqa_attention.cu for any sizes in bf16 and fp32; attention.cu and attention_tc.cu, the paged kernels of the
other decoders, for bf16).

The cache of a layer is a pair of paged tensors (keys [pages, page, kv heads, k_row], values [pages, page, kv heads, v_row]).
In bf16 the rows are padded with zeros to a head size of the paged kernels (64, 128 or 256) where there is one.

With pooled blocks the cache is two tensors more, the blocks' mean keys and values [pages, rows, kv heads, *]: a page holds the
blocks whose last position lies in it.  They are made once, when their last position is written.

A differential head has two maps, attentions of their own over common values; its result is `DiffMix` of the two.  To the
kernels they are two query heads of twice the size: a cached key is [map 1 | map 2], and a map's query is zero in the other
half, so keys and values are read once for both.
CPU tensors take the plain torch branch of each function.
"""
from __future__ import annotations

import ctypes as C
import math
from dataclasses import dataclass
from typing import Optional

import torch

from . import _lib

_p, _i, _ll, _f = C.c_void_p, C.c_int, C.c_longlong, C.c_float
_lib.register_signature("zb_gqa_prep", _i, [_p, _ll, _p, _p, _p, _p, _p, _p, _p, _p, _ll, _f, _i, _i, _i, _i, _i, _i, _i, _i, _i, _i, _p, _i, _i, _f,
                                            _i, _i, _p, _p, _p, _i, _i, _i, _i, _p])
_lib.register_signature("zb_gqa_pool", _i, [_p, _p, _p, _p, _i, _i, _p, _i, _i, _i, _i, _i, _p, _p, _i, _i, _i, _p])
_lib.register_signature("zb_gqa_attend", _i, [_p, _i, _p, _i, _p, _i, _p, _ll, _p, _ll, _i, _p, _i, _i, _i, _i, _i, _i, _i, _i, _i, _f, _f, _i, _i, _i,
                                              _p, _p, _f, _p, _p, _i, _i, _i, _p])
_lib.register_signature("zb_pair_combine", _i, [_p, _p, _ll, _i, _i, _i, _f, _f, _f, _i, _p])

PAGED_HEAD_SIZES = (64, 128, 256)


class AttnExt(C.Structure):
    """`ZbAttnExt` of csrc/host_api.h."""
    _fields_ = [("keep", C.c_int), ("cap", C.c_float), ("sink", C.c_int), ("vdim", C.c_int), ("gate", C.c_void_p), ("ldg", C.c_longlong),
                ("chunk", C.c_int), ("out_f32", C.c_int), ("pair", C.c_int), ("pair_lambda", C.c_float), ("pair_scale", C.c_float),
                ("pair_eps", C.c_float), ("pool", C.c_int), ("pool_rows", C.c_int), ("pool_k", C.c_void_p), ("pool_v", C.c_void_p),
                ("ldo", C.c_longlong), ("scaled", C.c_int), ("out_scale", C.c_float)]


@dataclass(frozen=True)
class Yarn:
    """Stretched positions (YaRN): pairs that turn fewer than `slow` times over `original` positions turn slower by `factor`, those
    that turn more than `fast` times as before, in between a blend; cosines and sines are multiplied by 0.1 ln(factor) + 1."""
    factor: float
    original: float
    fast: float
    slow: float

    @property
    def amplitude(self) -> float:
        return 0.1 * math.log(self.factor) + 1.0

    def shares(self, rot: int, base: float) -> torch.Tensor:
        """How much of the slow-down each pair takes, 0 to 1."""
        at = lambda turns: rot * math.log(self.original / (2 * math.pi * turns)) / (2 * math.log(base))
        lo, hi = max(math.floor(at(self.fast)), 0), min(math.ceil(at(self.slow)), rot - 1)
        return ((torch.arange(rot // 2, dtype=torch.float64) - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)


@dataclass(frozen=True)
class DiffMix:
    """What a differential head makes of its maps' results a1 and a2: o = a1 - lam * a2, then o / sqrt(mean(o^2) + eps) * scale."""
    lam: float
    scale: float
    eps: float

    def apply(self, a, heads: int):
        """a fp32 [T, 2 heads, vdim] -> [T, heads * vdim] fp32."""
        a = a.reshape(a.shape[0], heads, 2, -1)
        o = a[:, :, 0] - self.lam * a[:, :, 1]
        return (o / torch.sqrt((o * o).mean(-1, keepdim=True) + self.eps) * self.scale).reshape(a.shape[0], -1)


@dataclass(frozen=True)
class GqaSpec:
    """Position i sees j <= i when i - j < window (0: any) or j < keep; with `chunk`, when floor(i / chunk) = floor(j / chunk).
    With `pool`, block b (the positions b pool .. b pool + pool - 1) is one more key and value, their means, for every i with
    b pool + pool - 1 <= i - window; all share one softmax.
    score = q . k * scale, capped to cap * tanh(score / cap) unless cap is 0; with a sink the softmax denominator has an
    additional exp(0).  The first `rot` dimensions of queries and keys are rotated in pairs (i, i + rot / 2) by
    position * base^(-2i / rot) / factor, or as `yarn` has it.  maps = 2: differential heads, `dim` per map.  whole_norm: one norm
    over all query heads and one over all key heads."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    rot: int
    base: float = 10000.0
    factor: float = 1.0
    scale: float = 1.0
    cap: float = 0.0
    window: int = 0
    keep: int = 0
    sink: bool = False
    chunk: int = 0
    maps: int = 1
    pool: int = 0
    whole_norm: bool = False
    yarn: Optional[Yarn] = None

    def __post_init__(self):
        if self.kv_heads < 1 or self.heads % self.kv_heads:
            raise ValueError(f"{self.heads} query heads do not share {self.kv_heads} key / value heads")
        if self.rot % 2 or self.rot > self.dim:
            raise ValueError(f"cannot rotate {self.rot} of {self.dim} dimensions")
        if self.cap < 0 or self.window < 0 or self.keep < 0:
            raise ValueError("cap, window and keep are 0 (off) or positive")
        if self.chunk < 0 or (self.chunk and (self.window or self.keep)):
            raise ValueError("chunks take the place of a window")
        if self.maps not in (1, 2):
            raise ValueError("a head has one map or two")
        if self.pool < 0 or (self.pool and (not self.window or self.keep or self.maps != 1)):
            raise ValueError("pooled blocks go with a window, without kept tokens and differential heads")
        if self.whole_norm and self.maps != 1:
            raise ValueError("a norm over the whole projection takes heads of one map")

    @property
    def rows_q(self) -> int:
        """Query rows: heads, each map counted."""
        return self.heads * self.maps

    def columns(self) -> int:
        """Columns of q | k | v as projections write them."""
        return self.rows_q * self.dim + self.kv_heads * (self.maps * self.dim + self.vdim)

    def inv_freq(self, device) -> torch.Tensor:
        i = torch.arange(0, self.rot, 2, dtype=torch.float64)
        f = self.base ** (-i / max(self.rot, 1)) / self.factor
        if self.yarn is not None and self.rot:
            share = self.yarn.shares(self.rot, self.base)
            f = f / self.yarn.factor * share + f * (1 - share)
        return f.to(torch.float32).to(device)

    @property
    def amplitude(self) -> float:
        """Factor on the cosines and sines."""
        return self.yarn.amplitude if self.yarn is not None else 1.0

    def paged_size(self, dtype) -> int:
        """Head size of the paged tensor-core kernels this attention runs on, 0: none takes it."""
        if dtype != torch.bfloat16 or self.rows_q // self.kv_heads > 16:
            return 0
        return next((n for n in PAGED_HEAD_SIZES if n >= max(self.maps * self.dim, self.vdim)), 0)

    def rows(self, dtype) -> tuple[int, int]:
        """Elements per head of the key and the value cache."""
        n = self.paged_size(dtype)
        return (n, n) if n else (self.maps * self.dim, self.vdim)

    def alloc_cache(self, num_pages: int, page_size: int, dtype, device):
        slots = [page_size] + ([pool_rows(self.pool, page_size)] if self.pool else [])
        return tuple(torch.zeros((num_pages, r, self.kv_heads, n), dtype=dtype, device=device) for r in slots for n in self.rows(dtype))

    def visible(self, length: int) -> int:
        """Most keys that one position of a sequence of `length` tokens looks at, as far as splitting them goes."""
        span = self.chunk or self.window
        if not span:
            return length
        pooled = (length // self.pool + 63) // 64 * 64 if self.pool and length > self.window else 0
        return min(length, (span + self.keep + 126) // 64 * 64 + pooled)


def pool_rows(pool: int, page_size: int) -> int:
    """Blocks of `pool` positions whose last position can lie in one page."""
    return (page_size + pool - 1) // pool


def pool_row(block, pool: int, page_size: int):
    """(page's place in the block table, row in the page) of a pooled block."""
    at = (block * pool + pool - 1) // page_size
    return at, block - at * page_size // pool


def _ptr(t):
    return None if t is None else t.data_ptr()


# ------------------------------------------------------------------ norms, rotation, cache write
def _rotate(v, pos, inv_freq, rot: int, amp: float = 1.0):
    if rot == 0:
        return v
    a = pos.float()[:, None, None] * inv_freq[None, None]
    u, w = v[..., :rot // 2] * amp, v[..., rot // 2:rot] * amp
    return torch.cat([u * a.cos() - w * a.sin(), w * a.cos() + u * a.sin(), v[..., rot:]], -1)


def _pad_maps(z, n: int, s: GqaSpec):
    """[T, rows, dim] -> [T, rows, n] zeros behind, or with two maps in the other map's half."""
    if s.maps == 1:
        return torch.nn.functional.pad(z, (0, n - z.shape[-1]))
    t, rows, _ = z.shape
    z = torch.nn.functional.pad(z, (0, n // 2 - z.shape[-1])).reshape(t, rows // 2, 2, n // 2)
    out = torch.zeros((t, rows // 2, 2, 2, n // 2), dtype=z.dtype)
    for i in range(2):
        out[:, :, i, i] = z[:, :, i]
    return out.reshape(t, rows, n)


def _pool_cached(cache, spec: GqaSpec, block_table, q_start, seq_lens):
    """The blocks whose last position is new, from the cached rows."""
    kc, vc, pk, pv = cache
    page, P = kc.shape[1], spec.pool
    qs, sl = q_start.tolist(), seq_lens.tolist()
    for s, n in enumerate(sl):
        for b in range((n - (qs[s + 1] - qs[s])) // P, n // P):
            j = torch.arange(b * P, (b + 1) * P)
            rows = block_table[s, j // page].long() * page + j % page
            at, row = pool_row(b, P, page)
            for src, dst in ((kc, pk), (vc, pv)):
                dst[int(block_table[s, at]), row] = src.reshape(-1, *src.shape[2:])[rows].float().mean(0).to(dst.dtype)


def pool_new(cache, meta, spec: GqaSpec):
    """Pools the blocks that a varlen batch, whose keys and values are in the cache, has completed."""
    if not spec.pool:
        return
    kc, vc, pk, pv = cache
    if not kc.is_cuda:
        return _pool_cached(cache, spec, meta.block_table, meta.q_start, meta.seq_lens)
    nb = meta.positions.shape[0] // spec.pool + meta.seq_lens.shape[0]
    _lib.check(_lib.lib().zb_gqa_pool(
        _ptr(kc), _ptr(vc), _ptr(pk), _ptr(pv), spec.pool, pk.shape[1], _ptr(meta.block_table), meta.block_table.shape[1], kc.shape[1], spec.kv_heads,
        kc.shape[-1], vc.shape[-1], _ptr(meta.q_start), _ptr(meta.seq_lens), meta.seq_lens.shape[0], nb, int(kc.dtype == torch.float32),
        _lib.stream_ptr()), "zb_gqa_pool")


def sums_of_squares(proj, spec: GqaSpec):
    """fp32 [T, 2]: of the query and the key columns of proj, for `prep` to take once they are summed over the ranks."""
    nq, nk = spec.heads * spec.dim, spec.kv_heads * spec.dim
    x = proj[:, :nq + nk].float().square()
    return torch.stack([x[:, :nq].sum(1), x[:, nq:].sum(1)], 1)


def prep(proj, q_norm, k_norm, inv_freq, positions, slots, cache, eps: float, spec: GqaSpec, queries_only: bool = False, sumsq=None,
         totals: Optional[tuple] = None, step_table=None):
    """proj [T, >= `spec.columns()`] = q | k | v heads (maps of a head one after the other) -> normed (with norm weights fp32
    [dim], or [heads dim] and [kv_heads dim] with whole_norm; else not) and rotated queries [T, rows_q, k_row]; keys and values go
    to the cache rows `slots` (negative: none).
    `queries_only`: proj holds no keys and values and the cache, another layer's, is left alone.
    `sumsq` fp32 [T, 2] and `totals` (with whole_norm): `sums_of_squares` over all ranks and the elements behind them.
    `step_table`: the block table of a decode step, one token per sequence; pooled blocks that a token completes are made, too
    (a varlen batch calls `pool_new` instead)."""
    t, s = proj.shape[0], spec
    kc, vc = cache[:2]
    totals = totals or (s.heads * s.dim, s.kv_heads * s.dim)
    if s.whole_norm and sumsq is not None:
        sumsq = sumsq.contiguous()
    if not proj.is_cuda:
        x = proj.float()
        nq, nk = s.rows_q * s.dim, s.kv_heads * s.maps * s.dim
        rms = lambda v, w: v if w is None else v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps) * w
        xq, xk = x[:, :nq], x[:, nq:nq + nk]
        if s.whole_norm:
            ss = sums_of_squares(proj, s) if sumsq is None else sumsq
            xq, xk = (v / torch.sqrt(ss[:, i:i + 1] / totals[i] + eps) * w for i, (v, w) in enumerate(((xq, q_norm), (xk, k_norm))))
            rms = lambda v, w: v
        q = _pad_maps(_rotate(rms(xq.reshape(t, s.rows_q, s.dim), q_norm), positions, inv_freq, s.rot, s.amplitude), kc.shape[-1], s).to(proj.dtype)
        if queries_only:
            return q
        k = _rotate(rms(xk.reshape(t, s.kv_heads * s.maps, s.dim), k_norm), positions, inv_freq, s.rot, s.amplitude)
        v = x[:, nq + nk:nq + nk + s.kv_heads * s.vdim].reshape(t, s.kv_heads, s.vdim)
        ok = slots >= 0
        rows = slots[ok].long()
        pad = lambda z, n: torch.nn.functional.pad(z, (0, n - z.shape[-1])).to(proj.dtype)
        kc.view(-1, s.kv_heads, kc.shape[-1])[rows] = pad(k, kc.shape[-1] // s.maps)[ok].reshape(-1, s.kv_heads, kc.shape[-1])
        vc.view(-1, s.kv_heads, vc.shape[-1])[rows] = pad(v, vc.shape[-1])[ok]
        if s.pool and step_table is not None:
            n = positions + 1
            live = torch.cat([torch.zeros(1, dtype=torch.int64), ok.long().cumsum(0)])        # rows without a slot complete nothing
            _pool_cached(cache, s, step_table, live, n)
        return q
    assert proj.stride(1) == 1 and proj.dtype == kc.dtype == vc.dtype and kc.is_contiguous() and vc.is_contiguous()
    q = torch.empty((t, s.rows_q, kc.shape[-1]), dtype=proj.dtype, device=proj.device)
    pool = (0, 0, None, None, None, 0, 0)
    if s.pool and step_table is not None:
        pool = (s.pool, cache[2].shape[1], _ptr(cache[2]), _ptr(cache[3]), _ptr(step_table), step_table.shape[1], kc.shape[1])
    _lib.check(_lib.lib().zb_gqa_prep(
        _ptr(proj), proj.stride(0), _ptr(q_norm), _ptr(k_norm), _ptr(inv_freq), _ptr(positions), _ptr(slots), _ptr(q), _ptr(kc), _ptr(vc),
        kc.shape[0] * kc.shape[1], float(eps), s.rows_q, 0 if queries_only else s.kv_heads, s.dim, s.vdim, s.rot, s.maps, q.shape[-1],
        kc.shape[-1], vc.shape[-1], int(s.whole_norm), _ptr(sumsq), *totals, float(s.amplitude), *pool, int(proj.dtype == torch.float32), t,
        _lib.stream_ptr()), "zb_gqa_prep")
    return q


# ------------------------------------------------------------------ attention
def attention_reference(q, gate, cache, block_table, seq_lens, q_start, spec: GqaSpec, mix=None):
    s, (kc, vc) = spec, cache[:2]
    out = torch.zeros((q.shape[0], s.rows_q, s.vdim))
    page = kc.shape[1]
    rep = s.rows_q // s.kv_heads
    dk = s.dim if s.maps == 1 else kc.shape[-1]
    qs, sl = q_start.tolist(), seq_lens.tolist()
    for b in range(len(sl)):
        a, e, n = qs[b], qs[b + 1], sl[b]
        if e <= a or n <= 0:
            continue
        j = torch.arange(n)
        rows = block_table[b, j // page].long() * page + j % page
        k = kc.view(-1, s.kv_heads, kc.shape[-1])[rows][..., :dk].float().repeat_interleave(rep, 1)
        v = vc.view(-1, s.kv_heads, vc.shape[-1])[rows][..., :s.vdim].float().repeat_interleave(rep, 1)
        i = torch.arange(n - (e - a), n)[:, None]
        seen = j[None] <= i
        if s.window:
            seen &= (i - j[None] < s.window) | (j[None] < s.keep)
        if s.chunk:
            seen &= i // s.chunk == j[None] // s.chunk
        if s.pool:
            blocks = torch.arange(max(0, n - s.window) // s.pool)
            at, row = pool_row(blocks, s.pool, page)
            pages = block_table[b, at].long()
            k = torch.cat([k, cache[2][pages, row][..., :dk].float().repeat_interleave(rep, 1)], 0)
            v = torch.cat([v, cache[3][pages, row][..., :s.vdim].float().repeat_interleave(rep, 1)], 0)
            seen = torch.cat([seen, blocks[None] * s.pool + s.pool - 1 <= i - s.window], 1)
        z = torch.einsum("qhd,khd->hqk", q[a:e, :, :dk].float(), k) * s.scale
        if s.cap:
            z = s.cap * torch.tanh(z / s.cap)
        z = z.masked_fill(~seen[None], float("-inf"))
        if s.sink:
            z = torch.cat([z, torch.zeros_like(z[..., :1])], -1)
        p = torch.softmax(z, -1)[..., :k.shape[0]]
        out[a:e] = torch.einsum("hqk,khd->qhd", p, v)
    out = out.reshape(q.shape[0], -1) if mix is None else mix.apply(out, s.heads)
    if gate is not None:
        out = out * torch.sigmoid(gate.float())
    return out.to(q.dtype)


def _combine(a, s: GqaSpec, mix: DiffMix, dtype):
    out = torch.empty((a.shape[0], s.heads * s.vdim), dtype=dtype, device=a.device)
    _lib.check(_lib.lib().zb_pair_combine(_ptr(a), _ptr(out), out.stride(0), a.shape[0], s.heads, s.vdim, mix.lam, mix.scale, mix.eps,
                                          int(dtype == torch.float32), _lib.stream_ptr()), "zb_pair_combine")
    return out


def attention(q, gate, cache, meta, spec: GqaSpec, mix: Optional[DiffMix] = None, out=None, out_scale: float = 1.0):
    """Attention of the prepared queries over the cache (which holds the new tokens' keys and values already), times
    sigmoid(gate) where there is one and `out_scale`: [T, heads vdim], or into the columns `out` of a wider buffer.  `meta`: the
    engine's AttnMeta of the step.  Differential heads take `mix` and no gate, scale or `out`."""
    s, (kc, vc) = spec, cache[:2]
    t = q.shape[0]
    if (mix is None) != (s.maps == 1) or (mix is not None and gate is not None):
        raise ValueError("differential heads come with a mix of their maps and without a gate")
    if mix is not None and (out is not None or out_scale != 1.0):
        raise ValueError("differential heads have an output and a scale of their own")
    pk, pv = cache[2:] if s.pool else (None, None)
    pool_args = (s.pool, pk.shape[1] if s.pool else 0, _ptr(pk), _ptr(pv))
    assert out is None or (out.shape == (t, s.heads * s.vdim) and out.stride(1) == 1 and out.dtype == q.dtype)
    q_start = meta.q_start
    if q_start is None:
        q_start = torch.arange(t + 1, dtype=torch.int32, device=q.device)
    if not q.is_cuda:
        a = attention_reference(q, gate, cache, meta.block_table, meta.seq_lens, q_start, s, mix)
        a = a if out_scale == 1.0 else (a.float() * out_scale).to(a.dtype)
        return a if out is None else out.copy_(a)
    n = s.paged_size(q.dtype)
    if n:
        from . import paged_decode, paged_prefill, prefill_on_tc
        ext = AttnExt(s.keep, s.cap, int(s.sink), s.vdim, _ptr(gate), gate.stride(0) if gate is not None else 0, s.chunk)
        if mix is not None:
            ext.pair, ext.pair_lambda, ext.pair_scale, ext.pair_eps = 1, mix.lam, mix.scale, mix.eps
            if meta.is_prefill and not prefill_on_tc(q, kc, ext):                # the maps' results first, then their mix
                ext.pair, ext.out_f32 = 0, 1
                a = torch.empty((t, s.rows_q, s.vdim), dtype=torch.float32, device=q.device)
                paged_prefill(q, kc, vc, meta.block_table, meta.seq_lens, q_start, s.scale, s.window, out=a,
                              total_q_blocks=meta.total_q_blocks, impl="mma", ext=ext)
                return _combine(a, s, mix, q.dtype)
        else:
            ext.pool, ext.pool_rows, ext.pool_k, ext.pool_v = pool_args
            ext.scaled, ext.out_scale = int(out_scale != 1.0), out_scale
        if out is None:
            out = torch.empty((t, s.heads * s.vdim), dtype=q.dtype, device=q.device)
        elif out.stride(0) != s.heads * s.vdim:
            ext.ldo = out.stride(0)
        if meta.is_prefill:
            paged_prefill(q, kc, vc, meta.block_table, meta.seq_lens, q_start, s.scale, s.window, out=out,
                          total_q_blocks=meta.total_q_blocks, ext=ext)
        else:
            paged_decode(q, kc, vc, meta.block_table, meta.seq_lens, s.scale, s.window, num_splits=meta.num_splits,
                         max_seq_len=meta.max_seq_len, out=out, ext=ext)
        return out
    assert q.is_contiguous() and (gate is None or (gate.stride(1) == 1 and gate.dtype == q.dtype))
    if out is None:
        out = torch.empty((t, s.rows_q * s.vdim), dtype=torch.float32 if mix is not None else q.dtype, device=q.device)
    _lib.check(_lib.lib().zb_gqa_attend(
        _ptr(q), q.shape[-1], _ptr(kc), kc.shape[-1], _ptr(vc), vc.shape[-1], _ptr(gate), gate.stride(0) if gate is not None else 0, _ptr(out),
        out.stride(0), int(out.dtype == torch.float32), _ptr(meta.block_table), meta.block_table.shape[1], kc.shape[1], s.rows_q, s.kv_heads,
        s.maps * s.dim, s.vdim, s.window, s.keep, s.chunk, float(s.scale), float(s.cap), int(s.sink), *pool_args, float(out_scale), _ptr(q_start),
        _ptr(meta.seq_lens), meta.seq_lens.shape[0], t, int(q.dtype == torch.float32), _lib.stream_ptr()), "zb_gqa_attend")
    return out if mix is None else _combine(out, s, mix, q.dtype)
