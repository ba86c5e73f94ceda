"""Grouped-query attention with the options of `GqaSpec`: norms on queries and keys, partial rotation, a score cap, a sliding
window with kept first tokens or chunks, a sink, an output gate, differential heads, key and value sizes of their own
(libzb_cuda.so: gqa_attention.cu for any sizes in bf16 and fp32; attention.cu and attention_tc.cu, the paged kernels of the
other decoders, for bf16).

The cache of a layer is a pair of paged tensors (keys [pages, page, kv heads, k_row], values [pages, page, kv heads, v_row]).
In bf16 the rows are padded with zeros to a head size of the paged kernels (64, 128 or 256) where there is one.

A differential head has two maps, attentions of their own over common values; its result is `DiffMix` of the two.  To the
kernels they are two query heads of twice the size: a cached key is [map 1 | map 2], and a map's query is zero in the other
half, so keys and values are read once for both.
CPU tensors take the plain torch branch of each function.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import Optional

import torch

from . import _lib

_p, _i, _ll, _f = C.c_void_p, C.c_int, C.c_longlong, C.c_float
_lib.register_signature("zb_gqa_prep", _i, [_p, _ll, _p, _p, _p, _p, _p, _p, _p, _p, _ll, _f, _i, _i, _i, _i, _i, _i, _i, _i, _i, _i, _i, _p])
_lib.register_signature("zb_gqa_attend", _i, [_p, _i, _p, _i, _p, _i, _p, _ll, _p, _ll, _i, _p, _i, _i, _i, _i, _i, _i, _i, _i, _i, _f, _f, _i, _p, _p,
                                              _i, _i, _i, _p])
_lib.register_signature("zb_pair_combine", _i, [_p, _p, _ll, _i, _i, _i, _f, _f, _f, _i, _p])

PAGED_HEAD_SIZES = (64, 128, 256)


class AttnExt(C.Structure):
    """`ZbAttnExt` of csrc/host_api.h."""
    _fields_ = [("keep", C.c_int), ("cap", C.c_float), ("sink", C.c_int), ("vdim", C.c_int), ("gate", C.c_void_p), ("ldg", C.c_longlong),
                ("chunk", C.c_int), ("out_f32", C.c_int), ("pair", C.c_int), ("pair_lambda", C.c_float), ("pair_scale", C.c_float),
                ("pair_eps", C.c_float)]


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
    score = q . k * scale, capped to cap * tanh(score / cap) unless cap is 0; with a sink the softmax denominator has an
    additional exp(0).  The first `rot` dimensions of queries and keys are rotated in pairs (i, i + rot / 2) by
    position * base^(-2i / rot) / factor.  maps = 2: differential heads, `dim` per map."""
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

    @property
    def rows_q(self) -> int:
        """Query rows: heads, each map counted."""
        return self.heads * self.maps

    def columns(self) -> int:
        """Columns of q | k | v as projections write them."""
        return self.rows_q * self.dim + self.kv_heads * (self.maps * self.dim + self.vdim)

    def inv_freq(self, device) -> torch.Tensor:
        i = torch.arange(0, self.rot, 2, dtype=torch.float64)
        return (self.base ** (-i / max(self.rot, 1)) / self.factor).to(torch.float32).to(device)

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
        return tuple(torch.zeros((num_pages, page_size, self.kv_heads, n), dtype=dtype, device=device) for n in self.rows(dtype))

    def visible(self, length: int) -> int:
        """Most keys that one position of a sequence of `length` tokens looks at, as far as splitting them goes."""
        span = self.chunk or self.window
        return min(length, (span + self.keep + 126) // 64 * 64) if span else length


def _ptr(t):
    return None if t is None else t.data_ptr()


# ------------------------------------------------------------------ norms, rotation, cache write
def _rotate(v, pos, inv_freq, rot: int):
    if rot == 0:
        return v
    a = pos.float()[:, None, None] * inv_freq[None, None]
    u, w = v[..., :rot // 2], v[..., rot // 2:rot]
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


def prep(proj, q_norm, k_norm, inv_freq, positions, slots, cache, eps: float, spec: GqaSpec, queries_only: bool = False):
    """proj [T, >= `spec.columns()`] = q | k | v heads (maps of a head one after the other) -> normed (with norm weights fp32
    [dim], else not) and rotated queries [T, rows_q, k_row]; keys and values go to the cache rows `slots` (negative: none).
    `queries_only`: proj holds no keys and values and the cache, another layer's, is left alone."""
    t, s = proj.shape[0], spec
    kc, vc = cache
    if not proj.is_cuda:
        x = proj.float()
        nq, nk = s.rows_q * s.dim, s.kv_heads * s.maps * s.dim
        rms = lambda v, w: v if w is None else v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps) * w
        q = _pad_maps(_rotate(rms(x[:, :nq].reshape(t, s.rows_q, s.dim), q_norm), positions, inv_freq, s.rot), kc.shape[-1], s).to(proj.dtype)
        if queries_only:
            return q
        k = _rotate(rms(x[:, nq:nq + nk].reshape(t, s.kv_heads * s.maps, s.dim), k_norm), positions, inv_freq, s.rot)
        v = x[:, nq + nk:nq + nk + s.kv_heads * s.vdim].reshape(t, s.kv_heads, s.vdim)
        ok = slots >= 0
        rows = slots[ok].long()
        pad = lambda z, n: torch.nn.functional.pad(z, (0, n - z.shape[-1])).to(proj.dtype)
        kc.view(-1, s.kv_heads, kc.shape[-1])[rows] = pad(k, kc.shape[-1] // s.maps)[ok].reshape(-1, s.kv_heads, kc.shape[-1])
        vc.view(-1, s.kv_heads, vc.shape[-1])[rows] = pad(v, vc.shape[-1])[ok]
        return q
    assert proj.stride(1) == 1 and proj.dtype == kc.dtype == vc.dtype and kc.is_contiguous() and vc.is_contiguous()
    q = torch.empty((t, s.rows_q, kc.shape[-1]), dtype=proj.dtype, device=proj.device)
    _lib.check(_lib.lib().zb_gqa_prep(
        _ptr(proj), proj.stride(0), _ptr(q_norm), _ptr(k_norm), _ptr(inv_freq), _ptr(positions), _ptr(slots), _ptr(q), _ptr(kc), _ptr(vc),
        kc.shape[0] * kc.shape[1], float(eps), s.rows_q, 0 if queries_only else s.kv_heads, s.dim, s.vdim, s.rot, s.maps, q.shape[-1],
        kc.shape[-1], vc.shape[-1], int(proj.dtype == torch.float32), t, _lib.stream_ptr()), "zb_gqa_prep")
    return q


# ------------------------------------------------------------------ attention
def attention_reference(q, gate, cache, block_table, seq_lens, q_start, spec: GqaSpec, mix=None):
    s, (kc, vc) = spec, cache
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
        z = torch.einsum("qhd,khd->hqk", q[a:e, :, :dk].float(), k) * s.scale
        if s.cap:
            z = s.cap * torch.tanh(z / s.cap)
        z = z.masked_fill(~seen[None], float("-inf"))
        if s.sink:
            z = torch.cat([z, torch.zeros_like(z[..., :1])], -1)
        p = torch.softmax(z, -1)[..., :n]
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


def attention(q, gate, cache, meta, spec: GqaSpec, mix: Optional[DiffMix] = None):
    """Attention of the prepared queries over the cache (which holds the new tokens' keys and values already), times
    sigmoid(gate) where there is one: [T, heads vdim].  `meta`: the engine's AttnMeta of the step.  Differential heads take
    `mix` and no gate."""
    s, (kc, vc) = spec, cache
    t = q.shape[0]
    if (mix is None) != (s.maps == 1) or (mix is not None and gate is not None):
        raise ValueError("differential heads come with a mix of their maps and without a gate")
    q_start = meta.q_start
    if q_start is None:
        q_start = torch.arange(t + 1, dtype=torch.int32, device=q.device)
    if not q.is_cuda:
        return attention_reference(q, gate, cache, meta.block_table, meta.seq_lens, q_start, s, mix)
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
        out = torch.empty((t, s.heads, s.vdim), dtype=q.dtype, device=q.device)
        if meta.is_prefill:
            paged_prefill(q, kc, vc, meta.block_table, meta.seq_lens, q_start, s.scale, s.window, out=out,
                          total_q_blocks=meta.total_q_blocks, ext=ext)
        else:
            paged_decode(q, kc, vc, meta.block_table, meta.seq_lens, s.scale, s.window, num_splits=meta.num_splits,
                         max_seq_len=meta.max_seq_len, out=out, ext=ext)
        return out.reshape(t, s.heads * s.vdim)
    assert q.is_contiguous() and (gate is None or (gate.stride(1) == 1 and gate.dtype == q.dtype))
    out = torch.empty((t, s.rows_q * s.vdim), dtype=torch.float32 if mix is not None else q.dtype, device=q.device)
    _lib.check(_lib.lib().zb_gqa_attend(
        _ptr(q), q.shape[-1], _ptr(kc), kc.shape[-1], _ptr(vc), vc.shape[-1], _ptr(gate), gate.stride(0) if gate is not None else 0, _ptr(out),
        out.stride(0), int(out.dtype == torch.float32), _ptr(meta.block_table), meta.block_table.shape[1], kc.shape[1], s.rows_q, s.kv_heads,
        s.maps * s.dim, s.vdim, s.window, s.keep, s.chunk, float(s.scale), float(s.cap), int(s.sink), _ptr(q_start), _ptr(meta.seq_lens),
        meta.seq_lens.shape[0], t, int(q.dtype == torch.float32), _lib.stream_ptr()), "zb_gqa_attend")
    return out if mix is None else _combine(out, s, mix, q.dtype)
