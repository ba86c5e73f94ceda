"""Latent attention: keys and values are per-head projections of one low-rank latent per token.  The cache holds that
latent and a single rotary key vector, common to the heads (libzb_cuda.so: latent_attention.cu).

Two formulations of the same attention, chosen by `latent_attention`:

* in the latent space: the queries are taken through the key projection (`absorb_q`), attend to the cached latents as
  one key/value head, and the result goes through the value projection (`absorb_out`).  Reads each cached row once for
  all heads: decode.
* expanded (`prefill`): the visible latents of the batch are gathered from the pages and projected to keys and
  values of every head, which costs a third of the products in the latent space when a chunk has many queries per key.

The output gate and the sink (one learned number per head, a term exp(sink) of the softmax denominator) are optional, and so
is the low-rank latent of the queries.  Rotated parts are turned in neighbouring pairs (2i, 2i + 1); `halves_to_pairs` gives
the order of rows that brings projections of a design with pairs (i, i + rot / 2) into that layout.

bf16 runs on the tensor cores, fp32 on the FMA pipes; CPU tensors take the plain torch branch.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import Optional

import torch

from . import _lib

_p, _i, _ll, _f = C.c_void_p, C.c_int, C.c_longlong, C.c_float
_lib.register_signature("zb_latent_prep", _i, [_p, _ll, _p, _p, _p, _p, _p, _p, _ll, _p, _ll, _ll, _f, _i, _i, _i, _i, _i, _i, _p])
_lib.register_signature("zb_latent_absorb", _i, [_p, _ll, _ll, _p, _ll, _p, _ll, _ll, _p, _ll, _p, _p, _i, _i, _i, _i, _i, _i, _i, _i, _p])
_lib.register_signature("zb_latent_attend", _i, [_p, _p, _ll, _p, _ll, _p, _i, _i, _i, _i, _i, _i, _i, _f, _p, _p, _p, _i, _i, _i, _p])
_lib.register_signature("zb_latent_gather", _i, [_p, _ll, _p, _i, _i, _p, _p, _i, _p, _ll, _i, _i, _i, _i, _i, _p])
_lib.register_signature("zb_latent_q_pack", _i, [_p, _ll, _p, _p, _p, _i, _i, _i, _i, _i, _i, _p])
_lib.register_signature("zb_latent_prefill_tc_supported", _i, [_i, _i, _i, _i])
_lib.register_signature("zb_latent_prefill_tc", _i, [_p, _p, _ll, _p, _ll, _i, _p, _ll, _p, _ll, _p, _p, _i, _p, _p, _i, _i, _i, _i, _i, _i,
                                                     _i, _i, _f, _p, _p])
_lib.register_signature("zb_latent_decode_supported", _i, [_i, _i])
_lib.register_signature("zb_latent_decode_groups", _i, [_i])
_lib.register_signature("zb_latent_decode", _i, [_p, _p, _i, _p, _ll, _p, _i, _i, _p, _i, _i, _i, _i, _f, _p, _i, _p])


def _ptr(t: Optional[torch.Tensor]):
    return None if t is None else t.data_ptr()


def _ld(t: Optional[torch.Tensor]) -> int:
    return 0 if t is None else t.stride(0)


def _up(n: int, m: int) -> int:
    return (n + m - 1) // m * m


@dataclass(frozen=True)
class LatentDims:
    """Sizes and constants of one latent-attention layer (heads: this rank's)."""
    heads: int
    dim: int            # unrotated query / key dimensions per head
    rot: int            # rotated ones (keys: one such part for every head)
    vdim: int
    rank: int           # latent size
    q_rank: int         # of the queries' latent, 0: none
    window: int         # keys a position sees, itself included; <= 0: all
    scale: float
    base: float         # of the rotation frequencies

    @property
    def rot_off(self) -> int:
        return _up(self.rank, 16)

    @property
    def row(self) -> int:
        """Elements of a cache row: latent and rotated part, each padded to 16."""
        return self.rot_off + _up(self.rot, 16)

    def inv_freq(self, device) -> torch.Tensor:
        i = torch.arange(0, self.rot, 2, dtype=torch.float64)
        return (float(self.base) ** (-i / self.rot)).to(torch.float32).to(device)


def halves_to_pairs(rot: int) -> torch.Tensor:
    """Row order that turns a rotated part with pairs (i, i + rot / 2) into one with pairs (2i, 2i + 1)."""
    return torch.arange(rot).reshape(2, rot // 2).t().reshape(-1)


def rotate_reference(x, positions, inv_freq):
    """Adjacent pairs of x [..., T, rot] (T second from the right or with heads between) turned by position * frequency."""
    a = positions.float()[:, None] * inv_freq[None]
    shape = (x.shape[0],) + (1,) * (x.dim() - 2) + (inv_freq.shape[0],)
    cs, sn = torch.cos(a).reshape(shape), torch.sin(a).reshape(shape)
    u, v = x[..., 0::2].float(), x[..., 1::2].float()
    return torch.stack([u * cs - v * sn, v * cs + u * sn], -1).reshape(x.shape)


def _rms(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


# ---------------------------------------------------------------------------- norms, rotation, cache write
def prep(proj, q_norm, c_norm, inv_freq, positions, slots, cache, eps: float, d: LatentDims):
    """proj [T, >= q_rank + rank + rot] (query latent | latent | shared key part): returns the normed query latent
    [T, q_rank] (None without one) and writes the normed latent and the rotated key part into cache [pages, page, row] at
    `slots`."""
    t = proj.shape[0]
    if not proj.is_cuda:
        cq = _rms(proj[:, :d.q_rank].float(), q_norm, eps).to(proj.dtype) if d.q_rank else None
        c = _rms(proj[:, d.q_rank:d.q_rank + d.rank].float(), c_norm, eps)
        kr = rotate_reference(proj[:, d.q_rank + d.rank:d.q_rank + d.rank + d.rot], positions, inv_freq)
        flat = cache.view(-1, cache.shape[-1])
        ok = slots >= 0
        idx = slots[ok].long()
        flat[idx, :d.rank] = c[ok].to(cache.dtype)
        flat[idx, d.rot_off:d.rot_off + d.rot] = kr[ok].to(cache.dtype)
        return cq
    assert proj.stride(1) == 1 and cache.is_contiguous() and cache.dtype == proj.dtype and cache.shape[-1] == d.row
    cq = torch.empty((t, d.q_rank), dtype=proj.dtype, device=proj.device) if d.q_rank else None
    _lib.check(_lib.lib().zb_latent_prep(
        _ptr(proj), proj.stride(0), _ptr(q_norm), _ptr(c_norm), _ptr(inv_freq), _ptr(positions), _ptr(slots), _ptr(cq), d.q_rank,
        _ptr(cache), d.row, cache.shape[0] * cache.shape[1], float(eps), d.q_rank, d.rank, d.rot, d.rot_off,
        int(proj.dtype == torch.float32), t, _lib.stream_ptr()), "zb_latent_prep")
    return cq


# ---------------------------------------------------------------------------- latent space
def absorb_q(q, w_uk_t, inv_freq, positions, d: LatentDims):
    """q [T, H * (dim + rot)] -> [T, H, row]: the unrotated part through w_uk_t [H, rank, dim], the rotated part rotated."""
    t, hd = q.shape[0], d.dim + d.rot
    new = torch.empty if d.rot_off == d.rank and d.row == d.rot_off + d.rot else torch.zeros
    out = new((t, d.heads, d.row), dtype=q.dtype, device=q.device)
    if not q.is_cuda:
        qh = q.reshape(t, d.heads, hd)
        out[..., :d.rank] = torch.einsum("thk,hnk->thn", qh[..., :d.dim].float(), w_uk_t.float()).to(q.dtype)
        out[..., d.rot_off:d.rot_off + d.rot] = rotate_reference(qh[..., d.dim:], positions, inv_freq).to(q.dtype)
        return out
    assert q.stride(1) == 1 and w_uk_t.is_contiguous()
    _lib.check(_lib.lib().zb_latent_absorb(
        _ptr(q), q.stride(0), hd, _ptr(w_uk_t), d.dim, _ptr(out), out.stride(0), d.row, None, 0, _ptr(inv_freq), _ptr(positions), d.rot,
        d.dim, d.rot_off, t, d.heads, d.rank, d.dim, int(q.dtype == torch.float32), _lib.stream_ptr()), "zb_latent_absorb")
    return out


def absorb_out(o, w_uv, gate, d: LatentDims):
    """o [T, H, rot_off] (latent-space results) -> sigmoid(gate) * (o w_uv^T) [T, H * vdim]; w_uv [H, vdim, rank],
    gate [T, H * vdim] (row stride free) or None."""
    t = o.shape[0]
    if not o.is_cuda:
        y = torch.einsum("thk,hnk->thn", o[..., :d.rank].float(), w_uv.float()).reshape(t, -1)
        return (y if gate is None else y * torch.sigmoid(gate.float())).to(o.dtype)
    out = torch.empty((t, d.heads * d.vdim), dtype=o.dtype, device=o.device)
    assert w_uv.is_contiguous() and (gate is None or (gate.stride(1) == 1 and gate.dtype == o.dtype))
    _lib.check(_lib.lib().zb_latent_absorb(
        _ptr(o), o.stride(0), o.stride(1), _ptr(w_uv), d.rank, _ptr(out), out.stride(0), d.vdim, _ptr(gate), _ld(gate), None, None, 0,
        0, 0, t, d.heads, d.vdim, d.rank, int(o.dtype == torch.float32), _lib.stream_ptr()), "zb_latent_absorb")
    return out


def attend_reference(q, cache, block_table, q_start, seq_lens, d: LatentDims, sink=None):
    out = torch.zeros((q.shape[0], d.heads, d.rot_off), dtype=q.dtype, device=q.device)
    flat = cache.view(-1, cache.shape[-1])
    page = cache.shape[1]
    qs, sl = q_start.tolist(), seq_lens.tolist()
    for s in range(len(sl)):
        a, b, n = qs[s], qs[s + 1], sl[s]
        if b <= a or n <= 0:
            continue
        key = torch.arange(n)
        rows = flat[block_table[s].long()[key // page] * page + key % page].float()
        pos = torch.arange(n - (b - a), n)
        vis = key[None] <= pos[:, None]
        if d.window > 0:
            vis &= key[None] > pos[:, None] - d.window
        sc = torch.einsum("thc,kc->htk", q[a:b].float(), rows) * d.scale
        sc = sc.masked_fill(~vis[None], float("-inf"))
        if sink is not None:
            sc = torch.cat([sc, sink.float()[:, None, None].expand(-1, sc.shape[1], 1)], -1)
        pr = torch.softmax(sc, -1)[..., :n]
        out[a:b, :, :d.rank] = torch.einsum("htk,kc->thc", pr, rows[:, :d.rank]).to(q.dtype)
    return out


def attend(q, cache, block_table, q_start, seq_lens, d: LatentDims, decode: bool = False, num_splits: int = 1, sink=None):
    """Windowed causal attention of q [T, H, row] (`absorb_q`) against the cached rows; a sequence's queries are its last
    tokens; sink fp32 [H] or None.  Returns [T, H, rot_off]."""
    if not q.is_cuda:
        return attend_reference(q, cache, block_table, q_start, seq_lens, d, sink)
    t = q.shape[0]
    out = torch.empty((t, d.heads, d.rot_off), dtype=q.dtype, device=q.device)
    assert block_table.is_contiguous() and cache.dtype == q.dtype and q.is_contiguous()
    l = _lib.lib()
    if decode and q.dtype == torch.bfloat16 and l.zb_latent_decode_supported(d.row, d.rot_off):
        _lib.check(l.zb_latent_decode(
            _ptr(q), _ptr(cache), d.row, _ptr(out), d.rot_off, _ptr(block_table), block_table.shape[1], cache.shape[1], _ptr(seq_lens), t,
            d.heads, d.rot_off, d.window, float(d.scale), _ptr(sink), int(num_splits), _lib.stream_ptr()), "zb_latent_decode")
        return out
    _lib.check(l.zb_latent_attend(
        _ptr(q), _ptr(cache), d.row, _ptr(out), d.rot_off, _ptr(block_table), block_table.shape[1], cache.shape[1], d.heads, d.rank, d.rot,
        d.rot_off, d.window, float(d.scale), _ptr(sink), _ptr(q_start), _ptr(seq_lens), seq_lens.shape[0], t, int(q.dtype == torch.float32),
        _lib.stream_ptr()), "zb_latent_attend")
    return out


# tokens of a decode chunk: below this a chunk costs more in partial results than it gains in parallelism
_MIN_CHUNK = 64


def decode_plan_splits(batch: int, d: LatentDims, max_seq_len: int) -> int:
    """Chunks a sequence's visible tokens are cut into by a decode step: enough to give every SM a CTA."""
    l = _lib.lib()
    visible = min(max_seq_len, d.window) if d.window > 0 else max_seq_len
    ctas = max(1, batch * int(l.zb_latent_decode_groups(d.heads)))
    return max(1, min(l.zb_num_sms() // ctas, (visible + _MIN_CHUNK - 1) // _MIN_CHUNK, 64))


# ---------------------------------------------------------------------------- expanded keys and values
def _visible_plan(meta, window: int):
    """(first gathered row of every sequence and the total, position of that row's token) on the device, total rows: the
    tokens that this batch's queries see.  One upload per step and window, kept in `meta.plans`."""
    key = ("latent_visible", window)
    plan = meta.plans.get(key)
    if plan is None:
        qs, sl = meta.q_start_host, meta.seq_lens_host
        start, first = [0], []
        for a, b, n in zip(qs, qs[1:], sl):
            f = max(0, n - (b - a) - window + 1) if window > 0 else 0
            first.append(f)
            start.append(start[-1] + (n - f if b > a else 0))
        dev = torch.tensor(start + first, dtype=torch.int32).pin_memory().to(meta.seq_lens.device, non_blocking=True)
        plan = meta.plans[key] = (dev[:len(start)], dev[len(start):], start[-1])
    return plan


def expand(cache, w_ukv, meta, d: LatentDims):
    """Gathers the latents that this batch's queries see and projects them: (latents [rows, ..] with the rotated part at the
    returned column, kv [rows, H dim | H vdim], that column, the gather's plan)."""
    from . import gemm
    plan = key_start, first_key, rows = _visible_plan(meta, d.window)
    rot_out = _up(d.rot_off, 64)
    lat = torch.empty((rows, rot_out + _up(d.rot, 64)), dtype=cache.dtype, device=cache.device)
    _lib.check(_lib.lib().zb_latent_gather(
        _ptr(cache), d.row, _ptr(meta.block_table), meta.block_table.shape[1], cache.shape[1], _ptr(key_start), _ptr(first_key),
        first_key.shape[0], _ptr(lat), lat.shape[1], rows, d.rank, d.rot, d.rot_off, rot_out, _lib.stream_ptr()), "zb_latent_gather")
    return lat, gemm(lat[:, :d.rank], w_ukv, static_w=True), rot_out, plan


def pack_q(q, inv_freq, positions, d: LatentDims):
    """q [T, H * (dim + rot)] -> [T, H, dim | rot], the rotated part rotated and both padded with zeros to 64 columns."""
    t, dim_p, rot_p = q.shape[0], _up(d.dim, 64), _up(d.rot, 64)
    out = torch.empty((t, d.heads, dim_p + rot_p), dtype=q.dtype, device=q.device)
    _lib.check(_lib.lib().zb_latent_q_pack(_ptr(q), q.stride(0), _ptr(out), _ptr(inv_freq), _ptr(positions), t, d.heads, d.dim, d.rot, dim_p,
                                           rot_p, _lib.stream_ptr()), "zb_latent_q_pack")
    return out


def attend_expanded(qp, gate, lat, kv, rot_out: int, plan, meta, d: LatentDims, sink=None):
    """sigmoid(gate) * windowed causal attention of packed queries over expanded keys and values: [T, H * vdim]."""
    key_start, first_key, rows = plan
    t = qp.shape[0]
    out = torch.empty((t, d.heads * d.vdim), dtype=qp.dtype, device=qp.device)
    blocks = sum((b - a + 255) // 256 for a, b in zip(meta.q_start_host, meta.q_start_host[1:]))
    _lib.check(_lib.lib().zb_latent_prefill_tc(
        _ptr(qp), _ptr(kv), kv.stride(0), _ptr(lat), lat.stride(0), rot_out, _ptr(out), out.stride(0), _ptr(gate), _ld(gate),
        _ptr(meta.q_start), _ptr(meta.seq_lens), meta.seq_lens.shape[0], _ptr(key_start), _ptr(first_key), t, rows, blocks, d.heads, d.dim,
        d.rot, d.vdim, d.window, float(d.scale), _ptr(sink), _lib.stream_ptr()), "zb_latent_prefill_tc")
    return out


def prefill(q, gate, w_ukv, inv_freq, cache, meta, d: LatentDims, sink=None):
    """The expanded formulation on the tensor cores (bf16)."""
    lat, kv, rot_out, plan = expand(cache, w_ukv, meta, d)
    return attend_expanded(pack_q(q, inv_freq, meta.positions, d), gate, lat, kv, rot_out, plan, meta, d, sink)


def _expands(q, gate, meta, d: LatentDims) -> bool:
    return (q.is_cuda and q.dtype == torch.bfloat16 and meta.is_prefill and meta.q_start_host is not None and meta.seq_lens_host is not None
            and bool(_lib.lib().zb_latent_prefill_tc_supported(d.dim, d.rot, d.vdim, d.rank)) and q.stride(0) % 8 == 0
            and _ld(gate) % 8 == 0)


# ---------------------------------------------------------------------------- the layer's attention
def latent_attention(q, gate, w_uk_t, w_ukv, inv_freq, cache, meta, d: LatentDims, sink=None):
    """sigmoid(gate) * attention of one step: q [T, H * (dim + rot)] unrotated, gate [T, H * vdim] or None, w_uk_t [H, rank, dim],
    w_ukv [H dim + H vdim, rank], sink fp32 [H] or None; `meta` is the step's AttnMeta, the new tokens' cache rows are already
    written."""
    if _expands(q, gate, meta, d):
        return prefill(q, gate, w_ukv, inv_freq, cache, meta, d, sink)
    q_start = meta.q_start
    if q_start is None:
        q_start = torch.arange(q.shape[0] + 1, dtype=torch.int32, device=q.device)
    ql = absorb_q(q, w_uk_t, inv_freq, meta.positions, d)
    o = attend(ql, cache, meta.block_table, q_start, meta.seq_lens, d, decode=not meta.is_prefill, num_splits=meta.num_splits or 1, sink=sink)
    return absorb_out(o, w_ukv[d.heads * d.dim:].view(d.heads, d.vdim, d.rank), gate, d)
