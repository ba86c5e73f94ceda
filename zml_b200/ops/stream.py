"""Layer glue of decoders with an fp32 residual stream: embedding, the norms behind and in front of a sublayer, the
convolution in front of a mixer, and hyper-connections (several streams) (libzb_cuda.so: stream_f32.cu).

All of it works on the flattened varlen batch of the engine (`q_start`, `seq_lens`, `slots`, as in
`ops.linear_attn`).  Activations that a projection reads are written in the model's dtype (bf16 or fp32); the stream,
the norms, the convolution and its state are fp32.  CPU tensors take the plain torch branch of each function.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import Optional

import torch

from . import _lib

_p, _i, _ll, _f = C.c_void_p, C.c_int, C.c_longlong, C.c_float
_lib.register_signature("zb_embedding_f32", _i, [_p, _p, _i, _p, _i, _i, _i, _f, _i, _p])
_lib.register_signature("zb_hyper_norm", _i, [_p, _ll, _i, _p, _p, _i, _p, _i, _p, _p, _p, _p, _f, _p, _p, _ll, _i, _i, _i, _p])
_lib.register_signature("zb_sandwich_norm", _i, [_p, _ll, _i, _p, _p, _i, _p, _f, _p, _p, _f, _p, _p, _ll, _i, _i, _i, _p])
_lib.register_signature("zb_add_norm_conv_supported", _i, [_p, _ll, _i, _ll])
_lib.register_signature("zb_add_norm", _i, [_p, _ll, _i, _p, _p, _i, _p, _p, _p, _p, _f, _p, _ll, _i, _i, _i, _p, _p, _p, _i, _p, _p])
_lib.register_signature("zb_stream_conv", _i, [_p, _p, _p, _p, _p, _p, _i, _ll, _ll, _i, _i, _i, _i, _p, _p, _i, _i, _p])
_lib.register_signature("zb_post_norm", _i, [_p, _ll, _i, _p, _f, _p, _f, _p, _p, _ll, _i, _i, _i, _p, _p, _p, _p, _p, _ll, _ll,
                                             _i, _i, _i, _p, _p])

MAX_TAPS = 8
MAX_STREAMS = 8
CONV_BLOCK = 32          # tokens per block of the convolution kernel


def _ptr(t: Optional[torch.Tensor]):
    return None if t is None else t.data_ptr()


def embedding_f32(ids, table, scale: float = 1.0, streams: int = 0):
    """Rows of `table` (bf16 or fp32) times `scale`, as fp32 [T, d]; with `streams` as [T, streams, d], equal copies."""
    shape = (ids.shape[0], streams, table.shape[1]) if streams else (ids.shape[0], table.shape[1])
    if not table.is_cuda:
        x = table[ids.long()].float() * scale
        return x[:, None].expand(shape).contiguous() if streams else x
    assert ids.dtype == torch.int32 and table.is_contiguous()
    out = torch.empty(shape, dtype=torch.float32, device=table.device)
    _lib.check(_lib.lib().zb_embedding_f32(_ptr(ids), _ptr(table), int(table.dtype == torch.float32), _ptr(out), ids.shape[0],
                                           table.shape[1], table.shape[0], float(scale), max(1, streams), _lib.stream_ptr()), "zb_embedding_f32")
    return out


def layer_norm_reference(x, w, eps):
    d = x.float() - x.float().mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


@dataclass
class InputConv:
    """The convolution in front of a mixer and what follows it: h = x + conv(x), and with `mu` [nmix, d] the
    interpolations h + (h_prev - h) * mu_m of h with the previous token's h.  `state` is [slots, rows, d] fp32: the
    last inputs x of every sequence, `rows_for(taps, nmix)` of them."""
    w: torch.Tensor                       # [taps, d] fp32, tap taps - 1 on the current token
    state: torch.Tensor
    mu: Optional[torch.Tensor] = None

    @staticmethod
    def rows_for(taps: int, mixes: bool) -> int:
        return taps if mixes else taps - 1

    def nmix(self) -> int:
        return 0 if self.mu is None else self.mu.shape[0]

    def check(self) -> None:
        taps, d = self.w.shape
        if not 1 <= taps <= MAX_TAPS:
            raise ValueError(f"the input convolution takes 1 to {MAX_TAPS} taps, not {taps}")
        assert self.w.dtype == torch.float32 and self.w.is_contiguous() and self.state.is_contiguous()
        assert self.state.shape[1:] == (self.rows_for(taps, self.mu is not None), d), self.state.shape

    def alloc(self, tokens: int, dtype, device):
        shape = (tokens, self.w.shape[1]) if self.mu is None else (self.nmix(), tokens, self.w.shape[1])
        return torch.empty(shape, dtype=dtype, device=device)

    def alloc_padded(self, tokens: int, dtype, device):
        """h with zero columns up to a multiple of 8."""
        d = self.w.shape[1]
        make = torch.empty if d % 8 == 0 else torch.zeros
        return make((tokens, pad8(d)), dtype=dtype, device=device)

    def args(self, out):
        """The trailing kernel arguments: out pointer, row stride, plane stride, taps, rows, nmix."""
        return (_ptr(out), out.stride(-2), out.stride(0) if self.mu is not None else 0, self.w.shape[0], self.state.shape[1], self.nmix())


def _stream_conv_reference(x, conv: InputConv, q_start, seq_lens, slots, dtype):
    taps, d = conv.w.shape
    rows = conv.state.shape[1]
    out = conv.alloc(x.shape[0], dtype, x.device)
    qs, sl, so = q_start.tolist(), seq_lens.tolist(), slots.tolist()
    for s in range(len(sl)):
        a, b = qs[s], qs[s + 1]
        if b <= a:
            continue
        fresh = sl[s] - (b - a) <= 0
        hist = torch.zeros((rows, d)) if fresh else conv.state[so[s]]
        full = torch.cat([torch.zeros((taps - rows, d)), hist, x[a:b]], 0)             # [taps + n, d]
        h = full[taps - 1:] + (full.unfold(0, taps, 1) * conv.w.t()[None]).sum(-1)          # previous token's h, then n of them
        if conv.mu is None:
            out[a:b] = h[1:].to(dtype)
        else:
            out[:, a:b] = (h[None, 1:] + (h[:-1] - h[1:])[None] * conv.mu[:, None]).to(dtype)
        conv.state[so[s]] = full[full.shape[0] - rows:]
    return out


def stream_conv(x, conv: InputConv, q_start, seq_lens, slots, dtype, num_blocks: Optional[int] = None, padded: bool = False):
    """x [T, d] fp32 -> h [T, d] or the interpolations [nmix, T, d], in `dtype`; updates `conv.state`.  `padded` (h only): with
    zero columns up to a multiple of 8."""
    conv.check()
    if not x.is_cuda:
        h = _stream_conv_reference(x, conv, q_start, seq_lens, slots, dtype)
        return torch.nn.functional.pad(h, (0, pad8(h.shape[1]) - h.shape[1])) if padded else h
    t, d = x.shape
    assert x.is_contiguous() and x.dtype == torch.float32
    out = conv.alloc_padded(t, dtype, x.device) if padded else conv.alloc(t, dtype, x.device)
    nb = num_blocks if num_blocks is not None else t // CONV_BLOCK + seq_lens.shape[0]
    ptr, ld, plane, taps, rows, nmix = conv.args(out)
    _lib.check(_lib.lib().zb_stream_conv(_ptr(x), _ptr(conv.w), _ptr(conv.state), _ptr(slots), _ptr(conv.mu), ptr,
                                         int(dtype == torch.float32), ld, plane, taps, rows, nmix, d, _ptr(q_start), _ptr(seq_lens),
                                         seq_lens.shape[0], nb, _lib.stream_ptr()), "zb_stream_conv")
    return out


def post_norm(x, w, eps: float, y=None, alpha: float = 1.0, keep_x: bool = True, act_dtype=None,
              conv: Optional[InputConv] = None, seq_lens=None, slots=None):
    """layernorm(alpha * x + y) * w over rows of the fp32 stream x [T, d].  Returns (x_new or None, second):
    `second` is the same rows in `act_dtype` when that is given, or - for a decode step, one token per sequence - what
    `stream_conv` makes of them when `conv` is (then in `act_dtype` as well), all in one launch."""
    t, d = x.shape
    if not x.is_cuda:
        z = alpha * x.float()
        if y is not None:
            z = z + y.float()
        n = layer_norm_reference(z, w, eps)
        if conv is not None:
            q_start = torch.arange(t + 1, dtype=torch.int32)
            return (n if keep_x else None), _stream_conv_reference(n, conv, q_start, seq_lens, slots, act_dtype)
        return (n if keep_x else None), (n.to(act_dtype) if act_dtype is not None else None)
    assert x.dtype == torch.float32 and x.is_contiguous() and w.dtype == torch.float32
    assert y is None or (y.stride(1) == 1 and y.dtype in (torch.float32, torch.bfloat16))
    x_new = torch.empty_like(x) if keep_x else None
    act = out = None
    cargs = (None, 0, 0, 0, 0, 0)
    if conv is not None:
        conv.check()
        out = conv.alloc(t, act_dtype, x.device)
        cargs = conv.args(out)
    elif act_dtype is not None:
        act = torch.empty((t, d), dtype=act_dtype, device=x.device)
    c = conv
    _lib.check(_lib.lib().zb_post_norm(
        _ptr(y), y.stride(0) if y is not None else 0, int(y is not None and y.dtype == torch.float32), _ptr(x), float(alpha), _ptr(w),
        float(eps), _ptr(x_new), _ptr(act), d, int(act_dtype == torch.float32), t, d, _ptr(c.w) if c else None,
        _ptr(c.state) if c else None, _ptr(slots), _ptr(c.mu) if c else None, *cargs, _ptr(seq_lens), _lib.stream_ptr()), "zb_post_norm")
    return x_new, (out if conv is not None else act)


# ------------------------------------------------------------------ norms on both sides of a sublayer
def rms_norm_reference(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def pad8(n: int) -> int:
    return (n + 7) // 8 * 8


@dataclass
class ExpertRows:
    """Outputs of a routed mixture before they are summed: token t's value is sum_j weights[t, j] * rows[pair_pos[t, j]]
    over the pairs with a row here (`moe.expert_rows`).  `rows` may be wider than the stream."""
    rows: torch.Tensor                    # [*, >= d]
    pair_pos: torch.Tensor                # int32 [T * k]
    weights: torch.Tensor                 # float32 [T, k]

    def sum(self, d: int) -> torch.Tensor:
        t, k = self.weights.shape
        pos = self.pair_pos.reshape(t, k).long()
        w = self.weights.float() * (pos >= 0)
        return (self.rows[pos.clamp_min(0)][..., :d].float() * w[..., None]).sum(1)


def sandwich_norm(x, y=None, w=None, mult: float = 1.0, w_next=None, eps: float = 1e-6, act_dtype=None, keep_x: bool = True):
    """The residual sum of a sublayer with a norm behind it, and the norm in front of the next one, in one launch:
    x_new = x + mult * rmsnorm(y) * w and act = rmsnorm(x_new) * w_next in `act_dtype` ([T, d] with zero columns up to a
    multiple of 8).  x fp32 [T, d]; y [T, d] (bf16 or fp32) or `ExpertRows`; without y, act of x itself; without w_next,
    no act.  Returns (x_new or None, act or None); x is overwritten on CUDA."""
    t, d = x.shape
    if not x.is_cuda:
        if y is not None:
            v = y.sum(d) if isinstance(y, ExpertRows) else y[:, :d].float()
            x = x + mult * rms_norm_reference(v, w, eps)
        act = None
        if w_next is not None:
            act = torch.nn.functional.pad(rms_norm_reference(x, w_next, eps), (0, pad8(d) - d)).to(act_dtype)
        return (x if keep_x else None), act
    assert x.dtype == torch.float32 and x.is_contiguous()
    rows, pos, pw, k = y, None, None, 0
    if isinstance(y, ExpertRows):
        rows, pos, pw, k = y.rows, y.pair_pos, y.weights, y.weights.shape[1]
        assert pw.dtype == torch.float32 and pw.is_contiguous()
    assert rows is None or (rows.stride(1) == 1 and rows.shape[1] >= d and rows.dtype in (torch.float32, torch.bfloat16) and w.dtype == torch.float32)
    act = torch.empty((t, pad8(d)), dtype=act_dtype, device=x.device) if w_next is not None else None
    _lib.check(_lib.lib().zb_sandwich_norm(
        _ptr(rows), rows.stride(0) if rows is not None else 0, int(rows is not None and rows.dtype == torch.float32), _ptr(pos), _ptr(pw), k,
        _ptr(x), float(mult), _ptr(w), _ptr(w_next), float(eps), _ptr(x) if keep_x and rows is not None else None, _ptr(act), pad8(d),
        int(act_dtype == torch.float32), t, d, _lib.stream_ptr()), "zb_sandwich_norm")
    return (x if keep_x else None), act


# ------------------------------------------------------------------ norm in front of a sublayer
def _rows_of(y):
    """(rows, pair_pos, weights, k) of a sublayer's output, a tensor or `ExpertRows`."""
    if not isinstance(y, ExpertRows):
        return y, None, None, 0
    assert y.weights.dtype == torch.float32 and y.weights.is_contiguous()
    return y.rows, y.pair_pos, y.weights, y.weights.shape[1]


def add_norm(x, y=None, w=None, b=None, eps: float = 1e-6, act_dtype=None, conv: Optional[InputConv] = None, seq_lens=None, slots=None,
             inplace: bool = True, keep_x: bool = True, padded: bool = True):
    """The residual sum of a sublayer with a norm in front, and what the next one reads, in one launch: x_new = x + y and
    act = layernorm(x_new) * w + b in `act_dtype` ([T, d], `padded` with zero columns up to a multiple of 8) - for a decode step, one token
    per sequence, what `stream_conv` makes of that when `conv` is given.  Without w, act is x_new itself; without `act_dtype`, no
    act.  x fp32 [T, d]; y [T, >= d] (bf16 or fp32) or `ExpertRows`.  Returns (x_new or None, act or None); on CUDA x is
    overwritten unless `inplace` is off."""
    t, d = x.shape
    if not x.is_cuda:
        if y is not None:
            x = x + (y.sum(d) if isinstance(y, ExpertRows) else y[:, :d].float())
        act = None
        if act_dtype is not None:
            n = x if w is None else layer_norm_reference(x, w, eps) + b
            if conv is not None:
                n = _stream_conv_reference(n, conv, torch.arange(t + 1, dtype=torch.int32), seq_lens, slots, act_dtype)
            act = torch.nn.functional.pad(n, (0, pad8(d) - d if padded else 0)).to(act_dtype)
        return (x if keep_x else None), act
    assert x.dtype == torch.float32 and x.is_contiguous()
    rows, pos, pw, k = _rows_of(y)
    assert rows is None or (rows.stride(1) == 1 and rows.shape[1] >= d and rows.dtype in (torch.float32, torch.bfloat16))
    assert w is None or (w.dtype == b.dtype == torch.float32 and w.numel() == b.numel() == d)
    ldy, ptr, l = rows.stride(0) if rows is not None else 0, _ptr(rows), _lib.lib()
    apart = None
    if conv is not None:
        conv.check()
        if not l.zb_add_norm_conv_supported(ptr, ldy, d, pad8(d)):
            apart, conv, dtype, act_dtype = conv, None, act_dtype, torch.float32             # norm and convolution in two launches
    ld = d if apart is not None or not padded else pad8(d)
    act = torch.empty((t, ld), dtype=act_dtype, device=x.device) if act_dtype is not None else None
    x_new = None if not keep_x or (rows is None and inplace) else (x if inplace else torch.empty_like(x))
    c = conv
    _lib.check(l.zb_add_norm(
        ptr, ldy, int(rows is not None and rows.dtype == torch.float32), _ptr(pos), _ptr(pw), k, _ptr(x), _ptr(x_new), _ptr(w), _ptr(b), float(eps),
        _ptr(act), ld, int(act_dtype == torch.float32), t, d, _ptr(c.w) if c else None, _ptr(c.state) if c else None, _ptr(slots) if c else None,
        c.w.shape[0] if c else 0, _ptr(seq_lens) if c else None, _lib.stream_ptr()), "zb_add_norm")
    if apart is not None:
        act = stream_conv(act, apart, torch.arange(t + 1, dtype=torch.int32, device=x.device), seq_lens, slots, dtype, t, padded=True)
    if not keep_x:
        return None, act
    return (x if inplace else x_new), act


# ------------------------------------------------------------------ hyper-connections
@dataclass
class HyperMix:
    """Coefficients of one sublayer with hyper-connections, fp32: it reads sum_s inp[s] x_s, and its output y gives
    x_t <- sum_s mix[s, t] x_s + out[t] * y."""
    inp: torch.Tensor                     # [streams]
    mix: torch.Tensor                     # [streams, streams]
    out: torch.Tensor                     # [streams]


def hyper_norm(x, y=None, behind: Optional[HyperMix] = None, inp=None, w=None, eps: float = 1e-6, act_dtype=None):
    """The update of the streams behind a sublayer (`behind`) and the norm in front of the next one, which reads the mix `inp`
    [streams] of them, in one launch: act = rmsnorm(sum_s inp[s] x_s) * w in `act_dtype` ([T, d] with zero columns up to a
    multiple of 8).  x fp32 [T, streams, d]; y [T, >= d] (bf16 or fp32) or `ExpertRows`; without y, act of x itself; without w,
    no act.  Returns (x_new, act or None); x is overwritten on CUDA."""
    t, s, d = x.shape
    if not x.is_cuda:
        if y is not None:
            v = y.sum(d) if isinstance(y, ExpertRows) else y[:, :d].float()
            x = torch.einsum("st,nsd->ntd", behind.mix, x) + behind.out[None, :, None] * v[:, None]
        act = None
        if w is not None:
            act = rms_norm_reference(torch.einsum("s,nsd->nd", inp, x), w, eps)
            act = torch.nn.functional.pad(act, (0, pad8(d) - d)).to(act_dtype)
        return x, act
    assert x.dtype == torch.float32 and x.is_contiguous()
    rows, pos, pw, k = y, None, None, 0
    if isinstance(y, ExpertRows):
        rows, pos, pw, k = y.rows, y.pair_pos, y.weights, y.weights.shape[1]
        assert pw.dtype == torch.float32 and pw.is_contiguous()
    assert rows is None or (rows.stride(1) == 1 and rows.shape[1] >= d and rows.dtype in (torch.float32, torch.bfloat16))
    assert w is None or (w.dtype == inp.dtype == torch.float32 and inp.numel() == s and w.numel() == d)
    act = torch.empty((t, pad8(d)), dtype=act_dtype, device=x.device) if w is not None else None
    mix, out = (behind.mix, behind.out) if y is not None else (None, None)
    _lib.check(_lib.lib().zb_hyper_norm(
        _ptr(rows), rows.stride(0) if rows is not None else 0, int(rows is not None and rows.dtype == torch.float32), _ptr(pos), _ptr(pw), k,
        _ptr(x), s, _ptr(mix), _ptr(out), _ptr(inp if w is not None else None), _ptr(w), float(eps), _ptr(x) if rows is not None else None,
        _ptr(act), pad8(d), int(act_dtype == torch.float32), t, d, _lib.stream_ptr()), "zb_hyper_norm")
    return x, act
