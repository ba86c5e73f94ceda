"""Ops of the hybrid decoder layers: depthwise causal conv with a rolling cache, the gated
delta rule scan, and the sigmoid output gate (libzb_cuda.so: linear_attn.cu); the WKV
recurrence with its low-rank decay (wkv.cu); the delta rule with a decay per key channel, with its
convolutions, norms and gate (channel_delta.cu); the recurrence whose gates read the current token only
(gated_scan.cu).

All of them run over the flattened varlen token batch the engine uses everywhere else:
`q_start[S+1]` gives every sequence's token range in this launch, `seq_lens[S]` its length
including those tokens (so `seq_lens - count == 0` marks a sequence that starts here and
takes a zero state), `slots[S]` its row in the state pool.  On CPU tensors the functions
below evaluate the same math with plain torch in float32 - that is also the test oracle.

Reference: zml/nn.zig:1749-1874 (GatedDeltaNet), examples/llm/models/qwen3_5/model.zig:824-980,
examples/llm/models/lfm2/model.zig:441-500.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import Optional

import torch

from . import _lib

_p, _i, _ll, _f = C.c_void_p, C.c_int, C.c_longlong, C.c_float
_lib.register_signature("zb_causal_conv1d", _i, [_p, _ll, _p, _ll, _p, _ll, _p, _p, _ll, _p, _p, _p, _p, _i, _i,
                                                _i, _i, _p])
_lib.register_signature("zb_gated_delta_scan", _i, [_p, _ll, _p, _ll, _p, _p, _ll, _p, _p, _p, _f, _p, _p, _ll,
                                                   _p, _p, _p, _i, _i, _i, _i, _i, _p])
_lib.register_signature("zb_sigmoid_gate_mul", _i, [_p, _ll, _p, _ll, _i, _i, _p])


def _ptr(t: Optional[torch.Tensor]):
    return None if t is None else t.data_ptr()


def _bf16_round(x: torch.Tensor) -> torch.Tensor:
    return x.to(torch.bfloat16).float()


# ---------------------------------------------------------------------------- conv
def causal_conv1d_reference(x, w, state, q_start, seq_lens, slots, pre=None, post=None, silu=False):
    t, c = x.shape
    k = w.shape[1]
    out = torch.empty((t, c), dtype=x.dtype, device=x.device)
    wf = w.float()
    qs, sl, so = q_start.tolist(), seq_lens.tolist(), slots.tolist()
    for s in range(len(sl)):
        a, b = qs[s], qs[s + 1]
        if b <= a:
            continue
        xin = x[a:b].float()
        if pre is not None:
            xin = _bf16_round(xin * pre[a:b].float())
        hist = torch.zeros((k - 1, c)) if sl[s] - (b - a) <= 0 else state[so[s]].float()
        full = torch.cat([hist.to(xin.device), xin], 0)                     # [K-1+n, C]
        win = full.unfold(0, k, 1)                                           # [n, C, K]
        y = _bf16_round((win * wf[None]).sum(-1))
        if silu:
            y = y * torch.sigmoid(y)
        if post is not None:
            y = _bf16_round(y) * post[a:b].float()
        out[a:b] = y.to(x.dtype)
        state[so[s]] = full[-(k - 1):].to(state.dtype)
    return out


def causal_conv1d(x, w, state, q_start, seq_lens, slots, pre=None, post=None, silu: bool = False, out=None):
    """x [T, C] (row stride free), w [C, K] taps (tap K-1 on the current token), state
    [slots, K-1, C] updated in place.  Returns [T, C]."""
    if not x.is_cuda:
        return causal_conv1d_reference(x, w, state, q_start, seq_lens, slots, pre, post, silu)
    t, c = x.shape
    k = w.shape[1]
    assert w.is_contiguous() and state.is_contiguous() and state.shape[1:] == (k - 1, c)
    if out is None:
        out = torch.empty((t, c), dtype=torch.bfloat16, device=x.device)
    rc = _lib.lib().zb_causal_conv1d(
        _ptr(x), x.stride(0), _ptr(pre), pre.stride(0) if pre is not None else 0, _ptr(post),
        post.stride(0) if post is not None else 0, _ptr(w), _ptr(out), out.stride(0), _ptr(state),
        _ptr(q_start), _ptr(seq_lens), _ptr(slots), seq_lens.shape[0], c, k, 1 if silu else 0, _lib.stream_ptr())
    _lib.check(rc, "zb_causal_conv1d")
    return out


# ---------------------------------------------------------------------------- gated delta rule
def gated_delta_scan_reference(mix, z, a, b, a_log, dt_bias, norm_w, eps, state, q_start, seq_lens, slots,
                               hk, hv, dk, dv):
    t = mix.shape[0]
    key_dim = hk * dk
    rep = hv // hk
    out = torch.empty((t, hv * dv), dtype=mix.dtype, device=mix.device)
    q = mix[:, :key_dim].float().reshape(t, hk, dk).repeat_interleave(rep, 1)
    k = mix[:, key_dim:2 * key_dim].float().reshape(t, hk, dk).repeat_interleave(rep, 1)
    v = mix[:, 2 * key_dim:2 * key_dim + hv * dv].float().reshape(t, hv, dv)
    q = q * torch.rsqrt((q * q).sum(-1, keepdim=True) + 1e-6) * (dk ** -0.5)
    k = k * torch.rsqrt((k * k).sum(-1, keepdim=True) + 1e-6)
    alpha = torch.exp(-torch.exp(a_log.float())[None] * torch.nn.functional.softplus(a.float() + dt_bias.float()[None]))
    beta = torch.sigmoid(b.float())
    qs, sl, so = q_start.tolist(), seq_lens.tolist(), slots.tolist()
    for s in range(len(sl)):
        t0, t1 = qs[s], qs[s + 1]
        if t1 <= t0:
            continue
        st = torch.zeros((hv, dk, dv)) if sl[s] - (t1 - t0) <= 0 else state[so[s]].float().clone()
        st = st.to(mix.device)
        for i in range(t0, t1):
            vh = torch.einsum("hkv,hk->hv", st, k[i]) * alpha[i][:, None]
            delta = (v[i] - vh) * beta[i][:, None]
            st = st * alpha[i][:, None, None] + k[i][:, :, None] * delta[:, None, :]
            y = _bf16_round(torch.einsum("hkv,hk->hv", st, q[i]))
            inv = torch.rsqrt((y * y).mean(-1, keepdim=True) + eps)
            zg = z[i].float().reshape(hv, dv)
            out[i] = (y * inv * norm_w.float()[None] * (zg * torch.sigmoid(zg))).reshape(-1).to(mix.dtype)
        state[so[s]] = st.to(state.dtype)
    return out


def gated_delta_scan(mix, z, a, b, a_log, dt_bias, norm_w, eps, state, q_start, seq_lens, slots,
                     hk: int, hv: int, dk: int, dv: int, out=None):
    """mix [T, 2*hk*dk + hv*dv] = q | k | v after the conv; z [T, hv*dv]; a, b [T, hv] (same row
    stride); a_log, dt_bias float32 [hv]; norm_w [dv]; state float32 [slots, hv, dk, dv] updated
    in place.  Returns the gated, normalised output [T, hv*dv]."""
    if not mix.is_cuda:
        return gated_delta_scan_reference(mix, z, a, b, a_log, dt_bias, norm_w, eps, state, q_start, seq_lens,
                                          slots, hk, hv, dk, dv)
    t = mix.shape[0]
    assert a.stride(0) == b.stride(0) and state.dtype == torch.float32 and state.is_contiguous()
    assert a_log.dtype == torch.float32 and dt_bias.dtype == torch.float32
    if out is None:
        out = torch.empty((t, hv * dv), dtype=torch.bfloat16, device=mix.device)
    rc = _lib.lib().zb_gated_delta_scan(
        _ptr(mix), mix.stride(0), _ptr(z), z.stride(0), _ptr(a), _ptr(b), a.stride(0), _ptr(a_log), _ptr(dt_bias),
        _ptr(norm_w), float(eps), _ptr(state), _ptr(out), out.stride(0), _ptr(q_start), _ptr(seq_lens),
        _ptr(slots), seq_lens.shape[0], hk, hv, dk, dv, _lib.stream_ptr())
    _lib.check(rc, "zb_gated_delta_scan")
    return out


# ---------------------------------------------------------------------------- output gate
def sigmoid_gate_mul(x, gate):
    """x[r, c] * sigmoid(gate[r, c]); in place on CUDA tensors."""
    if not x.is_cuda:
        return (x.float() * torch.sigmoid(gate.float())).to(x.dtype)
    rows, cols = x.shape
    rc = _lib.lib().zb_sigmoid_gate_mul(_ptr(x), x.stride(0), _ptr(gate), gate.stride(0), rows, cols,
                                        _lib.stream_ptr())
    _lib.check(rc, "zb_sigmoid_gate_mul")
    return x


# ---------------------------------------------------------------------------- WKV
_lib.register_signature("zb_wkv_step_supported", _i, [_i])
_lib.register_signature("zb_wkv_scan", _i, [_p, _p, _p, _p, _ll, _p, _ll, _p, _p, _p, _f, _p, _p, _p, _ll, _p, _i, _i, _i, _p, _p, _i,
                                            _i, _p])
_lib.register_signature("zb_tanh_linear", _i, [_p, _ll, _p, _ll, _i, _p, _ll, _i, _i, _i, _p])
_lib.register_signature("zb_tanh_split", _i, [_p, _ll, _p, _i, _i, _i, _p])


def wkv_scan_reference(r, k, v, g, z, w0, u, norm_w, eps, state, q_start, seq_lens, slots, heads, dim):
    t = r.shape[0]
    hd = lambda x: x.float().reshape(-1, heads, dim)
    rf, kf, vf, gf = hd(r), hd(k), hd(v), hd(g)
    decay = torch.exp(-torch.exp(hd(z) + w0.reshape(1, heads, dim)))
    uu = u.reshape(heads, dim)
    o = torch.zeros((t, heads, dim))
    qs, sl, so = q_start.tolist(), seq_lens.tolist(), slots.tolist()
    for s in range(len(sl)):
        a, b = qs[s], qs[s + 1]
        if b <= a:
            continue
        st = torch.zeros((heads, dim, dim)) if sl[s] - (b - a) <= 0 else state[so[s]].clone()     # [H, value, key]
        for i in range(a, b):
            kv = vf[i][:, :, None] * kf[i][:, None, :]
            o[i] = torch.einsum("hvk,hk->hv", st + uu[:, None, :] * kv, rf[i])
            st = st * decay[i][:, None, :] + kv
        state[so[s]] = st
    o = o / torch.sqrt((o * o).mean(-1, keepdim=True) + eps) * norm_w.reshape(1, heads, dim) * (gf * torch.sigmoid(gf))
    return o.reshape(t, heads * dim).to(r.dtype)


def wkv_scan(r, k, v, g, z, w0, u, norm_w, eps, state, q_start, seq_lens, slots, heads: int, dim: int, decode: bool = False, out=None):
    """The WKV recurrence with its output norm and gate: r, k, v, g [T, heads * dim] (equal row strides), z fp32 the
    decay's pre-activation (w = exp(-exp(z + w0))), u the current token's bonus, norm_w the output norm's weight (fp32
    [heads * dim] each), state fp32 [slots, heads, dim (value), dim (key)] updated in place.  `decode`: one token per
    sequence.  Returns [T, heads * dim]."""
    if not r.is_cuda:
        return wkv_scan_reference(r, k, v, g, z, w0, u, norm_w, eps, state, q_start, seq_lens, slots, heads, dim)
    t, n = r.shape[0], heads * dim
    if dim > 256:
        raise ValueError(f"the WKV kernel takes heads of at most 256 channels, not {dim}")
    assert r.stride(0) == k.stride(0) == v.stride(0) == g.stride(0) and r.dtype == k.dtype == v.dtype == g.dtype
    assert z.dtype == torch.float32 and state.dtype == torch.float32 and state.is_contiguous()
    if out is None:
        out = torch.empty((t, n), dtype=r.dtype, device=r.device)
    o = None if decode and _lib.lib().zb_wkv_step_supported(dim) else torch.empty((t, n), dtype=torch.float32, device=r.device)
    _lib.check(_lib.lib().zb_wkv_scan(
        _ptr(r), _ptr(k), _ptr(v), _ptr(g), r.stride(0), _ptr(z), z.stride(0), _ptr(w0), _ptr(u), _ptr(norm_w), float(eps), _ptr(state),
        _ptr(slots), _ptr(out), out.stride(0), _ptr(o), int(r.dtype == torch.float32), heads, dim, _ptr(q_start), _ptr(seq_lens),
        seq_lens.shape[0], t, _lib.stream_ptr()), "zb_wkv_scan")
    return out


# tokens up to which the low-rank product runs as fp32 dot products instead of a GEMM
TANH_LINEAR_TOKENS = 64


def split_weight(w: torch.Tensor) -> torch.Tensor:
    """[N, R] -> [N, 2 R'] with R' = R rounded up to 8: the weight repeated, for `tanh_linear` on many tokens."""
    half = (w.shape[1] + 7) // 8 * 8
    p = torch.nn.functional.pad(w, (0, half - w.shape[1]))
    return torch.cat([p, p], 1).contiguous()


def tanh_linear(a, w_t, w_split=None):
    """tanh(a) @ w_t with an fp32 result from a fp32 [T, R] and w_t [R, N]: the activation is not rounded to bf16.  On the
    GPU few tokens take fp32 dot products, many take a bf16 GEMM over tanh(a) split into two bf16 pieces (`w_split`, see
    `split_weight`)."""
    if not a.is_cuda:
        return torch.tanh(a.float()) @ w_t.float()
    t, rank = a.shape
    n = w_t.shape[1]
    l = _lib.lib()
    if w_t.dtype == torch.bfloat16 and w_split is not None and t > TANH_LINEAR_TOKENS:
        from . import gemm
        half = w_split.shape[1] // 2
        s = torch.empty((t, 2 * half), dtype=torch.bfloat16, device=a.device)
        _lib.check(l.zb_tanh_split(_ptr(a), a.stride(0), _ptr(s), half, rank, t, _lib.stream_ptr()), "zb_tanh_split")
        return gemm(s, w_split, out_dtype=torch.float32, static_w=True)
    assert w_t.stride(1) == 1
    out = torch.empty((t, n), dtype=torch.float32, device=a.device)
    _lib.check(l.zb_tanh_linear(_ptr(a), a.stride(0), _ptr(w_t), w_t.stride(0), int(w_t.dtype == torch.float32), _ptr(out), out.stride(0), t, n,
                                rank, _lib.stream_ptr()), "zb_tanh_linear")
    return out


# ---------------------------------------------------------------------------- delta rule with a decay per key channel
_lib.register_signature("zb_channel_delta_block_floats", _i, [_i, _i])
_lib.register_signature("zb_channel_delta", _i, [_p, _ll, _i, _p, _ll, _p, _i, _p, _p, _p, _f, _p, _p, _p, _p, _p, _p, _ll, _i, _i, _i, _i, _i, _p, _p,
                                                 _i, _i, _i, _p])

DELTA_MAX_TAPS, DELTA_MAX_KEY, DELTA_BLOCK = 8, 256, 8


@dataclass
class ChannelDelta:
    """Parameters and state pools of one layer: `heads` value heads of `vdim` channels, `kv_heads` query / key heads of `dim`
    (head h uses h // (heads / kv_heads)).  Per head, with unit keys and queries (queries also times dim^-1/2):
    S <- g S by key channel, u = beta (v - S^T k), S <- S + k u^T, o = S^T q, out = o / rms(o) * norm * sigmoid(gate), where
    g = exp(-exp(a_log) softplus(z + dt_bias)).  q, k and v pass a causal convolution and silu first."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv_w: torch.Tensor                  # fp32 [taps, channels], channels = q | k | v, the last tap on the current token
    a_log: torch.Tensor                   # fp32 [heads]
    dt_bias: torch.Tensor                 # fp32 [heads dim]
    norm: torch.Tensor                    # fp32 [vdim]
    eps: float
    ring: Optional[torch.Tensor] = None   # [slots, taps, channels]: the input of position p at row p % taps
    state: Optional[torch.Tensor] = None  # fp32 [slots, heads, vdim, dim up to a multiple of 4]

    def __post_init__(self):
        if self.kv_heads < 1 or self.heads % self.kv_heads:
            raise ValueError(f"{self.heads} heads do not share {self.kv_heads} query / key heads")
        if not 1 <= self.taps <= DELTA_MAX_TAPS:
            raise ValueError(f"the convolution takes 1 to {DELTA_MAX_TAPS} taps, not {self.taps}")
        if self.dim > DELTA_MAX_KEY:
            raise ValueError(f"the delta rule takes at most {DELTA_MAX_KEY} key channels, not {self.dim}")
        assert self.conv_w.shape[1] == self.channels and self.conv_w.is_contiguous()

    @property
    def taps(self) -> int:
        return self.conv_w.shape[0]

    @property
    def channels(self) -> int:
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim

    def alloc(self, num_slots: int, dtype, device) -> None:
        self.ring = torch.zeros((num_slots, self.taps, self.channels), dtype=dtype, device=device)
        self.state = torch.zeros((num_slots, self.heads, self.vdim, (self.dim + 3) // 4 * 4), dtype=torch.float32, device=device)

    def slot_bytes(self) -> int:
        return sum(t[0].numel() * t.element_size() for t in (self.ring, self.state))


def channel_delta_reference(proj, beta_col, low, m: ChannelDelta, q_start, seq_lens, slots):
    t, H, G, dk, dv, taps = proj.shape[0], m.heads, m.kv_heads, m.dim, m.vdim, m.taps
    ch, rep = m.channels, m.heads // m.kv_heads
    z = low[:, :H * dk].float() + m.dt_bias
    decay = torch.exp(-torch.exp(m.a_log)[None, :, None] * torch.nn.functional.softplus(z).reshape(t, H, dk))
    beta = torch.sigmoid(proj[:, beta_col:beta_col + H].float())
    gate = torch.sigmoid(low[:, H * dk:H * (dk + dv)].float()).reshape(t, H, dv)
    out = torch.zeros((t, H, dv))
    unit = lambda v: v / torch.sqrt((v * v).sum(-1, keepdim=True) + 1e-6)
    qs, sl, so = q_start.tolist(), seq_lens.tolist(), slots.tolist()
    for s in range(len(sl)):
        a, b = qs[s], qs[s + 1]
        if b <= a:
            continue
        n, p0 = b - a, sl[s] - (b - a)
        raw = proj[a:b, :ch]
        hist = [m.ring[so[s], p % taps].float() if p >= 0 else torch.zeros(ch) for p in range(p0 - taps + 1, p0)]
        full = torch.cat([torch.stack(hist) if hist else torch.zeros((0, ch)), raw.float()], 0)
        x = (full.unfold(0, taps, 1) * m.conv_w.t()[None]).sum(-1)
        x = x * torch.sigmoid(x)
        q = unit(x[:, :G * dk].reshape(n, G, dk)).repeat_interleave(rep, 1) * dk ** -0.5
        k = unit(x[:, G * dk:2 * G * dk].reshape(n, G, dk)).repeat_interleave(rep, 1)
        v = x[:, 2 * G * dk:].reshape(n, H, dv)
        st = torch.zeros((H, dv, dk)) if p0 <= 0 else m.state[so[s], ..., :dk].clone()
        for i in range(n):
            st = st * decay[a + i][:, None, :]
            u = beta[a + i][:, None] * (v[i] - torch.einsum("hvk,hk->hv", st, k[i]))
            st = st + u[:, :, None] * k[i][:, None, :]
            out[a + i] = torch.einsum("hvk,hk->hv", st, q[i])
        m.state[so[s], ..., :dk] = st
        for i in range(max(0, n - taps), n):
            m.ring[so[s], (p0 + i) % taps] = raw[i]
    out = out / torch.sqrt((out * out).mean(-1, keepdim=True) + m.eps) * m.norm * gate
    return out.reshape(t, H * dv).to(proj.dtype)


def channel_delta(proj, beta_col: int, low, m: ChannelDelta, q_start, seq_lens, slots, decode: bool = False,
                  num_blocks: Optional[int] = None):
    """The mixer of `ChannelDelta` behind its input projections: proj [T, *] = q | k | v columns first, the write gates' logits
    at column `beta_col`; low fp32 [T, heads dim + heads vdim] = the decays' pre-activations and the output gates' logits.
    `decode`: one token per sequence; else `num_blocks` (optional) is the sum of ceil(tokens / 8) over the sequences.
    Updates the layer's ring and state at `slots`; returns [T, heads vdim]."""
    if not proj.is_cuda:
        return channel_delta_reference(proj, beta_col, low, m, q_start, seq_lens, slots)
    t, n, dev = proj.shape[0], m.heads * m.vdim, proj.device
    assert proj.stride(1) == 1 and low.stride(1) == 1 and low.dtype == torch.float32 and m.ring.dtype == proj.dtype
    l = _lib.lib()
    out = torch.empty((t, (n + 7) // 8 * 8), dtype=proj.dtype, device=dev)[:, :n]
    blocks = o = None
    nb = 0
    if not decode:
        nb = num_blocks if num_blocks is not None else t // DELTA_BLOCK + seq_lens.shape[0]
        blocks = torch.empty((nb, m.heads, l.zb_channel_delta_block_floats(m.dim, m.vdim)), dtype=torch.float32, device=dev)
        o = torch.empty((t, n), dtype=torch.float32, device=dev)
    _lib.check(l.zb_channel_delta(
        _ptr(proj), proj.stride(0), beta_col, _ptr(low), low.stride(0), _ptr(m.conv_w), m.taps, _ptr(m.a_log), _ptr(m.dt_bias), _ptr(m.norm),
        float(m.eps), _ptr(m.ring), _ptr(m.state), _ptr(slots), _ptr(blocks), _ptr(o), _ptr(out), out.stride(0), m.heads, m.kv_heads, m.dim,
        m.vdim, int(proj.dtype == torch.float32), _ptr(q_start), _ptr(seq_lens), seq_lens.shape[0], t, nb, _lib.stream_ptr()), "zb_channel_delta")
    return out


# ---------------------------------------------------------------------------- recurrence with gates of the current token
_lib.register_signature("zb_gated_scan_rows", _i, [])
_lib.register_signature("zb_gated_scan", _i, [_p, _p, _p, _ll, _p, _p, _p, _p, _p, _p, _ll, _f, _i, _i, _p, _p, _i, _i, _p])

GATED_ROWS = 64          # tokens per block of the kernel


def gated_scan_reference(z, x, gate, z_bias, x_bias, state, q_start, seq_lens, slots, scale):
    g, u, f = torch.sigmoid(z.float() + z_bias), x.float() + x_bias, gate.float()
    c = torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
    out = torch.zeros(z.shape)
    qs, sl, so = q_start.tolist(), seq_lens.tolist(), slots.tolist()
    for s in range(len(sl)):
        a, b = qs[s], qs[s + 1]
        if b <= a:
            continue
        st = torch.zeros(z.shape[1]) if sl[s] - (b - a) <= 0 else state[so[s]].clone()
        for i in range(a, b):
            st = (1 - g[i]) * st + g[i] * c[i]
            out[i] = st
        state[so[s]] = st
    return (out * f * torch.sigmoid(f) * scale).to(z.dtype)


def gated_scan(z, x, gate, z_bias, x_bias, state, q_start, seq_lens, slots, scale: float = 1.0, out=None, decode: bool = False,
               num_blocks: Optional[int] = None):
    """minGRU by channel: with g = sigmoid(z + z_bias), u = x + x_bias and the candidate c = u + 1/2 where u >= 0, else
    sigmoid(u): S <- (1 - g) S + g c, out = S * silu(gate) * scale.  z, x, gate [T, width] (equal row strides), biases fp32
    [width], state fp32 [slots, width] updated in place.  `decode`: one token per sequence; else `num_blocks` (optional) is the
    sum of ceil(tokens / 64) over the sequences.  `out`: [T, width] columns of a wider buffer to write to."""
    if not z.is_cuda:
        y = gated_scan_reference(z, x, gate, z_bias, x_bias, state, q_start, seq_lens, slots, scale)
        return y if out is None else out.copy_(y)
    t, n = z.shape
    l = _lib.lib()
    assert z.stride(0) == x.stride(0) == gate.stride(0) and z.stride(1) == 1 and z.dtype == x.dtype == gate.dtype
    assert state.dtype == z_bias.dtype == x_bias.dtype == torch.float32 and state.is_contiguous() and state.shape[1] == n
    if out is None:
        out = torch.empty((t, n), dtype=z.dtype, device=z.device)
    assert out.shape == (t, n) and out.stride(1) == 1 and out.dtype == z.dtype
    maps, nb = None, 0
    if not decode:
        rows = l.zb_gated_scan_rows()
        nb = num_blocks if num_blocks is not None and rows == GATED_ROWS else t // rows + seq_lens.shape[0]
        maps = torch.empty((nb, n, 2), dtype=torch.float32, device=z.device)
    _lib.check(l.zb_gated_scan(
        _ptr(z), _ptr(x), _ptr(gate), z.stride(0), _ptr(z_bias), _ptr(x_bias), _ptr(state), _ptr(slots), _ptr(maps), _ptr(out), out.stride(0),
        float(scale), n, int(z.dtype == torch.float32), _ptr(q_start), _ptr(seq_lens), seq_lens.shape[0], nb, _lib.stream_ptr()), "zb_gated_scan")
    return out
