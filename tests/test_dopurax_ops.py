"""The mechanisms of Dopurax one by one against the plain functions of `dopurax_oracle`, with inputs that make a wrong key,
a window edge or a lost state stand out."""
import os
import sys
from types import SimpleNamespace

import numpy as np
import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import dopurax_oracle as oracle  # noqa: E402
from zml_b200 import ops  # noqa: E402
from zml_b200.ops import latent as lat  # noqa: E402
from zml_b200.ops import linear_attn as la  # noqa: E402
from zml_b200.ops import stream  # noqa: E402

F32, BF16 = torch.float32, torch.bfloat16
TARGETS = [pytest.param(("cpu", F32), id="cpu-f32"), pytest.param(("cuda", F32), id="gpu-f32", marks=pytest.mark.gpu),
           pytest.param(("cuda", BF16), id="gpu-bf16", marks=pytest.mark.gpu)]
GPU_TARGETS = TARGETS[1:]
TOL = {F32: 2e-5, BF16: 2e-2}


def rnd(shape, seed, scale=1.0):
    """Values exact in bf16, as fp32."""
    return (scale * torch.randn(shape, generator=torch.Generator().manual_seed(seed))).to(BF16).float()


def npd(t):
    return t.detach().float().cpu().numpy().astype(np.float64)


def close(got, want, tol, what=""):
    err = np.abs(npd(got) - want)
    scale = max(np.sqrt((want * want).mean()), 1e-6)
    assert err.max() < tol * 6 * scale and np.sqrt((err * err).mean()) < tol * scale, (what, err.max() / scale, np.unravel_index(err.argmax(), err.shape))


def i32(x, dev):
    return torch.tensor(x, dtype=torch.int32, device=dev)


def varlen(counts, past, dev):
    qs = [0]
    for n in counts:
        qs.append(qs[-1] + n)
    return i32(qs, dev), i32([n + p for n, p in zip(counts, past)], dev)


# ------------------------------------------------------------------ norm behind a sublayer, input convolution
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("d", [8, 51, 260, 1028, 4100])
def test_post_norm(target, d):
    dev, dt = target
    x, y, w = rnd((5, d), 1) + 0.7, rnd((5, d), 2), rnd((d,), 3)
    want = oracle.layer_norm(1.9 * npd(x) + npd(y), npd(w), 1e-3)
    for yy in (y.to(dev), y.to(dev, dt)):
        new, act = stream.post_norm(x.to(dev).contiguous(), w.to(dev), 1e-3, yy, 1.9, act_dtype=dt)
        close(new, want, 2e-5)
        close(act, want, TOL[dt])
    new, act = stream.post_norm(x.to(dev), w.to(dev), 1e-3, keep_x=False, act_dtype=dt)
    assert new is None
    close(act, oracle.layer_norm(npd(x), npd(w), 1e-3), TOL[dt])


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 8])
@pytest.mark.parametrize("mixes", [False, True])
def test_input_convolution_in_portions_and_slots(target, taps, mixes):
    """Portions of two sequences in one batch, the state in slots that another sequence used before."""
    dev, dt = target
    d, total = 150, (71, 40)
    w = rnd((d, taps), 1)
    mu = rnd((5, d), 2) if mixes else None
    xs = [rnd((n, d), 3 + i) for i, n in enumerate(total)]
    want = []
    for x in xs:
        h = npd(x) + oracle.causal_taps(npd(x), npd(w))
        prev = np.concatenate([np.zeros_like(h[:1]), h[:-1]])
        want.append(h if mu is None else np.stack([h + (prev - h) * npd(mu[m]) for m in range(5)]))
    state = torch.full((4, stream.InputConv.rows_for(taps, mixes), d), 1e4, device=dev)       # whatever the slots held before
    conv = stream.InputConv(w.t().contiguous().to(dev), state, None if mu is None else mu.to(dev).contiguous())
    slots = i32([2, 1], dev)
    at = [0, 0]
    for ns in ((2, 3), (1, 1), (40, 2), (1, 33), (27, 1)):
        qs, sl = varlen(ns, at, dev)
        x = torch.cat([xs[s][at[s]:at[s] + ns[s]] for s in range(2)]).to(dev).contiguous()
        got = stream.stream_conv(x, conv, qs, sl, slots, dt)
        for s in range(2):
            a = int(qs[s])
            g = got[..., a:a + ns[s], :]
            close(g, want[s][..., at[s]:at[s] + ns[s], :], TOL[dt] if dt == BF16 else 2e-5, (taps, s, at[s]))
            at[s] += ns[s]
    assert at == list(total)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("taps", [1, 3, 8])
@pytest.mark.parametrize("mixes", [False, True])
@pytest.mark.parametrize("d", [64, 70, 2500])
def test_decode_step_norm_and_convolution_in_one_launch(target, taps, mixes, d):
    dev, dt = target
    w, nw = rnd((d, taps), 1), rnd((d,), 2)
    mu = rnd((5, d), 3).to(dev).contiguous() if mixes else None
    rows = stream.InputConv.rows_for(taps, mixes)
    a = stream.InputConv(w.t().contiguous().to(dev), torch.zeros((3, rows, d), device=dev), mu)
    b = stream.InputConv(w.t().contiguous().to(dev), torch.full((3, rows, d), 7.0, device=dev), mu)
    slots = i32([2, 0], dev)
    for t in range(taps + 3):
        x, y = rnd((2, d), 10 + t).to(dev), rnd((2, d), 50 + t).to(dev)
        qs, sl = varlen((1, 1), (t, t), dev)
        new, _ = stream.post_norm(x, nw.to(dev), 1e-5, y, 2.0)
        want = stream.stream_conv(new, a, qs, sl, slots, dt)
        new2, got = stream.post_norm(x, nw.to(dev), 1e-5, y, 2.0, act_dtype=dt, conv=b, seq_lens=sl, slots=slots)
        close(new2, npd(new), 1e-6)
        close(got, npd(want), TOL[dt])
        if rows:
            close(b.state[[2, 0]], npd(a.state[[2, 0]]), 1e-6)


# ------------------------------------------------------------------ WKV
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("heads,dim", [(1, 8), (3, 24), (2, 50), (2, 64), (1, 96), (2, 128), (1, 200), (300, 16)])
def test_wkv_recurrence(target, heads, dim):
    """Portions of two sequences with states in used slots; decays from none to almost everything, a bonus that stands out."""
    dev, dt = target
    if heads == 300 and dev == "cpu":
        pytest.skip("enough heads to take the one-launch form on the GPU")
    n, total = heads * dim, (37, 12)
    mk = lambda s, k, sc=1.0: rnd((total[s], n), 10 * s + k, sc)
    r, k, v, g = [[mk(s, j) for s in range(2)] for j in range(4)]
    z = [mk(s, 4, 2.0) for s in range(2)]
    w0, u, nw = rnd((n,), 70) - 1, rnd((n,), 71, 2.0), rnd((n,), 72)
    want = []
    for s in range(2):
        R, K, V = (npd(x[s]).reshape(-1, heads, dim) for x in (r, k, v))
        W = np.exp(-np.exp(npd(z[s]) + npd(w0))).reshape(-1, heads, dim)
        U, S, o = npd(u).reshape(heads, dim), np.zeros((heads, dim, dim)), np.zeros_like(R)
        for t in range(total[s]):
            kv = K[t][:, :, None] * V[t][:, None, :]
            o[t] = np.einsum("hk,hkv->hv", R[t], S + U[:, :, None] * kv)
            S = W[t][:, :, None] * S + kv
        want.append(oracle.rms(o, 1e-4).reshape(-1, n) * npd(nw) * oracle.silu(npd(g[s])))
    state = torch.full((3, heads, dim, dim), 1e5, device=dev)
    slots, at = i32([2, 0], dev), [0, 0]
    c = lambda p: torch.cat(p)
    for ns in ((2, 1), (1, 1), (17, 3), (1, 1), (16, 6)):
        qs, sl = varlen(ns, at, dev)
        pick = lambda x, t=dt: c([x[s][at[s]:at[s] + ns[s]] for s in range(2)]).to(dev, t).contiguous()
        got = la.wkv_scan(pick(r), pick(k), pick(v), pick(g), pick(z, F32), w0.to(dev), u.to(dev), nw.to(dev), 1e-4, state, qs, sl, slots,
                          heads, dim, decode=max(ns) == 1)
        for s in range(2):
            a = int(qs[s])
            close(got[a:a + ns[s]], want[s][at[s]:at[s] + ns[s]], TOL[dt] if dt == BF16 else 5e-5, (s, at[s]))
            at[s] += ns[s]
    assert at == list(total)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("t,rank,n", [(3, 1, 20), (5, 24, 200), (130, 20, 72), (100, 64, 256)])
def test_low_rank_decay_keeps_more_than_bf16(target, t, rank, n):
    dev, dt = target
    a, w = torch.randn((t, rank), generator=torch.Generator().manual_seed(1)).to(dev), rnd((n, rank), 2).to(dev, dt)
    got = la.tanh_linear(a, w.t().contiguous(), la.split_weight(w))
    close(got, np.tanh(npd(a)) @ npd(w).T, 2e-5)


# ------------------------------------------------------------------ GEMMs the design adds
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("m,n,k", [(1, 1, 1), (3, 130, 51), (70, 64, 96), (600, 256, 72), (600, 300, 100)])
def test_gemm_any_size_and_squared_relu(target, m, n, k):
    dev, dt = target
    a, w = rnd((m, k), 1).to(dev, dt), rnd((n, k), 2).to(dev, dt)
    want = npd(a) @ npd(w).T
    close(ops.gemm(a, w), want, TOL[dt] if dt == BF16 else 1e-5)
    close(ops.gemm(a, ops.pad_k(w), out_dtype=F32, static_w=True), want, 1e-5)
    close(ops.gemm(a, w, act="relu2"), np.maximum(want, 0) ** 2, TOL[dt] if dt == BF16 else 1e-5)


# ------------------------------------------------------------------ latent attention
def dims(heads=2, dim=16, rot=8, vdim=16, rank=32, q_rank=24, window=70, scale=0.2, base=1000.0):
    return lat.LatentDims(heads, dim, rot, vdim, rank, q_rank, window, scale, base)


DIMS = {"small": dims(), "odd": dims(3, 13, 6, 10, 21, 19, 29), "one": dims(1, 8, 2, 8, 8, 8, 1), "tiles": dims(4, 64, 64, 64, 128, 64, 65),
        "deep": dims(20, 128, 64, 128, 512, 64, 128, 0.05), "groups": dims(37, 24, 32, 40, 96, 40, 130, 0.1), "all": dims(2, 32, 16, 24, 48, 40, 0),
        "bigrot": dims(2, 64, 128, 72, 64, 64, 64, 0.05)}


class Setup:
    """A paged cache with `len(total)` sequences on scattered pages, everything computed from random projections."""

    def __init__(self, d, total, dev, dt, page=64, seed=0):
        self.d, self.dev, self.dt, self.page = d, dev, dt, page
        self.total = total
        n = sum((t + page - 1) // page for t in total)
        order = np.random.default_rng(seed).permutation(n) + 1
        width = max((t + page - 1) // page for t in total)
        bt, k = np.zeros((len(total), width), dtype=np.int32), 0
        for s, t in enumerate(total):
            c = (t + page - 1) // page
            bt[s, :c] = order[k:k + c]
            k += c
        self.bt = torch.tensor(bt, device=dev)
        self.cache = torch.zeros((n + 1, page, d.row), dtype=dt, device=dev)
        self.cache[0] = float("nan")                                   # the reserved page is not to be read for live rows
        # what other sequences left in the unused rows of the pages is finite and must not show
        self.cache[1:, :, :d.rank] = 3.0
        self.inv = d.inv_freq(dev)
        self.qn, self.cn = 1 + 0.3 * rnd((d.q_rank,), 1), 1 + 0.3 * rnd((d.rank,), 2)
        self.uq = rnd((d.heads * (d.dim + d.rot), d.q_rank), 3, 1.5 / d.q_rank ** 0.5)
        self.uk = rnd((d.heads * d.dim, d.rank), 4, 1.5 / d.rank ** 0.5)
        self.uv = rnd((d.heads * d.vdim, d.rank), 5, 1 / d.rank ** 0.5)
        cols = d.q_rank + d.rank + d.rot
        self.off = cols + -cols % 8
        self.proj = [rnd((t, self.off + d.heads * d.vdim), 100 + s) for s, t in enumerate(total)]

    def meta(self, counts, past, decode):
        qs, sl = varlen(counts, past, self.dev)
        pos = [p + i for n, p in zip(counts, past) for i in range(n)]
        bt = self.bt.cpu()
        slots = [int(bt[s, (p + i) // self.page]) * self.page + (p + i) % self.page for s, (n, p) in enumerate(zip(counts, past)) for i in range(n)]
        return SimpleNamespace(is_prefill=not decode, positions=i32(pos, self.dev), slot_mapping=i32(slots, self.dev), block_table=self.bt,
                               seq_lens=sl, q_start=qs, q_start_host=qs.tolist(), seq_lens_host=sl.tolist(), plans={}, num_splits=3)

    def run(self, counts, past, decode=False):
        d, dev, dt = self.d, self.dev, self.dt
        meta = self.meta(counts, past, decode)
        proj = torch.cat([self.proj[s][p:p + n] for s, (n, p) in enumerate(zip(counts, past))]).to(dev, dt)
        if proj.shape[1] % 8 and dt == BF16:
            proj = torch.nn.functional.pad(proj, (0, -proj.shape[1] % 8))[:, :proj.shape[1]]
        cq = lat.prep(proj, self.qn.to(dev), self.cn.to(dev), self.inv, meta.positions, meta.slot_mapping, self.cache, 1e-5, d)
        q = ops.gemm(cq, self.uq.to(dev, dt))
        uk_t = self.uk.reshape(d.heads, d.dim, d.rank).transpose(1, 2).contiguous().to(dev, dt)
        out = lat.latent_attention(q, proj[:, self.off:], uk_t, torch.cat([self.uk, self.uv]).to(dev, dt), self.inv, self.cache, meta, d)
        return [out[int(a):int(b)] for a, b in zip(meta.q_start, meta.q_start[1:])]

    def oracle(self, s):
        """The same up to the output projection, through the plain mixer with identity projections around it."""
        d, P = self.d, npd(self.proj[s])
        full = P.shape[1]
        eye = np.eye(full)
        W = {"dq": eye[:d.q_rank], "dq.norm": npd(self.qn), "uq": npd(self.uq), "dkv": eye[d.q_rank:d.q_rank + d.rank + d.rot],
             "dkv.norm": npd(self.cn), "uk": npd(self.uk), "uv": npd(self.uv), "g": eye[self.off:], "o": np.eye(d.heads * d.vdim)}
        m = {"heads": d.heads, "dim": d.dim, "rot_dim": d.rot, "vdim": d.vdim, "kv_rank": d.rank, "scale": d.scale,
             "mask": {"size": d.window if d.window > 0 else 1 << 30}, "rot": {"base": d.base, "dims": d.rot}}
        return oracle.latent_attention(P, W, m, 1e-5)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", sorted(DIMS))
def test_latent_attention_portions_and_decoding(target, name):
    dev, dt = target
    total = (200, 131)
    s = Setup(DIMS[name], total, dev, dt)
    want = [s.oracle(0), s.oracle(1)]
    tol = 4e-5 if dt == F32 else 3e-2
    at = [0, 0]
    plan = [((1, 2), False), ((1, 1), True), ((61, 60), False), ((1, 1), True), ((2, 3), False), ((130, 1), False), ((1, 1), True), ((3, 62), False)]
    for ns, decode in plan:
        got = s.run(ns, at, decode)
        for i in range(2):
            close(got[i], want[i][at[i]:at[i] + ns[i]], tol, (name, i, at[i], ns[i]))
            at[i] += ns[i]
    assert at == list(total)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("name", ["small", "tiles", "groups", "odd"])
def test_keys_at_the_window_edge_and_page_borders(target, decode, name):
    """One key per case is made to win the softmax outright; whether it is seen decides the output."""
    dev, dt = target
    d = DIMS[name]
    total = 3 * d.window + 70
    pos = total - 1
    seen = {}
    for planted in sorted({pos, pos - d.window + 1, pos - d.window, pos - 1, (pos // 64) * 64, (pos // 64) * 64 - 1, 0}):
        if planted < 0:
            continue
        s = Setup(d, (total,), dev, dt)
        # the latent that head 0's last query likes best, far above the others
        P, a = npd(s.proj[0]), slice(d.q_rank, d.q_rank + d.rank)
        q = (oracle.rms(P[pos, :d.q_rank], 1e-5) * npd(s.qn)) @ npd(s.uq).T
        liked = npd(s.uk)[:d.dim].T @ q[:d.dim]
        s.proj[0][planted, a] = torch.tensor(liked / np.abs(liked).max() * 4).to(BF16).float()
        big = 30.0 / max(d.scale * np.linalg.norm(liked), 1e-9) / np.sqrt(d.rank)
        s.cn = torch.full((d.rank,), 1.0)
        s.uq *= max(1.0, min(4.0, big))
        s.uq = s.uq.to(BF16).float()
        want = s.oracle(0)
        if pos:
            s.run((pos,), (0,))
        got = s.run((1,), (pos,), decode)[0]
        close(got, want[pos:], 4e-5 if dt == F32 else 6e-2, (planted - pos,))
        seen[planted - pos] = want[pos]
    inside, outside = seen[-d.window + 1], seen[-d.window]
    assert np.abs(inside - outside).max() > 0.05 * np.abs(inside).max()      # the case can tell the two apart


@pytest.mark.parametrize("target", GPU_TARGETS)
def test_latent_decode_chunks_and_padding_rows(target):
    """Long contexts cut into chunks of tokens, beside short ones and a row without a sequence."""
    dev, dt = target
    d = dims(5, 16, 16, 16, 64, 24, 900, 0.2)
    s = Setup(d, (1500, 70, 1), dev, dt)
    want = [s.oracle(i) for i in range(3)]
    s.run((1499, 69, 0), (0, 0, 0))
    for splits in (1, 2, 5, 64):
        meta = s.meta((1, 1, 1), (1499, 69, 0), True)
        meta.num_splits = splits
        s.meta = lambda *a, m=meta: m
        got = s.run((1, 1, 1), (1499, 69, 0), True)
        del s.meta
        for i in range(3):
            close(got[i], want[i][-1:], 4e-5 if dt == F32 else 3e-2, (splits, i))
    q = torch.randn((2, d.heads, d.row), device=dev).to(dt)
    o = lat.attend(q, s.cache, s.bt[:2].contiguous(), i32([0, 1, 2], dev), i32([0, 5], dev), d, decode=True, num_splits=2)
    assert (o[0, :, :d.rank] == 0).all() and torch.isfinite(o[1, :, :d.rank]).all()


@pytest.mark.gpu
def test_prefill_kernel_and_latent_space_agree_on_a_batch():
    """Several blocks of 256 queries, sequences that start inside a window, rows at every block's edge."""
    d = dims(6, 128, 64, 128, 256, 96, 300, 0.06)
    total = (700, 257, 3, 256)
    past = (190, 0, 1, 255)
    s = Setup(d, total, "cuda", BF16)
    s.run(tuple(max(p, 1) if p else 0 for p in past), (0, 0, 0, 0))
    counts = tuple(t - p for t, p in zip(total, past))
    fast = s.run(counts, past)
    keep, lat._expands = lat._expands, lambda *a: False
    try:
        slow = s.run(counts, past)
    finally:
        lat._expands = keep
    for f, g in zip(fast, slow):
        close(f, npd(g), 2e-2)
