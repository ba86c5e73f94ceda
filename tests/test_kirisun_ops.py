"""The mechanisms of Kirisun one by one against the plain functions of `kirisun_oracle`, with inputs that make a wrong key, a
window edge, a missing sink or a lost state stand out."""
import os
import sys
from types import SimpleNamespace

import numpy as np
import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import kirisun_oracle as oracle  # noqa: E402
from zml_b200.moe import ops as moe_ops  # noqa: E402
from zml_b200.ops import gqa, stream  # noqa: E402
from zml_b200.ops import linear_attn as la  # noqa: E402
from zml_b200 import ops  # noqa: E402

F32, BF16 = torch.float32, torch.bfloat16
TARGETS = [pytest.param(("cpu", F32), id="cpu-f32"), pytest.param(("cuda", F32), id="gpu-f32", marks=pytest.mark.gpu),
           pytest.param(("cuda", BF16), id="gpu-bf16", marks=pytest.mark.gpu)]
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


# ------------------------------------------------------------------ stream
@pytest.mark.parametrize("target", TARGETS)
def test_scaled_embedding(target):
    dev, dt = target
    table, ids = rnd((30, 51), 1), [3, 0, 29, 3]
    close(stream.embedding_f32(i32(ids, dev), table.to(dev, dt), 7.25), npd(table)[ids] * 7.25, 1e-6)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("d", [8, 51, 260, 1028, 2048, 4100, 3001, 9000])
def test_sandwich_norm(target, d):
    """The residual sum with a norm behind the sublayer, and the next sublayer's norm, each also alone; y in both types."""
    dev, dt = target
    x, y, w, wn = rnd((5, d), 1), rnd((5, d), 2, 3.0), rnd((d,), 3), rnd((d,), 4)
    new_x = npd(x) + 0.37 * oracle.rms_norm(npd(y), npd(w), 1e-2)
    act_want = oracle.rms_norm(new_x, npd(wn), 1e-2)
    for yy in (y.to(dev), y.to(dev, dt)):
        new, act = stream.sandwich_norm(x.to(dev).clone(), yy, w.to(dev), 0.37, wn.to(dev), 1e-2, act_dtype=dt)
        close(new, new_x, 2e-5)
        close(act[:, :d], act_want, TOL[dt])
        assert act.shape[1] % 8 == 0 and not act[:, d:].any()
    new, act = stream.sandwich_norm(x.to(dev).clone(), y.to(dev), w.to(dev), 0.37, eps=1e-2)
    assert act is None
    close(new, new_x, 2e-5)
    keep = x.to(dev).clone()
    _, act = stream.sandwich_norm(keep, w_next=wn.to(dev), eps=1e-2, act_dtype=dt)
    close(act[:, :d], oracle.rms_norm(npd(x), npd(wn), 1e-2), TOL[dt])
    assert torch.equal(keep.cpu(), x)
    small = 1e-3 * x                                         # eps counts
    _, act = stream.sandwich_norm(small.to(dev), w_next=wn.to(dev), eps=1e-6, act_dtype=dt)
    close(act[:, :d], oracle.rms_norm(npd(small), npd(wn), 1e-6), TOL[dt])


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("d,k", [(51, 3), (256, 1), (2048, 8), (1028, 40)])
def test_sandwich_norm_sums_expert_rows(target, d, k):
    """Rows wider than the stream, pairs without a row, more pairs than one pass takes."""
    dev, dt = target
    t = 6
    rows, weights = rnd((t * k + 3, (d + 127) // 128 * 128), 1), torch.rand((t, k), generator=torch.Generator().manual_seed(2))
    pos = torch.randperm(t * k + 3, generator=torch.Generator().manual_seed(3))[:t * k].to(torch.int32)
    pos[1::4] = -1
    x, w, wn = rnd((t, d), 4), rnd((d,), 5), rnd((d,), 6)
    y = np.zeros((t, d))
    for i in range(t * k):
        if pos[i] >= 0:
            y[i // k] += float(weights[i // k, i % k]) * npd(rows[pos[i]])[:d]
    new, act = stream.sandwich_norm(x.to(dev).clone(), stream.ExpertRows(rows.to(dev, dt), pos.to(dev), weights.to(dev)), w.to(dev), 1.3, wn.to(dev),
                                    1e-5, act_dtype=dt)
    want = npd(x) + 1.3 * oracle.rms_norm(y, npd(w), 1e-5)
    close(new, want, 2e-5)
    close(act[:, :d], oracle.rms_norm(want, npd(wn), 1e-5), TOL[dt])


# ------------------------------------------------------------------ queries, keys, values
PREP = {"even": (6, 2, 64, 64, 32, 2.0), "all": (2, 2, 128, 128, 128, 1.0), "none": (3, 1, 24, 40, 0, 1.0), "odd": (6, 3, 13, 10, 6, 4.0),
        "wide": (3, 3, 200, 256, 66, 8.0)}


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", sorted(PREP))
def test_norms_rotation_and_cache_write(target, name):
    dev, dt = target
    H, G, dk, dv, rot, factor = PREP[name]
    s = gqa.GqaSpec(H, G, dk, dv, rot, base=3000.0, factor=factor)
    pos, slots = [0, 1, 63, 64, 5000, 77], [130, 0, -1, 64, 65, 191]
    n = H * dk + G * (dk + dv)
    proj, qn, kn = rnd((len(pos), n + 11), 1), rnd((dk,), 2), rnd((dk,), 3)
    cache = s.alloc_cache(3, 64, dt, dev)
    for c in cache:
        c.fill_(7.0)
    q = gqa.prep(proj.to(dev, dt), qn.to(dev), kn.to(dev), s.inv_freq(dev), i32(pos, dev), i32(slots, dev), cache, 1e-3, s)
    x = npd(proj)
    turn = lambda v, w: np.stack([oracle.turn_halves(oracle.rms_norm(v[t], npd(w), 1e-3), p, rot, 3000.0, factor) for t, p in enumerate(pos)])
    tol = max(TOL[dt], 1e-3 if name != "none" else 0)         # fp32 angles of position 5000
    close(q[..., :dk], turn(x[:, :H * dk].reshape(-1, H, dk), qn), tol)
    assert not q[..., dk:].any()
    kc, vc = (c.view(192, G, -1) for c in cache)
    ok = [i for i, r in enumerate(slots) if r >= 0]
    rows = [slots[i] for i in ok]
    close(kc[rows][..., :dk], turn(x[:, H * dk:(H + G) * dk].reshape(-1, G, dk), kn)[ok], tol)
    close(vc[rows][..., :dv], x[:, (H + G) * dk:n].reshape(-1, G, dv)[ok], TOL[dt])
    assert not kc[rows][..., dk:].any() and not vc[rows][..., dv:].any()
    rest = [r for r in range(192) if r not in rows]
    assert bool((kc[rest] == 7).all()) and bool((vc[rest] == 7).all())


# ------------------------------------------------------------------ attention
#         heads kv dim vdim window keep cap sink
ATTN = {
    "small": (4, 2, 24, 16, 33, 3, 15.0, True),
    "tensor cores": (4, 1, 128, 128, 100, 5, 30.0, True),
    "tensor cores, narrower": (2, 1, 100, 72, 70, 64, 50.0, True),
    "tensor cores, no sink, no window": (4, 2, 128, 128, 0, 0, 20.0, False),
    "tensor cores, low cap": (4, 2, 128, 128, 100, 3, 7.0, True),
    "64": (3, 3, 64, 64, 64, 65, 8.0, True),
    "256": (2, 2, 256, 200, 130, 1, 30.0, True),
    "no cap": (2, 1, 128, 128, 90, 4, 0.0, True),
    "neither cap nor sink": (4, 2, 64, 32, 50, 10, 0.0, False),
    "large cap": (2, 1, 128, 128, 90, 4, 200.0, True),
    "one token": (2, 2, 40, 40, 1, 0, 10.0, True),
    "one token and the first": (2, 2, 40, 40, 1, 1, 10.0, True),
    "more kept than the window": (6, 3, 13, 10, 29, 140, 12.0, True),
    "many heads": (20, 1, 48, 24, 60, 2, 25.0, True),
    "large": (2, 1, 300, 264, 60, 2, 25.0, True),
}


def attend_case(name, n, seed):
    """(spec, q, k, v, gate) of one sequence.  Scores are small apart from those of single pairs, which stand out: keys a
    long way back, just inside and just outside the window, the last kept and the first dropped token, page borders."""
    H, G, dk, dv, window, keep, cap, sink = ATTN[name]
    s = gqa.GqaSpec(H, G, dk, dv, 0, scale=dk ** -0.5, cap=cap, window=window, keep=keep, sink=sink)
    q, k, v, gate = rnd((n, H, dk), seed), rnd((n, G, dk), seed + 1), rnd((n, G, dv), seed + 2), rnd((n, H * dv), seed + 3)
    k *= 0.3
    w = window or n
    places = [lambda i: i - w + 1, lambda i: i - w, lambda i: keep - 1, lambda i: keep, lambda i: i, lambda i: 64, lambda i: 63, lambda i: 0,
              lambda i: i - 1, lambda i: i - w - 40]
    for i in range(n):
        j = places[i % len(places)](i)
        if 0 <= j <= i:
            for h in range(H):                             # q leans towards key j of its group: one score of about 9
                key = k[j, h // (H // G)]
                q[i, h] = key * (9.0 / s.scale / float(key @ key))
    return s, q.to(BF16).float(), k.to(BF16).float(), v, gate


def run_attention(case, portions, dev, dt, page=64, extra_rows=0):
    s, q, k, v, gate = case
    n, G = q.shape[0], s.kv_heads
    pages = (n + page - 1) // page
    order = torch.randperm(pages + 2, generator=torch.Generator().manual_seed(9))[:pages]
    cache = s.alloc_cache(pages + 2, page, dt, dev)
    rows = (order[torch.arange(n) // page] * page + torch.arange(n) % page).to(dev)
    bt = torch.zeros((1 + extra_rows, pages + 1), dtype=torch.int32, device=dev)
    bt[0, :pages] = order.to(dev, torch.int32)
    kr = cache[0].shape[-1]
    out, at = [], 0
    for m in portions:
        e = at + m
        cache[0].view(-1, G, kr)[rows[at:e], :, :s.dim] = k[at:e].to(dev, dt)
        cache[1].view(-1, G, cache[1].shape[-1])[rows[at:e], :, :s.vdim] = v[at:e].to(dev, dt)
        qq = torch.zeros((m + extra_rows, s.heads, kr), dtype=dt, device=dev)
        qq[:m, :, :s.dim] = q[at:e].to(dev, dt)
        gg = torch.zeros((m + extra_rows, s.heads * s.vdim + 8), dtype=dt, device=dev)
        gg[:m, 8:] = gate[at:e].to(dev, dt)
        decode = m == 1
        qs, sl = varlen([m] + [1] * extra_rows, [at] + [-1] * extra_rows, dev)
        meta = SimpleNamespace(is_prefill=not decode, q_start=qs, seq_lens=sl, block_table=bt, total_q_blocks=(m + 63) // 64 + extra_rows,
                               num_splits=ops.decode_plan_splits(1, G, s.visible(n)) if dev == "cuda" else None, max_seq_len=n)
        out.append(gqa.attention(qq, gg[:, 8:], cache, meta, s)[:m])
        at = e
    return torch.cat(out)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", sorted(ATTN))
def test_attention_in_prompts_portions_and_decoding(target, name, monkeypatch):
    dev, dt = target
    n = 300
    case = attend_case(name, n, 11)
    s, q, k, v, gate = case
    if not s.sink:                                           # the oracle has a sink: without one, its score goes to minus infinity
        monkeypatch.setattr(oracle, "sink_softmax", lambda z: np.exp(z - z.max()) / np.exp(z - z.max()).sum())
    want = oracle.attend(npd(q), npd(k), npd(v), s.scale, s.cap, s.window, s.keep).reshape(n, -1) * oracle.sigmoid(npd(gate))
    for portions in ([n], [130] + [1] * 40 + [2, 128], [1] * 70 + [2, 3, 64, 5, 156]):
        got = npd(run_attention(case, portions, dev, dt))
        err = np.abs(got - want[:len(got)]).max(-1)
        assert err.max() < (1e-4 if dt == F32 else 5e-2), (portions[:3], err.max(), int(err.argmax()))


@pytest.mark.gpu
@pytest.mark.parametrize("name", ["small", "tensor cores", "256", "many heads"])
def test_long_contexts_are_split_and_padding_rows_are_ignored(name):
    """Decoding far into a sequence (several key chunks where there is no window) with a padding row in the batch."""
    case = attend_case(name, 1500, 21)
    s, q, k, v, gate = case
    for spec in (s, gqa.GqaSpec(**{**s.__dict__, "window": 0, "keep": 0})):
        first = 1490
        want = oracle.attend(npd(q)[first:], npd(k), npd(v), spec.scale, spec.cap, spec.window, spec.keep, first).reshape(10, -1) * oracle.sigmoid(npd(gate)[first:])
        got = npd(run_attention((spec, q, k, v, gate), [first] + [1] * 10, "cuda", BF16, extra_rows=1))[first:]
        assert np.abs(got - want).max() < 5e-2


@pytest.mark.parametrize("target", TARGETS[:2])
def test_a_cap_and_a_sink_change_what_they_should(target):
    """A sequence of one token: the only key competes with the sink, its score under the cap."""
    dev, dt = target
    for cap, raw in ((5.0, 40.0), (5.0, -40.0), (50.0, 1.0), (30.0, 0.0)):
        s = gqa.GqaSpec(1, 1, 8, 8, 0, scale=1.0, cap=cap, sink=True)
        q, k, v = torch.zeros((1, 1, 8)), torch.zeros((1, 1, 8)), rnd((1, 1, 8), 1)
        q[..., 0], k[..., 0] = raw, 1.0
        got = npd(run_attention((s, q, k, v, torch.full((1, 8), 40.0)), [1], dev, dt))
        e = np.exp(cap * np.tanh(raw / cap))
        close(torch.tensor(got), npd(v)[:, 0] * e / (1 + e), 2e-5)


# ------------------------------------------------------------------ delta rule
#         heads kv dim vdim taps
DELTA = {"small": (4, 2, 24, 16, 3), "ones": (1, 1, 1, 1, 1), "odd": (6, 3, 7, 5, 5), "square": (2, 2, 128, 128, 4), "wide values": (2, 1, 64, 200, 8),
         "wide keys": (2, 2, 160, 40, 6), "largest keys": (1, 1, 256, 33, 2), "shared": (8, 1, 40, 24, 2), "32": (3, 3, 32, 32, 4), "64": (2, 2, 64, 32, 3)}


def delta_case(name, n, seed, decay="mixed"):
    H, G, dk, dv, taps = DELTA[name]
    c = 2 * G * dk + H * dv
    t = dict(raw=rnd((n, c), seed), conv=rnd((c, taps), seed + 1, 0.6), beta=rnd((n, H), seed + 2), pre=rnd((n, H * dk), seed + 3),
             gate=rnd((n, H * dv), seed + 4), a_log=rnd((H,), seed + 5, 0.5), dt_bias=rnd((H * dk,), seed + 6), norm=rnd((dv,), seed + 7))
    if decay == "mixed":                                    # from forgetting at once to keeping nearly everything
        t["dt_bias"] = (torch.rand((H * dk,), generator=torch.Generator().manual_seed(seed + 6)) * 14 - 9).to(BF16).float()
    elif decay == "fast":
        t["dt_bias"] = torch.full((H * dk,), 40.0)
    return t


def delta_want(name, t):
    H, G, dk, dv, _ = DELTA[name]
    x, w = npd(t["raw"]), npd(t["conv"])
    cut = (0, G * dk, 2 * G * dk, x.shape[1])
    parts = [(x[:, a:b], w[a:b]) for a, b in zip(cut, cut[1:])]
    return oracle.delta_core(*(p[0] for p in parts), [p[1] for p in parts], npd(t["beta"]), npd(t["pre"]), npd(t["a_log"]), npd(t["dt_bias"]),
                             npd(t["gate"]), npd(t["norm"]), (H, G, dk, dv), 1e-3)


class DeltaLayer:
    def __init__(self, name, t, dev, dt, slots=3):
        H, G, dk, dv, _ = DELTA[name]
        self.m = la.ChannelDelta(H, G, dk, dv, t["conv"].t().contiguous().to(dev), t["a_log"].to(dev), t["dt_bias"].to(dev), t["norm"].to(dev), 1e-3)
        self.m.alloc(slots, dt, dev)
        self.m.ring.fill_(5.0)                               # what another sequence left
        self.m.state.fill_(5.0)
        self.dev, self.dt, self.H = dev, dt, H

    def run(self, pieces, past, slots, decode=False):
        """pieces: (case, from, to) per sequence."""
        pad = -pieces[0][0]["raw"].shape[1] % 8
        proj = torch.cat([torch.cat([torch.nn.functional.pad(t["raw"][a:b], (0, pad)), torch.nn.functional.pad(t["beta"][a:b], (0, -self.H % 8))], 1)
                          for t, a, b in pieces])
        low = torch.cat([torch.cat([t["pre"][a:b], t["gate"][a:b]], 1) for t, a, b in pieces])
        qs, sl = varlen([b - a for _, a, b in pieces], past, self.dev)
        return la.channel_delta(proj.to(self.dev, self.dt), self.m.channels + pad, low.to(self.dev), self.m, qs, sl, i32(slots, self.dev), decode)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", sorted(DELTA))
def test_delta_rule_in_prompts_portions_and_decoding(target, name):
    dev, dt = target
    n = 70
    t = delta_case(name, n, 31)
    want = delta_want(name, t)
    for sizes in ([n], [2, 3, 8, 1, 16, 7, 33], [9] + [1] * 61):
        L, out, at = DeltaLayer(name, t, dev, dt), [], 0
        for i, m in enumerate(sizes):
            decode = m == 1 and i > 0
            out.append(L.run([(t, at, at + m)], [at], [1], decode))
            at += m
        close(torch.cat([o.float().cpu() for o in out]), want, TOL[dt], sizes)
        assert bool((L.m.state[[0, 2]] == 5).all()) and bool((L.m.ring[[0, 2]] == 5).all())


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", ["small", "odd", "64"])
def test_delta_rule_of_unequal_sequences_in_one_batch(target, name):
    """Portions beside single tokens and sequences that start, in slots that are used again."""
    dev, dt = target
    a, b, c = (dict(delta_case(name, n, 41), raw=rnd(delta_case(name, n, 41)["raw"].shape, 50 + n)) for n in (45, 20, 30))
    L = DeltaLayer(name, a, dev, dt)
    got = {0: [], 1: [], 2: []}

    def go(pieces, past, slots, decode=False):
        out, at = L.run([(t, lo, hi) for _, t, lo, hi in pieces], past, slots, decode).float().cpu(), 0
        for i, _, lo, hi in pieces:
            got[i].append(out[at:at + hi - lo])
            at += hi - lo
    go([(0, a, 0, 13), (1, b, 0, 1)], [0, 0], [2, 0])
    go([(0, a, 13, 14), (1, b, 1, 19)], [13, 1], [2, 0])
    go([(1, b, 19, 20), (0, a, 14, 15)], [19, 14], [0, 2], decode=True)
    go([(2, c, 0, 17), (0, a, 15, 40)], [0, 15], [0, 2])                # c takes b's slot
    go([(0, a, 40, 45), (2, c, 17, 30)], [40, 17], [2, 0])
    for i, t in enumerate((a, b, c)):
        close(torch.cat(got[i]), delta_want(name, t), TOL[dt], i)


@pytest.mark.gpu
@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("name", ["32", "shared", "64", "square", "largest keys"])
def test_delta_rule_of_many_sequences(name, dt):
    """More sequences than a warp has lanes, every padded key size."""
    t = delta_case(name, 30, 81)
    want = delta_want(name, t)
    H, _, _, dv, _ = DELTA[name]
    m = 300 // (H * ((dv + 31) // 32)) + 2
    lens = [1 + (7 * i) % 23 for i in range(m)]
    L = DeltaLayer(name, t, "cuda", dt, slots=m)
    first = L.run([(t, 0, n) for n in lens], [0] * m, list(range(m))[::-1])
    second = L.run([(t, n, n + 7) for n in lens], lens, list(range(m))[::-1])
    close(first, np.concatenate([want[:n] for n in lens]), TOL[dt])
    close(second, np.concatenate([want[n:n + 7] for n in lens]), TOL[dt])


@pytest.mark.parametrize("target", TARGETS[:2])
@pytest.mark.parametrize("decay", ["fast", "slow"])
def test_extreme_decays(target, decay):
    """Channels that forget everything within a token, and channels that keep all of it over hundreds of tokens."""
    dev, dt = target
    t = delta_case("small", 400, 61, decay)
    if decay == "slow":
        t["dt_bias"] = torch.full_like(t["dt_bias"], -14.0)
        t["pre"] *= 0.1
    want = delta_want("small", t)
    assert np.isfinite(want).all()
    close(DeltaLayer("small", t, dev, dt).run([(t, 0, 400)], [0], [0]), want, 1e-4)


@pytest.mark.parametrize("target", TARGETS)
def test_a_decode_step_of_a_padding_row_leaves_other_slots_alone(target):
    dev, dt = target
    t = delta_case("small", 9, 71)
    L = DeltaLayer("small", t, dev, dt)
    L.run([(t, 0, 7)], [0], [1])
    before = L.m.state[1].clone(), L.m.ring[1].clone()
    L.run([(t, 7, 8)], [-1], [2], decode=True)               # length 0
    assert torch.equal(before[0], L.m.state[1]) and torch.equal(before[1], L.m.ring[1])
    close(L.run([(t, 7, 8)], [7], [1], decode=True), delta_want("small", t)[7:8], TOL[dt])


# ------------------------------------------------------------------ mixture
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("experts,top,ff,d,tokens", [(1, 1, 8, 40, 3), (5, 2, 33, 51, 70), (6, 6, 96, 96, 9), (40, 7, 24, 160, 50), (4, 2, 128, 128, 300),
                                                     (3, 1, 64, 264, 1)])
def test_router_and_experts(target, experts, top, ff, d, tokens):
    dev, dt = target
    x, router = rnd((tokens, d), 1), rnd((experts, d), 2, 2.0 * d ** -0.5)
    bias = rnd((experts,), 3, 2.0)
    gate, up, down = rnd((experts, ff, d), 4, d ** -0.5), rnd((experts, ff, d), 5, d ** -0.5), rnd((experts, d, ff), 6, ff ** -0.5)
    W = {"router": npd(router), "router.b": npd(bias)}
    for e in range(experts):
        W.update({f"e{e}.gate": npd(gate[e]), f"e{e}.up": npd(up[e]), f"e{e}.down": npd(down[e])})
    h = torch.nn.functional.pad(x, (0, -d % 8)).to(dev, dt)
    z = ops.gemm(h, ops.pad_k(router.to(dev, dt)), bias=bias.to(dev, dt), out_dtype=F32, static_w=True)
    ids, weights = moe_ops.router_topk(z, top)
    for t in range(tokens):
        pick, w = oracle.route(npd(x)[t], W, top)
        logits = np.sort(W["router"] @ npd(x)[t] + W["router.b"])[::-1]
        if top < experts and logits[top - 1] - logits[top] < 1e-3:
            continue                                         # a close call
        got = dict(zip(ids[t].tolist(), weights[t].tolist()))
        assert set(got) == set(pick.tolist())
        assert all(abs(got[int(e)] - v) < 1e-4 for e, v in zip(pick, w))
    gu, dn = moe_ops.pad_experts(gate.to(dev, dt), up.to(dev, dt), down.to(dev, dt))
    half = experts // 2
    parts = [(0, experts)] if half == 0 else [(0, experts), (0, half), (half, experts)]          # all experts; split over two ranks
    sums = []
    for e0, e1 in parts:
        rows, pos = moe_ops.expert_rows(h, ids, gu[e0:e1].contiguous(), dn[e0:e1].contiguous(), e0, experts)
        sums.append(npd(stream.ExpertRows(rows, pos, weights).sum(d)))
    want = np.zeros((tokens, d))
    for t in range(tokens):
        for e, w in zip(ids[t].tolist(), weights[t].tolist()):
            want[t] += w * oracle.expert(npd(x)[t], W[f"e{e}.gate"], W[f"e{e}.up"], W[f"e{e}.down"])
    close(torch.tensor(sums[0]), want, TOL[dt])
    if half:
        close(torch.tensor(sums[1] + sums[2]), want, TOL[dt])
