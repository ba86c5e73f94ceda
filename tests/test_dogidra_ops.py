"""The mechanisms of Dogidra one by one against the plain functions of `dogidra_oracle`, with inputs that make a wrong key, a
window's edge, a block that is seen too early or a lost state stand out."""
import dataclasses
import os
import sys
from types import SimpleNamespace

import numpy as np
import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import dogidra_oracle as oracle  # noqa: E402
from zml_b200 import ops  # noqa: E402
from zml_b200.moe import ops as moe_ops  # noqa: E402
from zml_b200.ops import gqa, stream  # noqa: E402
from zml_b200.ops import linear_attn as la  # noqa: E402

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


# ------------------------------------------------------------------ residual sum, norm with bias, input convolution
SIZES = [(8, 1), (51, 3), (260, 4), (1028, 8), (2048, 4), (4096, 5), (3001, 3), (5000, 4), (9000, 2)]


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("d", [8, 51, 260, 1028, 2048, 4100, 3001, 9000])
def test_residual_sum_and_layer_norm_with_bias(target, d):
    dev, dt = target
    t = 3
    x, y, w, b = rnd((t, d), 1) + 0.5, rnd((t, d), 2, 2.0), rnd((d,), 3), rnd((d,), 4)
    want = npd(x) + npd(y)
    act_want = oracle.layer_norm(want, npd(w), npd(b), 1e-2)
    for yy in (y.to(dev), y.to(dev, dt)):
        new, act = stream.add_norm(x.to(dev).clone(), yy, w.to(dev), b.to(dev), 1e-2, act_dtype=dt)
        close(new, want, 2e-6)
        close(act[:, :d], act_want, TOL[dt])
        assert act.shape[1] % 8 == 0 and not act[:, d:].any()
    old = x.to(dev)
    new, act = stream.add_norm(old, y.to(dev), w.to(dev), b.to(dev), 1e-2, act_dtype=F32, inplace=False, padded=False)
    assert act.shape == (t, d) and torch.equal(old.cpu(), x)
    close(new, want, 2e-6)
    close(act, act_want, TOL[F32])
    new, act = stream.add_norm(x.to(dev).clone(), y.to(dev))
    assert act is None
    close(new, want, 2e-6)
    new, act = stream.add_norm(x.to(dev).clone(), y.to(dev), act_dtype=dt)             # the stream itself, for the next pass
    close(act[:, :d], want, TOL[dt])
    assert not act[:, d:].any()
    small = 1e-3 * x                                          # eps counts
    _, act = stream.add_norm(small.to(dev), w=w.to(dev), b=b.to(dev), eps=1e-6, act_dtype=dt, keep_x=False)
    close(act[:, :d], oracle.layer_norm(npd(small), npd(w), npd(b), 1e-6), TOL[dt])


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("d,k", [(51, 3), (256, 1), (2048, 9), (1028, 40)])
def test_residual_sum_of_expert_rows(target, d, k):
    dev, dt = target
    t = 5
    rows, weights = rnd((t * k + 3, (d + 127) // 128 * 128), 1), torch.rand((t, k), generator=torch.Generator().manual_seed(2))
    pos = torch.randperm(t * k + 3, generator=torch.Generator().manual_seed(3))[:t * k].to(torch.int32)
    pos[1::4] = -1
    x, w, b = rnd((t, d), 4), rnd((d,), 5), rnd((d,), 6)
    want = npd(x).copy()
    for i in range(t * k):
        if pos[i] >= 0:
            want[i // k] += float(weights[i // k, i % k]) * npd(rows[pos[i]])[:d]
    new, act = stream.add_norm(x.to(dev).clone(), stream.ExpertRows(rows.to(dev, dt), pos.to(dev), weights.to(dev)), w.to(dev), b.to(dev), 1e-5, act_dtype=dt)
    close(new, want, 2e-5)
    close(act[:, :d], oracle.layer_norm(want, npd(w), npd(b), 1e-5), TOL[dt])


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("d,taps", SIZES)
def test_norm_and_convolution_step_by_step_and_in_portions(target, d, taps):
    """Three sequences in slots that others have used: whole, in portions down to one token, and as decode steps, where norm and
    convolution are one launch (two where a row does not fit)."""
    dev, dt = target
    n, S = 9, 3
    xs, w, b, taps_w = [rnd((n, d), 10 + s) for s in range(S)], rnd((d,), 3), rnd((d,), 4), rnd((d, taps), 5, 0.5)
    want = [oracle.with_past(oracle.layer_norm(npd(x), npd(w), npd(b), 1e-5), npd(taps_w)) for x in xs]
    slots = i32([4, 0, 2], dev)
    for portions in ([9], [2, 3, 4], [1] * 9, [4, 1, 1, 1, 2]):
        conv = stream.InputConv(taps_w.t().contiguous().to(dev), torch.full((5, taps - 1, d), 9.0, device=dev))      # what others have left
        at = 0
        for m in portions:
            x = torch.cat([x[at:at + m] for x in xs]).to(dev)
            qs, sl = varlen([m] * S, [at] * S, dev)
            kw = dict(w=w.to(dev), b=b.to(dev), eps=1e-5)
            if m == 1:
                _, h = stream.add_norm(x, act_dtype=dt, conv=conv, seq_lens=sl, slots=slots, **kw)
            else:
                _, norm = stream.add_norm(x, act_dtype=F32, padded=False, **kw)
                h = stream.stream_conv(norm, conv, qs, sl, slots, dt, padded=True)
            assert h.shape == (S * m, stream.pad8(d)) and not h[:, d:].any()
            for s in range(S):
                close(h[s * m:(s + 1) * m, :d], want[s][at:at + m], TOL[dt], (portions, at, s))
            at += m
        for unused in (1, 3):
            assert bool((conv.state[unused] == 9).all())


# ------------------------------------------------------------------ norms over a projection, rotation, cache write
#              heads kv dim vdim rot
PREP = {"even": (6, 2, 32, 64, 32), "128": (4, 2, 128, 128, 64), "narrower": (2, 1, 40, 72, 16), "none": (3, 1, 24, 40, 0), "odd": (6, 3, 13, 10, 6),
        "wide": (3, 3, 100, 256, 66), "beyond": (2, 1, 300, 30, 4), "many": (40, 2, 64, 64, 64)}
YARNS = {"plain": None, "stretched": gqa.Yarn(8.0, 300, 16.0, 0.5), "one": gqa.Yarn(1.0, 64, 4.0, 1.0), "short": gqa.Yarn(2.5, 9, 30.0, 20.0),
         "steep": gqa.Yarn(4.0, 4096, 2.0, 1.99)}


def rotation(rot, base, yarn):
    out = {"dims": rot, "base": base}
    return out if yarn is None else dict(out, scaling=dataclasses.asdict(yarn))


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("yarn", sorted(YARNS))
@pytest.mark.parametrize("name", sorted(PREP))
def test_whole_projection_norm_rotation_and_cache_write(target, name, yarn):
    dev, dt = target
    H, G, dk, dv, rot = PREP[name]
    s = gqa.GqaSpec(H, G, dk, dv, rot, base=3000.0, whole_norm=True, yarn=YARNS[yarn])
    pos, slots, t = [0, 1, 63, 64, 5000, 77], [130, 0, -1, 64, 65, 191], 6
    proj, qn, kn = rnd((t, s.columns() + 11), 1), rnd((H * dk,), 2), rnd((G * dk,), 3)
    proj[:, :dk] *= 3.0                                       # heads of different size: a norm per head would show
    x = npd(proj)
    turn = lambda v: v if rot == 0 else np.stack([oracle.turn(v[i], p, rotation(rot, 3000.0, YARNS[yarn])) for i, p in enumerate(pos)])
    q_want = turn((oracle.rms(x[:, :H * dk], 1e-3) * npd(qn)).reshape(t, H, dk))
    k_want = turn((oracle.rms(x[:, H * dk:(H + G) * dk], 1e-3) * npd(kn)).reshape(t, G, dk))
    tol = max(TOL[dt], 1e-3 if rot else 0)                    # fp32 angles of position 5000
    for split in (False, True):                               # sums of squares as several ranks add them up
        cache = s.alloc_cache(3, 64, dt, dev)
        for c in cache:
            c.fill_(7.0)
        p = proj.to(dev, dt)
        kw = dict(sumsq=3.0 * gqa.sums_of_squares(p, s), totals=(3 * H * dk, 3 * G * dk)) if split else {}
        q = gqa.prep(p, qn.to(dev), kn.to(dev), s.inv_freq(dev), i32(pos, dev), i32(slots, dev), cache, 1e-3, s, **kw)
        close(q[..., :dk], q_want, tol)
        kc, vc = (c.view(192, G, -1) for c in cache)
        ok = [i for i, r in enumerate(slots) if r >= 0]
        rows = [slots[i] for i in ok]
        close(kc[rows][..., :dk], k_want[ok], tol)
        close(vc[rows][..., :dv], x[:, (H + G) * dk:s.columns()].reshape(t, G, dv)[ok], TOL[dt])
        assert not kc[rows][..., dk:].any() and not vc[rows][..., dv:].any() and not q[..., dk:].any()
        rest = [r for r in range(192) if r not in rows]
        assert bool((kc[rest] == 7).all()) and bool((vc[rest] == 7).all())


@pytest.mark.parametrize("yarn", [y for y in sorted(YARNS) if y != "plain"])
@pytest.mark.parametrize("rot,base", [(64, 10000.0), (24, 500000.0), (2, 10.0), (128, 150.0)])
def test_stretched_frequencies(yarn, rot, base):
    s = gqa.GqaSpec(1, 1, 128, 8, rot, base=base, yarn=YARNS[yarn])
    f, amp = oracle.frequencies(rotation(rot, base, YARNS[yarn]))
    assert np.allclose(npd(s.inv_freq("cpu")), f, rtol=1e-6) and s.amplitude == pytest.approx(amp)


# ------------------------------------------------------------------ window and pooled blocks
#       heads kv dim vdim window pool cap
POOL = {
    "tensor cores": (4, 2, 128, 128, 70, 6, 20.0),
    "tensor cores, narrower": (6, 1, 88, 72, 100, 8, 40.0),
    "tensor cores, odd values": (2, 1, 90, 101, 64, 16, 20.0),
    "tensor cores, no cap": (4, 2, 128, 120, 33, 5, 0.0),
    "tensor cores, one token": (2, 1, 128, 128, 1, 1, 20.0),
    "tensor cores, page": (2, 2, 100, 128, 64, 64, 20.0),
    "tensor cores, many blocks": (2, 1, 128, 128, 5, 1, 20.0),
    "large cap": (4, 2, 128, 128, 70, 12, 90.0),
    "odd group": (3, 1, 128, 128, 50, 7, 20.0),
    "64": (8, 2, 64, 48, 90, 3, 20.0),
    "256": (2, 2, 200, 130, 40, 9, 20.0),
    "beyond a page": (4, 2, 40, 128, 30, 70, 20.0),
    "never": (2, 1, 64, 64, 100000, 4, 20.0),
    "odd": (6, 3, 13, 10, 29, 3, 20.0),
    "many heads": (18, 1, 16, 24, 60, 32, 20.0),
    "wide": (2, 1, 260, 30, 21, 10, 20.0),
}


def pool_spec(name):
    H, G, dk, dv, window, pool, cap = POOL[name]
    return gqa.GqaSpec(H, G, dk, dv, 0, scale=dk ** -0.5, window=window, pool=pool, cap=cap)


def pool_case(name, n, seed):
    """(spec, q, k, v) of one sequence.  Keys of a block are alike, so that each query can lean towards one block - the first, the last
    one that is seen, the next one, the blocks at the window's edge and at page borders, its own - and whatever of it is
    visible, single tokens or the mean, stands out."""
    s = pool_spec(name)
    H, G, dk, dv, w, P = s.heads, s.kv_heads, s.dim, s.vdim, s.window, s.pool
    base = rnd(((n + P) // P + 1, G, dk), seed)
    k = base[torch.arange(n) // P] + rnd((n, G, dk), seed + 1, 0.3)
    q, v = rnd((n, H, dk), seed + 2, 0.2), rnd((n, G, dv), seed + 3)
    block = lambda tok: tok // P
    places = [lambda i: 0, lambda i: block(i - w - P + 1), lambda i: block(i - w + 1), lambda i: block(i - w), lambda i: block(i), lambda i: block(i - w - P),
              lambda i: block(64), lambda i: block(63), lambda i: block(i // 2), lambda i: block(i // 64 * 64)]
    for i in range(n):
        b = places[i % len(places)](i)
        if 0 <= b <= i // P:
            for h in range(H):
                key = base[b, h // (H // G)]
                q[i, h] = key * (8.0 / s.scale / float(key @ key))
    return s, q.to(BF16).float(), k.to(BF16).float(), v


def pool_want(case, first=0):
    s, q, k, v = case
    cap = s.cap or 1e9
    return oracle.attend(npd(q)[first:], npd(k), npd(v), s.scale, cap, s.window, s.pool, first).reshape(len(q) - first, -1)


def run_pool(case, portions, dev, dt, extra_rows=0, scale=1.0, order_seed=9, cache=None, page=64):
    s, q, k, v = case
    n, G = q.shape[0], s.kv_heads
    pages = (n + page - 1) // page
    order = torch.randperm(pages + 2, generator=torch.Generator().manual_seed(order_seed))[:pages]
    if cache is None:
        cache = s.alloc_cache(pages + 2, page, dt, dev)
    rows = (order[torch.arange(n) // page] * page + torch.arange(n) % page).to(torch.int32).to(dev)
    bt = torch.zeros((1 + extra_rows, pages + 1), dtype=torch.int32, device=dev)
    bt[0, :pages] = order.to(dev, torch.int32)
    ones = torch.ones(8, device=dev)
    out, at = [], 0
    for m in portions:
        e = at + m
        proj = torch.cat([q[at:e].reshape(m, -1), k[at:e].reshape(m, -1), v[at:e].reshape(m, -1)], 1)
        proj = torch.cat([proj, torch.zeros((extra_rows, proj.shape[1]))], 0).to(dev, dt)
        slots = torch.cat([rows[at:e], torch.full((extra_rows,), -1, dtype=torch.int32, device=dev)])
        pos = i32(list(range(at, e)) + [0] * extra_rows, dev)
        step = m == 1
        qq = gqa.prep(proj, None, None, ones, pos, slots, cache, 1e-5, s, step_table=bt if step else None)
        qs, sl = varlen([m] + [1] * extra_rows, [at] + [-1] * extra_rows, dev)
        meta = SimpleNamespace(is_prefill=not step, q_start=qs, seq_lens=sl, block_table=bt, positions=pos, total_q_blocks=(m + 63) // 64 + extra_rows,
                               num_splits=ops.decode_plan_splits(1, G, s.visible(n)) if dev == "cuda" else None, max_seq_len=n)
        if not step:
            gqa.pool_new(cache, meta, s)
        width = s.heads * s.vdim
        wide = torch.full((m + extra_rows, width + 24), 5.0, dtype=dt, device=dev)
        got = gqa.attention(qq, None, cache, meta, s, out=wide[:, :width] if scale != 1.0 else None, out_scale=scale)
        assert scale == 1.0 or bool((wide[:, width:] == 5).all())
        out.append(got[:m])
        at = e
    return torch.cat(out)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", sorted(POOL))
def test_window_and_pooled_blocks_in_prompts_portions_and_decoding(target, name):
    dev, dt = target
    n = 300
    case = pool_case(name, n, 11)
    want = pool_want(case)
    for i, portions in enumerate(([n], [130] + [1] * 40 + [2, 128], [1] * 70 + [2, 3, 64, 5, 156])):
        scale = (1.0, 0.7, 0.0)[i]                            # with a scale: into a wider buffer
        got = npd(run_pool(case, portions, dev, dt, scale=scale))
        err = np.abs(got - scale * want).max(-1)
        assert err.max() < (3e-4 if dt == F32 else 9e-2), (portions[:3], err.max(), int(err.argmax()))


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", sorted(POOL))
def test_exactly_the_tokens_and_blocks_in_sight_count(target, name):
    """Flat scores: the mean of the visible values, in which a token or block too many or too few shows.  A window in the
    middle of blocks and pages, portions that start and end inside blocks, decoding over several edges."""
    dev, dt = target
    s = pool_spec(name)
    n = 230
    v = rnd((n, s.kv_heads, s.vdim), 5)
    case = (s, torch.zeros((n, s.heads, s.dim)), rnd((n, s.kv_heads, s.dim), 6), v)
    seen = [oracle.visible_rows(npd(v), npd(v), i, s.window, s.pool)[1] for i in range(n)]
    want = np.stack([np.repeat(x.mean(0), s.heads // s.kv_heads, 0).reshape(-1) for x in seen])
    for portions in ([n], [57, 2, 71, 3, 97], [101] + [1] * 129):
        got = npd(run_pool(case, portions, dev, dt))
        err = np.abs(got - want).max(-1) * np.sqrt([len(x) for x in seen])          # in units of one token's share
        assert err.max() < (1e-4 if dt == F32 else 8e-2), (portions[:2], err.max(), int(err.argmax()))


@pytest.mark.gpu
@pytest.mark.parametrize("name", ["tensor cores", "tensor cores, many blocks", "64", "256", "beyond a page"])
@pytest.mark.parametrize("window", [700, 1, 33])
def test_decoding_far_into_a_sequence_in_several_key_chunks(name, window):
    """A padding row in the batch; blocks over many pages; more chunks than the window alone would need."""
    case = pool_case(name, 1500, 21)
    case = (dataclasses.replace(case[0], window=window),) + case[1:]
    first = 1490
    got = npd(run_pool(case, [first] + [1] * 10, "cuda", BF16, extra_rows=1))[first:]
    assert np.abs(got - pool_want(case, first)).max() < 9e-2


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("page", [16, 48])
def test_other_page_sizes(target, page):
    dev, dt = target
    for name in ("64", "odd"):
        case = pool_case(name, 150, 31)
        got = npd(run_pool(case, [90] + [1] * 30 + [30], dev, dt, page=page))
        assert np.abs(got - pool_want(case)).max() < (3e-4 if dt == F32 else 9e-2)


@pytest.mark.parametrize("target", TARGETS)
def test_pages_of_another_sequence_are_overwritten(target):
    """A second sequence in the same pages, in another order: blocks of the first one must not be seen."""
    dev, dt = target
    for name in ("tensor cores", "odd"):
        a, b = pool_case(name, 200, 41), pool_case(name, 200, 51)
        cache = a[0].alloc_cache(6, 64, dt, dev)
        run_pool(a, [200], dev, dt, cache=cache)
        got = npd(run_pool(b, [65, 1, 1, 60, 73], dev, dt, cache=cache, order_seed=3))
        assert np.abs(got - pool_want(b)).max() < (3e-4 if dt == F32 else 9e-2)


@pytest.mark.parametrize("target", TARGETS)
def test_sequences_of_one_batch_see_their_own_blocks(target):
    """Unequal portions side by side, some of which complete no block."""
    dev, dt = target
    s = pool_spec("64")
    cases = [pool_case("64", n, 60 + n) for n in (150, 200, 131)]
    page, cache, bts, starts = 64, s.alloc_cache(12, 64, dt, dev), torch.arange(12, dtype=torch.int32).reshape(3, 4).to(dev), [0, 0, 0]
    got = [[], [], []]
    for counts in ((100, 2, 130), (2, 150, 1), (48, 48, 0)):
        live = [i for i in range(3) if counts[i]]
        proj = torch.cat([torch.cat([x[starts[i]:starts[i] + counts[i]].reshape(counts[i], -1) for x in cases[i][1:]], 1) for i in live]).to(dev, dt)
        pos = [p for i in live for p in range(starts[i], starts[i] + counts[i])]
        slots = [int(bts[i, p // page]) * page + p % page for i in live for p in range(starts[i], starts[i] + counts[i])]
        qq = gqa.prep(proj, None, None, torch.ones(8, device=dev), i32(pos, dev), i32(slots, dev), cache, 1e-5, s)
        qs, sl = varlen([counts[i] for i in live], [starts[i] for i in live], dev)
        meta = SimpleNamespace(is_prefill=True, q_start=qs, seq_lens=sl, block_table=bts[live].contiguous(), positions=i32(pos, dev),
                               total_q_blocks=sum((counts[i] + 63) // 64 for i in live), num_splits=None, max_seq_len=None)
        gqa.pool_new(cache, meta, s)
        out, at = gqa.attention(qq, None, cache, meta, s), 0
        for i in live:
            got[i].append(out[at:at + counts[i]])
            at += counts[i]
            starts[i] += counts[i]
    for i, case in enumerate(cases):
        assert np.abs(npd(torch.cat(got[i])) - pool_want(case)).max() < (3e-4 if dt == F32 else 9e-2), i


@pytest.mark.parametrize("pool,page", [(1, 64), (3, 64), (60, 64), (64, 64), (70, 64), (200, 64), (7, 16), (16, 16)])
def test_every_block_has_a_row_of_its_own(pool, page):
    rows, seen = gqa.pool_rows(pool, page), set()
    for b in range(400):
        at, row = gqa.pool_row(b, pool, page)
        assert 0 <= row < rows and at == (b * pool + pool - 1) // page and (at, row) not in seen
        seen.add((at, row))


def test_options_that_exclude_each_other():
    for kw in (dict(pool=4), dict(pool=4, window=8, keep=2), dict(pool=4, chunk=8), dict(pool=-1, window=8), dict(whole_norm=True, maps=2),
               dict(pool=2, window=8, maps=2)):
        with pytest.raises(ValueError):
            gqa.GqaSpec(2, 1, 8, 8, 0, **kw)


# ------------------------------------------------------------------ gated recurrence
def scan_case(n, width, seed):
    """Gates from shut to open, candidates on both sides of zero; states that must survive hundreds of tokens."""
    z, x, g, zb, xb = rnd((n, width), seed, 2.0) - 1.0, rnd((n, width), seed + 1), rnd((n, width), seed + 2), rnd((width,), seed + 3), rnd((width,), seed + 4)
    z[:, ::5] -= 6.0
    z[n // 2, ::7] = 120.0                                    # a gate fully open forgets everything,
    z[:, 1::9] = -120.0                                       # one fully shut takes nothing
    z[0, 1::9] = 0.0
    x[:, 2::11] = -xb[2::11]                                  # u = 0
    return [t.to(BF16).float() for t in (z, x, g, zb, xb)]


def scan_want(case, scale):
    z, x, g, zb, xb = (npd(t) for t in case)
    gate = 1.0 / (1.0 + np.exp(np.clip(-(z + zb), -700, 700)))
    return oracle.recur(gate, x + xb) * oracle.silu(g) * scale


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("width", [1, 37, 96, 300, 1026])
def test_gated_recurrence_in_prompts_portions_and_decoding(target, width):
    dev, dt = target
    n = 300
    case = scan_case(n, width, 5)
    want = scan_want(case, 1.3)
    for lead in (0, 3):                                       # columns in front: odd offsets take the narrow accesses
        for portions in ([n], [64, 64, 2, 62, 1, 107], [1] * 66 + [2, 65, 167], [63, 65, 1, 128, 43]):
            state, at, out = torch.full((4, width), 50.0, device=dev), 0, []
            for m in portions:
                proj = torch.cat([torch.zeros((m, lead))] + [c[at:at + m] for c in case[:3]], 1).to(dev, dt)
                z, x, g = (proj[:, lead + i * width:lead + (i + 1) * width] for i in range(3))
                wide = torch.full((m, width + 9), 5.0, dtype=dt, device=dev)
                qs, sl = varlen([m], [at], dev)
                la.gated_scan(z, x, g, case[3].to(dev), case[4].to(dev), state, qs, sl, i32([2], dev), 1.3, wide[:, lead:lead + width], decode=m == 1)
                out.append(wide[:, lead:lead + width])
                assert bool((wide[:, :lead] == 5).all()) and bool((wide[:, lead + width:] == 5).all())
                at += m
            close(torch.cat(out), want, TOL[dt], (width, portions[:3]))
            assert bool((state[[0, 1, 3]] == 50).all())


@pytest.mark.parametrize("target", TARGETS)
def test_gated_recurrence_of_unequal_sequences_in_one_batch(target):
    """Blocks of several sequences in one launch; slots used again start from zero."""
    dev, dt = target
    width, lens = 130, (200, 1, 64, 65, 130)
    cases = [scan_case(n, width, 20 + n) for n in lens]
    state = torch.full((8, width), 30.0, device=dev)
    for slots in ([5, 1, 0, 3, 7], [1, 5, 7, 0, 3]):
        first = [n // 3 for n in lens]
        got = [[] for _ in lens]
        for a, b in (([0] * 5, first), (first, lens)):
            live = [i for i in range(5) if b[i] > a[i]]
            cat = [torch.cat([cases[i][c][a[i]:b[i]] for i in live]).to(dev, dt) for c in range(3)]
            proj = torch.cat(cat, 1)
            qs, sl = varlen([b[i] - a[i] for i in live], [a[i] for i in live], dev)
            zb, xb = cases[0][3].to(dev), cases[0][4].to(dev)
            out, at = la.gated_scan(*(proj[:, c * width:(c + 1) * width] for c in range(3)), zb, xb, state, qs, sl, i32([slots[i] for i in live], dev)), 0
            for i in live:
                got[i].append(out[at:at + b[i] - a[i]])
                at += b[i] - a[i]
        for i, c in enumerate(cases):
            close(torch.cat(got[i]), scan_want(c[:3] + cases[0][3:], 1.0), TOL[dt], i)


@pytest.mark.parametrize("target", TARGETS)
def test_state_of_a_long_prompt(target):
    """Seventy blocks, gates that keep nearly everything: the first token is still there at the end."""
    dev, _ = target
    n, width = 4400, 8
    z, x, g = torch.full((n, width), -9.0), torch.full((n, width), -60.0), torch.full((n, width), 1.0)
    z[0], x[0] = 100.0, 7.5                                   # the state is 8 behind the first token, then fades towards 0
    state = torch.zeros((1, width), device=dev)
    zero = torch.zeros(width, device=dev)
    qs, sl = varlen([n], [0], dev)
    proj = torch.cat([z, x, g], 1).to(dev)
    la.gated_scan(*(proj[:, c * width:(c + 1) * width] for c in range(3)), zero, zero, state, qs, sl, i32([0], dev))
    gate = 1 / (1 + np.exp(9.0))
    want = 8.0 * (1 - gate) ** (n - 1)
    assert want > 4 and np.allclose(npd(state), want, rtol=1e-3)          # fp32 rounds the same factor 4400 times


# ------------------------------------------------------------------ mixture
@pytest.mark.parametrize("target", TARGETS[:2])
@pytest.mark.parametrize("experts,top,shared,e0,scale", [(1, 1, 1, 0, 1.0), (5, 2, 0, 0, 0.3), (16, 3, 2, 8, 2.5), (33, 32, 1, 11, 1.0), (200, 8, 3, 100, 1.5)])
def test_routing_by_sigmoid_scores(target, experts, top, shared, e0, scale):
    """Choice by score plus correction, weights by score alone and not divided by their sum, shared experts with weight one."""
    dev, _ = target
    t = 37
    z, corr = rnd((t, experts), 1, 2.0), rnd((experts,), 2, 0.3)
    ids, w = moe_ops.route(z.to(dev), top, experts, corr.to(dev), shared, e0, scores="sigmoid", normalize=False, scale=scale, shared_gate=False)
    assert ids.dtype == torch.int32 and ids.shape == w.shape == (t, top + shared)
    flips = 0
    for i in range(t):
        pick, want = oracle.choose(npd(z)[i], npd(corr), top, scale)
        flips += set(pick) != set(np.argsort(-npd(z)[i])[:top])
        got = {int(e): float(x) for e, x in zip(ids[i, :top], w[i, :top])}
        assert got.keys() == {shared + (int(e) - e0) % experts for e in pick}
        for e, x in zip(pick, want):
            assert abs(got[shared + (int(e) - e0) % experts] - x) < 1e-5
        assert ids[i, top:].tolist() == list(range(shared)) and bool((w[i, top:] == 1).all())
    assert flips > 0 or top >= experts - 1                    # the correction changed somebody's choice


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("t,d,ff,shared", [(3, 40, 24, 70), (70, 128, 64, 300), (700, 96, 130, 40)])
def test_experts_with_squared_units_and_a_shared_one_in_pieces(target, t, d, ff, shared):
    """Few and many rows per expert (both orientations of the grouped GEMM); the shared expert smaller and larger than a routed
    one."""
    dev, dt = target
    e, top = 4, 2
    x, up, down = rnd((t, d), 1), rnd((e, ff, d), 2, d ** -0.5), rnd((e, d, ff), 3, ff ** -0.5)
    su, sd = rnd((shared, d), 4, d ** -0.5), rnd((d, shared), 5, shared ** -0.5)
    ids = torch.stack([torch.randperm(e, generator=torch.Generator().manual_seed(i))[:top] for i in range(t)])
    w1, w2 = moe_ops.pad_plain_experts(up.to(dev, dt), down.to(dev, dt))
    s1, s2 = moe_ops.pad_plain_experts(*moe_ops.shared_pieces(su.to(dev, dt), sd.to(dev, dt), w1.shape[1]))
    n = s1.shape[0]
    assert n == -(-shared // w1.shape[1])
    all_ids = torch.cat([ids + n, torch.arange(n).expand(t, n)], 1).to(torch.int32).contiguous()
    rows, pos = moe_ops.expert_rows(x.to(dev, dt), all_ids.to(dev), torch.cat([s1, w1]), torch.cat([s2, w2]), 0, e + n, "relu2")
    got = npd(rows)[pos.cpu().long().numpy()][:, :d].reshape(t, top + n, d)
    want = np.stack([[oracle.expert(npd(x)[i], npd(up)[k], npd(down)[k]) for k in ids[i].tolist()] for i in range(t)])
    close(torch.tensor(got[:, :top]), want, TOL[dt])
    close(torch.tensor(got[:, top:].sum(1)), oracle.expert(npd(x), npd(su), npd(sd)), TOL[dt])
