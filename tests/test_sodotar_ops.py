"""The mechanisms of Sodotar one by one against the plain functions of `sodotar_oracle`, with inputs that make a wrong key, a
chunk's edge, a missing sink or a wrong map stand out."""
import os
import sys
from types import SimpleNamespace

import numpy as np
import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import sodotar_oracle as oracle  # noqa: E402
from zml_b200 import ops  # noqa: E402
from zml_b200.moe import ops as moe_ops  # noqa: E402
from zml_b200.ops import gqa, stream  # noqa: E402
from zml_b200.ops import latent as lat  # noqa: E402

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
    return i32(qs, dev), i32([n + p for n, p in zip(counts, past)], dev), qs, [n + p for n, p in zip(counts, past)]


# ------------------------------------------------------------------ hyper-connections
def hyper_mix(s, seed, dev):
    inp, mix, out = rnd((s,), seed), rnd((s, s), seed + 1), rnd((s,), seed + 2)
    return stream.HyperMix(inp.to(dev), mix.to(dev), out.to(dev)), npd(inp), npd(mix), npd(out)


@pytest.mark.parametrize("target", TARGETS)
def test_embedding_fills_every_stream(target):
    dev, dt = target
    table, ids = rnd((30, 51), 1), [3, 0, 29, 3]
    x = stream.embedding_f32(i32(ids, dev), table.to(dev, dt), streams=3)
    assert x.shape == (4, 3, 51) and x.dtype == F32
    close(x, np.repeat(npd(table)[ids][:, None], 3, 1), 1e-6)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("s,d", [(1, 8), (2, 51), (3, 260), (4, 1028), (5, 2048), (4, 4100), (8, 4096), (2, 3001), (3, 9000)])
def test_streams_update_and_next_norm(target, s, d):
    """mix is indexed from, to; all streams are written from the old ones; y in both types; no next norm; no sublayer."""
    dev, dt = target
    t = 3
    x, y, w = rnd((t, s, d), 1), rnd((t, d), 2, 2.0), rnd((d,), 3)
    behind, _, mix, out = hyper_mix(s, 10, dev)
    nxt, inp, _, _ = hyper_mix(s, 20, dev)
    want = np.einsum("ab,tad->tbd", mix, npd(x)) + out[None, :, None] * npd(y)[:, None]
    act_want = oracle.rms_norm(np.einsum("a,tad->td", inp, want), npd(w), 1e-2)
    for yy in (y.to(dev), y.to(dev, dt)):
        new, act = stream.hyper_norm(x.to(dev).clone(), yy, behind, nxt.inp, w.to(dev), 1e-2, act_dtype=dt)
        close(new, want, 2e-5)
        close(act[:, :d], act_want, TOL[dt])
        assert act.shape[1] % 8 == 0 and not act[:, d:].any()
    new, act = stream.hyper_norm(x.to(dev).clone(), y.to(dev), behind, eps=1e-2)
    assert act is None
    close(new, want, 2e-5)
    keep = x.to(dev).clone()
    _, act = stream.hyper_norm(keep, inp=nxt.inp, w=w.to(dev), eps=1e-2, act_dtype=dt)
    close(act[:, :d], oracle.rms_norm(np.einsum("a,tad->td", inp, npd(x)), npd(w), 1e-2), TOL[dt])
    assert torch.equal(keep.cpu(), x)
    small = 1e-3 * x                                         # eps counts
    _, act = stream.hyper_norm(small.to(dev), inp=nxt.inp, w=w.to(dev), eps=1e-6, act_dtype=dt)
    close(act[:, :d], oracle.rms_norm(np.einsum("a,tad->td", inp, npd(small)), npd(w), 1e-6), TOL[dt])


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("d,k", [(51, 3), (256, 1), (2048, 9), (1028, 40)])
def test_streams_take_summed_expert_rows(target, d, k):
    """Rows wider than the stream, pairs without a row, more pairs than one pass takes."""
    dev, dt = target
    t, s = 5, 3
    rows, weights = rnd((t * k + 3, (d + 127) // 128 * 128), 1), torch.rand((t, k), generator=torch.Generator().manual_seed(2))
    pos = torch.randperm(t * k + 3, generator=torch.Generator().manual_seed(3))[:t * k].to(torch.int32)
    pos[1::4] = -1
    x, w = rnd((t, s, d), 4), rnd((d,), 5)
    behind, _, mix, out = hyper_mix(s, 10, dev)
    nxt, inp, _, _ = hyper_mix(s, 20, dev)
    y = np.zeros((t, d))
    for i in range(t * k):
        if pos[i] >= 0:
            y[i // k] += float(weights[i // k, i % k]) * npd(rows[pos[i]])[:d]
    new, act = stream.hyper_norm(x.to(dev).clone(), stream.ExpertRows(rows.to(dev, dt), pos.to(dev), weights.to(dev)), behind, nxt.inp, w.to(dev), 1e-5,
                                 act_dtype=dt)
    want = np.einsum("ab,tad->tbd", mix, npd(x)) + out[None, :, None] * y[:, None]
    close(new, want, 2e-5)
    close(act[:, :d], oracle.rms_norm(np.einsum("a,tad->td", inp, want), npd(w), 1e-5), TOL[dt])


# ------------------------------------------------------------------ latent attention
#          heads dim rot vdim rank
LATENT = {"small": (3, 24, 8, 20, 40), "ones": (1, 8, 2, 8, 8), "odd": (5, 13, 6, 11, 21), "real": (4, 128, 64, 128, 512), "many heads": (33, 40, 16, 72, 96),
          "wide": (2, 192, 64, 104, 200)}


def latent_dims(name, scale=None, base=3000.0):
    H, dim, rot, vdim, rank = LATENT[name]
    return lat.LatentDims(H, dim, rot, vdim, rank, 0, 0, (dim + rot) ** -0.5 if scale is None else scale, base)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", sorted(LATENT))
def test_latent_norm_rotation_and_cache_write_without_a_query_latent(target, name):
    """The shared key part rotated in halves, its rows permuted into neighbouring pairs as at load."""
    dev, dt = target
    d = latent_dims(name)
    pos, slots = [0, 1, 63, 64, 5000, 77], [130, 0, -1, 64, 65, 191]
    raw, norm = rnd((len(pos), d.rank + d.rot), 1), rnd((d.rank,), 2)
    pairs = lat.halves_to_pairs(d.rot)
    proj = torch.cat([rnd((len(pos), 16), 3), raw[:, :d.rank], raw[:, d.rank:][:, pairs]], 1).to(dev, dt)
    cache = torch.full((3, 64, d.row), 7.0, dtype=dt, device=dev)
    assert lat.prep(proj[:, 16:], None, norm.to(dev), d.inv_freq(dev), i32(pos, dev), i32(slots, dev), cache, 1e-3, d) is None
    ok = [i for i, r in enumerate(slots) if r >= 0]
    rows = cache.view(192, -1)[[slots[i] for i in ok]]
    turned = np.stack([oracle.turn_halves(npd(raw)[i, d.rank:], pos[i], d.rot, d.base) for i in ok])
    close(rows[:, :d.rank], oracle.rms_norm(npd(raw)[ok, :d.rank], npd(norm), 1e-3), TOL[dt])
    close(rows[:, d.rot_off:d.rot_off + d.rot], turned[:, pairs.numpy()], max(TOL[dt], 1e-3))          # fp32 angles of position 5000
    rest = [r for r in range(192) if r not in slots]
    assert bool((cache.view(192, -1)[rest] == 7).all())


def latent_case(name, n, seed):
    """(dims, q, c, shared, uk, uv, sink) of one sequence; q and shared unrotated, in the layout of neighbouring pairs.  Scores are
    moderate apart from those of single keys far back, at page borders, the first and the last ones, which stand out."""
    d = latent_dims(name)
    H, hd = d.heads, d.dim + d.rot
    q, c, shared = rnd((n, H, hd), seed, 0.2), rnd((n, d.rank), seed + 1), rnd((n, d.rot), seed + 2, 0.1)
    uk, uv = rnd((H * d.dim, d.rank), seed + 3, d.rank ** -0.5), rnd((H * d.vdim, d.rank), seed + 4, d.rank ** -0.5)
    sink = rnd((H,), seed + 5) + 1.0
    key = (c @ uk.t()).reshape(n, H, d.dim)
    places = [lambda i: 0, lambda i: i, lambda i: 64, lambda i: 63, lambda i: i // 2, lambda i: 1, lambda i: i - 1, lambda i: 127, lambda i: 128]
    for i in range(n):
        j = places[i % len(places)](i)
        if 0 <= j <= i:
            for h in range(H):
                q[i, h, :d.dim] = key[j, h] * (8.0 / d.scale / float(key[j, h] @ key[j, h]))
    return d, q.to(BF16).float(), c, shared, uk, uv, sink.to(BF16).float()


def latent_want(case, first=0):
    d, q, c, shared, uk, uv, sink = case
    back = np.argsort(lat.halves_to_pairs(d.rot).numpy())
    qn, sn = npd(q)[first:], npd(shared)[:, back]
    q2 = np.concatenate([qn[..., :d.dim], oracle.turn_all(qn[..., d.dim:][..., back], d.rot, d.base, first)], -1)
    k, v = oracle.latent_keys_values(oracle.rms(npd(c), 1e-6), oracle.turn_all(sn, d.rot, d.base), npd(uk), npd(uv), d.heads)
    return oracle.latent_attend(q2, k, v, d.scale, npd(sink), first).reshape(len(qn), -1)


def run_latent(case, portions, dev, dt, extra_rows=0):
    d, q, c, shared, uk, uv, sink = case
    n, page = q.shape[0], 64
    pages = (n + page - 1) // page
    order = torch.randperm(pages + 2, generator=torch.Generator().manual_seed(9))[:pages]
    cache = torch.zeros((pages + 2, page, d.row), dtype=dt, device=dev)
    rows = (order[torch.arange(n) // page] * page + torch.arange(n) % page).to(torch.int32).to(dev)
    bt = torch.zeros((1 + extra_rows, pages + 1), dtype=torch.int32, device=dev)
    bt[0, :pages] = order.to(dev, torch.int32)
    uk_t = uk.reshape(d.heads, d.dim, d.rank).transpose(1, 2).contiguous().to(dev, dt)
    ukv, inv = torch.cat([uk, uv], 0).to(dev, dt), d.inv_freq(dev)
    ones = torch.ones(d.rank, device=dev)
    out, at = [], 0
    for m in portions:
        e = at + m
        lat.prep(torch.cat([c[at:e], shared[at:e]], 1).to(dev, dt), None, ones, inv, i32(list(range(at, e)), dev), rows[at:e], cache, 1e-6, d)
        ld = (d.heads * (d.dim + d.rot) + 7) // 8 * 8
        qq = torch.zeros((m + extra_rows, ld), dtype=dt, device=dev)
        qq[:m, :d.heads * (d.dim + d.rot)] = q[at:e].reshape(m, -1).to(dev, dt)
        qs, sl, qh, sh = varlen([m] + [1] * extra_rows, [at] + [-1] * extra_rows, dev)
        pos = i32(list(range(at, e)) + [0] * extra_rows, dev)
        meta = SimpleNamespace(is_prefill=m > 1, q_start=qs, seq_lens=sl, block_table=bt, positions=pos, q_start_host=qh, seq_lens_host=sh, plans={},
                               num_splits=lat.decode_plan_splits(1, d, n) if dev == "cuda" else None, max_seq_len=n)
        out.append(lat.latent_attention(qq[:, :d.heads * (d.dim + d.rot)], None, uk_t, ukv, inv, cache, meta, d, sink.to(dev))[:m])
        at = e
    return torch.cat(out)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", sorted(LATENT))
def test_latent_attention_with_sinks_in_prompts_portions_and_decoding(target, name):
    dev, dt = target
    n = 200
    case = latent_case(name, n, 31)
    want = latent_want(case)
    for portions in ([n], [130] + [1] * 40 + [2, 28], [1] * 70 + [2, 3, 64, 5, 56]):
        got = npd(run_latent(case, portions, dev, dt))
        err = np.abs(got - want).max(-1)
        assert err.max() < (2e-4 if dt == F32 else 8e-2), (portions[:3], err.max(), int(err.argmax()))


@pytest.mark.gpu
@pytest.mark.parametrize("name", ["small", "real", "many heads"])
def test_latent_decoding_far_into_a_sequence_counts_the_sink_once(name):
    """Several key chunks per sequence, a padding row in the batch, sinks as large as the largest scores."""
    n, first = 1500, 1490
    case = latent_case(name, n, 41)
    case = case[:6] + (case[6] + 6.0,)
    want = latent_want(case, first)
    got = npd(run_latent(case, [first] + [1] * 10, "cuda", BF16, extra_rows=1))[first:]
    assert np.abs(got - want).max() < 8e-2


@pytest.mark.parametrize("target", TARGETS)
def test_sink_of_a_sequence_of_one_token(target):
    """The only key competes with the sink, which is not scaled."""
    dev, dt = target
    d = lat.LatentDims(2, 8, 2, 8, 8, 0, 0, 0.25, 100.0)
    c = torch.zeros((1, 8))
    c[0, 0] = 8 ** 0.5                                        # unit root mean square
    uk, uv = torch.zeros((16, 8)), rnd((16, 8), 1)
    uk[0, 0] = uk[8, 0] = 1.0
    q = torch.zeros((1, 2, 10))
    q[0, :, 0] = 4.0
    for sinks in ((0.0, 3.0), (-2.0, 9.0)):
        got = npd(run_latent((d, q, c, torch.zeros((1, 2)), uk, uv, torch.tensor(sinks)), [1], dev, dt))[0].reshape(2, 8)
        v = 8 ** 0.5 * npd(uv)[:, 0].reshape(2, 8)
        e = np.exp(4.0 * 8 ** 0.5 * 0.25)
        close(torch.tensor(got), v * np.array([[e / (e + np.exp(x))] for x in sinks]), TOL[dt])


# ------------------------------------------------------------------ differential attention
#              heads kv dim vdim rot
PREP = {"even": (6, 2, 32, 64, 32), "tensor cores": (4, 2, 64, 128, 32), "narrower": (2, 1, 40, 72, 16), "none": (3, 1, 24, 40, 0), "odd": (6, 3, 13, 10, 6),
        "wide": (3, 3, 100, 256, 66), "beyond": (2, 1, 140, 30, 4)}


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("queries_only", [False, True])
@pytest.mark.parametrize("name", sorted(PREP))
def test_maps_rotation_and_cache_write(target, name, queries_only):
    dev, dt = target
    H, G, dk, dv, rot = PREP[name]
    s = gqa.GqaSpec(H, G, dk, dv, rot, base=3000.0, maps=2)
    pos, slots = [0, 1, 63, 64, 5000, 77], [130, 0, -1, 64, 65, 191]
    n = 2 * H * dk if queries_only else s.columns()
    proj = rnd((len(pos), n + 11), 1)
    cache = s.alloc_cache(3, 64, dt, dev)
    for c in cache:
        c.fill_(7.0)
    q = gqa.prep(proj.to(dev, dt), None, None, s.inv_freq(dev), i32(pos, dev), i32(slots, dev), cache, 1e-3, s, queries_only)
    x = npd(proj)
    turn = lambda v: np.stack([oracle.turn_halves(v[t], p, rot, 3000.0) for t, p in enumerate(pos)])
    tol = max(TOL[dt], 1e-3 if name != "none" else 0)         # fp32 angles of position 5000
    half = q.shape[-1] // 2
    want = turn(x[:, :2 * H * dk].reshape(-1, H, 2, dk))
    qv = q.reshape(len(pos), H, 2, 2, half)
    for i in (0, 1):
        close(qv[:, :, i, i, :dk], want[:, :, i], tol)
        assert not qv[:, :, i, 1 - i].any() and not qv[:, :, i, i, dk:].any()
    kc, vc = (c.view(192, G, -1) for c in cache)
    ok = [i for i, r in enumerate(slots) if r >= 0 and not queries_only]
    rows = [slots[i] for i in ok]
    if not queries_only:
        keys = turn(x[:, 2 * H * dk:2 * (H + G) * dk].reshape(-1, G, 2, dk))[ok]
        kv = kc[rows].reshape(len(rows), G, 2, -1)
        close(kv[..., :dk], keys, tol)
        close(vc[rows][..., :dv], x[:, 2 * (H + G) * dk:n].reshape(-1, G, dv)[ok], TOL[dt])
        assert not kv[..., dk:].any() and not vc[rows][..., dv:].any()
    rest = [r for r in range(192) if r not in rows]
    assert bool((kc[rest] == 7).all()) and bool((vc[rest] == 7).all())


#                          heads kv dim vdim chunk lambda diff
DIFF = {
    "small": (4, 2, 12, 20, 33, 0.4, 0.4),
    "tensor cores": (4, 2, 64, 128, 100, 0.3, 0.6),
    "tensor cores, pages": (4, 1, 64, 128, 128, 0.8, 0.2),
    "tensor cores, narrower": (2, 1, 50, 104, 70, -0.5, 0.5),
    "tensor cores, odd values": (2, 2, 64, 101, 64, 1.4, 0.1),
    "tensor cores, all": (6, 2, 64, 128, 100000, 0.5, 0.0),
    "64": (3, 3, 32, 64, 64, 0.45, 0.3),
    "64, eight": (8, 1, 24, 48, 90, 0.2, 0.9),
    "256": (2, 2, 100, 200, 130, 0.5, 0.3),
    "one token": (2, 2, 20, 40, 1, 0.5, 0.5),
    "two tokens": (2, 1, 64, 128, 2, 0.5, 0.5),
    "odd": (6, 3, 13, 10, 29, 0.7, 0.3),
    "many rows": (10, 1, 16, 24, 60, 0.4, 0.2),
    "beyond": (2, 1, 140, 30, 60, 0.6, 0.1),
}


def diff_case(name, n, seed):
    """(spec, mix, q, k, v) of one sequence.  Scores are small apart from those of single keys of one map, which stand out: the
    chunk's first key, the last one of the chunk before, page borders, the position itself, the sequence's first."""
    H, G, dk, dv, chunk, lam, diff = DIFF[name]
    s = gqa.GqaSpec(H, G, dk, dv, 0, scale=dk ** -0.5, chunk=chunk, maps=2)
    q, k, v = rnd((n, H, 2, dk), seed), rnd((n, G, 2, dk), seed + 1, 0.3), rnd((n, G, dv), seed + 2)
    places = [lambda i: i // chunk * chunk, lambda i: i // chunk * chunk - 1, lambda i: i, lambda i: 64, lambda i: 63, lambda i: 0, lambda i: i - 1,
              lambda i: i // 64 * 64, lambda i: i // chunk * chunk - 40]
    for i in range(n):
        j, a = places[i % len(places)](i), (i // len(places)) % 2
        if 0 <= j <= i:
            for h in range(H):                             # one map leans towards key j of its group: a score of about 9
                key = k[j, h // (H // G), a]
                q[i, h, a] = key * (9.0 / s.scale / float(key @ key))
    return s, gqa.DiffMix(lam, 1.0 - diff, 1e-5), q.to(BF16).float(), k.to(BF16).float(), v


def diff_want(case, first=0):
    s, mix, q, k, v = case
    q, k, v = npd(q)[first:], npd(k), npd(v)
    a1, a2 = (oracle.chunked_attend(q[:, :, i], k[:, :, i], v, s.scale, s.chunk, first) for i in (0, 1))
    return oracle.combine_maps(a1, a2, mix.lam, 1.0 - mix.scale, mix.eps).reshape(len(q), -1)


def run_diff(case, portions, dev, dt, extra_rows=0):
    s, mix, q, k, v = case
    n, G, page = q.shape[0], s.kv_heads, 64
    pages = (n + page - 1) // page
    order = torch.randperm(pages + 2, generator=torch.Generator().manual_seed(9))[:pages]
    cache = s.alloc_cache(pages + 2, page, dt, dev)
    rows = (order[torch.arange(n) // page] * page + torch.arange(n) % page).to(torch.int32).to(dev)
    bt = torch.zeros((1 + extra_rows, pages + 1), dtype=torch.int32, device=dev)
    bt[0, :pages] = order.to(dev, torch.int32)
    out, at = [], 0
    for m in portions:
        e = at + m
        proj = torch.cat([q[at:e].reshape(m, -1), k[at:e].reshape(m, -1), v[at:e].reshape(m, -1)], 1)
        proj = torch.cat([proj, torch.zeros((extra_rows, proj.shape[1]))], 0).to(dev, dt)
        slots = torch.cat([rows[at:e], torch.full((extra_rows,), -1, dtype=torch.int32, device=dev)])
        qq = gqa.prep(proj, None, None, s.inv_freq(dev), i32(list(range(at, e)) + [0] * extra_rows, dev), slots, cache, 1e-5, s)
        qs, sl, _, _ = varlen([m] + [1] * extra_rows, [at] + [-1] * extra_rows, dev)
        meta = SimpleNamespace(is_prefill=m > 1, q_start=qs, seq_lens=sl, block_table=bt, total_q_blocks=(m + 63) // 64 + extra_rows,
                               num_splits=ops.decode_plan_splits(1, G, s.visible(n)) if dev == "cuda" else None, max_seq_len=n)
        out.append(gqa.attention(qq, None, cache, meta, s, mix)[:m])
        at = e
    return torch.cat(out)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", sorted(DIFF))
def test_differential_attention_in_prompts_portions_and_decoding(target, name):
    dev, dt = target
    n = 300
    case = diff_case(name, n, 11)
    want = diff_want(case)
    for portions in ([n], [130] + [1] * 40 + [2, 128], [1] * 70 + [2, 3, 64, 5, 156]):
        got = npd(run_diff(case, portions, dev, dt))
        err = np.abs(got - want).max(-1)
        assert err.max() < (2e-4 if dt == F32 else 8e-2), (portions[:3], err.max(), int(err.argmax()))


@pytest.mark.gpu
@pytest.mark.parametrize("name", ["tensor cores, all", "64", "256", "64, eight"])
@pytest.mark.parametrize("chunk", [100000, 700, 640])
def test_differential_decoding_in_key_chunks_ignores_padding_rows(name, chunk):
    """Far into a sequence: the maps are combined by the last key chunk to finish."""
    import dataclasses
    case = diff_case(name, 1500, 21)
    case = (dataclasses.replace(case[0], chunk=chunk),) + case[1:]
    first = 1490
    got = npd(run_diff(case, [first] + [1] * 10, "cuda", BF16, extra_rows=1))[first:]
    assert np.abs(got - diff_want(case, first)).max() < 8e-2


@pytest.mark.parametrize("target", TARGETS)
def test_chunks_count_from_the_start_of_the_sequence(target):
    """A portion that starts inside a chunk, and a chunk whose start lies in the middle of a page: exactly the keys of the own
    chunk, each with its share."""
    dev, dt = target
    s = gqa.GqaSpec(1, 1, 8, 16, 0, scale=1.0, chunk=40, maps=2)
    n = 130
    q, k = torch.zeros((n, 1, 2, 8)), torch.zeros((n, 1, 2, 8))
    k[:, 0, 0, 0] = 1.0
    q[:, 0, 0, 0] = 0.0                                       # flat scores: the mean of the visible values
    v = rnd((n, 1, 16), 5)
    mix = gqa.DiffMix(0.25, 1.0, 1e-5)
    for portions in ([n], [57, 2, 71], [50] + [1] * 80):
        got = npd(run_diff((s, mix, q, k, v), portions, dev, dt))
        for i in (0, 39, 40, 41, 63, 64, 79, 80, 119, 120, 129):
            lo = i // 40 * 40
            o = 0.75 * npd(v)[lo:i + 1, 0].mean(0)
            assert np.abs(got[i] - o / np.sqrt((o * o).mean() + 1e-5)).max() < (1e-4 if dt == F32 else 5e-2), (portions[:2], i)


def test_differential_heads_need_their_mix_and_chunks_exclude_windows():
    with pytest.raises(ValueError):
        gqa.GqaSpec(2, 1, 8, 8, 0, chunk=4, window=4)
    with pytest.raises(ValueError):
        gqa.GqaSpec(2, 1, 8, 8, 0, maps=3)
    s = gqa.GqaSpec(2, 1, 8, 8, 0, maps=2)
    with pytest.raises(ValueError):
        gqa.attention(torch.zeros((1, 4, 16)), None, s.alloc_cache(1, 64, F32, "cpu"), None, s)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("window,keep,sink,dims", [(70, 5, True, (4, 2, 128, 128)), (0, 0, True, (4, 2, 128, 72)), (33, 100, False, (2, 1, 100, 128))])
def test_uncapped_attention_of_other_designs_on_the_same_kernels(target, window, keep, sink, dims):
    """One map, no cap, with and without kept tokens and a sink, against a chunk-free plain form."""
    dev, dt = target
    H, G, dk, dv = dims
    s = gqa.GqaSpec(H, G, dk, dv, 0, scale=dk ** -0.5, window=window, keep=keep, sink=sink)
    n = 200
    q, k, v = rnd((n, H, dk), 1, 2.0), rnd((n, G, dk), 2), rnd((n, G, dv), 3)
    cache = s.alloc_cache(5, 64, dt, dev)
    pos = i32(list(range(n)), dev)
    proj = torch.cat([x.reshape(n, -1) for x in (q, k, v)], 1).to(dev, dt)
    qq = gqa.prep(proj, None, None, s.inv_freq(dev), pos, pos + 64, cache, 1e-5, s)
    qs, sl, _, _ = varlen([n], [0], dev)
    meta = SimpleNamespace(is_prefill=True, q_start=qs, seq_lens=sl, block_table=i32([[1, 2, 3, 4]], dev), total_q_blocks=4, num_splits=1, max_seq_len=n)
    got = npd(gqa.attention(qq, None, cache, meta, s)).reshape(n, H, dv)
    for i in range(n):
        js = [j for j in range(i + 1) if window == 0 or i - j < window or j < keep]
        for h in range(H):
            z = npd(k)[js, h // (H // G)] @ npd(q)[i, h] * s.scale
            p = oracle.sink_softmax(z, 0.0) if sink else oracle.softmax(z)
            assert np.abs(got[i, h] - p @ npd(v)[js, h // (H // G)]).max() < (1e-4 if dt == F32 else 5e-2), (i, h)


# ------------------------------------------------------------------ mixture
@pytest.mark.parametrize("target", TARGETS[:2])
@pytest.mark.parametrize("experts,top,shared,e0", [(1, 1, 1, 0), (5, 2, 0, 0), (16, 3, 2, 8), (33, 32, 1, 11), (200, 8, 3, 100), (512, 6, 40, 0)])
def test_routing(target, experts, top, shared, e0):
    """Choice by score plus correction, weights by score alone, shared experts with the sigmoid of their own logit."""
    dev, _ = target
    t = 37
    z, corr = rnd((t, experts + 1), 1, 2.0), rnd((experts,), 2, 0.3)
    ids, w = moe_ops.route(z.to(dev), top, experts, corr.to(dev), shared, e0)
    assert ids.dtype == torch.int32 and ids.shape == w.shape == (t, top + shared)
    flips = 0
    for i in range(t):
        pick, want = oracle.choose(npd(z)[i, :experts], npd(corr), top)
        flips += set(pick) != set(np.argsort(-npd(z)[i, :experts])[:top])
        got = {int(e): float(x) for e, x in zip(ids[i, :top], w[i, :top])}
        assert got.keys() == {shared + (int(e) - e0) % experts for e in pick}
        for e, x in zip(pick, want):
            assert abs(got[shared + (int(e) - e0) % experts] - x) < 1e-5
        assert ids[i, top:].tolist() == list(range(shared))
        assert not shared or np.abs(npd(w[i, top:]) - oracle.sigmoid(npd(z)[i, experts])).max() < 1e-6
    assert flips > 0 or top >= experts                        # the correction changed somebody's choice


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("t,d,ff", [(3, 40, 24), (70, 128, 64), (700, 96, 130)])
def test_experts_with_clipped_units_and_limits_of_their_own(target, t, d, ff):
    """Units on both sides of every limit; few and many rows per expert (both orientations of the grouped GEMM)."""
    dev, dt = target
    e, top = 4, 2
    limits = [0.5, 1.0, 2.5, 100.0]
    x, gate, up, down = rnd((t, d), 1), rnd((e, ff, d), 2, 2.0 * d ** -0.5), rnd((e, ff, d), 3, 2.0 * d ** -0.5), rnd((e, d, ff), 4, ff ** -0.5)
    ids = torch.stack([torch.randperm(e, generator=torch.Generator().manual_seed(i))[:top] for i in range(t)]).to(torch.int32)
    w1, w2 = moe_ops.pad_experts(gate.to(dev, dt), up.to(dev, dt), down.to(dev, dt))
    rows, pos = moe_ops.expert_rows(x.to(dev, dt), ids.to(dev), w1, w2, 0, e, "clipped_glu", torch.tensor(limits, device=dev))
    got = npd(rows)[pos.cpu().long().numpy()][:, :d].reshape(t, top, d)
    want = np.stack([[oracle.expert(npd(x)[i], npd(gate)[k], npd(up)[k], npd(down)[k], limits[k]) for k in ids[i].tolist()] for i in range(t)])
    close(torch.tensor(got), want, TOL[dt])


def test_clipped_units_far_outside_their_limit():
    g, u = torch.tensor([[-50.0, 50.0, 50.0, -3.0]]), torch.tensor([[50.0, 50.0, -50.0, 0.25]])
    got = moe_ops._gated_unit(g, u, 5, 7.0)
    close(got, oracle.clipped_glu(npd(g), npd(u), 7.0), 1e-6)
    assert got[0, 1] == pytest.approx(7.0 * 8.0, rel=1e-4) and got[0, 2] == pytest.approx(-7.0 * 6.0, rel=1e-4)


def test_a_limit_is_required_where_it_is_used():
    xs, w = torch.zeros((1, 8)), torch.zeros((1, 128, 8))
    meta = torch.tensor([0, 1, 0, 0], dtype=torch.int32)
    with pytest.raises(AssertionError):
        moe_ops.grouped_gemm(xs, w, meta, swiglu="clipped_glu")
    with pytest.raises(AssertionError):
        moe_ops.grouped_gemm(xs, w, meta, swiglu="swiglu", limits=torch.ones(1))
