"""A plain, slow implementation of the Dogidra decoder for the tests: one function per mechanism, float64, one sequence at a
time, no cache, no batching, nothing from the package under test."""
import math

import numpy as np

from dopurax_oracle import causal_taps, read_safetensors, rms, sigmoid, silu  # noqa: F401


# ------------------------------------------------------------------ elementary pieces
def layer_norm(z, weight, bias, eps):
    d = z - z.mean(-1, keepdims=True)
    return d / np.sqrt((d * d).mean(-1, keepdims=True) + eps) * weight + bias


def with_past(h, w):
    """h plus its causal convolution, w [width, taps]."""
    return h + causal_taps(h, w)


def frequencies(rot):
    """(turning rates of the pairs, factor on cosines and sines) of a rotation with or without stretched positions."""
    dims, base, sc = rot["dims"], rot["base"], rot.get("scaling")
    f = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)])
    if not sc:
        return f, 1.0
    turns_to_dim = lambda turns: dims * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(turns_to_dim(sc["fast"])), 0), min(math.ceil(turns_to_dim(sc["slow"])), dims - 1)
    out = []
    for i, rate in enumerate(f):
        share = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(rate / sc["factor"] * share + rate * (1 - share))
    return np.array(out), 0.1 * math.log(sc["factor"]) + 1.0


def turn(v, pos, rot):
    """The first rot["dims"] entries of v [..., n]: entry i and entry i + dims/2 are a pair."""
    f, amp = frequencies(rot)
    out, half = v.copy(), rot["dims"] // 2
    for i in range(half):
        c, s = amp * math.cos(pos * f[i]), amp * math.sin(pos * f[i])
        x, y = v[..., i], v[..., i + half]
        out[..., i] = x * c - y * s
        out[..., i + half] = y * c + x * s
    return out


def turn_all(v, rot, first=0):
    """v [T, ...] at positions first, first + 1, .."""
    return np.stack([turn(v[t], first + t, rot) for t in range(v.shape[0])])


def softmax(s):
    e = np.exp(s - s.max())
    return e / e.sum()


# ------------------------------------------------------------------ attention over a window and pooled blocks
def tokens_seen(i, size):
    return [j for j in range(i + 1) if i - j < size]


def blocks_seen(i, size, pool):
    """Blocks of `pool` tokens whose last one has left the window of position i."""
    return [b for b in range(i + 1) if b * pool + pool - 1 <= i - size]


def visible_rows(k, v, i, size, pool):
    """Keys and values that position i attends to: k [T, G, *], v [T, G, *] by token."""
    ks, vs = [k[j] for j in tokens_seen(i, size)], [v[j] for j in tokens_seen(i, size)]
    for b in blocks_seen(i, size, pool):
        ks.append(k[b * pool:(b + 1) * pool].mean(0))
        vs.append(v[b * pool:(b + 1) * pool].mean(0))
    return np.stack(ks), np.stack(vs)


def capped(s, cap):
    return cap * np.tanh(s / cap)


def attend(q, k, v, scale, cap, size, pool, first=0):
    """Rows first .. of a sequence: q [n, H, dim], k [>= first + n, G, dim], v [.., G, vdim] -> [n, H, vdim]."""
    H, G = q.shape[1], k.shape[1]
    out = np.zeros(q.shape[:2] + (v.shape[-1],))
    for r in range(q.shape[0]):
        kk, vv = visible_rows(k, v, first + r, size, pool)
        for a in range(H):
            g = a // (H // G)
            out[r, a] = softmax(capped(kk[:, g] @ q[r, a] * scale, cap)) @ vv[:, g]
    return out


def window_attention(h, W, m, eps):
    """W: tensors by short name; m: the sizes of this side."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = rms(h @ W["q"].T, eps) * W["q.norm"]                       # over all heads at once
    k = rms(h @ W["k"].T, eps) * W["k.norm"]
    q, k = turn_all(q.reshape(T, H, m["dim"]), m["rot"]), turn_all(k.reshape(T, G, m["dim"]), m["rot"])
    v = (h @ W["v"].T).reshape(T, G, m["vdim"])
    a = attend(q, k, v, m["scale"], m["softcap"], m["mask"]["size"], m["mask"]["pool"])
    return a.reshape(T, -1) @ W["o"].T


# ------------------------------------------------------------------ gated recurrence
def candidate(u):
    return np.where(u >= 0, u + 0.5, sigmoid(u))


def recur(z, u, state=None):
    """z: gates in (0, 1), u: pre-activations of the candidates, [T, width] -> states behind every token."""
    s = np.zeros(z.shape[1]) if state is None else state.copy()
    out = np.zeros_like(z)
    for t in range(z.shape[0]):
        s = (1 - z[t]) * s + z[t] * candidate(u[t])
        out[t] = s
    return out


def gated_recurrence(h, W):
    s = recur(sigmoid(h @ W["z"].T + W["z.b"]), h @ W["x"].T + W["x.b"])
    return (s * silu(h @ W["g"].T)) @ W["o"].T


def side(W, name):
    return {n[len(name) + 1:]: t for n, t in W.items() if n.startswith(name + ".")}


def parallel(h, W, m, eps):
    return m["left_scale"] * window_attention(h, side(W, "left"), m["left"], eps) + m["right_scale"] * gated_recurrence(h, side(W, "right"))


# ------------------------------------------------------------------ feed-forward
def expert(x, up, down):
    return np.maximum(x @ up.T, 0) ** 2 @ down.T


def choose(z, correction, top, scale):
    """(indices, weights) of one token's experts out of the router's logits."""
    s = sigmoid(z)
    pick = np.argsort(-(s + correction), kind="stable")[:top]
    return pick, s[pick] * scale


def mixture(x, W, mlp):
    y = np.zeros_like(x)
    r = mlp["router"]
    for t in range(x.shape[0]):
        for e, w in zip(*choose(W["router"] @ x[t], W["correction"], r["top"], r["scale"])):
            y[t] += w * expert(x[t], W[f"e{e}.up"], W[f"e{e}.down"])
    return y + expert(x, W["shared.up"], W["shared.down"]) if mlp.get("shared") else y


# ------------------------------------------------------------------ the stack
def runs(cfg):
    """(layer, whether a pass of the loop begins in front of it) in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    return [(i, False) for i in range(a)] + [(i, i == a) for _ in range(loop["times"]) for i in range(a, b)] + [(i, False) for i in range(b, n)]


def forward(cfg, W, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence; `layers_out` (a list) receives the stream behind every layer that ran."""
    eps = cfg["norm"]["eps"]
    x = x0 = W["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    for i, begins in runs(cfg):
        p, layer = f"l{i}.", cfg["layers"][i]
        if begins:
            x = np.concatenate([x, x0], -1) @ W["loop.in"].T
        h = with_past(layer_norm(x, W[p + "norm1"], W[p + "norm1.b"], eps), W[p + "canon1"])
        x = x + parallel(h, side(W, f"l{i}.mix"), layer["mixer"], eps)
        if layer["mlp"] is not None:
            h = with_past(layer_norm(x, W[p + "norm2"], W[p + "norm2.b"], eps), W[p + "canon2"])
            x = x + mixture(h, side(W, f"l{i}.mlp"), layer["mlp"])
        if layers_out is not None:
            layers_out.append(x)
    return layer_norm(x, W["final.norm"], W["final.norm.b"], eps) @ W["embed"].T


def greedy(cfg, W, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(np.argmax(forward(cfg, W, toks)[-1])))
    return toks[len(prompt):]
