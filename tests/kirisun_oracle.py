"""A plain, slow implementation of the Kirisun decoder for the tests: one function per mechanism, float64, one sequence at
a time, no cache, no batching, nothing from the package under test."""
import numpy as np

from dopurax_oracle import causal_taps, mixer_tensors, read_safetensors, rms, sigmoid, silu  # noqa: F401


# ------------------------------------------------------------------ elementary pieces
def rms_norm(z, weight, eps):
    return rms(z, eps) * weight


def softplus(z):
    return np.logaddexp(0.0, z)


def turn_halves(v, pos, dims, base, factor=1.0):
    """The first `dims` entries of v [..., n]: entry i and entry i + dims/2 turned together by pos * base^(-2i/dims) / factor."""
    out = v.copy()
    half = dims // 2
    for i in range(half):
        a = pos * base ** (-2.0 * i / dims) / factor
        c, s = np.cos(a), np.sin(a)
        x, y = v[..., i], v[..., i + half]
        out[..., i] = x * c - y * s
        out[..., i + half] = y * c + x * s
    return out


def soft_cap(s, cap):
    return cap * np.tanh(s / cap)


def sees(i, j, window, keep):
    """Whether position i looks at position j."""
    return j <= i and (i - j < window or j < keep)


def sink_softmax(s):
    """exp(s) / (1 + sum exp(s)) over the last axis."""
    top = max(0.0, float(s.max()))
    e = np.exp(s - top)
    return e / (np.exp(-top) + e.sum())


def unit(z):
    return z / np.sqrt((z * z).sum(-1, keepdims=True) + 1e-6)


# ------------------------------------------------------------------ mixers
def attention(h, W, m, eps):
    """W: tensors of the mixer by short name; m: its sizes.  Returns [T, width]."""
    T, H, G, dk, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    window, keep = m["mask"]["size"], m["mask"]["keep_first"]
    rot = m["rot"]
    q = rms_norm((h @ W["q"].T).reshape(T, H, dk), W["q.norm"], eps)
    k = rms_norm((h @ W["k"].T).reshape(T, G, dk), W["k.norm"], eps)
    v = (h @ W["v"].T).reshape(T, G, dv)
    factor = rot["scaling"]["factor"]
    q = np.stack([turn_halves(q[t], t, rot["dims"], rot["base"], factor) for t in range(T)])
    k = np.stack([turn_halves(k[t], t, rot["dims"], rot["base"], factor) for t in range(T)])
    out = np.zeros((T, H, dv))
    for t in range(T):
        js = [j for j in range(t + 1) if sees(t, j, window, keep)]
        for a in range(H):
            g = a // (H // G)
            p = sink_softmax(soft_cap(k[js, g] @ q[t, a] * m["scale"], m["softcap"]))
            out[t, a] = p @ v[js, g]
    return (out.reshape(T, H * dv) * sigmoid(h @ W["g"].T)) @ W["o"].T


def channel_delta(h, W, m, eps):
    T, H, G, dk, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    assert W["q.conv"].shape[1] == W["k.conv"].shape[1] == W["v.conv"].shape[1] == m["conv"]
    q, k, v = (silu(causal_taps(h @ W[n].T, W[n + ".conv"])) for n in "qkv")
    q = unit(q.reshape(T, G, dk)) * dk ** -0.5
    k = unit(k.reshape(T, G, dk))
    v = v.reshape(T, H, dv)
    beta = sigmoid(h @ W["b"].T)
    rate = softplus((h @ W["a1"].T) @ W["a2"].T + W["dt_bias"]).reshape(T, H, dk)
    decay = np.exp(-np.exp(W["A_log"])[None, :, None] * rate)
    S = np.zeros((H, dk, dv))
    o = np.zeros((T, H, dv))
    for t in range(T):
        for a in range(H):
            g = a // (H // G)
            S[a] = decay[t, a][:, None] * S[a]
            u = beta[t, a] * (v[t, a] - S[a].T @ k[t, g])
            S[a] = S[a] + np.outer(k[t, g], u)
            o[t, a] = S[a].T @ q[t, g]
    gate = sigmoid((h @ W["g1"].T) @ W["g2"].T)
    return ((rms(o, eps) * W["norm"]).reshape(T, H * dv) * gate) @ W["o"].T


MIXERS = {"attention": attention, "channel_delta": channel_delta}


# ------------------------------------------------------------------ feed-forward
def expert(x, gate, up, down):
    return (silu(x @ gate.T) * (x @ up.T)) @ down.T


def route(x, W, top):
    """(indices, weights) of the `top` experts of one token."""
    z = W["router"] @ x + W["router.b"]
    pick = np.argsort(-z, kind="stable")[:top]
    e = np.exp(z[pick] - z[pick].max())
    return pick, e / e.sum()


def mixture(x, W, top):
    y = np.zeros_like(x)
    for t in range(x.shape[0]):
        for e, w in zip(*route(x[t], W, top)):
            y[t] += w * expert(x[t], W[f"e{e}.gate"], W[f"e{e}.up"], W[f"e{e}.down"])
    return y


# ------------------------------------------------------------------ the stack
def forward(cfg, W, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence; `layers_out` (a list) receives the stream after every layer."""
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x = W["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        y = MIXERS[layer["type"]](rms_norm(x, W[p + "norm1"], eps), mixer_tensors(W, i), layer["mixer"], eps)
        x = x + mult * rms_norm(y, W[p + "norm1b"], eps)
        if layer["mlp"] is not None:
            ff = {n[len(p) + 4:]: t for n, t in W.items() if n.startswith(p + "mlp.")}
            y = mixture(rms_norm(x, W[p + "norm2"], eps), ff, layer["mlp"]["router"]["top"])
            x = x + mult * rms_norm(y, W[p + "norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x)
    return rms_norm(x, W["final.norm"], eps) @ W["head"].T


def greedy(cfg, W, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(np.argmax(forward(cfg, W, toks)[-1])))
    return toks[len(prompt):]
