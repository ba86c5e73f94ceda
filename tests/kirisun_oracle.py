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
    return cap * np.tanh(s / cap) if cap else s


def sees(i, j, window, keep):
    """Whether position i looks at position j (window 0: no window)."""
    return j <= i and (window == 0 or i - j < window or j < keep)


def sink_softmax(s):
    """exp(s) / (1 + sum exp(s)) over the last axis."""
    top = max(0.0, float(s.max()))
    e = np.exp(s - top)
    return e / (np.exp(-top) + e.sum())


def unit(z):
    return z / np.sqrt((z * z).sum(-1, keepdims=True) + 1e-6)


# ------------------------------------------------------------------ mixers
def attend(q, k, v, scale, cap, window, keep, first=0):
    """Rows first .. of a sequence: q [n, H, dk] at positions first + row, k, v [>= first + n, G, *] of all positions."""
    n, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = np.zeros((n, H, v.shape[-1]))
    for r in range(n):
        i = first + r
        js = [j for j in range(i + 1) if sees(i, j, window, keep)]
        for a in range(H):
            g = a // (H // G)
            out[r, a] = sink_softmax(soft_cap(k[js, g] @ q[r, a] * scale, cap)) @ v[js, g]
    return out


def attention(h, W, m, eps):
    """W: tensors of the mixer by short name; m: its sizes.  Returns [T, width]."""
    T, H, G, dk, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    rot = m["rot"]
    q = rms_norm((h @ W["q"].T).reshape(T, H, dk), W["q.norm"], eps)
    k = rms_norm((h @ W["k"].T).reshape(T, G, dk), W["k.norm"], eps)
    v = (h @ W["v"].T).reshape(T, G, dv)
    factor = rot["scaling"]["factor"]
    q = np.stack([turn_halves(q[t], t, rot["dims"], rot["base"], factor) for t in range(T)])
    k = np.stack([turn_halves(k[t], t, rot["dims"], rot["base"], factor) for t in range(T)])
    out = attend(q, k, v, m["scale"], m["softcap"], m["mask"]["size"], m["mask"]["keep_first"])
    return (out.reshape(T, H * dv) * sigmoid(h @ W["g"].T)) @ W["o"].T


def delta_rule(q, k, v, beta, decay):
    """q, k [T, G, dk], v [T, H, dv], beta [T, H], decay [T, H, dk], one token after the other from a zero state."""
    (T, G, dk), (H, dv) = k.shape, v.shape[1:]
    S = np.zeros((H, dk, dv))
    o = np.zeros((T, H, dv))
    for t in range(T):
        for a in range(H):
            g = a // (H // G)
            S[a] = decay[t, a][:, None] * S[a]
            u = beta[t, a] * (v[t, a] - S[a].T @ k[t, g])
            S[a] = S[a] + np.outer(k[t, g], u)
            o[t, a] = S[a].T @ q[t, g]
    return o


def delta_core(q, k, v, convs, beta, pre, a_log, dt_bias, gate, norm, sizes, eps):
    """Everything between the input projections and the output projection: q, k, v before their convolutions, logits of the
    write gates [T, H] and of the output gates [T, H dv], pre-activations of the decays [T, H dk]."""
    H, G, dk, dv = sizes
    T = q.shape[0]
    q, k, v = (silu(causal_taps(x, w)) for x, w in zip((q, k, v), convs))
    q = unit(q.reshape(T, G, dk)) * dk ** -0.5
    k = unit(k.reshape(T, G, dk))
    rate = softplus(pre + dt_bias).reshape(T, H, dk)
    o = delta_rule(q, k, v.reshape(T, H, dv), sigmoid(beta), np.exp(-np.exp(a_log)[None, :, None] * rate))
    return (rms(o, eps) * norm).reshape(T, H * dv) * sigmoid(gate)


def channel_delta(h, W, m, eps):
    assert W["q.conv"].shape[1] == W["k.conv"].shape[1] == W["v.conv"].shape[1] == m["conv"]
    o = delta_core(*(h @ W[n].T for n in "qkv"), [W[n + ".conv"] for n in "qkv"], h @ W["b"].T, (h @ W["a1"].T) @ W["a2"].T, W["A_log"],
                   W["dt_bias"], (h @ W["g1"].T) @ W["g2"].T, W["norm"], (m["heads"], m["kv_heads"], m["dim"], m["vdim"]), eps)
    return o @ W["o"].T


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
