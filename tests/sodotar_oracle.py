"""A plain, slow implementation of the Sodotar decoder for the tests: one function per mechanism, float64, one sequence at a
time, no cache, no batching, nothing from the package under test."""
import numpy as np

from dopurax_oracle import mixer_tensors, read_safetensors, rms, sigmoid  # noqa: F401


# ------------------------------------------------------------------ elementary pieces
def rms_norm(z, weight, eps):
    return rms(z, eps) * weight


def turn_halves(v, pos, dims, base):
    """The first `dims` entries of v [..., n]: entry i and entry i + dims/2 turned together by pos * base^(-2i/dims)."""
    out = v.copy()
    half = dims // 2
    for i in range(half):
        a = pos * base ** (-2.0 * i / dims)
        c, s = np.cos(a), np.sin(a)
        x, y = v[..., i], v[..., i + half]
        out[..., i] = x * c - y * s
        out[..., i + half] = y * c + x * s
    return out


def turn_all(v, dims, base, first=0):
    """v [T, ...] at positions first, first + 1, .."""
    return np.stack([turn_halves(v[t], first + t, dims, base) for t in range(v.shape[0])])


def softmax(s):
    e = np.exp(s - s.max())
    return e / e.sum()


def sink_softmax(s, sink):
    """exp(s) / (exp(sink) + sum exp(s))."""
    top = max(float(sink), float(s.max()))
    e = np.exp(s - top)
    return e / (np.exp(sink - top) + e.sum())


# ------------------------------------------------------------------ latent attention
def latent_attend(q, k, v, scale, sink, first=0):
    """Rows first .. of a sequence: q [n, H, *], k [>= first + n, H, *], v [.., H, *]; sink [H]."""
    out = np.zeros(q.shape[:2] + (v.shape[-1],))
    for r in range(q.shape[0]):
        n = first + r + 1
        for a in range(q.shape[1]):
            out[r, a] = sink_softmax(k[:n, a] @ q[r, a] * scale, sink[a]) @ v[:n, a]
    return out


def latent_keys_values(c, shared, uk, uv, H):
    """Keys [T, H, dim + rot] and values [T, H, vdim] out of normed latents c [T, rank] and the turned part `shared` [T, rot]."""
    T = c.shape[0]
    k = (c @ uk.T).reshape(T, H, -1)
    return np.concatenate([k, np.repeat(shared[:, None], H, 1)], -1), (c @ uv.T).reshape(T, H, -1)


def latent_attention(h, W, m, eps):
    """W: tensors of the mixer by short name; m: its sizes.  Returns [T, width]."""
    T, H, dim, rot, rank, base = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["kv_rank"], m["rot"]["base"]
    q = (h @ W["q"].T).reshape(T, H, dim + rot)
    q = np.concatenate([q[..., :dim], turn_all(q[..., dim:], rot, base)], -1)
    d = h @ W["dkv"].T
    k, v = latent_keys_values(rms_norm(d[:, :rank], W["dkv.norm"], eps), turn_all(d[:, rank:], rot, base), W["uk"], W["uv"], H)
    return latent_attend(q, k, v, m["scale"], W["sink"]).reshape(T, -1) @ W["o"].T


# ------------------------------------------------------------------ differential attention
def sees(i, j, chunk):
    return j <= i and i // chunk == j // chunk


def chunked_attend(q, k, v, scale, chunk, first=0):
    """One map: rows first .. of a sequence, q [n, H, dk], k [.., G, dk], v [.., G, dv]."""
    n, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = np.zeros((n, H, v.shape[-1]))
    for r in range(n):
        i = first + r
        js = [j for j in range(i + 1) if sees(i, j, chunk)]
        for a in range(H):
            g = a // (H // G)
            out[r, a] = softmax(k[js, g] @ q[r, a] * scale) @ v[js, g]
    return out


def map_weight(W, diff):
    return np.exp((W["lq1"] * W["lk1"]).sum()) - np.exp((W["lq2"] * W["lk2"]).sum()) + diff


def combine_maps(a1, a2, lam, diff, eps):
    return rms(a1 - lam * a2, eps) * (1.0 - diff)


def keys_values(h, W, m):
    """What a layer caches: turned keys [T, G, 2, dk] and values [T, G, dv]."""
    T, G = h.shape[0], m["kv_heads"]
    k = turn_all((h @ W["k"].T).reshape(T, G, 2, m["dim"]), m["rot"]["dims"], m["rot"]["base"])
    return k, (h @ W["v"].T).reshape(T, G, m["vdim"])


def diff_attention(h, W, m, eps, kv):
    T, H = h.shape[0], m["heads"]
    q = turn_all((h @ W["q"].T).reshape(T, H, 2, m["dim"]), m["rot"]["dims"], m["rot"]["base"])
    k, v = kv
    a1, a2 = (chunked_attend(q[:, :, i], k[:, :, i], v, m["scale"], m["mask"]["size"]) for i in (0, 1))
    return combine_maps(a1, a2, map_weight(W, m["diff"]), m["diff"], eps).reshape(T, -1) @ W["o"].T


# ------------------------------------------------------------------ feed-forward
def clipped_glu(gate, up, limit):
    g, u = np.minimum(gate, limit), np.clip(up, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def expert(x, gate, up, down, limit):
    return clipped_glu(x @ gate.T, x @ up.T, limit) @ down.T


def choose(z, correction, top):
    """(indices, weights) of one token's experts out of the router's logits."""
    s = softmax(z)
    pick = np.argsort(-(s + correction), kind="stable")[:top]
    return pick, s[pick] / (s[pick].sum() + 1e-20)


def mixture(x, W, mlp):
    y = np.zeros_like(x)
    for t in range(x.shape[0]):
        for e, w in zip(*choose(W["router"] @ x[t], W["correction"], mlp["router"]["top"])):
            y[t] += w * expert(x[t], W[f"e{e}.gate"], W[f"e{e}.up"], W[f"e{e}.down"], mlp["expert"]["limit"])
    if mlp.get("shared"):
        s = expert(x, W["shared.gate"], W["shared.up"], W["shared.down"], mlp["shared"]["limit"])
        y = y + sigmoid(x @ W["shared.sg"].T) * s
    return y


# ------------------------------------------------------------------ the stack
def sublayer(xs, W, hc, norm, eps, f):
    """xs [streams, T, d] through one sublayer: read a mix of the streams, write them all."""
    y = f(rms_norm(np.einsum("s,std->td", W[hc + "in"], xs), W[norm], eps))
    return np.einsum("st,snd->tnd", W[hc + "mix"], xs) + W[hc + "out"][:, None, None] * y[None]


def forward(cfg, W, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence; `layers_out` (a list) receives the sum of the streams behind every layer."""
    eps = cfg["norm"]["eps"]
    xs = np.repeat(W["embed"][np.asarray(tokens)][None], cfg["streams"], 0)
    cached = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        mix = mixer_tensors(W, i)

        def mixer(h):
            if layer["type"] == "latent_attention":
                return latent_attention(h, mix, m, eps)
            if m.get("kv_from") is None:
                cached[i] = keys_values(h, mix, m)
            return diff_attention(h, mix, m, eps, cached[i if m.get("kv_from") is None else m["kv_from"]])

        xs = sublayer(xs, W, p + "hc1.", p + "norm1", eps, mixer)
        if layer["mlp"] is not None:
            ff = {n[len(p) + 4:]: t for n, t in W.items() if n.startswith(p + "mlp.")}
            xs = sublayer(xs, W, p + "hc2.", p + "norm2", eps, lambda h: mixture(h, ff, layer["mlp"]))
        if layers_out is not None:
            layers_out.append(xs.sum(0))
    return rms_norm(xs.sum(0), W["final.norm"], eps) @ W["embed"].T * cfg["logit_scale"]


def greedy(cfg, W, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(np.argmax(forward(cfg, W, toks)[-1])))
    return toks[len(prompt):]
