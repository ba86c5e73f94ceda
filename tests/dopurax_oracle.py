"""A plain, slow implementation of the Dopurax decoder for the tests: one function per mechanism, float64, one
sequence at a time, no cache, no batching, nothing from the package under test."""
import json
import math
import struct

import numpy as np


# ------------------------------------------------------------------ files
def read_safetensors(path):
    """{name: float64 / int array} of a .safetensors file (BF16, F32 and I32 entries)."""
    raw = open(path, "rb").read()
    n = struct.unpack("<Q", raw[:8])[0]
    head = json.loads(raw[8:8 + n])
    out = {}
    for name, ent in head.items():
        if name == "__metadata__":
            continue
        a, b = ent["data_offsets"]
        buf = raw[8 + n + a:8 + n + b]
        if ent["dtype"] == "BF16":
            v = (np.frombuffer(buf, "<u2").astype(np.uint32) << 16).view(np.float32).astype(np.float64)
        elif ent["dtype"] == "F32":
            v = np.frombuffer(buf, "<f4").astype(np.float64)
        elif ent["dtype"] == "I32":
            v = np.frombuffer(buf, "<i4")
        else:
            raise ValueError(ent["dtype"])
        out[name] = v.reshape(ent["shape"])
    return out


# ------------------------------------------------------------------ elementary pieces
def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def rms(z, eps):
    """z at unit root mean square over the last axis."""
    return z / np.sqrt((z * z).mean(-1, keepdims=True) + eps)


def layer_norm(z, weight, eps):
    d = z - z.mean(-1, keepdims=True)
    return d / np.sqrt((d * d).mean(-1, keepdims=True) + eps) * weight


def causal_taps(h, w):
    """Depthwise causal convolution, tap K-1 on the current token, zeros before the first token."""
    out = np.zeros_like(h)
    taps = w.shape[1]
    for t in range(h.shape[0]):
        for j in range(taps):
            s = t - (taps - 1) + j
            if s >= 0:
                out[t] += w[:, j] * h[s]
    return out


def rotate_pairs(v, pos, base):
    """Adjacent dimensions (2i, 2i+1) of v [..., dims] turned by pos * base^(-2i / dims)."""
    out = v.copy()
    dims = v.shape[-1]
    for i in range(dims // 2):
        a = pos * base ** (-2.0 * i / dims)
        u, w = v[..., 2 * i], v[..., 2 * i + 1]
        out[..., 2 * i] = u * math.cos(a) - w * math.sin(a)
        out[..., 2 * i + 1] = w * math.cos(a) + u * math.sin(a)
    return out


# ------------------------------------------------------------------ mixers
def latent_attention(h, W, m, eps, first_pos=0):
    """W: tensors of the mixer by short name; m: its sizes.  Returns [T, width]."""
    T = h.shape[0]
    H, dn, dr, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    window, base = m["mask"]["size"], m["rot"]["base"]
    assert m["rot"]["dims"] == dr
    q = (rms(h @ W["dq"].T, eps) * W["dq.norm"]) @ W["uq"].T
    q = q.reshape(T, H, dn + dr)
    down = h @ W["dkv"].T
    c = rms(down[:, :rank], eps) * W["dkv.norm"]
    kr = down[:, rank:]
    kr = np.stack([rotate_pairs(kr[t], first_pos + t, base) for t in range(T)]) if T else kr
    qr = np.stack([rotate_pairs(q[t, :, dn:], first_pos + t, base) for t in range(T)]) if T else q[..., dn:]
    kn = (c @ W["uk"].T).reshape(T, H, dn)
    v = (c @ W["uv"].T).reshape(T, H, dv)
    out = np.zeros((T, H, dv))
    for t in range(T):
        lo = max(0, t - window + 1)
        for a in range(H):
            s = (kn[lo:t + 1, a] @ q[t, a, :dn] + kr[lo:t + 1] @ qr[t, a]) * m["scale"]
            e = np.exp(s - s.max())
            out[t, a] = (e / e.sum()) @ v[lo:t + 1, a]
    return (out.reshape(T, H * dv) * sigmoid(h @ W["g"].T)) @ W["o"].T


def wkv(h, W, m, eps):
    T = h.shape[0]
    H, D = m["heads"], m["dim"]
    prev = np.concatenate([np.zeros_like(h[:1]), h[:-1]], 0)
    mix = {s: h + (prev - h) * W["mu." + s] for s in "rkvgw"}
    r, k, v = (np.reshape(mix[s] @ W[s].T, (T, H, D)) for s in "rkv")
    gate = silu(mix["g"] @ W["g"].T)
    decay = np.exp(-np.exp(np.tanh(mix["w"] @ W["w1"].T) @ W["w2"].T + W["w0"])).reshape(T, H, D)
    S = np.zeros((H, D, D))                    # [head, key channel, value channel]
    o = np.zeros((T, H, D))
    for t in range(T):
        for a in range(H):
            kv = np.outer(k[t, a], v[t, a])
            o[t, a] = r[t, a] @ (S[a] + W["u"][a][:, None] * kv)
            S[a] = decay[t, a][:, None] * S[a] + kv
    return (rms(o, eps).reshape(T, H * D) * W["norm"] * gate) @ W["o"].T


MIXERS = {"latent_attention": latent_attention, "wkv": wkv}


def dense_ff(x, up, down):
    return np.maximum(x @ up.T, 0.0) ** 2 @ down.T


# ------------------------------------------------------------------ the stack
def mixer_tensors(W, i):
    p = f"l{i}.mix."
    return {n[len(p):]: t for n, t in W.items() if n.startswith(p)}


def forward(cfg, W, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence; `layers_out` (a list) receives the stream after every layer."""
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    x = W["embed"][np.asarray(tokens)]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        assert W[p + "canon1"].shape[1] == cfg["canon"]["taps"]
        h = x + causal_taps(x, W[p + "canon1"])
        y = MIXERS[layer["type"]](h, mixer_tensors(W, i), layer["mixer"], eps)
        x = layer_norm(alpha * x + y, W[p + "norm1"], eps)
        if layer["mlp"] is not None:
            x = layer_norm(alpha * x + dense_ff(x, W[p + "mlp.up"], W[p + "mlp.down"]), W[p + "norm2"], eps)
        if layers_out is not None:
            layers_out.append(x)
    return layer_norm(x, W["final.norm"], eps) @ W["head"].T


def greedy(cfg, W, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(np.argmax(forward(cfg, W, toks)[-1])))
    return toks[len(prompt):]
