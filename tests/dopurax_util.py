"""Small Dopurax configurations, random checkpoints and engine drivers for the tests."""
import json
import os

import numpy as np
import torch

from zml_b200 import safetensors
from zml_b200.models import hub
from zml_b200.models.dopurax import DopuraxConfig, DopuraxModel
from zml_b200.serving import Engine

PAGE = 64


def latent(heads=3, dim=24, rot=8, vdim=16, rank=40, q_rank=32, window=50, scale=None, base=5000.0):
    return {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "q_rank": q_rank, "mask": {"size": window},
            "scale": (dim + rot) ** -0.5 if scale is None else scale, "rot": {"base": base, "dims": rot}}


def config(layers, width=96, vocab=130, taps=3, alpha=1.7, eps=1e-5, decay_rank=12):
    """`layers`: (mixer dict, ff or None) pairs; a mixer without `kv_rank` is WKV."""
    out = [{"type": "latent_attention" if "kv_rank" in m else "wkv", "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None}
           for m, ff in layers]
    return {"architecture": "Dopurax", "vocab": vocab, "width": width, "layers": out, "norm": {"eps": eps}, "postln_alpha": alpha,
            "canon": {"taps": taps}, "decay_rank": decay_rank}


WKV = {"heads": 3, "dim": 24}
CONFIGS = {
    # both mixers with and without a feed-forward, WKV first
    "mixed": config([(WKV, 80), (latent(), 72), (WKV, None), (latent(window=33, scale=0.4), None)]),
    # one head, one tap (the convolution has no past), a window of one token, attention first
    "ones": config([(latent(heads=1, dim=8, rot=8, vdim=8, rank=16, q_rank=8, window=1), 8), ({"heads": 1, "dim": 16}, 16)], width=40, vocab=65,
                   taps=1, alpha=1.0, decay_rank=1),
    # nothing is a multiple of 8: the kernels for any size
    "odd": config([(latent(heads=3, dim=13, rot=6, vdim=10, rank=21, q_rank=19, window=29), 45), ({"heads": 5, "dim": 7}, 33)], width=51, vocab=77,
                  taps=5, decay_rank=5),
    # layers of different sizes, whole sub-tiles, a window over a page border, eight taps
    "wide": config([(latent(heads=4, dim=64, rot=32, vdim=64, rank=128, q_rank=96, window=70), 256), ({"heads": 4, "dim": 96}, None),
                    (latent(heads=2, dim=128, rot=64, vdim=128, rank=256, q_rank=64, window=100000), 64)], width=160, vocab=203, taps=8, decay_rank=24),
    # two groups of heads in decode, 512 latent columns, WKV heads with a launch of its own for the norm
    "heads": config([(latent(heads=40, dim=16, rot=16, vdim=8, rank=512, q_rank=48, window=90), None), ({"heads": 1, "dim": 160}, None),
                     ({"heads": 2, "dim": 64}, 40)], width=128, vocab=96, taps=2),
}


def weights(cfg, seed):
    """A random checkpoint: {name: float64 array}, every value exact in bf16, spread so that each mechanism matters."""
    model = DopuraxModel(DopuraxConfig.from_hf(cfg), device="cpu", dtype=torch.float32)
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in model.checkpoint_shapes().items():
        leaf = name.rsplit(".", 1)[-1]
        r = torch.randn(shape, generator=g)
        if ".mu." in name:
            t = torch.rand(shape, generator=g)
        elif leaf in ("norm", "norm1", "norm2"):
            t = 1 + 0.2 * r
        elif leaf == "w0":
            t = torch.rand(shape, generator=g) * 5 - 6           # decays from near 1 to about 0.7
        elif leaf == "canon1":
            t = 0.4 * r
        elif leaf == "u":
            t = r
        elif name == "embed":
            t = r
        elif leaf in ("uq", "uk"):
            t = 2.0 * r / shape[-1] ** 0.5                       # scores of a few units: attention is not flat
        else:
            t = 1.2 * r / shape[-1] ** 0.5
        out[name] = t.to(torch.bfloat16)
    return out


def checkpoint(path, name_or_cfg, seed=0):
    """Writes config.json + model.safetensors and returns (config, float64 weights)."""
    cfg = CONFIGS[name_or_cfg] if isinstance(name_or_cfg, str) else name_or_cfg
    w = weights(cfg, seed)
    os.makedirs(path, exist_ok=True)
    safetensors.save_file(w, os.path.join(path, "model.safetensors"))
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    return cfg, {k: v.double().numpy() for k, v in w.items()}


def engine(path, device, dtype, max_tokens=1024, max_batch=4, slots=None, page=PAGE, **kw):
    model, _ = hub.load_model(str(path), device=device, dtype=dtype)
    pages = (max_tokens + page - 1) // page
    return Engine(model, pages + 1, page, max_batch, pages * page, num_state_slots=slots, **kw)


def tokens(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


def run_portions(eng, toks, sizes):
    """All logits of one request brought in portions of the given sizes (the last one repeats)."""
    r, out, at, i = eng.open_request(), [], 0, 0
    while at < len(toks):
        n = min(sizes[min(i, len(sizes) - 1)], len(toks) - at)
        out.append(eng.step([(r, toks[at:at + n])], [list(range(n))]).float().cpu())
        at += n
        i += 1
    eng.release(r)
    return torch.cat(out).numpy().astype(np.float64)


def error(got, want):
    """Root mean square of the difference over that of the expected logits, means taken off, worst row."""
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    c = want - want.mean(-1, keepdims=True)
    return float(np.sqrt((d * d).mean(-1)).max() / np.sqrt((c * c).mean()))


TOL = {torch.float32: 3e-5, torch.bfloat16: 6e-2}
