"""Small Kirisun configurations and random checkpoints for the tests."""
import json
import os

import torch

from dopurax_util import engine, error, run_portions, tokens  # noqa: F401
from zml_b200 import safetensors
from zml_b200.models.kirisun import KirisunConfig, KirisunModel


def attn(heads=4, kv_heads=2, dim=24, vdim=16, rot=12, window=33, keep=3, cap=15.0, base=4000.0, factor=2.0, scale=None):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": rot, "scaling": {"factor": factor}},
            "scale": dim ** -0.5 if scale is None else scale, "softcap": cap, "mask": {"size": window, "keep_first": keep}}


def delta(heads=4, kv_heads=2, dim=24, vdim=16, taps=3):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": taps}


def config(layers, width=96, vocab=130, eps=1e-5, scale=3.0, mult=0.4, decay_rank=12, gate_rank=20):
    """`layers`: (mixer, (experts, top, ff) or None) pairs."""
    out = [{"type": "channel_delta" if "conv" in m else "attention", "mixer": m,
            "mlp": {"kind": "moe", "expert": {"ff": f[2]}, "router": {"experts": f[0], "top": f[1]}} if f else None} for m, f in layers]
    return {"architecture": "Kirisun", "vocab": vocab, "width": width, "layers": out, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "residual_mult": mult, "decay_rank": decay_rank, "gate_rank": gate_rank}


CONFIGS = {
    # both mixers with and without a feed-forward, the delta rule first
    "mixed": config([(delta(), (6, 2, 40)), (attn(), (5, 3, 72)), (delta(heads=3, kv_heads=3, taps=4), None), (attn(window=50, keep=1, cap=4.0), None)]),
    # one of everything: one head, one expert, one tap, a window of one token and no kept ones, all factors one
    "ones": config([(attn(heads=1, kv_heads=1, dim=8, vdim=8, rot=2, window=1, keep=0, factor=1.0), (1, 1, 8)),
                    (delta(heads=1, kv_heads=1, dim=16, vdim=8, taps=1), (2, 2, 16))], width=40, vocab=65, scale=1.0, mult=1.0, decay_rank=1, gate_rank=1),
    # nothing is a multiple of 8; more kept tokens than the window has
    "odd": config([(attn(heads=6, kv_heads=3, dim=13, vdim=10, rot=6, window=29, keep=70), (5, 2, 33)), (delta(heads=6, kv_heads=2, dim=7, vdim=5, taps=5), (3, 1, 45))],
                  width=51, vocab=77, decay_rank=5, gate_rank=3),
    # head sizes of the tensor-core kernels and between them, windows over page borders, eight taps
    "wide": config([(attn(heads=4, kv_heads=2, dim=128, vdim=128, rot=64, window=70, keep=5, cap=30.0), (8, 4, 128)),
                    (delta(heads=4, kv_heads=4, dim=128, vdim=96, taps=8), None),
                    (attn(heads=2, kv_heads=1, dim=100, vdim=72, rot=100, window=100000, keep=0, cap=50.0), (4, 2, 64)),
                    (delta(heads=2, kv_heads=1, dim=64, vdim=128, taps=2), (40, 6, 24))], width=160, vocab=203),
    # many query heads on one key, sizes up to 256, a cap too large for a fixed reference, keys and values of different sizes
    "heads": config([(attn(heads=20, kv_heads=1, dim=16, vdim=24, rot=16, window=90, keep=66), None), (delta(heads=2, kv_heads=2, dim=160, vdim=40, taps=6), None),
                     (attn(heads=4, kv_heads=4, dim=200, vdim=256, rot=32, window=64, keep=64, cap=90.0), (3, 2, 40))], width=128, vocab=96),
}


def weights(cfg, seed):
    """A random checkpoint: {name: float64 array}, every value exact in bf16, spread so that each mechanism matters."""
    model = KirisunModel(KirisunConfig.from_hf(cfg), device="cpu", dtype=torch.float32)
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in model.checkpoint_shapes().items():
        leaf = name.rsplit(".", 1)[-1]
        r = torch.randn(shape, generator=g)
        if leaf in ("norm1", "norm2", "norm1b", "norm2b") or name.endswith("mix.norm") or name == "final.norm":
            t = 1 + 0.2 * r
        elif leaf == "norm":
            t = 1.8 + 0.3 * r                                    # of queries and keys: scores of a few units, attention is not flat
        elif leaf == "A_log":
            t = torch.rand(shape, generator=g) - 1.0
        elif leaf == "dt_bias":
            t = torch.rand(shape, generator=g) * 4 - 5           # decays from near 1 to about 0.7
        elif leaf == "conv":
            t = 0.5 * r
        elif name == "embed":
            t = r
        elif leaf == "b" and ".router." in name:
            t = 0.5 * r
        elif leaf == "router":
            t = 3.0 * r / shape[-1] ** 0.5                       # no close calls between experts
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


TOL = {torch.float32: 5e-5, torch.bfloat16: 8e-2}
