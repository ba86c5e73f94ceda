"""Small Sodotar configurations and random checkpoints for the tests."""
import json
import os

import torch

from dopurax_util import engine, run_portions, tokens  # noqa: F401
from zml_b200 import safetensors
from zml_b200.models.sodotar import SodotarConfig


def latent(heads=3, dim=24, rot=8, vdim=20, rank=40, base=3000.0, scale=None):
    return {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "rot": {"base": base, "dims": rot},
            "scale": (dim + rot) ** -0.5 if scale is None else scale}


def attn(heads=4, kv_heads=2, dim=12, vdim=20, rot=8, chunk=33, diff=0.4, base=4000.0, scale=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": rot},
         "scale": dim ** -0.5 if scale is None else scale, "mask": {"size": chunk}, "diff": diff}
    return m if kv_from is None else dict(m, kv_from=kv_from)


def moe(experts=5, top=2, ff=40, limit=0.9, shared=24, shared_limit=1.7):
    out = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    return dict(out, shared={"ff": shared, "limit": shared_limit}) if shared else out


def config(layers, width=96, vocab=130, eps=1e-5, streams=3, logit_scale=0.7):
    """`layers`: (mixer, feed-forward or None) pairs."""
    out = [{"type": "latent_attention" if "kv_rank" in m else "attention", "mixer": m, "mlp": f} for m, f in layers]
    return {"architecture": "Sodotar", "vocab": vocab, "width": width, "layers": out, "norm": {"eps": eps}, "streams": streams, "logit_scale": logit_scale}


CONFIGS = {
    # both mixers with and without a feed-forward; keys of layers that are not the one before, under another mask
    "mixed": config([(attn(), moe()), (latent(), moe(6, 3, 72, 1.2, 90, 0.6)), (attn(chunk=50, diff=0.7), None), (attn(chunk=80, kv_from=0), None),
                     (latent(heads=2, vdim=40), None), (attn(heads=2, chunk=20, diff=0.1, kv_from=2), moe(shared=0))]),
    # one of everything: one head, one expert, one stream, chunks of one token, all factors one
    "ones": config([(latent(heads=1, dim=8, rot=2, vdim=8, rank=8, base=1.0, scale=1.0), moe(1, 1, 8, 1.0, 8, 1.0)),
                    (attn(heads=1, kv_heads=1, dim=8, vdim=8, rot=2, chunk=1, scale=1.0), moe(2, 2, 16, 1.0, 8, 1.0))], width=40, vocab=65, streams=1,
                   logit_scale=1.0),
    # nothing is a multiple of 8
    "odd": config([(latent(heads=5, dim=13, rot=6, vdim=11, rank=21), moe(5, 2, 33, 0.8, 70)),
                   (attn(heads=6, kv_heads=3, dim=13, vdim=10, rot=6, chunk=29), moe(3, 1, 45, 2.0, 7))], width=51, vocab=77, streams=2),
    # head sizes of the tensor-core kernels and between them, chunks over page borders, a shared expert of several pieces
    "wide": config([(latent(heads=4, dim=128, rot=64, vdim=128, rank=256), moe(8, 4, 128, 1.5, 300)),
                    (attn(heads=4, kv_heads=2, dim=64, vdim=128, rot=32, chunk=128), None),
                    (attn(heads=4, kv_heads=2, dim=64, vdim=128, rot=64, chunk=70, diff=0.6, kv_from=1), moe(40, 6, 24, 1.0, 64)),
                    (latent(heads=20, dim=40, rot=16, vdim=72, rank=96), None),
                    (attn(heads=2, kv_heads=1, dim=50, vdim=104, rot=50, chunk=100000), moe(4, 2, 64, 3.0, 40))], width=160, vocab=203, streams=4),
    # more query rows per key than a tile holds, sizes up to 256, many streams
    "heads": config([(attn(heads=10, kv_heads=1, dim=16, vdim=24, rot=16, chunk=90), None), (latent(heads=33, dim=16, rot=16, vdim=8, rank=32), None),
                     (attn(heads=4, kv_heads=4, dim=100, vdim=256, rot=32, chunk=64), moe(3, 2, 40)), (attn(heads=2, kv_heads=1, dim=140, vdim=30, chunk=96), None)],
                    width=128, vocab=96, streams=7),
}


def all_experts(cfg):
    """The same with every expert chosen (at most 32, what the router takes)."""
    cfg = json.loads(json.dumps(cfg))
    for e in cfg["layers"]:
        if e["mlp"] is not None:
            r = e["mlp"]["router"]
            r["experts"] = r["top"] = min(32, r["experts"])
    return cfg


CONFIGS.update({f"{name}, all experts": all_experts(cfg) for name, cfg in list(CONFIGS.items())})


def case_for(name, dtype):
    """In bf16 a close call between two experts may fall the other way, and all later positions see it: logits of whole models are
    compared with all experts chosen (the choice itself is tested in fp32, and the router's kernel by itself)."""
    return name if dtype == torch.float32 else f"{name}, all experts"


def weights(cfg, seed):
    """A random checkpoint: {name: tensor}, every value exact in bf16, spread so that each mechanism matters."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in SodotarConfig.from_hf(cfg).checkpoint_shapes().items():
        leaf = name.rsplit(".", 1)[-1]
        r = torch.randn(shape, generator=g)
        if leaf in ("norm1", "norm2", "norm"):
            t = 1 + 0.2 * r
        elif ".hc" in name:
            t = {"in": 1.0 / shape[0] + 0.3 * r, "out": 0.7 + 0.4 * r, "mix": 0.8 * torch.eye(shape[0]) + 0.25 * r if leaf == "mix" else None}[leaf]
        elif name == "embed":
            t = r
        elif leaf == "sink":
            t = 1.0 + r
        elif leaf in ("lq1", "lk1", "lq2", "lk2"):
            t = 0.4 * r / shape[0] ** 0.25                       # not near 1, where flat maps would cancel to noise
        elif leaf == "correction":
            t = 0.2 * r
        elif leaf == "router":
            t = 3.0 * r / shape[-1] ** 0.5                       # no close calls between experts
        elif leaf == "q":
            t = 1.6 * r / shape[-1] ** 0.5                       # scores of a few units: attention is not flat
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


TOL = {torch.float32: 5e-5, torch.bfloat16: 0.12}
