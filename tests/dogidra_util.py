"""Small Dogidra configurations and random checkpoints for the tests."""
import json
import os

import torch

from dopurax_util import engine, run_portions, tokens  # noqa: F401
from zml_b200 import safetensors
from zml_b200.models.dogidra import DogidraConfig


def mixer(heads=4, kv_heads=2, dim=24, vdim=20, rot=16, window=37, pool=5, width=56, cap=15.0, base=5000.0, yarn=(3.0, 60, 8.0, 0.7), left=0.6,
          right=1.3, scale=None):
    r = {"base": base, "dims": rot}
    if yarn:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    side = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": r, "scale": dim ** -0.5 if scale is None else scale, "softcap": cap,
            "mask": {"size": window, "pool": pool}}
    return {"left": side, "left_scale": left, "right": {"width": width}, "right_scale": right}


def moe(experts=5, top=2, ff=40, scale=0.8, shared=24):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}}
    return dict(out, shared={"ff": shared}) if shared else out


def config(layers, width=96, vocab=130, eps=1e-5, taps=3, scale=1.6, loop=None):
    """`layers`: (mixer, feed-forward or None) pairs; `loop`: (start, stop, times)."""
    out = {"architecture": "Dogidra", "vocab": vocab, "width": width, "layers": [{"type": "parallel", "mixer": m, "mlp": f} for m, f in layers],
           "norm": {"eps": eps}, "embedding": {"scale": scale}, "canon": {"taps": taps}}
    return dict(out, loop=dict(zip(("start", "stop", "times"), loop))) if loop else out


CONFIGS = {
    # layers of different sizes, one without a feed-forward, three passes over the middle
    "mixed": config([(mixer(), moe()), (mixer(heads=3, kv_heads=1, window=50, pool=16, width=40, left=1.1, right=0.4), None),
                     (mixer(dim=32, rot=32, vdim=48, pool=7, window=64, width=72), moe(6, 3, 72, 1.2, 90)), (mixer(window=21, pool=4), moe(shared=0))],
                    loop=(1, 3, 3)),
    # one of everything: one head, one expert, a window of one token, blocks of one token, one tap, all factors one, the loop once
    "ones": config([(mixer(heads=1, kv_heads=1, dim=8, vdim=8, rot=2, window=1, pool=1, width=8, cap=1.0, base=10.0, yarn=(1.0, 1, 1.0, 1.0), left=1.0,
                           right=1.0, scale=1.0), moe(1, 1, 8, 1.0, 8))], width=40, vocab=65, taps=1, scale=1.0, loop=(0, 1, 1)),
    # nothing is a multiple of 8; no loop; positions that are not stretched; a scale of zero for the recurrence
    "odd": config([(mixer(heads=6, kv_heads=3, dim=13, vdim=10, rot=6, window=29, pool=3, width=37, yarn=None), moe(5, 2, 33, 0.8, 70)),
                   (mixer(heads=5, kv_heads=5, dim=11, vdim=17, rot=10, window=66, pool=11, width=51, right=0.0), moe(3, 1, 45, 2.0, 7))], width=51, vocab=77,
                  taps=5),
    # head sizes of the tensor-core kernels, blocks larger than a page, all layers loop, eight taps
    "wide": config([(mixer(heads=4, kv_heads=2, dim=128, vdim=128, rot=64, window=70, pool=6, width=160), moe(8, 4, 128, 0.5, 300)),
                    (mixer(heads=6, kv_heads=1, dim=100, vdim=72, rot=100, window=40, pool=16, width=96, cap=80.0), None),
                    (mixer(heads=2, kv_heads=1, dim=50, vdim=104, rot=24, window=30, pool=70, width=256), moe(40, 6, 24, 1.0, 64))], width=160, vocab=203,
                   taps=8, loop=(0, 3, 2)),
    # more query heads per key than a tile holds, sizes up to 256 and beyond the paged kernels, the loop at the end
    "heads": config([(mixer(heads=18, kv_heads=1, dim=16, vdim=24, rot=16, window=33, pool=8, width=64), None),
                     (mixer(heads=4, kv_heads=4, dim=100, vdim=256, rot=32, window=48, pool=32, width=24), moe(3, 2, 40, 1.0, 40)),
                     (mixer(heads=2, kv_heads=1, dim=260, vdim=30, rot=64, window=25, pool=9, width=200), None),
                     (mixer(heads=4, kv_heads=2, dim=64, vdim=40, rot=20, window=200, pool=2, width=32), None)], width=128, vocab=96, loop=(2, 4, 2)),
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
    for name, shape in DogidraConfig.from_hf(cfg).checkpoint_shapes().items():
        leaf = name.rsplit(".", 1)[-1]
        r = torch.randn(shape, generator=g)
        if name.endswith(".z.b"):
            t = -1.5 + r                                         # states that last a few tokens
        elif leaf in ("b", "correction"):
            t = 0.3 * r
        elif leaf.startswith("norm"):
            t = 1 + 0.2 * r
        elif leaf.startswith("canon"):
            t = 0.35 * r
        elif name == "embed":
            t = r
        elif leaf == "router":
            t = 3.0 * r / shape[-1] ** 0.5                       # no close calls between experts
        else:
            t = 1.2 * r / shape[-1] ** 0.5
        if name.endswith("q.norm"):
            t = 1.7 * t                                          # scores of a few units: attention is not flat
        if leaf in ("down", "in"):
            t = 0.5 * t                                          # squared units and repeated passes stay in range
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


TOL = {torch.float32: 3e-5, torch.bfloat16: 0.12}
