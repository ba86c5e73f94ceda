"""Dogidra: a decoder whose layers mix tokens by windowed attention and by a gated recurrence side by side, some of them run
several times, each followed by a routed mixture of experts with a shared one (or by nothing).

* The residual stream is fp32.  Every sublayer reads n + conv(n) with n = layernorm(x), a short causal convolution per channel.
* Attention (`ops.gqa`): one norm over all query heads and one over all key heads, partial rotation with stretched positions, a
  score cap, a sliding window and beside it the mean key and value of every block of tokens in front of the window.
* Gated recurrence (`ops.linear_attn.gated_scan`): gates and candidates from the current token only, a silu gate behind.
* Loop: a range of layers runs several times with the same weights; a pass begins with x <- W [x; x0], x0 the embedding.  Every
  pass has caches and states of its own.
* Mixture: the `top` experts by sigmoid score plus a correction, weighted by the scores alone; down(relu(up x)^2).

The input projections of both mixers are one GEMM; both write into one buffer, scaled, so their output projections and their sum
are one GEMM too.  The residual sum, the norm in front of the next sublayer and, in a decode step, its convolution are one launch;
behind a mixture it also sums the experts' rows.  W x0 is formed once for all passes.  Tensor parallelism splits heads, recurrent
channels, experts and the shared expert's hidden units; the loop's projection is replicated, partial sums are all-reduced in fp32.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Optional

import torch

from .. import ops
from ..moe import ops as moe_ops
from ..ops import gqa
from ..ops import linear_attn as la
from ..ops import stream
from ..parallel.comm import Comm
from . import common
from .decoder import AttnMeta, DecoderModel

PARALLEL = "parallel"
pad8 = stream.pad8


@dataclass
class MoeSpec:
    experts: int
    top: int
    ff: int
    scale: float
    shared_ff: int = 0              # 0: no shared expert

    @staticmethod
    def from_json(mlp: dict) -> "MoeSpec":
        if mlp.get("kind") != "moe":
            raise ValueError(f"unknown feed-forward kind {mlp.get('kind')!r}")
        r = mlp["router"]
        s = MoeSpec(int(r["experts"]), int(r["top"]), int(mlp["expert"]["ff"]), float(r["scale"]), int((mlp.get("shared") or {"ff": 0})["ff"]))
        if not 1 <= s.top <= s.experts:
            raise ValueError(f"cannot choose {s.top} of {s.experts} experts")
        return s

    def to_json(self) -> dict:
        out = {"kind": "moe", "expert": {"ff": self.ff}, "router": {"experts": self.experts, "top": self.top, "scale": self.scale}}
        if self.shared_ff:
            out["shared"] = {"ff": self.shared_ff}
        return out


@dataclass
class LayerSpec:
    """One entry of config.json's `layers`."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    width: int                      # channels of the recurrence
    left_scale: float
    right_scale: float
    rot: int
    base: float
    scale: float
    cap: float = 0.0                # 0: scores are not capped
    window: int = 0                 # 0: all earlier tokens
    pool: int = 0                   # tokens per pooled block, 0: none
    yarn: Optional[gqa.Yarn] = None
    moe: Optional[MoeSpec] = None

    @staticmethod
    def from_json(e: dict) -> "LayerSpec":
        if e["type"] != PARALLEL:
            raise ValueError(f"unknown layer type {e['type']!r}")
        m, a = e["mixer"], e["mixer"]["left"]
        rot, mask, sc = a["rot"], a.get("mask") or {}, a["rot"].get("scaling")
        s = LayerSpec(int(a["heads"]), int(a["kv_heads"]), int(a["dim"]), int(a["vdim"]), int(m["right"]["width"]), float(m["left_scale"]),
                      float(m["right_scale"]), int(rot["dims"]), float(rot["base"]), float(a["scale"]), float(a.get("softcap") or 0.0),
                      int(mask.get("size", 0)), int(mask.get("pool") or 0),
                      gqa.Yarn(*(float(sc[k]) for k in ("factor", "original", "fast", "slow"))) if sc else None,
                      MoeSpec.from_json(e["mlp"]) if e.get("mlp") is not None else None)
        if mask and s.window < 1:
            raise ValueError("mask.size must be positive")
        return s

    def to_json(self) -> dict:
        rot = {"base": self.base, "dims": self.rot}
        if self.yarn is not None:
            rot["scaling"] = {k: getattr(self.yarn, k) for k in ("factor", "original", "fast", "slow")}
        left = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "rot": rot, "scale": self.scale}
        if self.cap:
            left["softcap"] = self.cap
        if self.window:
            left["mask"] = {"size": self.window, **({"pool": self.pool} if self.pool else {})}
        mixer = {"left": left, "left_scale": self.left_scale, "right": {"width": self.width}, "right_scale": self.right_scale}
        return {"type": PARALLEL, "mixer": mixer, "mlp": self.moe.to_json() if self.moe is not None else None}

    def gqa_spec(self, heads: int, kv_heads: int) -> gqa.GqaSpec:
        return gqa.GqaSpec(heads, kv_heads, self.dim, self.vdim, self.rot, self.base, scale=self.scale, cap=self.cap, window=self.window,
                           pool=self.pool, whole_norm=True, yarn=self.yarn)


@dataclass
class DogidraConfig:
    vocab_size: int
    hidden_size: int
    layers: list                    # of LayerSpec
    norm_eps: float
    embed_scale: float
    taps: int
    loop: Optional[tuple] = None    # (start, stop, times)
    bos_token_id: Optional[int] = None
    eos_token_id: object = None
    max_position_embeddings: int = 1 << 20
    model_type: str = "dogidra"
    extra: dict = field(default_factory=dict)

    def __post_init__(self):
        if self.loop is not None:
            a, b, n = self.loop
            if not 0 <= a < b <= len(self.layers) or n < 1:
                raise ValueError(f"cannot loop layers {a} to {b} of {len(self.layers)} {n} times")
        if not 1 <= self.taps <= stream.MAX_TAPS:
            raise ValueError(f"the input convolutions take 1 to {stream.MAX_TAPS} taps, not {self.taps}")

    @classmethod
    def from_hf(cls, obj: dict) -> "DogidraConfig":
        for need in ("vocab", "width", "layers", "norm", "embedding", "canon"):
            if need not in obj:
                raise ValueError(f"config.json lacks {need}")
        kw = {k: obj[k] for k in ("bos_token_id", "eos_token_id") if obj.get(k) is not None}
        loop = obj.get("loop")
        return cls(int(obj["vocab"]), int(obj["width"]), [LayerSpec.from_json(e) for e in obj["layers"]], float(obj["norm"]["eps"]),
                   float(obj["embedding"]["scale"]), int(obj["canon"]["taps"]),
                   (int(loop["start"]), int(loop["stop"]), int(loop["times"])) if loop else None, **kw)

    def to_json(self) -> dict:
        out = {"architecture": "Dogidra", "vocab": self.vocab_size, "width": self.hidden_size, "layers": [s.to_json() for s in self.layers],
               "norm": {"eps": self.norm_eps}, "embedding": {"scale": self.embed_scale}, "canon": {"taps": self.taps}}
        if self.loop is not None:
            out["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        return out

    def runs(self) -> list[tuple[int, bool]]:
        """(layer, whether a pass of the loop begins with it) in the order the layers run."""
        n = len(self.layers)
        a, b, times = self.loop or (n, n, 1)
        return [(i, False) for i in range(a)] + [(i, i == a) for _ in range(times) for i in range(a, b)] + [(i, False) for i in range(b, n)]

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def eos_ids(self) -> list[int]:
        return common.eos_list(self.eos_token_id)

    def checkpoint_shapes(self) -> dict:
        """Names and shapes of a checkpoint of this configuration."""
        d = self.hidden_size
        out = {"embed": (self.vocab_size, d)}
        if self.loop is not None:
            out["loop.in"] = (d, 2 * d)
        for i, s in enumerate(self.layers):
            t, a, r, f = f"l{i}.", f"l{i}.mix.left.", f"l{i}.mix.right.", f"l{i}.mlp."
            nq, nk = s.heads * s.dim, s.kv_heads * s.dim
            for q in (1, 2) if s.moe is not None else (1,):
                out.update({t + f"norm{q}": (d,), t + f"norm{q}.b": (d,), t + f"canon{q}": (d, self.taps)})
            out.update({a + "q": (nq, d), a + "k": (nk, d), a + "v": (s.kv_heads * s.vdim, d), a + "q.norm": (nq,), a + "k.norm": (nk,),
                        a + "o": (d, s.heads * s.vdim)})
            for x in "zx":
                out.update({r + x: (s.width, d), r + x + ".b": (s.width,)})
            out.update({r + "g": (s.width, d), r + "o": (d, s.width)})
            if s.moe is not None:
                e = s.moe
                for k in range(e.experts):
                    out.update({f + f"e{k}.up": (e.ff, d), f + f"e{k}.down": (d, e.ff)})
                out.update({f + "router": (e.experts, d), f + "correction": (e.experts,)})
                if e.shared_ff:
                    out.update({f + "shared.up": (e.shared_ff, d), f + "shared.down": (d, e.shared_ff)})
        out.update({"final.norm": (d,), "final.norm.b": (d,)})
        return out

    def num_params(self) -> int:
        n = 0
        for shape in self.checkpoint_shapes().values():
            k = 1
            for a in shape:
                k *= a
            n += k
        return n


def _preset(width, vocab, pattern, mixer, moe, taps=4, loop=None, scale=1.0, **kw):
    """`pattern`: one letter per layer, P, lower case without a feed-forward."""
    layers = [{"type": PARALLEL, "mixer": mixer, "mlp": moe if ch.isupper() else None} for ch in pattern]
    out = dict(architecture="Dogidra", width=width, vocab=vocab, layers=layers, norm={"eps": 1e-6}, embedding={"scale": scale}, canon={"taps": taps}, **kw)
    return dict(out, loop=dict(zip(("start", "stop", "times"), loop))) if loop else out


def _mixer(heads, kv_heads, dim, vdim, rot, window, pool, width, cap=50.0, base=1e6, factor=4.0, original=4096, left=0.7, right=0.7):
    return {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5, "softcap": cap,
                     "rot": {"base": base, "dims": rot, "scaling": {"factor": factor, "original": original, "fast": 32.0, "slow": 1.0}},
                     "mask": {"size": window, "pool": pool}},
            "left_scale": left, "right": {"width": width}, "right_scale": right}


def _moe(experts, top, ff, shared, scale=1.0):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}, "shared": {"ff": shared}}


PRESETS = {
    # shapes of the benchmark (random-init): 12 layers of which four run twice, 32 experts of which four run, and a shared one
    "dogidra-3b": _preset(2048, 65536, "P" * 12, _mixer(16, 4, 128, 128, 64, 1024, 16, 2048), _moe(32, 4, 1536, 1536), loop=(4, 8, 2)),
    "dogidra-10b": _preset(4096, 65536, "P" * 12, _mixer(32, 8, 128, 128, 64, 1024, 16, 4096), _moe(32, 4, 2304, 2304), loop=(4, 8, 2)),
    "tiny-dogidra-test": _preset(192, 320, "PpP", _mixer(6, 2, 48, 32, 24, 70, 6, 120, cap=20.0, base=20000.0, original=64), _moe(6, 3, 80, 112, 1.5),
                                 taps=3, loop=(1, 3, 2), scale=2.0),
}


class _Moe:
    __slots__ = ("router", "correction", "up", "down", "shared")


class _Layer:
    """Weights of one layer, this rank's heads, channels and experts; `mix` holds the mixer's matrices."""

    def __init__(self, spec: LayerSpec):
        self.spec = spec
        self.norm1 = self.norm2 = None                # (weight, bias)
        self.conv1 = self.conv2 = None                # fp32 [taps, d]
        self.mix: dict = {}
        self.moe: Optional[_Moe] = None
        self.attn: Optional[gqa.GqaSpec] = None
        self.inv_freq = None
        self.width = 0                                # recurrent channels here

    def tensors(self):
        ts = [*self.norm1, *(self.norm2 or ()), self.conv1, self.conv2, *self.mix.values()]
        if self.moe is not None:
            ts += [self.moe.router, self.moe.correction, self.moe.up, self.moe.down]
        return [t for t in ts if isinstance(t, torch.Tensor)]


class _Run:
    """One run of a layer: the per-sequence state that it has to itself."""

    def __init__(self, layer: _Layer, begins: bool):
        self.layer, self.begins = layer, begins
        self.conv1: Optional[stream.InputConv] = None
        self.conv2: Optional[stream.InputConv] = None
        self.state = None                             # fp32 [slots, width]

    def states(self):
        return [t for t in (self.conv1.state, self.conv2.state if self.conv2 is not None else None, self.state) if t is not None]


class DogidraModel(DecoderModel):
    KERNEL_SOURCES = ("runtime", "gemm_bf16", "gemm_2cta", "gemm_f32", "elementwise", "stream_f32", "attention", "attention_tc", "gqa_attention",
                      "gated_scan", "moe", "moe_f32")
    FP32_ON_GPU = True
    # as for the other decoders with an fp32 stream: the prefill's kernels are long, overlapping their launches gains nothing
    SERIAL_PREFILL = True

    def __init__(self, config: DogidraConfig, comm: Optional[Comm] = None, device="cpu", dtype=torch.bfloat16):
        super().__init__(config, comm, device, dtype)
        p = self.comm.world
        for i, s in enumerate(config.layers):
            if s.heads % p or s.width % p or (s.moe is not None and (s.moe.experts % p or s.moe.shared_ff % p)):
                raise ValueError(f"layer {i}: heads, recurrent channels, experts or the shared expert's hidden units do not split over {p} ranks")
        self.layers: list[_Layer] = []
        self.runs: list[_Run] = []
        self.final_bias = self.loop_x = self.loop_x0 = None
        self._splits: dict = {}

    # ------------------------------------------------------------------ weights
    def _assemble(self, get) -> "DogidraModel":
        """Builds the layers from `get(name, rows=None, cols=None, f32=False)`, which returns a tensor of the checkpoint's
        layout (optionally this rank's rows or columns) in the model's dtype or in fp32."""
        c, (r, p) = self.config, (self.comm.rank, self.comm.world)
        d = c.hidden_size
        self.embed = get("embed").contiguous()
        self.final_norm, self.final_bias = get("final.norm", f32=True), get("final.norm.b", f32=True)
        self.lm_head = ops.pad_k(self.embed[self.v_rng[0]:self.v_rng[1]])
        self._pad_lm_head()
        if c.loop is not None:
            w = get("loop.in")
            self.loop_x, self.loop_x0 = ops.pad_k(w[:, :d]).contiguous(), ops.pad_k(w[:, d:]).contiguous()
        for i, s in enumerate(c.layers):
            L, t = _Layer(s), f"l{i}."
            L.norm1, L.conv1 = (get(t + "norm1", f32=True), get(t + "norm1.b", f32=True)), self._taps(get, t + "canon1")
            self._assemble_mixer(L, get, t + "mix.", common.shard_range(s.heads, r, p), common.kv_head_shard(s.kv_heads, r, p),
                                 common.shard_range(s.width, r, p))
            if s.moe is not None:
                L.norm2, L.conv2 = (get(t + "norm2", f32=True), get(t + "norm2.b", f32=True)), self._taps(get, t + "canon2")
                L.moe = self._assemble_moe(s.moe, get, t + "mlp.")
            self.layers.append(L)
        self.runs = [_Run(self.layers[i], begins) for i, begins in c.runs()]
        return self

    def _taps(self, get, name: str):
        w = get(name, f32=True).t().contiguous()
        if w.shape[0] != self.config.taps:
            raise ValueError(f"{name}: {w.shape[0]} convolution taps in the checkpoint, {self.config.taps} in config.json")
        return w

    def _assemble_mixer(self, L: _Layer, get, m: str, heads, kv, chan) -> None:
        s, a, b = L.spec, m + "left.", m + "right."
        L.attn, L.width = s.gqa_spec(heads[1] - heads[0], kv[1] - kv[0]), chan[1] - chan[0]
        L.inv_freq = L.attn.inv_freq(self.device)
        nq, nk, nv = (tuple(n * x for x in r) for r, n in ((heads, s.dim), (kv, s.dim), (heads, s.vdim)))
        qkv = [get(a + "q", rows=nq), get(a + "k", rows=nk), get(a + "v", rows=(kv[0] * s.vdim, kv[1] * s.vdim))]
        cols = sum(w.shape[0] for w in qkv)
        fill = torch.zeros((pad8(cols) - cols, qkv[0].shape[1]), dtype=self.dtype, device=self.device)     # the other side's columns start on 16 bytes
        L.mix["proj"] = ops.pad_k(torch.cat(qkv + [fill] + [get(b + x, rows=chan) for x in "zxg"], 0))
        L.mix["q_norm"], L.mix["k_norm"] = (get(a + x, f32=True)[n[0]:n[1]].contiguous() for x, n in (("q.norm", nq), ("k.norm", nk)))
        L.mix["z_bias"], L.mix["x_bias"] = (get(b + x, f32=True)[chan[0]:chan[1]].contiguous() for x in ("z.b", "x.b"))
        L.mix["o"] = ops.pad_k(torch.cat([get(a + "o", cols=nv), get(b + "o", cols=chan)], 1)).contiguous()

    def _assemble_moe(self, e: MoeSpec, get, m: str) -> _Moe:
        r, p = self.comm.rank, self.comm.world
        w = _Moe()
        w.router, w.correction, w.shared = ops.pad_k(get(m + "router")), get(m + "correction", f32=True).contiguous(), 0
        up, down = (torch.stack([get(m + f"e{k}.{x}") for k in range(*common.shard_range(e.experts, r, p))]) for x in ("up", "down"))
        w.up, w.down = moe_ops.pad_plain_experts(up, down)
        if e.shared_ff:
            units = common.shard_range(e.shared_ff, r, p)
            pieces = moe_ops.shared_pieces(get(m + "shared.up", rows=units), get(m + "shared.down", cols=units), w.up.shape[1])
            su, sd = moe_ops.pad_plain_experts(*pieces)
            w.shared, w.up, w.down = su.shape[0], torch.cat([su, w.up], 0), torch.cat([sd, w.down], 0)
        return w

    def load(self, store, prefix: str = "") -> "DogidraModel":
        def get(name, rows=None, cols=None, f32=False):
            return store.load_tensor(prefix + name, device=self.device, dtype=torch.float32 if f32 else self.dtype, rows=rows, cols=cols)
        return self._assemble(get)

    def init_random(self, seed: int = 0, std: float = 0.02) -> "DogidraModel":
        """Random-init weights of this architecture: matrices N(0, std), norms around one, gates that keep most of the state."""
        shapes = self.config.checkpoint_shapes()
        order = {n: k for k, n in enumerate(shapes)}

        def get(name, rows=None, cols=None, f32=False):
            shape, leaf = shapes[name], name.rsplit(".", 1)[-1]
            g = torch.Generator(device=self.device).manual_seed((seed * 1000003 + order[name] * 7919 + 1) % (2 ** 63))
            w = torch.empty(shape, dtype=torch.float32 if len(shape) == 1 or f32 else self.dtype, device=self.device)
            if leaf.startswith("norm"):
                w.normal_(1.0, 0.05, generator=g)
            elif leaf.startswith("canon"):
                w.normal_(0.0, 0.2, generator=g)
            elif name.endswith(".z.b"):
                w.uniform_(-4.0, 0.0, generator=g)
            elif len(shape) == 1:
                w.normal_(0.0, 0.1, generator=g)
            else:
                w.normal_(0.0, std, generator=g)
            if rows is not None:
                w = w[rows[0]:rows[1]]
            if cols is not None:
                w = w[:, cols[0]:cols[1]]
            w = w.to(torch.bfloat16)                      # the values a checkpoint could hold
            return w.to(torch.float32 if f32 else self.dtype)
        return self._assemble(get)

    def checkpoint_shapes(self) -> dict:
        return self.config.checkpoint_shapes()

    def state_dict_hf(self) -> dict:
        """This rank's weights under their checkpoint names, in bf16; a complete checkpoint when TP == 1."""
        d = self.config.hidden_size
        out = {"embed": self.embed, "final.norm": self.final_norm, "final.norm.b": self.final_bias}
        if self.loop_x is not None:
            out["loop.in"] = torch.cat([self.loop_x[:, :d], self.loop_x0[:, :d]], 1)
        for i, L in enumerate(self.layers):
            s, t, a, b, x, n = L.spec, f"l{i}.", f"l{i}.mix.left.", f"l{i}.mix.right.", L.mix, L.attn
            for q, norm, conv in ((1, L.norm1, L.conv1), (2, L.norm2, L.conv2)):
                if norm is not None:
                    out.update({t + f"norm{q}": norm[0], t + f"norm{q}.b": norm[1], t + f"canon{q}": conv.t()})
            w, nq, nk, nv = x["proj"][:, :d], n.heads * s.dim, n.kv_heads * s.dim, n.heads * s.vdim
            out.update({a + "q": w[:nq], a + "k": w[nq:nq + nk], a + "v": w[nq + nk:n.columns()], a + "q.norm": x["q_norm"], a + "k.norm": x["k_norm"],
                        a + "o": x["o"][:, :nv], b + "o": x["o"][:, nv:nv + L.width], b + "z.b": x["z_bias"], b + "x.b": x["x_bias"]})
            for name, cols in zip("zxg", self._recurrent(L, w.t())):
                out[b + name] = cols.t()
            if L.moe is not None:
                out.update(self._moe_state(s.moe, L.moe, f"l{i}.mlp."))
        return {k: v.to(torch.bfloat16).contiguous() for k, v in out.items()}

    def _moe_state(self, e: MoeSpec, w: _Moe, f: str) -> dict:
        d, n = self.config.hidden_size, w.shared
        out = {f + "router": w.router[:, :d], f + "correction": w.correction}
        e0 = self.comm.rank * (w.up.shape[0] - n)
        for k in range(w.up.shape[0] - n):
            out.update({f + f"e{e0 + k}.up": w.up[n + k, :e.ff, :d], f + f"e{e0 + k}.down": w.down[n + k, :d, :e.ff]})
        if n:
            units = e.shared_ff // self.comm.world
            out.update({f + "shared.up": w.up[:n].flatten(0, 1)[:units, :d],
                        f + "shared.down": w.down[:n, :d].transpose(0, 1).flatten(1)[:, :units]})
        return out

    def weight_bytes(self) -> int:
        ts = [t for t in (self.embed, self.final_norm, self.final_bias, self.loop_x, self.loop_x0) if t is not None] + [t for L in self.layers for t in L.tensors()]
        if self.lm_head.data_ptr() != self.embed[self.v_rng[0]:].data_ptr():
            ts.append(self.lm_head)
        return sum(t.numel() * t.element_size() for t in ts)

    # ------------------------------------------------------------------ cache and state
    def alloc_kv_cache(self, num_pages: int, page_size: int):
        """Per run of a layer its keys, values and pooled blocks."""
        return [r.layer.attn.alloc_cache(num_pages, page_size, self.dtype, self.device) for r in self.runs]

    def alloc_state(self, num_slots: int) -> None:
        """Per-sequence state of every run: the last inputs of its convolutions and the recurrence."""
        d, rows = self.config.hidden_size, self.config.taps - 1
        zeros = lambda *shape: torch.zeros((num_slots, *shape), dtype=torch.float32, device=self.device)
        for r in self.runs:
            L = r.layer
            r.conv1 = stream.InputConv(L.conv1, zeros(rows, d))
            r.conv2 = stream.InputConv(L.conv2, zeros(rows, d)) if L.conv2 is not None else None
            r.state = zeros(L.width)

    def state_bytes_per_slot(self) -> int:
        return sum(t[0].numel() * t.element_size() for r in self.runs for t in r.states())

    def _layer_splits(self, L: _Layer, batch: int, max_seq_len: int) -> int:
        key = (L.attn, batch, max_seq_len)
        if key not in self._splits:
            self._splits[key] = ops.decode_plan_splits(batch, L.attn.kv_heads, L.attn.visible(max_seq_len))
        return self._splits[key]

    def decode_splits(self, batch: int, max_seq_len: int) -> int:
        return max((self._layer_splits(L, batch, max_seq_len) for L in self.layers), default=1)

    # ------------------------------------------------------------------ forward
    def _recurrent(self, L: _Layer, proj):
        """The recurrence's columns z, x, gate of a projection."""
        at, n = pad8(L.attn.columns()), L.width
        return tuple(proj[:, at + i * n:at + (i + 1) * n] for i in range(3))

    def mixer(self, run: _Run, h, meta: AttnMeta, q_start, cache):
        L, s, m = run.layer, run.layer.attn, run.layer.mix
        t, step = h.shape[0], not meta.is_prefill
        proj = ops.gemm(h, m["proj"], static_w=True)
        sumsq, totals = None, None
        if self.comm.world > 1:                       # the norms go over all ranks' heads
            sumsq = self.comm.all_reduce_(gqa.sums_of_squares(proj, s))
            totals = (s.heads * s.dim * self.comm.world, s.kv_heads * s.dim * self.comm.world)
        q = gqa.prep(proj, m["q_norm"], m["k_norm"], L.inv_freq, meta.positions, meta.slot_mapping, cache, self.config.norm_eps, s, sumsq=sumsq,
                     totals=totals, step_table=meta.block_table if step else None)
        if not step:
            gqa.pool_new(cache, meta, s)
        nv, n = s.heads * s.vdim, s.heads * s.vdim + L.width
        both = (torch.empty if n % 8 == 0 else torch.zeros)((t, pad8(n)), dtype=self.dtype, device=self.device)
        plan = self.layer_plan(meta, lambda length: self._layer_splits(L, t, length))
        gqa.attention(q, None, cache, plan, s, out=both[:, :nv], out_scale=L.spec.left_scale)
        la.gated_scan(*self._recurrent(L, proj), m["z_bias"], m["x_bias"], run.state, q_start, meta.seq_lens, meta.state_slots,
                      L.spec.right_scale, both[:, nv:n], decode=step, num_blocks=self._blocks(meta, la.GATED_ROWS))
        y = ops.gemm(both, m["o"], out_dtype=torch.float32, static_w=True)
        return y if self.comm.world == 1 else self.comm.all_reduce_(y)

    def mixture(self, L: _Layer, h):
        """The experts' outputs, still to be summed with their weights (summed over the ranks with more than one)."""
        e, w = L.spec.moe, L.moe
        z = ops.gemm(h, w.router, out_dtype=torch.float32, static_w=True)
        ids, weights = moe_ops.route(z, e.top, e.experts, w.correction, w.shared, self.comm.rank * (w.up.shape[0] - w.shared), scores="sigmoid",
                                     normalize=False, scale=e.scale, shared_gate=False)
        rows, pos = moe_ops.expert_rows(h, ids, w.up, w.down, 0, e.experts + w.shared, "relu2")
        y = stream.ExpertRows(rows, pos, weights)
        return y if self.comm.world == 1 else self.comm.all_reduce_(y.sum(self.config.hidden_size))

    @staticmethod
    def _blocks(meta: AttnMeta, rows: int) -> Optional[int]:
        """Blocks of `rows` tokens of the step's sequences (None: not known on the host)."""
        if not meta.is_prefill or meta.q_start_host is None:
            return None
        n = meta.plans.get(("blocks", rows))
        if n is None:
            qs = meta.q_start_host
            n = meta.plans[("blocks", rows)] = sum((b - a + rows - 1) // rows for a, b in zip(qs, qs[1:]))
        return n

    def _read(self, x, y, norm, conv, meta: AttnMeta, q_start, inplace: bool = True):
        """The stream x + y and what a sublayer reads of it: the norm plus its convolution."""
        kw = dict(w=norm[0], b=norm[1], eps=self.config.norm_eps, inplace=inplace)
        if not meta.is_prefill:
            return stream.add_norm(x, y, act_dtype=self.dtype, conv=conv, seq_lens=meta.seq_lens, slots=meta.state_slots, **kw)
        x, n = stream.add_norm(x, y, act_dtype=torch.float32, padded=False, **kw)
        return x, stream.stream_conv(n, conv, q_start, meta.seq_lens, meta.state_slots, self.dtype, self._blocks(meta, stream.CONV_BLOCK), padded=True)

    def layer_steps(self, ids, meta: AttnMeta, kv_cache):
        """The stack, one run of a layer at a time: yields the fp32 stream behind every run (a buffer the next one overwrites)."""
        if meta.state_slots is None:
            raise ValueError("Dogidra needs AttnMeta.state_slots (one state slot per sequence)")
        if self.runs and self.runs[0].conv1 is None:
            self.alloc_state(int(meta.state_slots.max().item()) + 1)
        q_start = meta.q_start
        if q_start is None:
            q_start = torch.arange(ids.shape[0] + 1, dtype=torch.int32, device=self.device)
        wide = dict(out_dtype=torch.float32, static_w=True)
        x, part = stream.embedding_f32(ids, self.embed, self.config.embed_scale), None
        if self.loop_x is not None:
            _, xa = stream.add_norm(x, act_dtype=self.dtype)
            part = ops.gemm(xa, self.loop_x0, **wide)                      # what x0 adds at the start of every pass

        def enter(run, x, y, xa):
            """(stream, input of the run's mixer) in front of a run, y still to be added to x; xa: x in the model's dtype."""
            if run.begins:
                x, y = part, ops.gemm(xa, self.loop_x, **wide)
            return self._read(x.contiguous(), y, run.layer.norm1, run.conv1, meta, q_start, inplace=not run.begins)

        if self.runs:
            x, h = enter(self.runs[0], x, None, xa if self.loop_x is not None else None)
        for i, run in enumerate(self.runs):
            L = run.layer
            y = self.mixer(run, h, meta, q_start, kv_cache[i])
            if L.moe is not None:
                x, h = self._read(x, y, L.norm2, run.conv2, meta, q_start)
                y = self.mixture(L, h)
            nxt = self.runs[i + 1] if i + 1 < len(self.runs) else None
            if nxt is None:
                x, _ = stream.add_norm(x, y)
                yield x
            elif nxt.begins:
                x, xa = stream.add_norm(x, y, act_dtype=self.dtype)
                yield x
                x, h = enter(nxt, x, None, xa)
            else:
                x, h = enter(nxt, x, y, None)
                yield x

    def hidden_states(self, ids, meta: AttnMeta, kv_cache):
        x = stream.embedding_f32(ids, self.embed, self.config.embed_scale) if not self.runs else None
        for x in self.layer_steps(ids, meta, kv_cache):
            pass
        return x

    def logits(self, x, rows=None):
        if rows is not None:
            x = x.index_select(0, rows.long() if rows.dtype != torch.int64 else rows)
        _, n = stream.add_norm(x, w=self.final_norm, b=self.final_bias, eps=self.config.norm_eps, act_dtype=self.dtype, keep_x=False)
        return self.head_logits(n)
