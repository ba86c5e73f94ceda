"""Sodotar: a decoder with several residual streams (hyper-connections) whose layers mix tokens by latent attention or by
chunked differential attention, in any order, each followed by a routed mixture of experts with a shared one (or by nothing).

* Hyper-connections (`ops.stream.hyper_norm`): fp32 streams x_1 .. x_s per token, all the embedding at the start.  A sublayer
  reads norm(sum_s in[s] x_s); its output y gives x_t <- sum_s mix[s, t] x_s + out[t] y.  The head reads the streams' sum.
* Latent attention (`ops.latent`): keys and values from one cached latent per token plus a rotary key part common to the
  heads, queries straight from the input, a learned sink per head.
* Differential attention (`ops.gqa`, two maps per head): the maps' results are subtracted and normalised; a position sees its
  own chunk of the sequence; a layer may use the keys and values of an earlier one (`kv_from`).
* Mixture: the `top` experts by softmax score plus a correction, weighted by the scores alone; clipped gated units; a shared
  expert times a sigmoid gate.

The input projections of a layer are one GEMM.  The streams' update behind a sublayer, the mix and the norm in front of the next
one are one launch; behind a mixture it also sums the experts' rows.  The shared expert's hidden units are cut into pieces of
an expert's size that every token is routed to, so router, shared gate, routed and shared experts take the launches of a plain
mixture.  Tensor parallelism splits heads, experts and the shared expert's hidden units; partial sums are all-reduced in fp32.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Optional

import torch

from .. import ops
from ..moe import ops as moe_ops
from ..ops import gqa
from ..ops import latent as lat
from ..ops import stream
from ..parallel.comm import Comm
from . import common
from .decoder import AttnMeta, DecoderModel

LATENT, ATTENTION = "latent_attention", "attention"


@dataclass
class MoeSpec:
    experts: int
    top: int
    ff: int
    limit: float
    shared_ff: int = 0              # 0: no shared expert
    shared_limit: float = 0.0

    @staticmethod
    def from_json(mlp: dict) -> "MoeSpec":
        if mlp.get("kind") != "moe":
            raise ValueError(f"unknown feed-forward kind {mlp.get('kind')!r}")
        sh = mlp.get("shared") or {"ff": 0, "limit": 0.0}
        s = MoeSpec(int(mlp["router"]["experts"]), int(mlp["router"]["top"]), int(mlp["expert"]["ff"]), float(mlp["expert"]["limit"]), int(sh["ff"]),
                    float(sh["limit"]))
        if not 1 <= s.top <= s.experts:
            raise ValueError(f"cannot choose {s.top} of {s.experts} experts")
        return s

    def to_json(self) -> dict:
        out = {"kind": "moe", "expert": {"ff": self.ff, "limit": self.limit}, "router": {"experts": self.experts, "top": self.top}}
        if self.shared_ff:
            out["shared"] = {"ff": self.shared_ff, "limit": self.shared_limit}
        return out


@dataclass
class LayerSpec:
    """One entry of config.json's `layers`."""
    kind: str
    heads: int
    dim: int                        # latent attention: unrotated dimensions; attention: per map
    vdim: int
    rot: int
    base: float
    scale: float
    rank: int = 0                   # latent attention
    kv_heads: int = 0               # attention
    chunk: int = 0
    diff: float = 0.0
    kv_from: Optional[int] = None   # layer whose keys and values this one uses
    moe: Optional[MoeSpec] = None

    @staticmethod
    def from_json(e: dict) -> "LayerSpec":
        kind, m = e["type"], e["mixer"]
        if kind not in (LATENT, ATTENTION):
            raise ValueError(f"unknown layer type {kind!r}")
        kw = dict(moe=MoeSpec.from_json(e["mlp"]) if e.get("mlp") is not None else None)
        if kind == LATENT:
            if m["rot"]["dims"] != m["rot_dim"] or m["rot_dim"] % 2:
                raise ValueError("latent attention rotates the whole rotated part: rot.dims must equal rot_dim, an even number")
            kw.update(rank=int(m["kv_rank"]))
        else:
            kw.update(kv_heads=int(m["kv_heads"]), chunk=int(m["mask"]["size"]), diff=float(m["diff"]),
                      kv_from=int(m["kv_from"]) if m.get("kv_from") is not None else None)
            if kw["chunk"] < 1:
                raise ValueError("mask.size must be positive")
        return LayerSpec(kind, int(m["heads"]), int(m["dim"]), int(m["vdim"]), int(m["rot"]["dims"]), float(m["rot"]["base"]), float(m["scale"]), **kw)

    def to_json(self) -> dict:
        m = {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "rot": {"base": self.base, "dims": self.rot}, "scale": self.scale}
        if self.kind == LATENT:
            m.update(kv_rank=self.rank, rot_dim=self.rot)
        else:
            m.update(kv_heads=self.kv_heads, mask={"size": self.chunk}, diff=self.diff)
            if self.kv_from is not None:
                m["kv_from"] = self.kv_from
        return {"type": self.kind, "mixer": m, "mlp": self.moe.to_json() if self.moe is not None else None}


@dataclass
class SodotarConfig:
    vocab_size: int
    hidden_size: int
    layers: list                    # of LayerSpec
    norm_eps: float
    streams: int
    logit_scale: float
    bos_token_id: Optional[int] = None
    eos_token_id: object = None
    max_position_embeddings: int = 1 << 20
    model_type: str = "sodotar"
    extra: dict = field(default_factory=dict)

    def __post_init__(self):
        if not 1 <= self.streams <= stream.MAX_STREAMS:
            raise ValueError(f"{self.streams} streams; 1 to {stream.MAX_STREAMS} are supported")
        for i, s in enumerate(self.layers):
            if s.kv_from is None:
                continue
            src = self.layers[s.kv_from] if 0 <= s.kv_from < i else None
            if src is None or src.kind != ATTENTION or src.kv_from is not None:
                raise ValueError(f"layer {i}: kv_from {s.kv_from} is not an earlier attention layer with keys of its own")
            if (src.kv_heads, src.dim, src.vdim) != (s.kv_heads, s.dim, s.vdim):
                raise ValueError(f"layer {i} cannot use the keys of layer {s.kv_from}: other sizes")

    @classmethod
    def from_hf(cls, obj: dict) -> "SodotarConfig":
        for need in ("vocab", "width", "layers", "norm", "streams", "logit_scale"):
            if need not in obj:
                raise ValueError(f"config.json lacks {need}")
        kw = {k: obj[k] for k in ("bos_token_id", "eos_token_id") if obj.get(k) is not None}
        return cls(int(obj["vocab"]), int(obj["width"]), [LayerSpec.from_json(e) for e in obj["layers"]], float(obj["norm"]["eps"]),
                   int(obj["streams"]), float(obj["logit_scale"]), **kw)

    def to_json(self) -> dict:
        return {"architecture": "Sodotar", "vocab": self.vocab_size, "width": self.hidden_size, "layers": [s.to_json() for s in self.layers],
                "norm": {"eps": self.norm_eps}, "streams": self.streams, "logit_scale": self.logit_scale}

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def eos_ids(self) -> list[int]:
        return common.eos_list(self.eos_token_id)

    def checkpoint_shapes(self) -> dict:
        """Names and shapes of a checkpoint of this configuration."""
        d, n = self.hidden_size, self.streams
        out = {"embed": (self.vocab_size, d)}
        for i, s in enumerate(self.layers):
            t, m, f = f"l{i}.", f"l{i}.mix.", f"l{i}.mlp."
            out[t + "norm1"] = (d,)
            if s.kind == LATENT:
                out.update({m + "q": (s.heads * (s.dim + s.rot), d), m + "dkv": (s.rank + s.rot, d), m + "dkv.norm": (s.rank,),
                            m + "uk": (s.heads * s.dim, s.rank), m + "uv": (s.heads * s.vdim, s.rank), m + "sink": (s.heads,)})
            else:
                out[m + "q"] = (s.heads * 2 * s.dim, d)
                if s.kv_from is None:
                    out.update({m + "k": (s.kv_heads * 2 * s.dim, d), m + "v": (s.kv_heads * s.vdim, d)})
                out.update({m + x: (s.dim,) for x in ("lq1", "lk1", "lq2", "lk2")})
            out[m + "o"] = (d, s.heads * s.vdim)
            if s.moe is not None:
                e = s.moe
                out[t + "norm2"] = (d,)
                for k in range(e.experts):
                    out.update({f + f"e{k}.gate": (e.ff, d), f + f"e{k}.up": (e.ff, d), f + f"e{k}.down": (d, e.ff)})
                out.update({f + "router": (e.experts, d), f + "correction": (e.experts,)})
                if e.shared_ff:
                    out.update({f + "shared.gate": (e.shared_ff, d), f + "shared.up": (e.shared_ff, d), f + "shared.down": (d, e.shared_ff),
                                f + "shared.sg": (1, d)})
            for q in (1, 2) if s.moe is not None else (1,):
                out.update({t + f"hc{q}.in": (n,), t + f"hc{q}.out": (n,), t + f"hc{q}.mix": (n, n)})
        out["final.norm"] = (d,)
        return out

    def num_params(self) -> int:
        n = 0
        for shape in self.checkpoint_shapes().values():
            k = 1
            for a in shape:
                k *= a
            n += k
        return n


def _preset(width, vocab, pattern, latent, attn, moe, streams=4, logit_scale=1.0, **kw):
    """`pattern`: one letter per layer - L (latent attention), A (attention) or S (attention with the keys and values of the last
    A), lower case without a feed-forward."""
    layers, last = [], None
    for i, ch in enumerate(pattern):
        mixer = dict(latent if ch in "Ll" else attn)
        if ch in "Aa":
            last = i
        elif ch in "Ss":
            mixer["kv_from"] = last
        layers.append({"type": LATENT if ch in "Ll" else ATTENTION, "mixer": mixer, "mlp": moe if ch.isupper() else None})
    return dict(architecture="Sodotar", width=width, vocab=vocab, layers=layers, norm={"eps": 1e-6}, streams=streams, logit_scale=logit_scale, **kw)


def _latent(heads, dim, rot, vdim, rank, base=1e6):
    return dict(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=rank, rot={"base": base, "dims": rot}, scale=(dim + rot) ** -0.5)


def _attn(heads, kv_heads, dim, vdim, rot, chunk, diff=0.5, base=1e6):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, rot={"base": base, "dims": rot}, scale=dim ** -0.5, mask={"size": chunk}, diff=diff)


def _moe(experts, top, ff, shared, limit=7.0):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}, "shared": {"ff": shared, "limit": limit}}


PRESETS = {
    # shapes of the benchmark (random-init): latent and differential attention in turn, every other one of the latter with the keys
    # and values of the one before, 32 experts of which four run, and a shared one
    "sodotar-3b": _preset(2048, 65536, "LALS" * 4, _latent(16, 128, 64, 128, 512), _attn(16, 4, 64, 128, 32, 4096), _moe(32, 4, 1024, 1024)),
    "sodotar-10b": _preset(4096, 65536, "LALS" * 4, _latent(32, 128, 64, 128, 512), _attn(32, 8, 64, 128, 32, 4096), _moe(32, 4, 1536, 1536)),
    "tiny-sodotar-test": _preset(192, 320, "LAsA", _latent(4, 40, 24, 32, 72), _attn(6, 2, 24, 40, 12, 60), _moe(6, 2, 80, 112, 2.0), streams=3,
                                 logit_scale=1.5),
}


class _Moe:
    __slots__ = ("router", "correction", "gate_up", "down", "limits", "shared")


class _Layer:
    """Weights of one layer, this rank's heads and experts; `mix` holds the mixer's matrices."""

    def __init__(self, spec: LayerSpec):
        self.spec = spec
        self.norm1 = self.norm2 = None
        self.hc1: Optional[stream.HyperMix] = None
        self.hc2: Optional[stream.HyperMix] = None
        self.mix: dict = {}
        self.moe: Optional[_Moe] = None
        self.latent: Optional[lat.LatentDims] = None
        self.attn: Optional[gqa.GqaSpec] = None
        self.diff: Optional[gqa.DiffMix] = None
        self.inv_freq = None

    def tensors(self):
        ts = [self.norm1, self.norm2] + list(self.mix.values())
        for h in (self.hc1, self.hc2):
            if h is not None:
                ts += [h.inp, h.mix, h.out]
        if self.moe is not None:
            ts += [self.moe.router, self.moe.correction, self.moe.gate_up, self.moe.down, self.moe.limits]
        return [t for t in ts if isinstance(t, torch.Tensor)]


class SodotarModel(DecoderModel):
    KERNEL_SOURCES = ("runtime", "gemm_bf16", "gemm_2cta", "gemm_f32", "elementwise", "stream_f32", "attention", "attention_tc", "gqa_attention",
                      "latent_attention", "latent_prefill_tc", "latent_decode", "moe", "moe_f32")
    FP32_ON_GPU = True
    # as for the other decoders with an fp32 stream: the prefill's kernels are long, overlapping their launches gains nothing
    SERIAL_PREFILL = True

    def __init__(self, config: SodotarConfig, comm: Optional[Comm] = None, device="cpu", dtype=torch.bfloat16):
        super().__init__(config, comm, device, dtype)
        p = self.comm.world
        for i, s in enumerate(config.layers):
            if s.heads % p or (s.moe is not None and (s.moe.experts % p or s.moe.shared_ff % p)):
                raise ValueError(f"layer {i}: heads, experts or the shared expert's hidden units do not split over {p} ranks")
        self.layers: list[_Layer] = []
        self.head_norm = self.all_streams = None
        self._splits: dict = {}

    # ------------------------------------------------------------------ weights
    def _assemble(self, get) -> "SodotarModel":
        """Builds the layers from `get(name, rows=None, cols=None, f32=False)`, which returns a tensor of the checkpoint's
        layout (optionally this rank's rows or columns) in the model's dtype or in fp32."""
        c, (r, p) = self.config, (self.comm.rank, self.comm.world)
        self.embed = get("embed").contiguous()
        self.final_norm = get("final.norm", f32=True)
        self.head_norm = self.final_norm * c.logit_scale               # the logits' factor rides on the last norm
        self.all_streams = torch.ones(c.streams, dtype=torch.float32, device=self.device)
        self.lm_head = ops.pad_k(self.embed[self.v_rng[0]:self.v_rng[1]])
        self._pad_lm_head()
        for i, s in enumerate(c.layers):
            L, t = _Layer(s), f"l{i}."
            L.norm1, L.hc1 = get(t + "norm1", f32=True), self._hyper(get, t + "hc1.")
            (self._assemble_latent if s.kind == LATENT else self._assemble_attention)(L, get, t + "mix.", common.shard_range(s.heads, r, p))
            if s.moe is not None:
                L.norm2, L.hc2 = get(t + "norm2", f32=True), self._hyper(get, t + "hc2.")
                L.moe = self._assemble_moe(s.moe, get, t + "mlp.")
            self.layers.append(L)
        return self

    def _hyper(self, get, h: str) -> stream.HyperMix:
        return stream.HyperMix(get(h + "in", f32=True).contiguous(), get(h + "mix", f32=True).contiguous(), get(h + "out", f32=True).contiguous())

    def _assemble_latent(self, L: _Layer, get, m: str, heads) -> None:
        s, H = L.spec, heads[1] - heads[0]
        L.latent = lat.LatentDims(H, s.dim, s.rot, s.vdim, s.rank, 0, 0, s.scale, s.base)
        L.inv_freq = L.latent.inv_freq(self.device)
        pairs = lat.halves_to_pairs(s.rot).to(self.device)
        q = get(m + "q", rows=(heads[0] * (s.dim + s.rot), heads[1] * (s.dim + s.rot))).reshape(H, s.dim + s.rot, -1)
        dkv = get(m + "dkv")
        L.mix["proj"] = ops.pad_k(torch.cat([torch.cat([q[:, :s.dim], q[:, s.dim:][:, pairs]], 1).flatten(0, 1), dkv[:s.rank], dkv[s.rank:][pairs]], 0))
        L.mix["c_norm"] = get(m + "dkv.norm", f32=True)
        L.mix["sink"] = get(m + "sink", f32=True)[heads[0]:heads[1]].contiguous()
        uk = get(m + "uk", rows=(heads[0] * s.dim, heads[1] * s.dim))
        uv = get(m + "uv", rows=(heads[0] * s.vdim, heads[1] * s.vdim))
        L.mix["uk_t"] = uk.reshape(H, s.dim, s.rank).transpose(1, 2).contiguous()                 # [H, rank, dim]
        L.mix["ukv"] = torch.cat([uk, uv], 0).contiguous()                                        # [H (dim + vdim), rank]
        L.mix["o"] = ops.pad_k(get(m + "o", cols=(heads[0] * s.vdim, heads[1] * s.vdim)))

    def _assemble_attention(self, L: _Layer, get, m: str, heads) -> None:
        s = L.spec
        kv = common.kv_head_shard(s.kv_heads, self.comm.rank, self.comm.world)
        L.attn = gqa.GqaSpec(heads[1] - heads[0], kv[1] - kv[0], s.dim, s.vdim, s.rot, s.base, scale=s.scale, chunk=s.chunk, maps=2)
        L.inv_freq = L.attn.inv_freq(self.device)
        proj = [get(m + "q", rows=(heads[0] * 2 * s.dim, heads[1] * 2 * s.dim))]
        if s.kv_from is None:
            proj += [get(m + "k", rows=(kv[0] * 2 * s.dim, kv[1] * 2 * s.dim)), get(m + "v", rows=(kv[0] * s.vdim, kv[1] * s.vdim))]
        L.mix["proj"] = ops.pad_k(torch.cat(proj, 0))
        for x in ("lq1", "lk1", "lq2", "lk2"):
            L.mix[x] = get(m + x, f32=True)
        dot = lambda a, b: float((L.mix[a].double() * L.mix[b].double()).sum().exp())
        L.diff = gqa.DiffMix(dot("lq1", "lk1") - dot("lq2", "lk2") + s.diff, 1.0 - s.diff, self.config.norm_eps)
        L.mix["o"] = ops.pad_k(get(m + "o", cols=(heads[0] * s.vdim, heads[1] * s.vdim)))

    def _assemble_moe(self, e: MoeSpec, get, m: str) -> _Moe:
        r, p = self.comm.rank, self.comm.world
        w = _Moe()
        experts = common.shard_range(e.experts, r, p)
        rows = [get(m + "router")]
        gate, up, down = (torch.stack([get(m + f"e{k}.{x}") for k in range(*experts)]) for x in ("gate", "up", "down"))
        w.gate_up, w.down = moe_ops.pad_experts(gate, up, down)
        w.correction = get(m + "correction", f32=True).contiguous()
        limits, w.shared = [e.limit] * (experts[1] - experts[0]), 0
        if e.shared_ff:
            rows.append(get(m + "shared.sg"))
            units = common.shard_range(e.shared_ff, r, p)
            n, size = units[1] - units[0], w.down.shape[2]                     # hidden units here, units of an expert as stored
            w.shared = (n + size - 1) // size
            fill, d = w.shared * size - n, gate.shape[2]
            pad = torch.nn.functional.pad
            cut = lambda x: pad(get(m + "shared." + x, rows=units), (0, 0, 0, fill)).reshape(w.shared, size, d)
            sd = pad(get(m + "shared.down", cols=units), (0, fill)).reshape(d, w.shared, size).transpose(0, 1)
            sg, sd = moe_ops.pad_experts(cut("gate"), cut("up"), sd)
            w.gate_up, w.down = torch.cat([sg, w.gate_up], 0), torch.cat([sd, w.down], 0)
            limits = [e.shared_limit] * w.shared + limits
        w.router = ops.pad_k(torch.cat(rows, 0))
        w.limits = torch.tensor(limits, dtype=torch.float32, device=self.device)
        return w

    def load(self, store, prefix: str = "") -> "SodotarModel":
        def get(name, rows=None, cols=None, f32=False):
            return store.load_tensor(prefix + name, device=self.device, dtype=torch.float32 if f32 else self.dtype, rows=rows, cols=cols)
        return self._assemble(get)

    def init_random(self, seed: int = 0, std: float = 0.02) -> "SodotarModel":
        """Random-init weights of this architecture: matrices N(0, std), norms around one, streams that mostly keep themselves."""
        shapes = self.config.checkpoint_shapes()
        order = {n: k for k, n in enumerate(shapes)}

        def get(name, rows=None, cols=None, f32=False):
            shape, leaf = shapes[name], name.rsplit(".", 1)[-1]
            g = torch.Generator(device=self.device).manual_seed((seed * 1000003 + order[name] * 7919 + 1) % (2 ** 63))
            w = torch.empty(shape, dtype=torch.float32 if len(shape) == 1 or f32 else self.dtype, device=self.device)
            if leaf.startswith("norm"):
                w.normal_(1.0, 0.05, generator=g)
            elif ".hc" in name:
                w.normal_(0.0, 0.1, generator=g)
                if leaf == "mix":
                    w += torch.eye(shape[0], device=self.device)
                else:
                    w += 1.0 / shape[0] if leaf == "in" else 1.0
            elif leaf in ("lq1", "lk1", "lq2", "lk2", "correction"):
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
        out = {"embed": self.embed, "final.norm": self.final_norm}
        for i, L in enumerate(self.layers):
            s, t, m, x = L.spec, f"l{i}.", f"l{i}.mix.", L.mix
            out[t + "norm1"] = L.norm1
            w = x["proj"][:, :d]
            if L.latent is not None:
                H, hd = L.latent.heads, s.dim + s.rot
                halves = torch.argsort(lat.halves_to_pairs(s.rot)).to(w.device)
                q, dkv = w[:H * hd].reshape(H, hd, d), w[H * hd:]
                out.update({m + "q": torch.cat([q[:, :s.dim], q[:, s.dim:][:, halves]], 1).flatten(0, 1),
                            m + "dkv": torch.cat([dkv[:s.rank], dkv[s.rank:][halves]], 0), m + "dkv.norm": x["c_norm"], m + "sink": x["sink"],
                            m + "uk": x["ukv"][:H * s.dim], m + "uv": x["ukv"][H * s.dim:], m + "o": x["o"][:, :H * s.vdim]})
            else:
                a = L.attn
                nq, nk = a.rows_q * s.dim, a.kv_heads * 2 * s.dim
                out.update({m + "q": w[:nq], m + "o": x["o"][:, :a.heads * s.vdim]})
                out.update({m + k: x[k] for k in ("lq1", "lk1", "lq2", "lk2")})
                if s.kv_from is None:
                    out.update({m + "k": w[nq:nq + nk], m + "v": w[nq + nk:]})
            for q, h in ((1, L.hc1), (2, L.hc2)):
                if h is not None:
                    out.update({t + f"hc{q}.in": h.inp, t + f"hc{q}.out": h.out, t + f"hc{q}.mix": h.mix})
            if L.moe is not None:
                out[t + "norm2"] = L.norm2
                out.update(self._moe_state(s.moe, L.moe, f"l{i}.mlp."))
        return {k: v.to(torch.bfloat16).contiguous() for k, v in out.items()}

    def _moe_state(self, e: MoeSpec, w: _Moe, f: str) -> dict:
        d, n = self.config.hidden_size, w.shared
        out = {f + "router": w.router[:e.experts, :d], f + "correction": w.correction}
        gate, up = moe_ops.deinterleave_gate_up(w.gate_up)
        e0 = self.comm.rank * (gate.shape[0] - n)
        for k in range(gate.shape[0] - n):
            out.update({f + f"e{e0 + k}.gate": gate[n + k, :e.ff, :d], f + f"e{e0 + k}.up": up[n + k, :e.ff, :d], f + f"e{e0 + k}.down": w.down[n + k, :d, :e.ff]})
        if n:
            units = e.shared_ff // self.comm.world
            whole = lambda x: x[:n].flatten(0, 1)[:units, :d]
            out.update({f + "shared.gate": whole(gate), f + "shared.up": whole(up), f + "shared.sg": w.router[e.experts:, :d],
                        f + "shared.down": w.down[:n, :d].transpose(0, 1).flatten(1)[:, :units]})
        return out

    def weight_bytes(self) -> int:
        ts = [self.embed, self.final_norm] + [t for L in self.layers for t in L.tensors()]
        if self.lm_head.data_ptr() != self.embed[self.v_rng[0]:].data_ptr():
            ts.append(self.lm_head)
        return sum(t.numel() * t.element_size() for t in ts)

    # ------------------------------------------------------------------ cache
    def alloc_kv_cache(self, num_pages: int, page_size: int):
        """Per layer one paged tensor of latents or a pair of keys and values; a layer with `kv_from` has that layer's."""
        out = []
        for L in self.layers:
            if L.latent is not None:
                out.append(torch.zeros((num_pages, page_size, L.latent.row), dtype=self.dtype, device=self.device))
            elif L.spec.kv_from is not None:
                out.append(out[L.spec.kv_from])
            else:
                out.append(L.attn.alloc_cache(num_pages, page_size, self.dtype, self.device))
        return out

    def _layer_splits(self, L: _Layer, batch: int, max_seq_len: int) -> int:
        if L.latent is not None:
            return lat.decode_plan_splits(batch, L.latent, max_seq_len)
        return ops.decode_plan_splits(batch, L.attn.kv_heads, L.attn.visible(max_seq_len))

    def decode_splits(self, batch: int, max_seq_len: int) -> int:
        return max((self._layer_splits(L, batch, max_seq_len) for L in self.layers), default=1)

    def _plan(self, i: int, batch: int, meta: AttnMeta) -> AttnMeta:
        L = self.layers[i]

        def splits(max_seq_len):
            key = (L.latent or L.attn, batch, max_seq_len)
            if key not in self._splits:
                self._splits[key] = self._layer_splits(L, batch, max_seq_len)
            return self._splits[key]
        return self.layer_plan(meta, splits)

    # ------------------------------------------------------------------ forward
    def _out_proj(self, a, w):
        """A mixer's output projection, the partial sums of all ranks added: what the streams take."""
        y = ops.gemm(a, w, out_dtype=torch.float32, static_w=True)
        return y if self.comm.world == 1 else self.comm.all_reduce_(y)

    def latent_attention(self, L: _Layer, h, meta: AttnMeta, cache):
        d, m = L.latent, L.mix
        proj = ops.gemm(h, m["proj"], static_w=True)
        nq = d.heads * (d.dim + d.rot)
        lat.prep(proj[:, nq:], None, m["c_norm"], L.inv_freq, meta.positions, meta.slot_mapping, cache, self.config.norm_eps, d)
        a = lat.latent_attention(proj[:, :nq], None, m["uk_t"], m["ukv"], L.inv_freq, cache, meta, d, m["sink"])
        return self._out_proj(a, m["o"])

    def attention(self, L: _Layer, h, meta: AttnMeta, cache):
        a, m = L.attn, L.mix
        proj = ops.gemm(h, m["proj"], static_w=True)
        q = gqa.prep(proj, None, None, L.inv_freq, meta.positions, meta.slot_mapping, cache, self.config.norm_eps, a,
                     queries_only=L.spec.kv_from is not None)
        return self._out_proj(gqa.attention(q, None, cache, meta, a, L.diff), m["o"])

    def mixture(self, L: _Layer, h):
        """The experts' outputs, still to be summed with their weights (summed over the ranks with more than one)."""
        e, w = L.spec.moe, L.moe
        z = ops.gemm(h, w.router, out_dtype=torch.float32, static_w=True)
        local = w.down.shape[0] - w.shared
        ids, weights = moe_ops.route(z, e.top, e.experts, w.correction, w.shared, self.comm.rank * local)
        rows, pos = moe_ops.expert_rows(h, ids, w.gate_up, w.down, 0, e.experts + w.shared, "clipped_glu", w.limits)
        y = stream.ExpertRows(rows, pos, weights)
        return y if self.comm.world == 1 else self.comm.all_reduce_(y.sum(self.config.hidden_size))

    def layer_steps(self, ids, meta: AttnMeta, kv_cache):
        """The stack, one layer at a time: yields the fp32 streams [T, streams, d] behind every layer (a buffer the next layer
        overwrites)."""
        c = self.config
        norm = dict(eps=c.norm_eps, act_dtype=self.dtype)
        x = stream.embedding_f32(ids, self.embed, streams=c.streams)
        h = None
        if self.layers:
            x, h = stream.hyper_norm(x, inp=self.layers[0].hc1.inp, w=self.layers[0].norm1, **norm)
        for i, L in enumerate(self.layers):
            plan = self._plan(i, ids.shape[0], meta)
            y = (self.latent_attention if L.latent is not None else self.attention)(L, h, plan, kv_cache[i])
            nxt = self.layers[i + 1] if i + 1 < len(self.layers) else None
            nxt = dict(inp=nxt.hc1.inp, w=nxt.norm1) if nxt is not None else {}
            if L.moe is not None:
                x, h = stream.hyper_norm(x, y, L.hc1, L.hc2.inp, L.norm2, **norm)
                x, h = stream.hyper_norm(x, self.mixture(L, h), L.hc2, **nxt, **norm)
            else:
                x, h = stream.hyper_norm(x, y, L.hc1, **nxt, **norm)
            yield x

    def hidden_states(self, ids, meta: AttnMeta, kv_cache):
        x = stream.embedding_f32(ids, self.embed, streams=self.config.streams) if not self.layers else None
        for x in self.layer_steps(ids, meta, kv_cache):
            pass
        return x

    def logits(self, x, rows=None):
        if rows is not None:
            x = x.index_select(0, rows.long() if rows.dtype != torch.int64 else rows)
        _, n = stream.hyper_norm(x, inp=self.all_streams, w=self.head_norm, eps=self.config.norm_eps, act_dtype=self.dtype)
        return self.head_logits(n)
