"""Kirisun: a decoder whose layers mix tokens by gated attention or by a delta rule with a decay per key channel, in any order,
each followed by a routed mixture of experts (or by nothing).

* The residual stream is fp32; every sublayer has a norm in front and one behind: x <- x + m * norm(f(norm(x))).
* Attention (`ops.gqa`): normalised queries and keys, partial rotation with linearly scaled angles, a score cap, a sliding
  window with kept first tokens, a sink, a sigmoid gate on the result.
* Channel delta (`ops.linear_attn.ChannelDelta`): short convolutions, unit keys and queries, low-rank decays and output gates.
* Mixture: the `top` experts by biased router logits, weighted by the softmax over the chosen logits; swiglu experts.

The input projections of a layer are one GEMM (attention: [q | k | v | gate]; delta: [q | k | v | write gate | both low-rank
inputs], then both low-rank outputs as one GEMM with a block-diagonal weight).  The norm behind a sublayer, the residual sum
and the norm in front of the next one are one launch; behind a mixture it also sums the experts' rows.  Tensor parallelism
splits heads and experts; low-rank inputs are replicated, partial sums are all-reduced in fp32.
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

ATTENTION, DELTA = "attention", "channel_delta"
pad8 = stream.pad8


@dataclass
class LayerSpec:
    """One entry of config.json's `layers`."""
    kind: str
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    experts: int = 0                # 0: no feed-forward
    top: int = 0
    ff: int = 0
    taps: int = 0                   # channel_delta
    attn: dict = field(default_factory=dict)      # attention: the other fields of ops.gqa.GqaSpec

    @staticmethod
    def from_json(e: dict) -> "LayerSpec":
        kind, m, mlp = e["type"], e["mixer"], e.get("mlp")
        kw = {}
        if mlp is not None:
            if mlp.get("kind") != "moe":
                raise ValueError(f"unknown feed-forward kind {mlp.get('kind')!r}")
            kw.update(experts=int(mlp["router"]["experts"]), top=int(mlp["router"]["top"]), ff=int(mlp["expert"]["ff"]))
            if not 1 <= kw["top"] <= kw["experts"]:
                raise ValueError(f"cannot choose {kw['top']} of {kw['experts']} experts")
        if kind == DELTA:
            kw.update(taps=int(m["conv"]))
        elif kind == ATTENTION:
            rot, mask = m["rot"], m.get("mask") or {}
            kw.update(attn=dict(rot=int(rot["dims"]), base=float(rot["base"]), factor=float((rot.get("scaling") or {}).get("factor", 1.0)),
                                scale=float(m["scale"]), cap=float(m.get("softcap") or 0.0), window=int(mask.get("size", 0)),
                                keep=int(mask.get("keep_first", 0)), sink=True))
        else:
            raise ValueError(f"unknown layer type {kind!r}")
        return LayerSpec(kind, int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), **kw)

    def to_json(self) -> dict:
        m = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim}
        if self.kind == DELTA:
            m["conv"] = self.taps
        else:
            a = self.attn
            m.update(rot={"base": a["base"], "dims": a["rot"], "scaling": {"factor": a["factor"]}}, scale=a["scale"], softcap=a["cap"],
                     mask={"size": a["window"], "keep_first": a["keep"]})
        mlp = {"kind": "moe", "expert": {"ff": self.ff}, "router": {"experts": self.experts, "top": self.top}} if self.experts else None
        return {"type": self.kind, "mixer": m, "mlp": mlp}


@dataclass
class KirisunConfig:
    vocab_size: int
    hidden_size: int
    layers: list                    # of LayerSpec
    norm_eps: float
    embed_scale: float
    residual_mult: float
    decay_rank: int = 64            # ranks of random-init models; checkpoints give them by the shapes of mix.a1 and mix.g1
    gate_rank: int = 64
    bos_token_id: Optional[int] = None
    eos_token_id: object = None
    max_position_embeddings: int = 1 << 20
    model_type: str = "kirisun"
    extra: dict = field(default_factory=dict)

    @classmethod
    def from_hf(cls, obj: dict) -> "KirisunConfig":
        for need in ("vocab", "width", "layers", "norm", "embedding", "residual_mult"):
            if need not in obj:
                raise ValueError(f"config.json lacks {need}")
        kw = {k: obj[k] for k in ("bos_token_id", "eos_token_id", "decay_rank", "gate_rank") if obj.get(k) is not None}
        return cls(int(obj["vocab"]), int(obj["width"]), [LayerSpec.from_json(e) for e in obj["layers"]], float(obj["norm"]["eps"]),
                   float(obj["embedding"]["scale"]), float(obj["residual_mult"]), **kw)

    def to_json(self) -> dict:
        return {"architecture": "Kirisun", "vocab": self.vocab_size, "width": self.hidden_size, "layers": [s.to_json() for s in self.layers],
                "norm": {"eps": self.norm_eps}, "embedding": {"scale": self.embed_scale}, "residual_mult": self.residual_mult}

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def eos_ids(self) -> list[int]:
        return common.eos_list(self.eos_token_id)

    def num_params(self) -> int:
        d, n = self.hidden_size, 2 * self.vocab_size * self.hidden_size + self.hidden_size
        for s in self.layers:
            n += 2 * d + (2 * d + s.experts * (3 * d * s.ff + d + 1) if s.experts else 0)
            nq, nk, nv = s.heads * s.dim, s.kv_heads * s.dim, s.heads * s.vdim
            if s.kind == ATTENTION:
                n += d * (nq + nk + s.kv_heads * s.vdim + 2 * nv) + 2 * s.dim
            else:
                n += (d + s.taps) * (2 * nk + nv) + d * (s.heads + nv) + self.decay_rank * (d + nq) + self.gate_rank * (d + nv) + s.heads + nq + s.vdim
        return n


def _preset(width, vocab, pattern, attn, delta, moe, scale=None, mult=0.5, **kw):
    """`pattern`: one letter per layer - A (attention) or D (channel delta), lower case without a feed-forward."""
    layers = []
    for ch in pattern:
        mlp = {"kind": "moe", "expert": {"ff": moe[2]}, "router": {"experts": moe[0], "top": moe[1]}} if ch.isupper() else None
        layers.append({"type": ATTENTION, "mixer": attn, "mlp": mlp} if ch in "Aa" else {"type": DELTA, "mixer": delta, "mlp": mlp})
    return dict(architecture="Kirisun", width=width, vocab=vocab, layers=layers, norm={"eps": 1e-6},
                embedding={"scale": width ** 0.5 if scale is None else scale}, residual_mult=mult, **kw)


def _attn(heads, kv_heads, dim, vdim, rot, window, keep, cap=50.0, base=1e6, factor=2.0):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, rot={"base": base, "dims": rot, "scaling": {"factor": factor}},
                scale=dim ** -0.5, softcap=cap, mask={"size": window, "keep_first": keep})


def _delta(heads, kv_heads, dim, vdim, taps):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=taps)


PRESETS = {
    # shapes of the benchmark (random-init): attention and delta layers in turn, 32 experts of which four run
    "kirisun-3b": _preset(2048, 65536, "AD" * 8, _attn(16, 4, 128, 128, 64, 4096, 16), _delta(16, 16, 128, 128, 4), (32, 4, 1024), decay_rank=128,
                          gate_rank=128),
    "kirisun-10b": _preset(4096, 65536, "AD" * 8, _attn(32, 8, 128, 128, 64, 4096, 16), _delta(32, 32, 128, 128, 4), (32, 4, 1536), decay_rank=128,
                           gate_rank=128),
    "tiny-kirisun-test": _preset(192, 320, "ADdA", _attn(6, 2, 48, 32, 24, 70, 3, cap=20.0, base=20000.0), _delta(4, 2, 40, 24, 3), (6, 3, 80),
                                 decay_rank=20, gate_rank=12),
}


class _Moe:
    __slots__ = ("router", "bias", "gate_up", "down")


class _Layer:
    """Weights of one layer, this rank's heads and experts; `mix` holds the mixer's matrices."""

    def __init__(self, spec: LayerSpec):
        self.spec = spec
        self.norm1 = self.norm1b = self.norm2 = self.norm2b = None
        self.mix: dict = {}
        self.moe: Optional[_Moe] = None
        self.attn: Optional[gqa.GqaSpec] = None
        self.inv_freq = None
        self.delta: Optional[la.ChannelDelta] = None
        self.ranks = (0, 0)                           # delta: low-rank sizes of the decay and of the output gate

    def tensors(self):
        ts = [self.norm1, self.norm1b, self.norm2, self.norm2b] + list(self.mix.values())
        if self.moe is not None:
            ts += [self.moe.router, self.moe.bias, self.moe.gate_up, self.moe.down]
        if self.delta is not None:
            ts += [self.delta.conv_w, self.delta.a_log, self.delta.dt_bias, self.delta.norm]
        return [t for t in ts if isinstance(t, torch.Tensor)]


class KirisunModel(DecoderModel):
    KERNEL_SOURCES = ("runtime", "gemm_bf16", "gemm_2cta", "gemm_f32", "elementwise", "stream_f32", "attention", "attention_tc",
                      "gqa_attention", "channel_delta", "moe", "moe_f32")
    FP32_ON_GPU = True
    # as for the other decoder with an fp32 stream: the prefill's kernels are long, overlapping their launches gains nothing
    SERIAL_PREFILL = True

    def __init__(self, config: KirisunConfig, comm: Optional[Comm] = None, device="cpu", dtype=torch.bfloat16):
        super().__init__(config, comm, device, dtype)
        p = self.comm.world
        for i, s in enumerate(config.layers):
            if s.heads % p or s.experts % p:
                raise ValueError(f"layer {i}: {s.heads} heads / {s.experts} experts do not split over {p} ranks")
        self.layers: list[_Layer] = []

    # ------------------------------------------------------------------ weights
    def _assemble(self, get) -> "KirisunModel":
        """Builds the layers from `get(name, rows=None, cols=None, f32=False)`, which returns a tensor of the checkpoint's
        layout (optionally this rank's rows or columns) in the model's dtype or in fp32."""
        c, (r, p) = self.config, (self.comm.rank, self.comm.world)
        self.embed = get("embed").contiguous()
        self.final_norm = get("final.norm", f32=True)
        self.lm_head = ops.pad_k(get("head", rows=self.v_rng))
        self._pad_lm_head()
        for i, s in enumerate(c.layers):
            L, t = _Layer(s), f"l{i}."
            heads, kv = common.shard_range(s.heads, r, p), common.kv_head_shard(s.kv_heads, r, p)
            L.norm1, L.norm1b = get(t + "norm1", f32=True), get(t + "norm1b", f32=True)
            (self._assemble_attention if s.kind == ATTENTION else self._assemble_delta)(L, get, t + "mix.", heads, kv)
            if s.experts:
                L.norm2, L.norm2b = get(t + "norm2", f32=True), get(t + "norm2b", f32=True)
                L.moe = self._assemble_moe(s, get, t + "mlp.", common.shard_range(s.experts, r, p))
            self.layers.append(L)
        return self

    def _assemble_attention(self, L: _Layer, get, m: str, heads, kv) -> None:
        s, H, G = L.spec, heads[1] - heads[0], kv[1] - kv[0]
        L.attn = gqa.GqaSpec(H, G, s.dim, s.vdim, **s.attn)
        L.inv_freq = L.attn.inv_freq(self.device)
        nv = (heads[0] * s.vdim, heads[1] * s.vdim)
        qkv = [get(m + "q", rows=(heads[0] * s.dim, heads[1] * s.dim)), get(m + "k", rows=(kv[0] * s.dim, kv[1] * s.dim)),
               get(m + "v", rows=(kv[0] * s.vdim, kv[1] * s.vdim))]
        cols = sum(w.shape[0] for w in qkv)
        fill = torch.zeros((pad8(cols) - cols, qkv[0].shape[1]), dtype=self.dtype, device=self.device)         # the gate's columns start on 16 bytes
        L.mix["proj"] = ops.pad_k(torch.cat(qkv + [fill, get(m + "g", rows=nv)], 0))
        L.mix["q_norm"], L.mix["k_norm"] = get(m + "q.norm", f32=True), get(m + "k.norm", f32=True)
        L.mix["o"] = ops.pad_k(get(m + "o", cols=nv))

    def _assemble_delta(self, L: _Layer, get, m: str, heads, kv) -> None:
        s, H, G = L.spec, heads[1] - heads[0], kv[1] - kv[0]
        nk, nh, nv = ((a * n, b * n) for (a, b), n in ((kv, s.dim), (heads, s.dim), (heads, s.vdim)))
        conv = torch.cat([get(m + f"{x}.conv", rows=n, f32=True) for x, n in (("q", nk), ("k", nk), ("v", nv))], 0).t().contiguous()
        if conv.shape[0] != s.taps:
            raise ValueError(f"{m}: {conv.shape[0]} convolution taps in the checkpoint, {s.taps} in config.json")
        L.delta = la.ChannelDelta(H, G, s.dim, s.vdim, conv, get(m + "A_log", f32=True)[heads[0]:heads[1]].contiguous(),
                                  get(m + "dt_bias", f32=True)[nh[0]:nh[1]].contiguous(), get(m + "norm", f32=True), self.config.norm_eps)
        a1, g1, a2, g2 = get(m + "a1"), get(m + "g1"), get(m + "a2", rows=nh), get(m + "g2", rows=nv)
        zeros = lambda rows, like: torch.zeros((rows, like.shape[1]), dtype=like.dtype, device=like.device)
        L.ranks = (a1.shape[0], g1.shape[0])
        ranks, mixed = sum(L.ranks), L.delta.channels + H
        L.mix["proj"] = ops.pad_k(torch.cat([get(m + "q", rows=nk), get(m + "k", rows=nk), get(m + "v", rows=nv), get(m + "b", rows=heads),
                                             zeros(pad8(mixed) - mixed, a1), a1, g1, zeros(pad8(ranks) - ranks, a1)], 0))
        low = torch.zeros((a2.shape[0] + g2.shape[0], pad8(ranks)), dtype=a2.dtype, device=a2.device)          # block diagonal
        low[:a2.shape[0], :a1.shape[0]] = a2
        low[a2.shape[0]:, a1.shape[0]:ranks] = g2
        L.mix["low"] = low
        L.mix["o"] = ops.pad_k(get(m + "o", cols=nv))

    def _assemble_moe(self, s: LayerSpec, get, m: str, experts) -> _Moe:
        w = _Moe()
        w.router = ops.pad_k(get(m + "router"))
        w.bias = get(m + "router.b")
        gate, up, down = (torch.stack([get(m + f"e{e}.{x}") for e in range(*experts)]) for x in ("gate", "up", "down"))
        w.gate_up, w.down = moe_ops.pad_experts(gate, up, down)
        return w

    def load(self, store, prefix: str = "") -> "KirisunModel":
        def get(name, rows=None, cols=None, f32=False):
            return store.load_tensor(prefix + name, device=self.device, dtype=torch.float32 if f32 else self.dtype, rows=rows, cols=cols)
        return self._assemble(get)

    def init_random(self, seed: int = 0, std: float = 0.02) -> "KirisunModel":
        """Random-init weights of this architecture: matrices N(0, std), norms around one, decays spread over time scales."""
        shapes = self.checkpoint_shapes()
        order = {n: k for k, n in enumerate(shapes)}

        def get(name, rows=None, cols=None, f32=False):
            shape, leaf = shapes[name], name.rsplit(".", 1)[-1]
            g = torch.Generator(device=self.device).manual_seed((seed * 1000003 + order[name] * 7919 + 1) % (2 ** 63))
            w = torch.empty(shape, dtype=torch.float32 if len(shape) == 1 or f32 else self.dtype, device=self.device)
            if leaf.startswith("norm"):
                w.normal_(1.0, 0.05, generator=g)
            elif leaf == "A_log":
                w.uniform_(0.0, 2.0, generator=g)
            elif leaf == "dt_bias":
                w.uniform_(-6.0, -1.0, generator=g)
            elif leaf == "conv":
                w.normal_(0.0, 0.4, generator=g)
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
        """Names and shapes of a checkpoint of this configuration."""
        c, d = self.config, self.config.hidden_size
        out = {"embed": (c.vocab_size, d)}
        for i, s in enumerate(c.layers):
            t, m, f = f"l{i}.", f"l{i}.mix.", f"l{i}.mlp."
            nq, nk, nv = s.heads * s.dim, s.kv_heads * s.dim, s.heads * s.vdim
            out.update({t + "norm1": (d,), t + "norm1b": (d,)})
            if s.kind == ATTENTION:
                out.update({m + "q": (nq, d), m + "k": (nk, d), m + "v": (s.kv_heads * s.vdim, d), m + "q.norm": (s.dim,), m + "k.norm": (s.dim,),
                            m + "g": (nv, d), m + "o": (d, nv)})
            else:
                for x, n in (("q", nk), ("k", nk), ("v", nv)):
                    out.update({m + x: (n, d), m + x + ".conv": (n, s.taps)})
                out.update({m + "b": (s.heads, d), m + "A_log": (s.heads,), m + "norm": (s.vdim,), m + "a1": (c.decay_rank, d),
                            m + "a2": (nq, c.decay_rank), m + "dt_bias": (nq,), m + "g1": (c.gate_rank, d), m + "g2": (nv, c.gate_rank), m + "o": (d, nv)})
            if s.experts:
                out.update({t + "norm2": (d,), t + "norm2b": (d,), f + "router": (s.experts, d), f + "router.b": (s.experts,)})
                for e in range(s.experts):
                    out.update({f + f"e{e}.gate": (s.ff, d), f + f"e{e}.up": (s.ff, d), f + f"e{e}.down": (d, s.ff)})
        out.update({"final.norm": (d,), "head": (c.vocab_size, d)})
        return out

    def state_dict_hf(self) -> dict:
        """This rank's weights under their checkpoint names, in bf16; a complete checkpoint when TP == 1."""
        d = self.config.hidden_size
        out = {"embed": self.embed, "final.norm": self.final_norm, "head": self.lm_head[:self.v_rng[1] - self.v_rng[0], :d]}
        for i, L in enumerate(self.layers):
            s, t, m, f, x = L.spec, f"l{i}.", f"l{i}.mix.", f"l{i}.mlp.", L.mix
            out.update({t + "norm1": L.norm1, t + "norm1b": L.norm1b})
            if s.kind == ATTENTION:
                a = L.attn
                nq, nk, nv = a.heads * s.dim, a.kv_heads * s.dim, a.kv_heads * s.vdim
                w = x["proj"][:, :d]
                out.update({m + "q": w[:nq], m + "k": w[nq:nq + nk], m + "v": w[nq + nk:nq + nk + nv], m + "g": w[pad8(nq + nk + nv):],
                            m + "q.norm": x["q_norm"], m + "k.norm": x["k_norm"], m + "o": x["o"][:, :a.heads * s.vdim]})
            else:
                a = L.delta
                nk, nh, nv = a.kv_heads * s.dim, a.heads * s.dim, a.heads * s.vdim
                w, conv, low = x["proj"][:, :d], a.conv_w.t(), x["low"]
                ra, rg = L.ranks
                at = pad8(a.channels + a.heads)
                for name, r0, r1 in (("q", 0, nk), ("k", nk, 2 * nk), ("v", 2 * nk, a.channels)):
                    out.update({m + name: w[r0:r1], m + name + ".conv": conv[r0:r1]})
                out.update({m + "b": w[a.channels:a.channels + a.heads], m + "a1": w[at:at + ra], m + "g1": w[at + ra:at + ra + rg],
                            m + "a2": low[:nh, :ra], m + "g2": low[nh:, ra:ra + rg], m + "A_log": a.a_log, m + "dt_bias": a.dt_bias,
                            m + "norm": a.norm, m + "o": x["o"][:, :nv]})
            if L.moe is not None:
                out.update({t + "norm2": L.norm2, t + "norm2b": L.norm2b, f + "router": L.moe.router[:, :d], f + "router.b": L.moe.bias})
                gate, up = moe_ops.deinterleave_gate_up(L.moe.gate_up)
                e0 = self.comm.rank * gate.shape[0]
                for e in range(gate.shape[0]):
                    out.update({f + f"e{e0 + e}.gate": gate[e, :s.ff, :d], f + f"e{e0 + e}.up": up[e, :s.ff, :d],
                                f + f"e{e0 + e}.down": L.moe.down[e, :d, :s.ff]})
        return {k: v.to(torch.bfloat16).contiguous() for k, v in out.items()}

    def weight_bytes(self) -> int:
        ts = [self.embed, self.final_norm, self.lm_head] + [t for L in self.layers for t in L.tensors()]
        return sum(t.numel() * t.element_size() for t in ts)

    # ------------------------------------------------------------------ cache and state
    def alloc_kv_cache(self, num_pages: int, page_size: int):
        """Per attention layer its pair of paged tensors (layers may differ in size), None for the others."""
        return [L.attn.alloc_cache(num_pages, page_size, self.dtype, self.device) if L.attn is not None else None for L in self.layers]

    def alloc_state(self, num_slots: int) -> None:
        """Per-sequence state of the delta layers: convolution inputs and the per-head matrices."""
        for L in self.layers:
            if L.delta is not None:
                L.delta.alloc(num_slots, self.dtype, self.device)

    def state_bytes_per_slot(self) -> int:
        return sum(L.delta.slot_bytes() for L in self.layers if L.delta is not None)

    def decode_splits(self, batch: int, max_seq_len: int) -> int:
        return max((ops.decode_plan_splits(batch, L.attn.kv_heads, L.attn.visible(max_seq_len)) for L in self.layers if L.attn is not None), default=1)

    # ------------------------------------------------------------------ forward
    def _out_proj(self, a, w):
        """A mixer's output projection, the partial sums of all ranks added: what the residual sum takes."""
        y = ops.gemm(a, w, out_dtype=torch.float32, static_w=True)
        return y if self.comm.world == 1 else self.comm.all_reduce_(y)

    def attention(self, L: _Layer, h, meta: AttnMeta, cache):
        a, m = L.attn, L.mix
        proj = ops.gemm(h, m["proj"], static_w=True)
        q = gqa.prep(proj, m["q_norm"], m["k_norm"], L.inv_freq, meta.positions, meta.slot_mapping, cache, self.config.norm_eps, a)
        gate = proj[:, pad8(a.heads * a.dim + a.kv_heads * (a.dim + a.vdim)):]
        return self._out_proj(gqa.attention(q, gate, cache, meta, a), m["o"])

    def delta(self, L: _Layer, h, meta: AttnMeta, q_start):
        a, m = L.delta, L.mix
        proj = ops.gemm(h, m["proj"], static_w=True)
        at = pad8(a.channels + a.heads)
        low = ops.gemm(proj[:, at:at + m["low"].shape[1]], m["low"], out_dtype=torch.float32, static_w=True)
        nb = None
        if meta.is_prefill and meta.q_start_host is not None:
            qs = meta.q_start_host
            nb = meta.plans.get("delta_blocks")
            if nb is None:
                nb = meta.plans["delta_blocks"] = sum((y - x + la.DELTA_BLOCK - 1) // la.DELTA_BLOCK for x, y in zip(qs, qs[1:]))
        y = la.channel_delta(proj, a.channels, low, a, q_start, meta.seq_lens, meta.state_slots, decode=not meta.is_prefill, num_blocks=nb)
        return self._out_proj(y, m["o"])

    def mixture(self, L: _Layer, h):
        """The routed experts' outputs, still to be summed with their weights (summed over the ranks with more than one)."""
        s, w = L.spec, L.moe
        z = ops.gemm(h, w.router, bias=w.bias, out_dtype=torch.float32, static_w=True)
        ids, weights = moe_ops.router_topk(z, s.top)
        rows, pos = moe_ops.expert_rows(h, ids, w.gate_up, w.down, self.comm.rank * w.down.shape[0], s.experts)
        y = stream.ExpertRows(rows, pos, weights)
        return y if self.comm.world == 1 else self.comm.all_reduce_(y.sum(self.config.hidden_size))

    def layer_steps(self, ids, meta: AttnMeta, kv_cache):
        """The stack, one layer at a time: yields the fp32 stream behind every layer (a buffer the next layer overwrites)."""
        if meta.state_slots is None:
            raise ValueError("Kirisun needs AttnMeta.state_slots (one state slot per sequence)")
        if any(L.delta is not None and L.delta.state is None for L in self.layers):
            self.alloc_state(int(meta.state_slots.max().item()) + 1)
        c = self.config
        q_start = meta.q_start
        if q_start is None:
            q_start = torch.arange(ids.shape[0] + 1, dtype=torch.int32, device=self.device)
        norm = dict(eps=c.norm_eps, act_dtype=self.dtype)
        x = stream.embedding_f32(ids, self.embed, c.embed_scale)
        if self.layers:
            _, h = stream.sandwich_norm(x, w_next=self.layers[0].norm1, **norm)
        for i, L in enumerate(self.layers):
            y = self.delta(L, h, meta, q_start) if L.delta is not None else self.attention(L, h, meta, kv_cache[i])
            nxt = self.layers[i + 1].norm1 if i + 1 < len(self.layers) else None
            if L.moe is not None:
                x, h = stream.sandwich_norm(x, y, L.norm1b, c.residual_mult, L.norm2, **norm)
                x, h = stream.sandwich_norm(x, self.mixture(L, h), L.norm2b, c.residual_mult, nxt, **norm)
            else:
                x, h = stream.sandwich_norm(x, y, L.norm1b, c.residual_mult, nxt, **norm)
            yield x

    def hidden_states(self, ids, meta: AttnMeta, kv_cache):
        x = None
        for x in self.layer_steps(ids, meta, kv_cache):
            pass
        return x

    def logits(self, x, rows=None):
        if rows is not None:
            x = x.index_select(0, rows.long() if rows.dtype != torch.int64 else rows)
        _, n = stream.sandwich_norm(x, w_next=self.final_norm, eps=self.config.norm_eps, act_dtype=self.dtype, keep_x=False)
        return self.head_logits(n)
