"""Dopurax: a decoder whose layers mix tokens by latent attention or by a WKV recurrence, in any order.

* The residual stream is fp32 and normalised behind every sublayer: x <- layernorm(alpha x + mixer(h)), then, where the
  layer has a feed-forward, x <- layernorm(alpha x + ff(x)); there is no norm in front of a sublayer.
* What a mixer reads is h = x + conv(x), a short causal convolution per channel over time.
* Latent attention (`ops.latent`): queries through a low-rank latent, keys and values from one cached latent per token
  plus a rotary key vector common to the heads, a sliding window, a sigmoid gate on the result.
* WKV (`ops.linear_attn.wkv_scan`): per-head matrix state with a data-dependent decay, a bonus for the current token, token
  shift in front of every projection, a per-head RMS norm and a silu gate behind.
* Feed-forward: down(relu(up x)^2).

A decode step runs the norm behind a layer, the convolution in front of the next one and its token-shift interpolations as
one launch; the input projections of a layer are one GEMM (latent attention: [query latent | key latent | gate]) or one
grouped GEMM (WKV: r, k, v and the gate, each on its own interpolation).  Tensor parallelism splits heads and the
feed-forward's hidden units; the latent projections are replicated, partial sums are all-reduced in fp32.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Optional

import torch

from .. import ops
from ..moe import ops as moe_ops
from ..ops import latent as lat
from ..ops import linear_attn as la
from ..ops import stream
from ..parallel.comm import Comm
from . import common
from .decoder import AttnMeta, DecoderModel

LATENT, WKV = "latent_attention", "wkv"
MIX_ORDER = "rkvgw"                 # planes of the token-shift interpolations


@dataclass
class LayerSpec:
    """One entry of config.json's `layers`."""
    kind: str
    heads: int
    dim: int                        # latent attention: unrotated query / key dimensions; WKV: key and value channels
    ff: int = 0                     # 0: no feed-forward
    rot: int = 0
    vdim: int = 0
    rank: int = 0
    q_rank: int = 0
    window: int = 0
    scale: float = 1.0
    rot_base: float = 10000.0

    @staticmethod
    def from_json(e: dict) -> "LayerSpec":
        kind, m, mlp = e["type"], e["mixer"], e.get("mlp")
        if mlp is not None and mlp.get("kind", "dense") != "dense":
            raise ValueError(f"unknown feed-forward kind {mlp['kind']!r}")
        ff = int(mlp["ff"]) if mlp is not None else 0
        if kind == WKV:
            return LayerSpec(WKV, int(m["heads"]), int(m["dim"]), ff)
        if kind != LATENT:
            raise ValueError(f"unknown layer type {kind!r}")
        if m["rot"]["dims"] != m["rot_dim"]:
            raise ValueError("latent attention rotates the whole rotated part: rot.dims must equal rot_dim")
        if m["rot_dim"] % 2:
            raise ValueError("rot_dim must be even")
        mask = m.get("mask") or {}
        return LayerSpec(LATENT, int(m["heads"]), int(m["dim"]), ff, int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"]), int(m["q_rank"]),
                         int(mask.get("size", 0)), float(m["scale"]), float(m["rot"]["base"]))

    def to_json(self) -> dict:
        mlp = {"kind": "dense", "ff": self.ff} if self.ff else None
        m = {"heads": self.heads, "dim": self.dim}
        if self.kind == LATENT:
            m.update(rot_dim=self.rot, vdim=self.vdim, kv_rank=self.rank, q_rank=self.q_rank, mask={"size": self.window}, scale=self.scale,
                     rot={"base": self.rot_base, "dims": self.rot})
        return {"type": self.kind, "mixer": m, "mlp": mlp}


@dataclass
class DopuraxConfig:
    vocab_size: int
    hidden_size: int
    layers: list                    # of LayerSpec
    norm_eps: float
    alpha: float
    taps: int
    decay_rank: int = 64            # of random-init models; checkpoints give it by the shape of mix.w1
    bos_token_id: Optional[int] = None
    eos_token_id: object = None
    max_position_embeddings: int = 1 << 20
    model_type: str = "dopurax"
    extra: dict = field(default_factory=dict)

    @classmethod
    def from_hf(cls, obj: dict) -> "DopuraxConfig":
        for need in ("vocab", "width", "layers", "norm", "postln_alpha", "canon"):
            if need not in obj:
                raise ValueError(f"config.json lacks {need}")
        kw = {k: obj[k] for k in ("bos_token_id", "eos_token_id", "decay_rank") if obj.get(k) is not None}
        return cls(int(obj["vocab"]), int(obj["width"]), [LayerSpec.from_json(e) for e in obj["layers"]], float(obj["norm"]["eps"]),
                   float(obj["postln_alpha"]), int(obj["canon"]["taps"]), **kw)

    def to_json(self) -> dict:
        return {"architecture": "Dopurax", "vocab": self.vocab_size, "width": self.hidden_size, "layers": [s.to_json() for s in self.layers],
                "norm": {"eps": self.norm_eps}, "postln_alpha": self.alpha, "canon": {"taps": self.taps}}

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def eos_ids(self) -> list[int]:
        return common.eos_list(self.eos_token_id)

    def num_params(self) -> int:
        d, n = self.hidden_size, 2 * self.vocab_size * self.hidden_size + self.hidden_size
        for s in self.layers:
            n += d * (1 + self.taps) + (2 * d * s.ff + d if s.ff else 0)
            if s.kind == LATENT:
                n += d * (s.q_rank + s.rank + s.rot + 2 * s.heads * s.vdim) + s.q_rank * s.heads * (s.dim + s.rot)
                n += s.rank * s.heads * (s.dim + s.vdim) + s.q_rank + s.rank
            else:
                n += 5 * d * s.heads * s.dim + self.decay_rank * (d + s.heads * s.dim) + 5 * d + 3 * s.heads * s.dim
        return n


def _preset(width, vocab, pattern, ff, latent, wkv, taps=4, alpha=2.0, **kw):
    """`pattern`: one letter per layer - L (latent attention) or W (WKV), lower case without a feed-forward."""
    layers = []
    for ch in pattern:
        mlp = {"kind": "dense", "ff": ff} if ch.isupper() else None
        layers.append({"type": LATENT, "mixer": latent, "mlp": mlp} if ch in "Ll" else {"type": WKV, "mixer": wkv, "mlp": mlp})
    return dict(architecture="Dopurax", width=width, vocab=vocab, layers=layers, norm={"eps": 1e-5}, postln_alpha=alpha, canon={"taps": taps}, **kw)


def _latent(heads, dim, rot, vdim, rank, q_rank, window, base=500000.0):
    return dict(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=rank, q_rank=q_rank, mask={"size": window}, scale=(dim + rot) ** -0.5,
                rot={"base": base, "dims": rot})


PRESETS = {
    # the 1B- and 8B-class shapes of the benchmark (random-init): latent attention and WKV in turn
    "dopurax-1b": _preset(2048, 65536, "LW" * 8, 8192, _latent(16, 128, 64, 128, 512, 1536, 4096), dict(heads=32, dim=64)),
    "dopurax-8b": _preset(4096, 65536, "LW" * 16, 16384, _latent(32, 128, 64, 128, 512, 1536, 4096), dict(heads=32, dim=128)),
    "tiny-dopurax-test": _preset(192, 320, "WlL", 384, _latent(4, 40, 16, 24, 56, 72, 100, 10000.0), dict(heads=4, dim=40), taps=3,
                                 decay_rank=24),
}


class _Ff:
    __slots__ = ("up", "down")


class _Layer:
    """Weights of one layer, this rank's heads and hidden units; `mix` holds the mixer's tensors."""

    def __init__(self, spec: LayerSpec):
        self.spec = spec
        self.norm1 = self.norm2 = self.conv_w = None
        self.ff: Optional[_Ff] = None
        self.mix: dict = {}
        self.dims: Optional[lat.LatentDims] = None
        self.inv_freq = None
        self.conv: Optional[stream.InputConv] = None
        self.wkv_state = None

    def tensors(self):
        ts = [self.norm1, self.norm2, self.conv_w] + list(self.mix.values())
        if self.ff is not None:
            ts += [self.ff.up, self.ff.down]
        return [t for t in ts if isinstance(t, torch.Tensor)]


class DopuraxModel(DecoderModel):
    KERNEL_SOURCES = ("runtime", "gemm_bf16", "gemm_2cta", "gemm_f32", "elementwise", "stream_f32", "latent_attention",
                      "latent_prefill_tc", "latent_decode", "wkv", "moe")
    FP32_ON_GPU = True
    # With overlapping launches a prefill of several chunks queued back to back has stopped making progress (some kernel of
    # the chain waits for resources that a later one holds); serial launches cost nothing here, the kernels are long.
    SERIAL_PREFILL = True

    def __init__(self, config: DopuraxConfig, comm: Optional[Comm] = None, device="cpu", dtype=torch.bfloat16):
        super().__init__(config, comm, device, dtype)
        p = self.comm.world
        for i, s in enumerate(config.layers):
            if s.heads % p or s.ff % p:
                raise ValueError(f"layer {i}: {s.heads} heads / {s.ff} hidden units do not split over {p} ranks")
        self.layers: list[_Layer] = []
        self._offsets: dict = {}

    # ------------------------------------------------------------------ weights
    def _assemble(self, get) -> "DopuraxModel":
        """Builds the layers from `get(name, rows=None, cols=None, f32=False)`, which returns a tensor of the checkpoint's
        layout (optionally this rank's rows or columns) in the model's dtype or in fp32."""
        c, (r, p) = self.config, (self.comm.rank, self.comm.world)
        self.embed = get("embed").contiguous()
        self.final_norm = get("final.norm", f32=True)
        self.lm_head = ops.pad_k(get("head", rows=self.v_rng))
        self._pad_lm_head()
        for i, s in enumerate(c.layers):
            L, t = _Layer(s), f"l{i}."
            h0, h1 = common.shard_range(s.heads, r, p)
            L.norm1 = get(t + "norm1", f32=True)
            L.conv_w = get(t + "canon1", f32=True).t().contiguous()                              # [taps, d]
            if L.conv_w.shape[0] != c.taps:
                raise ValueError(f"layer {i}: {L.conv_w.shape[0]} convolution taps in the checkpoint, {c.taps} in config.json")
            m = t + "mix."
            if s.kind == LATENT:
                self._assemble_latent(L, get, m, h0, h1)
            else:
                self._assemble_wkv(L, get, m, h0, h1)
            if s.ff:
                L.norm2 = get(t + "norm2", f32=True)
                L.ff = _Ff()
                f = common.shard_range(s.ff, r, p)
                L.ff.up = ops.pad_k(get(t + "mlp.up", rows=f))
                L.ff.down = ops.pad_k(get(t + "mlp.down", cols=f))
            self.layers.append(L)
        return self

    def _assemble_latent(self, L: _Layer, get, m: str, h0: int, h1: int) -> None:
        s, H = L.spec, h1 - h0
        L.dims = lat.LatentDims(H, s.dim, s.rot, s.vdim, s.rank, s.q_rank, s.window, s.scale, s.rot_base)
        L.inv_freq = L.dims.inv_freq(self.device)
        gate = get(m + "g", rows=(h0 * s.vdim, h1 * s.vdim))
        down = s.q_rank + s.rank + s.rot
        fill = torch.zeros((-down % 8, gate.shape[1]), dtype=gate.dtype, device=gate.device)      # the gate's columns start on 16 bytes
        L.mix["proj"] = ops.pad_k(torch.cat([get(m + "dq"), get(m + "dkv"), fill, gate], 0))
        L.mix["q_norm"] = get(m + "dq.norm", f32=True)
        L.mix["c_norm"] = get(m + "dkv.norm", f32=True)
        L.mix["uq"] = ops.pad_k(get(m + "uq", rows=(h0 * (s.dim + s.rot), h1 * (s.dim + s.rot))))
        uk = get(m + "uk", rows=(h0 * s.dim, h1 * s.dim))
        uv = get(m + "uv", rows=(h0 * s.vdim, h1 * s.vdim))
        L.mix["uk_t"] = uk.reshape(H, s.dim, s.rank).transpose(1, 2).contiguous()                 # [H, rank, dim]
        L.mix["ukv"] = torch.cat([uk, uv], 0).contiguous()                                        # [H (dim + vdim), rank]
        L.mix["o"] = ops.pad_k(get(m + "o", cols=(h0 * s.vdim, h1 * s.vdim)))

    def _assemble_wkv(self, L: _Layer, get, m: str, h0: int, h1: int) -> None:
        s, n = L.spec, (h0 * L.spec.dim, h1 * L.spec.dim)
        L.mix["mu"] = torch.stack([get(m + "mu." + x, f32=True) for x in MIX_ORDER]).contiguous()
        L.mix["rkvg"] = torch.stack([ops.pad_k(get(m + x, rows=n)) for x in MIX_ORDER[:4]]).contiguous()     # [4, H dim, d]
        L.mix["w1"] = ops.pad_k(get(m + "w1"))
        w2 = get(m + "w2", rows=n)
        L.mix["w2_t"] = w2.t().contiguous()
        if self.dtype == torch.bfloat16:
            L.mix["w2_split"] = la.split_weight(w2)
        for name, key in (("w0", "w0"), ("norm", "norm")):
            L.mix[name] = get(m + key, f32=True)[n[0]:n[1]].contiguous()
        L.mix["u"] = get(m + "u", f32=True)[h0:h1].reshape(-1).contiguous()
        L.mix["o"] = ops.pad_k(get(m + "o", cols=n))

    def load(self, store, prefix: str = "") -> "DopuraxModel":
        def get(name, rows=None, cols=None, f32=False):
            return store.load_tensor(prefix + name, device=self.device, dtype=torch.float32 if f32 else self.dtype, rows=rows, cols=cols)
        return self._assemble(get)

    def init_random(self, seed: int = 0, std: float = 0.02) -> "DopuraxModel":
        """Random-init weights of this architecture: matrices N(0, std), norms around one, decays spread over time scales."""
        shapes = self.checkpoint_shapes()
        order = {n: k for k, n in enumerate(shapes)}

        def get(name, rows=None, cols=None, f32=False):
            shape, leaf = shapes[name], name.rsplit(".", 1)[-1]
            g = torch.Generator(device=self.device).manual_seed((seed * 1000003 + order[name] * 7919 + 1) % (2 ** 63))
            w = torch.empty(shape, dtype=torch.float32 if len(shape) == 1 or f32 else self.dtype, device=self.device)
            if ".mu." in name:
                w.uniform_(0.0, 1.0, generator=g)
            elif leaf in ("norm1", "norm2", "norm"):
                w.normal_(1.0, 0.05, generator=g)
            elif leaf == "w0":
                w.uniform_(-5.0, -0.5, generator=g)
            elif leaf == "canon1":
                w.normal_(0.0, 0.2, generator=g)
            elif leaf == "u":
                w.normal_(0.0, 0.5, generator=g)
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
            t, m = f"l{i}.", f"l{i}.mix."
            out.update({t + "norm1": (d,), t + "canon1": (d, c.taps)})
            if s.kind == LATENT:
                out.update({m + "dq": (s.q_rank, d), m + "dq.norm": (s.q_rank,), m + "uq": (s.heads * (s.dim + s.rot), s.q_rank),
                            m + "dkv": (s.rank + s.rot, d), m + "dkv.norm": (s.rank,), m + "uk": (s.heads * s.dim, s.rank),
                            m + "uv": (s.heads * s.vdim, s.rank), m + "g": (s.heads * s.vdim, d), m + "o": (d, s.heads * s.vdim)})
            else:
                n = s.heads * s.dim
                out.update({m + "mu." + x: (d,) for x in MIX_ORDER})
                out.update({m + x: (n, d) for x in MIX_ORDER[:4]})
                out.update({m + "w1": (c.decay_rank, d), m + "w2": (n, c.decay_rank), m + "w0": (n,), m + "u": (s.heads, s.dim), m + "norm": (n,),
                            m + "o": (d, n)})
            if s.ff:
                out.update({t + "norm2": (d,), t + "mlp.up": (s.ff, d), t + "mlp.down": (d, s.ff)})
        out.update({"final.norm": (d,), "head": (c.vocab_size, d)})
        return out

    def state_dict_hf(self) -> dict:
        """This rank's weights under their checkpoint names, in bf16; a complete checkpoint when TP == 1."""
        c, d = self.config, self.config.hidden_size
        out = {"embed": self.embed, "final.norm": self.final_norm, "head": self.lm_head[:self.v_rng[1] - self.v_rng[0], :d]}
        for i, L in enumerate(self.layers):
            s, t, m, x = L.spec, f"l{i}.", f"l{i}.mix.", L.mix
            out.update({t + "norm1": L.norm1, t + "canon1": L.conv_w.t()})
            if s.kind == LATENT:
                H, down = L.dims.heads, s.q_rank + s.rank + s.rot
                out.update({m + "dq": x["proj"][:s.q_rank, :d], m + "dkv": x["proj"][s.q_rank:down, :d], m + "g": x["proj"][down + -down % 8:, :d],
                            m + "dq.norm": x["q_norm"], m + "dkv.norm": x["c_norm"], m + "uq": x["uq"][:, :s.q_rank],
                            m + "uk": x["ukv"][:H * s.dim], m + "uv": x["ukv"][H * s.dim:], m + "o": x["o"][:, :H * s.vdim]})
            else:
                n = x["w0"].shape[0]
                out.update({m + "mu." + k: x["mu"][j] for j, k in enumerate(MIX_ORDER)})
                out.update({m + k: x["rkvg"][j][:, :d] for j, k in enumerate(MIX_ORDER[:4])})
                out.update({m + "w1": x["w1"][:, :d], m + "w2": x["w2_t"].t(), m + "w0": x["w0"], m + "u": x["u"].reshape(-1, s.dim), m + "norm": x["norm"],
                            m + "o": x["o"][:, :n]})
            if L.ff is not None:
                out.update({t + "norm2": L.norm2, t + "mlp.up": L.ff.up[:, :d], t + "mlp.down": L.ff.down[:, :s.ff // self.comm.world]})
        return {k: v.to(torch.bfloat16).contiguous() for k, v in out.items()}

    def weight_bytes(self) -> int:
        ts = [self.embed, self.final_norm, self.lm_head] + [t for L in self.layers for t in L.tensors()]
        return sum(t.numel() * t.element_size() for t in ts)

    # ------------------------------------------------------------------ cache and state
    def alloc_kv_cache(self, num_pages: int, page_size: int):
        """One [pages, page, row] tensor per latent-attention layer (layers may differ in size), None for the others."""
        return [torch.zeros((num_pages, page_size, L.dims.row), dtype=self.dtype, device=self.device) if L.dims is not None else None
                for L in self.layers]

    def alloc_state(self, num_slots: int) -> None:
        """Per-sequence state: the last inputs of every layer's convolution, and the WKV matrices ([value, key] per head)."""
        d, taps = self.config.hidden_size, self.config.taps
        f32 = dict(dtype=torch.float32, device=self.device)
        for L in self.layers:
            mixes = L.spec.kind == WKV
            st = torch.zeros((num_slots, stream.InputConv.rows_for(taps, mixes), d), **f32)
            L.conv = stream.InputConv(L.conv_w, st, L.mix["mu"] if mixes else None)
            if mixes:
                L.wkv_state = torch.zeros((num_slots, L.spec.heads // self.comm.world, L.spec.dim, L.spec.dim), **f32)

    def state_bytes_per_slot(self) -> int:
        return sum(4 * (L.conv.state[0].numel() + (L.wkv_state[0].numel() if L.wkv_state is not None else 0)) for L in self.layers)

    def decode_splits(self, batch: int, max_seq_len: int) -> int:
        dims = [L.dims for L in self.layers if L.dims is not None]
        return max((lat.decode_plan_splits(batch, d, max_seq_len) for d in dims), default=1)

    # ------------------------------------------------------------------ forward
    def _reduce(self, y):
        return y if self.comm.world == 1 else self.comm.all_reduce_(y)

    def _out_proj(self, a, w):
        """A sublayer's output projection, the partial sums of all ranks added: what the residual sum takes."""
        return self._reduce(ops.gemm(a, w, out_dtype=torch.float32, static_w=True))

    def latent_attention(self, L: _Layer, h, meta: AttnMeta, cache):
        d, m = L.dims, L.mix
        proj = ops.gemm(h, m["proj"], static_w=True)
        cq = lat.prep(proj, m["q_norm"], m["c_norm"], L.inv_freq, meta.positions, meta.slot_mapping, cache, self.config.norm_eps, d)
        q = ops.gemm(cq, m["uq"], static_w=True)
        down = d.q_rank + d.rank + d.rot
        gate = proj[:, down + -down % 8:]
        a = lat.latent_attention(q, gate, m["uk_t"], m["ukv"], L.inv_freq, cache, meta, d)
        return self._out_proj(a, m["o"])

    def _stacked(self, x, w):
        """x [4, T, d] times w [4, N, d] plane by plane: one grouped GEMM for decode-sized steps, else one GEMM each."""
        e, t, n = x.shape[0], x.shape[1], w.shape[1]
        if x.is_cuda and x.dtype == torch.bfloat16 and t <= 128 and n % 128 == 0 and x.shape[2] % 8 == 0:
            off = self._offsets.get(t)
            if off is None:
                off = self._offsets[t] = torch.arange(0, (e + 1) * t, t, dtype=torch.int32, device=x.device)
            return moe_ops.grouped_gemm(x.reshape(e * t, -1), w, off, avg_tokens=t).reshape(e, t, n)
        ld = (n + 7) // 8 * 8 if x.dtype == torch.bfloat16 else n
        out = torch.empty((e, t, ld), dtype=x.dtype, device=x.device)[..., :n]
        for i in range(e):
            ops.gemm(x[i], w[i], out=out[i], static_w=True)
        return out

    def wkv(self, L: _Layer, mix, meta: AttnMeta, q_start):
        s, m = L.spec, L.mix
        r, k, v, g = self._stacked(mix[:4], m["rkvg"])
        low = ops.gemm(mix[4], m["w1"], out_dtype=torch.float32, static_w=True)
        z = la.tanh_linear(low, m["w2_t"], m.get("w2_split"))
        a = la.wkv_scan(r, k, v, g, z, m["w0"], m["u"], m["norm"], self.config.norm_eps, L.wkv_state, q_start, meta.seq_lens, meta.state_slots,
                        s.heads // self.comm.world, s.dim, decode=not meta.is_prefill)
        return self._out_proj(a, m["o"])

    def _conv(self, L: _Layer, x, meta: AttnMeta, q_start):
        nb = None
        if meta.is_prefill and meta.q_start_host is not None:
            qs, blk = meta.q_start_host, stream.CONV_BLOCK
            nb = meta.plans.get("conv_blocks")
            if nb is None:
                nb = meta.plans["conv_blocks"] = sum((b - a + blk - 1) // blk for a, b in zip(qs, qs[1:]))
        elif not meta.is_prefill:
            nb = x.shape[0]
        return stream.stream_conv(x, L.conv, q_start, meta.seq_lens, meta.state_slots, self.dtype, nb)

    def layer_steps(self, ids, meta: AttnMeta, kv_cache):
        """The stack, one layer at a time: yields the fp32 stream behind every layer."""
        if meta.state_slots is None:
            raise ValueError("Dopurax needs AttnMeta.state_slots (one state slot per sequence)")
        if self.layers and self.layers[0].conv is None:
            self.alloc_state(int(meta.state_slots.max().item()) + 1)
        c, dt = self.config, self.dtype
        q_start = meta.q_start
        if q_start is None:
            q_start = torch.arange(ids.shape[0] + 1, dtype=torch.int32, device=self.device)
        x = stream.embedding_f32(ids, self.embed)
        h = None
        for i, L in enumerate(self.layers):
            if h is None:
                h = self._conv(L, x, meta, q_start)
            y = self.wkv(L, h, meta, q_start) if L.spec.kind == WKV else self.latent_attention(L, h, meta, kv_cache[i])
            w = L.norm1
            if L.ff is not None:
                x, a = stream.post_norm(x, w, c.norm_eps, y, c.alpha, act_dtype=dt)
                y = self._out_proj(ops.gemm(a, L.ff.up, static_w=True, act="relu2"), L.ff.down)
                w = L.norm2
            nxt = self.layers[i + 1] if i + 1 < len(self.layers) else None
            h = None
            if nxt is not None and not meta.is_prefill:
                x, h = stream.post_norm(x, w, c.norm_eps, y, c.alpha, act_dtype=dt, conv=nxt.conv, seq_lens=meta.seq_lens, slots=meta.state_slots)
            else:
                x, _ = stream.post_norm(x, w, c.norm_eps, y, c.alpha)
            yield x

    def hidden_states(self, ids, meta: AttnMeta, kv_cache):
        x = None
        for x in self.layer_steps(ids, meta, kv_cache):
            pass
        return x

    def logits(self, x, rows=None):
        if rows is not None:
            x = x.index_select(0, rows.long() if rows.dtype != torch.int64 else rows)
        _, n = stream.post_norm(x, self.final_norm, self.config.norm_eps, keep_x=False, act_dtype=self.dtype)
        return self.head_logits(n)
