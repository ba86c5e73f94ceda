"""What every decoder of the zoo shares with the engine: the per-step metadata, the split of the vocabulary over ranks,
the output head, sampling, and the cache / plan hooks a model may override.
"""
from __future__ import annotations

import dataclasses
from dataclasses import dataclass, field
from typing import Optional

import torch

from .. import ops
from ..parallel.comm import Comm
from . import common


@dataclass
class AttnMeta:
    """Per-step attention metadata in the shapes of the reference's paged API
    (zml/attention/paged_attention.zig:19-293): block_table {b,p}, seq_lens {b},
    query_start_len {b+1}, slot_mapping {tokens}."""
    is_prefill: bool
    positions: torch.Tensor
    slot_mapping: torch.Tensor
    block_table: torch.Tensor
    seq_lens: torch.Tensor
    q_start: Optional[torch.Tensor] = None
    total_q_blocks: Optional[int] = None
    num_splits: Optional[int] = None
    max_seq_len: Optional[int] = None
    logits_rows: Optional[torch.Tensor] = None    # rows of the hidden state that need logits
    state_slots: Optional[torch.Tensor] = None    # {b} slot of every sequence in a model's recurrent-state pool
    q_start_host: Optional[list] = None           # host copy of q_start (prefill), for splitting a chunk by sequences
    seq_lens_host: Optional[list] = None          # host copy of seq_lens (prefill)
    plans: dict = field(default_factory=dict)     # what the layers derive from this step's metadata once (by their own keys)


class DecoderModel:
    """Base of the decoder models: one tensor-parallel rank.  A model provides `hidden_states(ids, meta, kv_cache)` and
    `logits(x, rows)`; models with per-sequence state besides KV pages also `alloc_state(num_slots)`."""

    # sources of csrc/ that the model's kernels need; None: the whole library
    KERNEL_SOURCES: Optional[tuple] = None
    # True when the model's kernels also run in fp32 on the GPU
    FP32_ON_GPU = False
    # True: varlen batches (prompts and portions of them) run without programmatic dependent launch
    SERIAL_PREFILL = False

    def __init__(self, config, comm: Optional[Comm] = None, device="cpu", dtype=torch.bfloat16):
        self.config = config
        self.comm = comm or Comm.single()
        self.device = torch.device(device)
        self.dtype = dtype
        p, r, v = self.comm.world, self.comm.rank, config.vocab_size
        # vocab-parallel lm_head: every rank holds v_per rows; rows past the vocabulary (last ranks, when the
        # vocabulary does not divide) are zero rows whose logits are masked to -inf
        self.v_per = (v + p - 1) // p
        self.v_rng = (min(v, r * self.v_per), min(v, (r + 1) * self.v_per))
        self.v_pad = self.v_per - (self.v_rng[1] - self.v_rng[0])
        self.embed = None
        self.final_norm = None
        self.lm_head = None

    # ------------------------------------------------------------------ engine hooks
    def alloc_kv_cache(self, num_pages: int, page_size: int):
        """The paged cache, as `hidden_states` takes it."""
        return torch.zeros(self.kv_cache_shape(num_pages, page_size), dtype=self.dtype, device=self.device)

    def decode_splits(self, batch: int, max_seq_len: int) -> int:
        """KV chunks per sequence of a decode step (part of the key of captured graphs)."""
        return ops.decode_plan_splits(batch, self.hkv, max_seq_len)

    def layer_plan(self, meta: AttnMeta, splits) -> AttnMeta:
        """The metadata of a decode step with a layer's own number of key chunks, at most the step's: a layer that sees a part of
        the sequence is cut into fewer pieces than one that sees all of it.  `splits(max_seq_len)`: that number."""
        if meta.is_prefill or meta.num_splits is None or meta.max_seq_len is None or self.device.type != "cuda":
            return meta
        n = min(meta.num_splits, splits(meta.max_seq_len))
        plan = meta.plans.get(("splits", n))
        if plan is None:
            plan = meta.plans[("splits", n)] = dataclasses.replace(meta, num_splits=n)
        return plan

    # ------------------------------------------------------------------ output head
    def _pad_lm_head(self) -> None:
        if self.v_pad > 0 and self.comm.world > 1 and self.lm_head.shape[0] < self.v_per:
            pad = torch.zeros((self.v_pad, self.lm_head.shape[1]), dtype=self.lm_head.dtype, device=self.lm_head.device)
            self.lm_head = torch.cat([self.lm_head, pad], 0)

    def head_logits(self, n):
        """float32 logits of this rank's vocab shard from the normed hidden state."""
        if self.v_pad > 0 and self.comm.world > 1 and self.lm_head.shape[0] < self.v_per:
            self._pad_lm_head()         # model families that fill `lm_head` themselves
        lg = ops.gemm(n, self.lm_head, out_dtype=torch.float32, static_w=True)
        if self.v_pad > 0 and self.comm.world > 1:
            lg[:, self.v_per - self.v_pad:] = float("-inf")
        return lg

    def sample(self, logits, strategy: common.SamplingStrategy, seed: int = 0, step: int = 0, rng=None):
        """Token ids int32 [B] from vocab-parallel logits.  `rng`: device-side {seed, draw counter} of
        `ops.topk_sample` (the serving engine's, so that graph replays draw fresh noise)."""
        comm = self.comm
        rng = rng if (rng is not None and logits.is_cuda) else None
        if comm.world == 1:
            if strategy.topk <= 1:
                return ops.argmax(logits)
            return ops.topk_sample(logits, strategy.topk, strategy.temperature, seed, step, rng=rng)
        if strategy.topk <= 1:
            if comm.fused is not None and logits.is_cuda and comm.fused.can_argmax_tp(logits.shape[0]):
                return comm.fused.argmax_tp(logits, comm.rank * self.v_per)     # candidates exchanged inside the kernel
            idx = ops.argmax(logits)
            val = logits.gather(1, idx.long()[:, None])[:, 0]
            vals = comm.all_gather(val[None])                   # [P, B]
            idxs = comm.all_gather((idx + self.comm.rank * self.v_per)[None])
            best = vals.argmax(0)
            return idxs.gather(0, best[None])[0].to(torch.int32)
        # Every rank ranks its own columns (column j of rank r is token r * v_per + j; padding columns are -inf) and
        # only the k best (value, token) pairs per row travel: the k best of their union are the k best of the whole
        # vocabulary, in the same order, so the draw below equals the draw on gathered logits at 1 / (v_per / k) of the bytes.
        k = min(strategy.topk, logits.shape[1])
        vals, idx = ops.topk(logits, k)
        cand_v = comm.all_gather(vals.contiguous(), dim=1).contiguous()
        cand_i = comm.all_gather((idx + comm.rank * self.v_per).to(torch.int32).contiguous(), dim=1)
        pos = ops.topk_sample(cand_v, strategy.topk if strategy.topk <= cand_v.shape[1] else cand_v.shape[1],
                              strategy.temperature, seed, step, rng=rng)
        return cand_i.gather(1, pos.long()[:, None])[:, 0].to(torch.int32)

    def forward(self, ids, meta: AttnMeta, kv_cache, strategy: Optional[common.SamplingStrategy] = None,
                seed: int = 0, step: int = 0, rng=None):
        """ids int32 [T] -> sampled tokens int32 [rows] (one per sequence)."""
        x = self.hidden_states(ids, meta, kv_cache)
        lg = self.logits(x, meta.logits_rows)
        return self.sample(lg, strategy or common.SamplingStrategy(), seed, step, rng)
