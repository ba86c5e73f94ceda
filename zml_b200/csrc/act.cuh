// Activations in bf16 or fp32 behind one pair of accessors, and the varlen batch description shared by the kernels
// of decoders whose residual stream is fp32.
#pragma once

#include "common.cuh"

ZB_DEVICE float zb_ld_act(const __nv_bfloat16* p) { return __bfloat162float(*p); }
ZB_DEVICE float zb_ld_act(const float* p) { return *p; }
ZB_DEVICE void zb_st_act(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }
ZB_DEVICE void zb_st_act(float* p, float v) { *p = v; }

// A flattened batch: tokens [q_start[s], q_start[s + 1]) belong to sequence s, whose length including them is
// seq_lens[s].
struct ZbVarlen {
  const int32_t* q_start;
  const int32_t* seq_lens;
  int num_seqs;
};

// (sequence, block) number `idx` when every sequence is cut into blocks of `rows` tokens; false past the last one.
ZB_DEVICE bool zb_find_block(const ZbVarlen& b, int rows, int idx, int& seq, int& block) {
  for (int s = 0; s < b.num_seqs; ++s) {
    const int nb = (b.q_start[s + 1] - b.q_start[s] + rows - 1) / rows;
    if (idx < nb) {
      seq = s;
      block = idx;
      return true;
    }
    idx -= nb;
  }
  return false;
}

// The same by all 32 lanes of a warp together, 32 sequences at a time.
ZB_DEVICE bool zb_find_block_warp(const ZbVarlen& b, int rows, int idx, int& seq, int& block) {
  const int lane = threadIdx.x & 31;
  for (int base = 0; base < b.num_seqs; base += 32) {
    const int s = base + lane;
    const int nb = s < b.num_seqs ? (b.q_start[s + 1] - b.q_start[s] + rows - 1) / rows : 0;
    int incl = nb;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int v = __shfl_up_sync(0xffffffffu, incl, o);
      if (lane >= o) incl += v;
    }
    const unsigned hit = __ballot_sync(0xffffffffu, idx < incl);
    if (hit != 0u) {
      const int l = __ffs(hit) - 1;
      seq = base + l;
      block = idx - __shfl_sync(0xffffffffu, incl - nb, l);
      return true;
    }
    idx -= __shfl_sync(0xffffffffu, incl, 31);
  }
  return false;
}

// Blocks in front of sequence `seq`, by a warp.
ZB_DEVICE int zb_blocks_before(const ZbVarlen& b, int rows, int seq) {
  int n = 0;
  for (int s = threadIdx.x & 31; s < seq; s += 32) n += (b.q_start[s + 1] - b.q_start[s] + rows - 1) / rows;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) n += __shfl_xor_sync(0xffffffffu, n, o);
  return n;
}

// The sequence of token t, by a warp.
ZB_DEVICE int zb_sequence_of(const ZbVarlen& b, int t) {
  int n = 0;
  for (int base = 1; base < b.num_seqs; base += 32) {
    const int s = base + (threadIdx.x & 31);
    n += __popc(__ballot_sync(0xffffffffu, s < b.num_seqs && b.q_start[s] <= t));
  }
  return n;
}
