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
