// Gated recurrence whose gates read the current token only (minGRU), over a varlen batch, channel by channel:
//
//   g = sigmoid(z + z_bias), u = x + x_bias, c = u + 1/2 where u >= 0, else sigmoid(u)
//   S <- (1 - g) S + g c,  out = S * silu(gate) * scale
//
// z, x and gate are columns of one projection.  The recurrence is a composition of affine maps, so prompts are cut into blocks of
// kRows tokens: the first launch composes the maps of every block but a sequence's last, the second one applies those in front of
// a block to the sequence's state and walks the block.  A decode step is one token per sequence and one launch.
// Gates, candidates and the state are fp32; the state of a sequence is one fp32 per channel.
#include "act.cuh"
#include "host_api.h"

namespace {
constexpr uint32_t kKernelGatedScan = 38;
constexpr int kRows = 64;

struct GatedScanArgs {
  const void* z;             // [T, ld]
  const void* x;
  const void* gate;
  long long ld;
  const float* z_bias;       // [width]
  const float* x_bias;
  float* state;              // [slots, width]
  const int32_t* slots;
  float2* maps;              // [blocks, width]: a block's entry is what comes in front of it, (0, state) or the map of the block before
  void* out;                 // [T, ld_out]
  long long ld_out;
  float scale;
  int width;
};

// 1 / (1 + e^-v) and 1 - that; EXACT: fp32 functions, else their fast forms.
template <bool EXACT>
ZB_DEVICE float exp_of(float v) { return EXACT ? expf(v) : __expf(v); }
template <bool EXACT>
ZB_DEVICE float over(float a, float b) { return EXACT ? a / b : __fdividef(a, b); }
template <bool EXACT>
ZB_DEVICE void gates(float v, float& open, float& keep) {
  const float e = exp_of<EXACT>(-fmaxf(v, -80.f));       // e^80 and its reciprocal are in range
  const float r = over<EXACT>(1.f, 1.f + e);
  open = r;
  keep = e * r;
}
template <bool EXACT>
ZB_DEVICE float sigmoid_of(float v) { return over<EXACT>(1.f, 1.f + exp_of<EXACT>(-fmaxf(v, -80.f))); }
template <bool EXACT>
ZB_DEVICE float candidate(float u) { return u >= 0.f ? u + 0.5f : sigmoid_of<EXACT>(u); }

template <int V>
ZB_DEVICE void ld_cols(float (&v)[V], const __nv_bfloat16* p) {
  if constexpr (V == 2) {
    const float2 f = zb_unpack_bf16x2(*reinterpret_cast<const uint32_t*>(p));
    v[0] = f.x; v[1] = f.y;
  } else {
    v[0] = zb_ld_act(p);
  }
}
template <int V>
ZB_DEVICE void ld_cols(float (&v)[V], const float* p) {
  if constexpr (V == 2) {
    const float2 f = *reinterpret_cast<const float2*>(p);
    v[0] = f.x; v[1] = f.y;
  } else {
    v[0] = *p;
  }
}
template <int V>
ZB_DEVICE void st_cols(__nv_bfloat16* p, const float (&v)[V]) {
  if constexpr (V == 2) *reinterpret_cast<uint32_t*>(p) = zb_pack_bf16x2(v[0], v[1]);
  else zb_st_act(p, v[0]);
}
template <int V>
ZB_DEVICE void st_cols(float* p, const float (&v)[V]) {
  if constexpr (V == 2) *reinterpret_cast<float2*>(p) = make_float2(v[0], v[1]);
  else *p = v[0];
}

// State of sequence s in front of the launch; zero for one that starts here.
template <int V>
ZB_DEVICE void first_state(const GatedScanArgs& p, const ZbVarlen& b, int s, int slot, int c, float (&st)[V]) {
  const bool fresh = b.seq_lens[s] - (b.q_start[s + 1] - b.q_start[s]) <= 0;
#pragma unroll
  for (int e = 0; e < V; ++e) st[e] = fresh ? 0.f : p.state[static_cast<size_t>(slot) * p.width + c + e];
}

constexpr int kBatch = 8;      // tokens whose loads are in flight together

template <typename A, int V, bool EXACT>
__global__ void __launch_bounds__(128) zb_gated_maps_kernel(const GatedScanArgs p, const ZbVarlen b) {
  zb_pdl_launch();
  zb_pdl_wait();
  const int c = (blockIdx.x * 128 + threadIdx.x) * V, idx = blockIdx.y;
  int s, blk;
  if (!zb_find_block(b, kRows, idx, s, blk) || c >= p.width) return;
  const int t0 = b.q_start[s], n = b.q_start[s + 1] - t0;
  float2* maps = p.maps + static_cast<size_t>(idx) * p.width + c;
  if (blk == 0) {
    const int slot = p.slots[s];
    float st[V];
#pragma unroll
    for (int e = 0; e < V; ++e) st[e] = 0.f;
    if (ZB_BC_OK(slot, ZB_BC_STATE_SLOTS, kKernelGatedScan, 1)) first_state<V>(p, b, s, slot, c, st);
#pragma unroll
    for (int e = 0; e < V; ++e) maps[e] = make_float2(0.f, st[e]);
  }
  if ((blk + 1) * kRows >= n) return;
  const A* z = reinterpret_cast<const A*>(p.z) + static_cast<long long>(t0 + blk * kRows) * p.ld + c;
  const A* x = reinterpret_cast<const A*>(p.x) + static_cast<long long>(t0 + blk * kRows) * p.ld + c;
  float zb[V], xb[V], mul[V], add[V];
#pragma unroll
  for (int e = 0; e < V; ++e) {
    zb[e] = p.z_bias[c + e];
    xb[e] = p.x_bias[c + e];
    mul[e] = 1.f;
    add[e] = 0.f;
  }
#pragma unroll 1
  for (int i = 0; i < kRows; i += kBatch) {
    float zv[kBatch][V], xv[kBatch][V];
#pragma unroll
    for (int j = 0; j < kBatch; ++j) {
      ld_cols<V>(zv[j], z + (i + j) * p.ld);
      ld_cols<V>(xv[j], x + (i + j) * p.ld);
    }
#pragma unroll
    for (int j = 0; j < kBatch; ++j)
#pragma unroll
      for (int e = 0; e < V; ++e) {
        float open, keep;
        gates<EXACT>(zv[j][e] + zb[e], open, keep);
        mul[e] *= keep;
        add[e] = fmaf(keep, add[e], open * candidate<EXACT>(xv[j][e] + xb[e]));
      }
  }
#pragma unroll
  for (int e = 0; e < V; ++e) maps[p.width + e] = make_float2(mul[e], add[e]);
}

template <typename A, int V, bool EXACT>
__global__ void __launch_bounds__(128) zb_gated_walk_kernel(const GatedScanArgs p, const ZbVarlen b) {
  zb_pdl_launch();
  zb_pdl_wait();
  const int c = (blockIdx.x * 128 + threadIdx.x) * V, idx = blockIdx.y;
  int s, blk;
  if (!zb_find_block(b, kRows, idx, s, blk) || c >= p.width) return;
  const int t0 = b.q_start[s], n = b.q_start[s + 1] - t0;
  const float2* maps = p.maps + static_cast<size_t>(idx - blk) * p.width + c;
  float st[V];
#pragma unroll
  for (int e = 0; e < V; ++e) st[e] = 0.f;
#pragma unroll 8
  for (int j = 0; j <= blk; ++j) {
#pragma unroll
    for (int e = 0; e < V; ++e) {
      const float2 m = maps[static_cast<size_t>(j) * p.width + e];
      st[e] = fmaf(m.x, st[e], m.y);
    }
  }
  const int i0 = blk * kRows, rows = min(kRows, n - i0);
  const long long at = static_cast<long long>(t0 + i0);
  const A* z = reinterpret_cast<const A*>(p.z) + at * p.ld + c;
  const A* x = reinterpret_cast<const A*>(p.x) + at * p.ld + c;
  const A* g = reinterpret_cast<const A*>(p.gate) + at * p.ld + c;
  A* out = reinterpret_cast<A*>(p.out) + at * p.ld_out + c;
  float zb[V], xb[V];
#pragma unroll
  for (int e = 0; e < V; ++e) {
    zb[e] = p.z_bias[c + e];
    xb[e] = p.x_bias[c + e];
  }
#pragma unroll 1
  for (int i = 0; i < rows; i += kBatch) {
    float zv[kBatch][V], xv[kBatch][V], gv[kBatch][V];
#pragma unroll
    for (int j = 0; j < kBatch; ++j) {
      const long long r = min(i + j, rows - 1) * p.ld;
      ld_cols<V>(zv[j], z + r);
      ld_cols<V>(xv[j], x + r);
      ld_cols<V>(gv[j], g + r);
    }
#pragma unroll
    for (int j = 0; j < kBatch; ++j) {
      if (i + j >= rows) break;
      float o[V];
#pragma unroll
      for (int e = 0; e < V; ++e) {
        float open, keep;
        gates<EXACT>(zv[j][e] + zb[e], open, keep);
        st[e] = fmaf(keep, st[e], open * candidate<EXACT>(xv[j][e] + xb[e]));
        o[e] = st[e] * (gv[j][e] * sigmoid_of<EXACT>(gv[j][e])) * p.scale;
      }
      st_cols<V>(out + (i + j) * p.ld_out, o);
    }
  }
  if (i0 + rows < n) return;                             // the sequence's last block leaves the state behind
  const int slot = p.slots[s];
  if (!ZB_BC_OK(slot, ZB_BC_STATE_SLOTS, kKernelGatedScan, 2)) return;
#pragma unroll
  for (int e = 0; e < V; ++e) p.state[static_cast<size_t>(slot) * p.width + c + e] = st[e];
}

// One token per sequence.
template <typename A, int V, bool EXACT>
__global__ void __launch_bounds__(128) zb_gated_step_kernel(const GatedScanArgs p, const ZbVarlen b) {
  zb_pdl_launch();
  const int c = (blockIdx.x * 128 + threadIdx.x) * V, s = blockIdx.y;
  if (c >= p.width) return;
  float zb[V], xb[V];
#pragma unroll
  for (int e = 0; e < V; ++e) {
    zb[e] = p.z_bias[c + e];
    xb[e] = p.x_bias[c + e];
  }
  zb_pdl_wait();
  const int t = b.q_start[s], slot = p.slots[s];
  if (b.q_start[s + 1] <= t || !ZB_BC_OK(slot, ZB_BC_STATE_SLOTS, kKernelGatedScan, 3)) return;
  float st[V], zv[V], xv[V], gv[V];
  first_state<V>(p, b, s, slot, c, st);
  ld_cols<V>(zv, reinterpret_cast<const A*>(p.z) + t * p.ld + c);
  ld_cols<V>(xv, reinterpret_cast<const A*>(p.x) + t * p.ld + c);
  ld_cols<V>(gv, reinterpret_cast<const A*>(p.gate) + t * p.ld + c);
  float o[V];
#pragma unroll
  for (int e = 0; e < V; ++e) {
    float open, keep;
    gates<EXACT>(zv[e] + zb[e], open, keep);
    st[e] = fmaf(keep, st[e], open * candidate<EXACT>(xv[e] + xb[e]));
    o[e] = st[e] * (gv[e] * sigmoid_of<EXACT>(gv[e])) * p.scale;
    p.state[static_cast<size_t>(slot) * p.width + c + e] = st[e];
  }
  st_cols<V>(reinterpret_cast<A*>(p.out) + t * p.ld_out + c, o);
}

template <typename A, int V>
cudaError_t launch_scan(const GatedScanArgs& p, const ZbVarlen& b, int num_blocks, cudaStream_t s) {
  constexpr bool kExact = sizeof(A) == 4;
  const int cols = (p.width + 128 * V - 1) / (128 * V);
  if (num_blocks <= 0) {
    zb_count_launch(1);
    return zb_launch(zb_gated_step_kernel<A, V, kExact>, dim3(cols, b.num_seqs), dim3(128), 0, s, p, b);
  }
  cudaError_t e = zb_launch(zb_gated_maps_kernel<A, V, kExact>, dim3(cols, num_blocks), dim3(128), 0, s, p, b);
  if (e != cudaSuccess) return e;
  zb_count_launch(2);
  return zb_launch(zb_gated_walk_kernel<A, V, kExact>, dim3(cols, num_blocks), dim3(128), 0, s, p, b);
}
template <typename A>
cudaError_t launch_scan(const GatedScanArgs& p, const ZbVarlen& b, int num_blocks, cudaStream_t s) {
  const uintptr_t at = reinterpret_cast<uintptr_t>(p.z) | reinterpret_cast<uintptr_t>(p.x) | reinterpret_cast<uintptr_t>(p.gate) | reinterpret_cast<uintptr_t>(p.out);
  const bool vec = p.width % 2 == 0 && p.ld % 2 == 0 && p.ld_out % 2 == 0 && (at & (2 * sizeof(A) - 1)) == 0;
  return vec ? launch_scan<A, 2>(p, b, num_blocks, s) : launch_scan<A, 1>(p, b, num_blocks, s);
}
}  // namespace

extern "C" {

// Tokens per block of a varlen batch.
int zb_gated_scan_rows() { return kRows; }

// num_blocks >= sum over sequences of ceil(tokens / zb_gated_scan_rows()), `maps` holds num_blocks * width pairs of floats; or 0 and
// null for one token per sequence.
int zb_gated_scan(const void* z, const void* x, const void* gate, long long ld, const float* z_bias, const float* x_bias, float* state, const int32_t* slots,
                  float* maps, void* out, long long ld_out, float scale, int width, int act_f32, const int32_t* q_start, const int32_t* seq_lens,
                  int num_seqs, int num_blocks, void* stream) {
  if (num_seqs <= 0 || width <= 0) return 0;
  if (num_blocks > 65535 || num_seqs > 65535 || (num_blocks > 0 && maps == nullptr)) return -70;
  const GatedScanArgs p = {z, x, gate, ld, z_bias, x_bias, state, slots, reinterpret_cast<float2*>(maps), out, ld_out, scale, width};
  const ZbVarlen b = {q_start, seq_lens, num_seqs};
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const cudaError_t e = act_f32 ? launch_scan<float>(p, b, num_blocks, s) : launch_scan<__nv_bfloat16>(p, b, num_blocks, s);
  return static_cast<int>(e != cudaSuccess ? e : cudaGetLastError());
}

}  // extern "C"
