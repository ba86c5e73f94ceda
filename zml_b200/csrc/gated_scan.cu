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

// Of one token and two channels (the second one idle where a thread has one): S <- keep S + add, gate = silu(g).
struct Terms {
  ZbF2 keep, add, gate;
};
constexpr float kLog2e = 1.4426950408889634f;
// EXACT: each sigmoid 1 / (1 + e^-v) by itself, in fp32 functions.  Else by powers of two (the caller's z_bias is times -log2 e)
// and one reciprocal of the product of the denominators.  There arguments are cut at -29: three factors stay below 2^126, and
// a gate that is shut further adds less than 3e-13 of a candidate.
template <bool EXACT, bool WITH_GATE>
ZB_DEVICE Terms terms_of(const float (&z)[2], const float (&x)[2], const float (&g)[2], ZbF2 z_bias, ZbF2 x_bias) {
  Terms o;
  if constexpr (EXACT) {
    float zb[2], xb[2], keep[2], add[2], gate[2];
    zb_unpack2(z_bias, zb[0], zb[1]);
    zb_unpack2(x_bias, xb[0], xb[1]);
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const float e = expf(-fmaxf(z[i] + zb[i], -80.f)), open = 1.f / (1.f + e), u = x[i] + xb[i];
      keep[i] = e * open;
      add[i] = open * (u >= 0.f ? u + 0.5f : 1.f / (1.f + expf(-fmaxf(u, -80.f))));
      gate[i] = WITH_GATE ? g[i] / (1.f + expf(-fmaxf(g[i], -80.f))) : 0.f;
    }
    o.keep = zb_pack2(keep[0], keep[1]);
    o.add = zb_pack2(add[0], add[1]);
    o.gate = zb_pack2(gate[0], gate[1]);
  } else {
    const ZbF2 one = zb_pack2(1.f, 1.f), half = zb_pack2(0.5f, 0.5f), minus = zb_pack2(-kLog2e, -kLog2e);
    auto power = [](ZbF2 v) {
      float v0, v1;
      zb_unpack2(v, v0, v1);
      return zb_pack2(zb_ex2(fminf(v0, 29.f * kLog2e)), zb_ex2(fminf(v1, 29.f * kLog2e)));
    };
    auto inverse = [](ZbF2 v) {
      float v0, v1;
      zb_unpack2(v, v0, v1);
      return zb_pack2(zb_rcp(v0), zb_rcp(v1));
    };
    const ZbF2 u = zb_add2(zb_pack2(x[0], x[1]), x_bias), g2 = zb_pack2(g[0], g[1]);
    const ZbF2 e = power(zb_fma2(zb_pack2(z[0], z[1]), minus, z_bias)), a = zb_add2(e, one), b = zb_add2(power(zb_mul2(u, minus)), one), ab = zb_mul2(a, b);
    ZbF2 r, rab;
    if constexpr (WITH_GATE) {
      const ZbF2 c = zb_add2(power(zb_mul2(g2, minus)), one);
      r = inverse(zb_mul2(ab, c));
      rab = zb_mul2(r, c);
      o.gate = zb_mul2(g2, zb_mul2(r, ab));
    } else {
      r = rab = inverse(ab);
      o.gate = 0ull;
    }
    const ZbF2 open = zb_mul2(rab, b);
    float u0, u1, p0, p1, s0, s1;
    zb_unpack2(u, u0, u1);
    zb_unpack2(zb_add2(u, half), p0, p1);
    zb_unpack2(zb_mul2(rab, a), s0, s1);
    o.keep = zb_mul2(e, open);
    o.add = zb_mul2(open, zb_pack2(u0 >= 0.f ? p0 : s0, u1 >= 0.f ? p1 : s1));
  }
  return o;
}

// This thread's biases as `terms_of` takes them.
template <int V, bool EXACT>
ZB_DEVICE void load_biases(const GatedScanArgs& p, int c, ZbF2& z_bias, ZbF2& x_bias) {
  const float f = EXACT ? 1.f : -kLog2e;
  z_bias = zb_pack2(f * p.z_bias[c], V == 2 ? f * p.z_bias[c + V - 1] : 0.f);
  x_bias = zb_pack2(p.x_bias[c], V == 2 ? p.x_bias[c + V - 1] : 0.f);
}

// V neighbouring columns as they are stored.
template <typename A, int V>
struct Cols;
template <>
struct Cols<__nv_bfloat16, 2> {
  uint32_t raw;
  ZB_DEVICE void load(const __nv_bfloat16* p) { raw = *reinterpret_cast<const uint32_t*>(p); }
  ZB_DEVICE void get(float (&v)[2]) const {
    const float2 f = zb_unpack_bf16x2(raw);
    v[0] = f.x; v[1] = f.y;
  }
};
template <>
struct Cols<float, 2> {
  float2 raw;
  ZB_DEVICE void load(const float* p) { raw = *reinterpret_cast<const float2*>(p); }
  ZB_DEVICE void get(float (&v)[2]) const { v[0] = raw.x; v[1] = raw.y; }
};
template <typename A>
struct Cols<A, 1> {
  A raw;
  ZB_DEVICE void load(const A* p) { raw = *p; }
  ZB_DEVICE void get(float (&v)[2]) const {
    v[0] = zb_ld_act(&raw);
    v[1] = 0.f;
  }
};
template <int V>
ZB_DEVICE void st_cols(__nv_bfloat16* p, ZbF2 v) {
  float a, b;
  zb_unpack2(v, a, b);
  if constexpr (V == 2) *reinterpret_cast<uint32_t*>(p) = zb_pack_bf16x2(a, b);
  else zb_st_act(p, a);
}
template <int V>
ZB_DEVICE void st_cols(float* p, ZbF2 v) {
  float a, b;
  zb_unpack2(v, a, b);
  if constexpr (V == 2) *reinterpret_cast<float2*>(p) = make_float2(a, b);
  else *p = a;
}

// State of sequence s in front of the launch; zero for one that starts here.
template <int V>
ZB_DEVICE ZbF2 first_state(const GatedScanArgs& p, const ZbVarlen& b, int s, int slot, int c) {
  if (b.seq_lens[s] - (b.q_start[s + 1] - b.q_start[s]) <= 0) return 0ull;
  const float* st = p.state + static_cast<size_t>(slot) * p.width + c;
  return zb_pack2(st[0], V == 2 ? st[V - 1] : 0.f);
}
template <int V>
ZB_DEVICE void store_state(const GatedScanArgs& p, int slot, int c, ZbF2 st) {
  st_cols<1>(p.state + static_cast<size_t>(slot) * p.width + c, st);
  float a, b;
  zb_unpack2(st, a, b);
  if (V == 2) p.state[static_cast<size_t>(slot) * p.width + c + 1] = b;
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
  auto put = [&](float2* to, ZbF2 mul, ZbF2 add) {
    float m0, m1, a0, a1;
    zb_unpack2(mul, m0, m1);
    zb_unpack2(add, a0, a1);
    to[0] = make_float2(m0, a0);
    if (V == 2) to[V - 1] = make_float2(m1, a1);
  };
  if (blk == 0) {
    const int slot = p.slots[s];
    put(maps, 0ull, ZB_BC_OK(slot, ZB_BC_STATE_SLOTS, kKernelGatedScan, 1) ? first_state<V>(p, b, s, slot, c) : 0ull);
  }
  if ((blk + 1) * kRows >= n) return;
  const A* z = reinterpret_cast<const A*>(p.z) + static_cast<long long>(t0 + blk * kRows) * p.ld + c;
  const A* x = reinterpret_cast<const A*>(p.x) + static_cast<long long>(t0 + blk * kRows) * p.ld + c;
  ZbF2 zb, xb, mul = zb_pack2(1.f, 1.f), add = 0ull;
  load_biases<V, EXACT>(p, c, zb, xb);
#pragma unroll 1
  for (int i = 0; i < kRows; i += kBatch) {
    Cols<A, V> zc[kBatch], xc[kBatch];
#pragma unroll
    for (int j = 0; j < kBatch; ++j) {
      zc[j].load(z);
      xc[j].load(x);
      z += p.ld;
      x += p.ld;
    }
#pragma unroll
    for (int j = 0; j < kBatch; ++j) {
      float zv[2], xv[2];
      zc[j].get(zv);
      xc[j].get(xv);
      const Terms g = terms_of<EXACT, false>(zv, xv, xv, zb, xb);
      mul = zb_mul2(mul, g.keep);
      add = zb_fma2(g.keep, add, g.add);
    }
  }
  put(maps + p.width, mul, add);
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
  ZbF2 st = 0ull;
#pragma unroll 8
  for (int j = 0; j <= blk; ++j) {
    const float2 m0 = maps[static_cast<size_t>(j) * p.width], m1 = V == 2 ? maps[static_cast<size_t>(j) * p.width + V - 1] : m0;
    st = zb_fma2(zb_pack2(m0.x, m1.x), st, zb_pack2(m0.y, m1.y));
  }
  const int i0 = blk * kRows, rows = min(kRows, n - i0);
  const long long at = static_cast<long long>(t0 + i0);
  const A* z = reinterpret_cast<const A*>(p.z) + at * p.ld + c;
  const A* x = reinterpret_cast<const A*>(p.x) + at * p.ld + c;
  const A* g = reinterpret_cast<const A*>(p.gate) + at * p.ld + c;
  A* out = reinterpret_cast<A*>(p.out) + at * p.ld_out + c;
  const ZbF2 scale = zb_pack2(p.scale, p.scale);
  ZbF2 zb, xb;
  load_biases<V, EXACT>(p, c, zb, xb);
  auto token = [&](const Cols<A, V>& zc, const Cols<A, V>& xc, const Cols<A, V>& gc) {
    float zv[2], xv[2], gv[2];
    zc.get(zv);
    xc.get(xv);
    gc.get(gv);
    const Terms t = terms_of<EXACT, true>(zv, xv, gv, zb, xb);
    st = zb_fma2(t.keep, st, t.add);
    st_cols<V>(out, zb_mul2(zb_mul2(st, t.gate), scale));
    out += p.ld_out;
  };
  int i = 0;
#pragma unroll 1
  for (; i + kBatch <= rows; i += kBatch) {
    Cols<A, V> zc[kBatch], xc[kBatch], gc[kBatch];
#pragma unroll
    for (int j = 0; j < kBatch; ++j) {
      zc[j].load(z);
      xc[j].load(x);
      gc[j].load(g);
      z += p.ld;
      x += p.ld;
      g += p.ld;
    }
#pragma unroll
    for (int j = 0; j < kBatch; ++j) token(zc[j], xc[j], gc[j]);
  }
#pragma unroll 1
  for (; i < rows; ++i) {
    Cols<A, V> zc, xc, gc;
    zc.load(z);
    xc.load(x);
    gc.load(g);
    z += p.ld;
    x += p.ld;
    g += p.ld;
    token(zc, xc, gc);
  }
  if (i0 + rows < n) return;                             // the sequence's last block leaves the state behind
  const int slot = p.slots[s];
  if (ZB_BC_OK(slot, ZB_BC_STATE_SLOTS, kKernelGatedScan, 2)) store_state<V>(p, slot, c, st);
}

// One token per sequence.
template <typename A, int V, bool EXACT>
__global__ void __launch_bounds__(128) zb_gated_step_kernel(const GatedScanArgs p, const ZbVarlen b) {
  zb_pdl_launch();
  const int c = (blockIdx.x * 128 + threadIdx.x) * V, s = blockIdx.y;
  if (c >= p.width) return;
  ZbF2 zb, xb;
  load_biases<V, EXACT>(p, c, zb, xb);
  zb_pdl_wait();
  const int t = b.q_start[s], slot = p.slots[s];
  if (b.q_start[s + 1] <= t || !ZB_BC_OK(slot, ZB_BC_STATE_SLOTS, kKernelGatedScan, 3)) return;
  Cols<A, V> zc, xc, gc;
  zc.load(reinterpret_cast<const A*>(p.z) + t * p.ld + c);
  xc.load(reinterpret_cast<const A*>(p.x) + t * p.ld + c);
  gc.load(reinterpret_cast<const A*>(p.gate) + t * p.ld + c);
  ZbF2 st = first_state<V>(p, b, s, slot, c);
  float zv[2], xv[2], gv[2];
  zc.get(zv);
  xc.get(xv);
  gc.get(gv);
  const Terms g = terms_of<EXACT, true>(zv, xv, gv, zb, xb);
  st = zb_fma2(g.keep, st, g.add);
  store_state<V>(p, slot, c, st);
  st_cols<V>(reinterpret_cast<A*>(p.out) + t * p.ld_out + c, zb_mul2(zb_mul2(st, g.gate), zb_pack2(p.scale, p.scale)));
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
