// Layer glue of decoders that keep the residual stream in fp32:
//
//   zb_embedding_f32   gathers table rows (bf16 or fp32), times a constant, into the fp32 stream (or several copies of it)
//   zb_post_norm       x <- layernorm(alpha * x + y) * w, the normalisation behind a sublayer;
//                      without y a plain layer norm.  For decode steps the same launch continues with the input
//                      convolution of the next layer (one token per sequence: everything it needs is in the row and
//                      in the sequence's state)
//   zb_sandwich_norm   x <- x + m * rmsnorm(y) * w, the residual sum of a sublayer with a norm behind it, and in the same
//                      launch rmsnorm(x) * w_next, what the next sublayer reads.  y is a row, or the weighted sum of a
//                      token's expert rows
//   zb_add_norm        x <- x + y, the residual sum of a sublayer with a norm in front (y as above), and in the same launch what
//                      the next sublayer reads: layernorm(x) * w + b, for decode steps on through its input convolution, or x
//                      itself in the activation type
//   zb_hyper_norm      hyper-connections: S streams per token instead of one.  x_t <- sum_s mix[s, t] x_s + out[t] y behind a
//                      sublayer (y as above), and in the same launch rmsnorm(sum_s in[s] x_s) * w, what the next one reads
//   zb_stream_conv     that input convolution over a varlen batch: h = x + conv(x), causal and per channel, and for
//                      token-shift mixers the interpolations h + (h_prev - h) * mu of h with the previous token's h
//
// Sums, norms and convolutions are fp32; what a projection reads is written as bf16 or fp32.  The state of a sequence
// is the last `rows` rows of x (taps - 1 of them, or taps when the previous token's h is needed: it is computed again
// from x rather than stored).
#include "act.cuh"
#include "host_api.h"

namespace {
constexpr uint32_t kKernelEmbeddingF32 = 26;
constexpr uint32_t kKernelStreamConv = 27;
constexpr int kMaxMix = 5;
constexpr int kMaxTaps = 8;

template <typename W>
__global__ void __launch_bounds__(256) zb_embedding_f32_kernel(const int32_t* __restrict__ ids, const W* __restrict__ table,
                                                               float* __restrict__ out, int d, int vocab, float scale, int copies) {
  zb_pdl_launch();
  zb_pdl_wait();
  const int t = blockIdx.x;
  int id = ids[t];
  if (id < 0 || id >= vocab) {
    (void)ZB_BC_OK(id, vocab, kKernelEmbeddingF32, 1);
    id = 0;
  }
  const W* src = table + static_cast<size_t>(id) * d;
  float* dst = out + static_cast<size_t>(t) * copies * d;
  for (int i = threadIdx.x; i < d; i += 256) {
    const float v = scale * zb_ld_act(src + i);
    for (int c = 0; c < copies; ++c) dst[static_cast<size_t>(c) * d + i] = v;
  }
}

// ------------------------------------------------------------------------------------------ convolution
struct ConvArgs {
  const float* w;          // [taps, d], tap taps - 1 on the current token
  float* state;            // [slots, rows, d]: the last `rows` inputs, oldest first
  const int32_t* slots;    // [num_seqs]
  const float* mu;         // [nmix, d] or null
  void* out;               // h [T, ld], or the nmix interpolations [nmix][T, ld]
  long long ld;
  long long plane;         // elements between interpolations
  int taps;
  int rows;
  int nmix;                // 0: h itself
  int d;
};

template <typename A>
ZB_DEVICE void emit_h(const ConvArgs& a, long long t, int c, float h, float h_prev) {
  A* out = reinterpret_cast<A*>(a.out) + t * a.ld + c;
  if (a.nmix == 0) {
    zb_st_act(out, h);
    return;
  }
  const float delta = h_prev - h;
  for (int m = 0; m < a.nmix; ++m) zb_st_act(out + m * a.plane, h + delta * a.mu[static_cast<size_t>(m) * a.d + c]);
}

template <int V>
ZB_DEVICE void ld_vec(float (&v)[V], const float* p) {
  if constexpr (V == 4) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
  } else {
    v[0] = *p;
  }
}
template <typename A, int V>
ZB_DEVICE void st_vec(A* p, const float (&v)[V]) {
  if constexpr (V == 4 && sizeof(A) == 2) *reinterpret_cast<uint2*>(p) = make_uint2(zb_pack_bf16x2(v[0], v[1]), zb_pack_bf16x2(v[2], v[3]));
  else if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  else zb_st_act(p, v[0]);
}

// One thread owns V neighbouring channels and walks a block of kConvRows tokens of one sequence; T >= taps bounds the
// unrolled window.
constexpr int kConvRows = 32;

template <typename A, int T, int V, bool MIX>
__global__ void __launch_bounds__(128) zb_stream_conv_kernel(const float* __restrict__ x, const ConvArgs a, const ZbVarlen b) {
  zb_pdl_launch();
  zb_pdl_wait();
  const int c = (blockIdx.x * 128 + threadIdx.x) * V;
  int s, blk;
  if (c >= a.d || !zb_find_block(b, kConvRows, blockIdx.y, s, blk)) return;
  const int slot = a.slots[s];
  if (!ZB_BC_OK(slot, ZB_BC_STATE_SLOTS, kKernelStreamConv, 1)) return;
  const int t0 = b.q_start[s], n = b.q_start[s + 1] - t0;
  const bool fresh = b.seq_lens[s] - n <= 0;
  const int taps = a.taps, rows = a.rows;
  float* st = a.state + static_cast<size_t>(slot) * rows * a.d + c;
  const float* xs = x + static_cast<size_t>(t0) * a.d + c;
  // input `i` tokens after the launch's first token of this sequence (negative: before it)
  auto input = [&](int i, float (&v)[V]) {
#pragma unroll
    for (int e = 0; e < V; ++e) v[e] = 0.f;
    if (i >= 0) ld_vec<V>(v, xs + static_cast<size_t>(i) * a.d);
    else if (!fresh && i >= -rows) ld_vec<V>(v, st + static_cast<size_t>(rows + i) * a.d);
  };
  float w[T][V], win[T][V];                   // win[j]: the input T - 1 - j tokens before the current one; the last taps count
#pragma unroll
  for (int j = 0; j < T; ++j)
#pragma unroll
    for (int e = 0; e < V; ++e) w[j][e] = j >= T - taps ? a.w[static_cast<size_t>(j - (T - taps)) * a.d + c + e] : 0.f;
  float mu[MIX ? kMaxMix : 1][V];
  if constexpr (MIX) {
#pragma unroll
    for (int m = 0; m < kMaxMix; ++m)
      if (m < a.nmix) ld_vec<V>(mu[m], a.mu + static_cast<size_t>(m) * a.d + c);
  }
  const int i0 = blk * kConvRows, i1 = min(n, i0 + kConvRows);
  auto conv = [&](float (&h)[V]) {            // the newest input plus the weighted window
#pragma unroll
    for (int e = 0; e < V; ++e) {
      float acc = 0.f;
#pragma unroll
      for (int j = 0; j < T; ++j) acc = fmaf(w[j][e], win[j][e], acc);
      h[e] = win[T - 1][e] + acc;
    }
  };
#pragma unroll
  for (int j = 0; j < T; ++j) {
    if (j >= T - taps) input(i0 - T + j, win[j]);
    else
#pragma unroll
      for (int e = 0; e < V; ++e) win[j][e] = 0.f;
  }
  float h_prev[V];
  conv(h_prev);                               // (used with interpolations only: there the state reaches far enough back)
  A* out = reinterpret_cast<A*>(a.out) + static_cast<long long>(t0) * a.ld + c;
#pragma unroll 4
  for (int i = i0; i < i1; ++i) {
    float cur[V], h[V];
    ld_vec<V>(cur, xs + static_cast<size_t>(i) * a.d);
#pragma unroll
    for (int j = 0; j < T; ++j)
#pragma unroll
      for (int e = 0; e < V; ++e) win[j][e] = j + 1 < T ? win[j + 1 < T ? j + 1 : j][e] : cur[e];
    conv(h);
    A* o = out + i * a.ld;
    if constexpr (MIX) {
#pragma unroll
      for (int m = 0; m < kMaxMix; ++m) {
        if (m >= a.nmix) break;
        float v[V];
#pragma unroll
        for (int e = 0; e < V; ++e) v[e] = fmaf(h_prev[e] - h[e], mu[m][e], h[e]);
        st_vec<A, V>(o + m * a.plane, v);
      }
#pragma unroll
      for (int e = 0; e < V; ++e) h_prev[e] = h[e];
    } else {
      st_vec<A, V>(o, h);
    }
  }
  // The block that reads the old state also writes the new one: no other thread touches these channels' state.
  if (blk == 0) {
    float keep[kMaxTaps][V];
#pragma unroll
    for (int j = 0; j < kMaxTaps; ++j)
      if (j < rows) input(n - rows + j, keep[j]);
#pragma unroll
    for (int j = 0; j < kMaxTaps; ++j)
      if (j < rows) st_vec<float, V>(st + static_cast<size_t>(j) * a.d, keep[j]);
  }
}

template <typename A, int V, bool MIX>
cudaError_t launch_conv(const float* x, const ConvArgs& a, const ZbVarlen& b, int num_blocks, cudaStream_t s) {
  const dim3 grid((a.d + 128 * V - 1) / (128 * V), num_blocks);
  if (a.taps <= 3) return zb_launch(zb_stream_conv_kernel<A, 3, V, MIX>, grid, dim3(128), 0, s, x, a, b);
  if (a.taps == 4) return zb_launch(zb_stream_conv_kernel<A, 4, V, MIX>, grid, dim3(128), 0, s, x, a, b);
  return zb_launch(zb_stream_conv_kernel<A, kMaxTaps, V, MIX>, grid, dim3(128), 0, s, x, a, b);
}
template <typename A>
cudaError_t launch_conv(const float* x, const ConvArgs& a, const ZbVarlen& b, int num_blocks, cudaStream_t s) {
  const bool vec = a.d % 4 == 0 && a.ld % 4 == 0 && a.plane % 4 == 0;
  if (a.nmix > 0) return vec ? launch_conv<A, 4, true>(x, a, b, num_blocks, s) : launch_conv<A, 1, true>(x, a, b, num_blocks, s);
  return vec ? launch_conv<A, 4, false>(x, a, b, num_blocks, s) : launch_conv<A, 1, false>(x, a, b, num_blocks, s);
}

// ------------------------------------------------------------------------------------------ post norm
struct PostNormArgs {
  const void* y;           // sublayer output, bf16 or fp32, or null
  long long ldy;
  int y_f32;
  const float* x;          // [T, d]
  float alpha;
  const float* w;          // [d]
  float eps;
  float* x_out;            // [T, d] or null (may be x)
  void* act;               // [T, ld_act] or null: the same rows in the activation type
  long long ld_act;
  int d;
  int conv;                // 1: one token per sequence, continue with the convolution
};

ZB_DEVICE float block_sum_256(float v, float* red) {
  v = zb_warp_sum(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float tot = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) tot += red[i];
  return tot;
}

// NV values per thread; VEC: groups of four consecutive channels (d a multiple of 4), else one channel each.
template <typename A, int NV, bool VEC>
__global__ void __launch_bounds__(256) zb_post_norm_kernel(const PostNormArgs p, const ConvArgs a, const ZbVarlen b) {
  zb_pdl_launch();
  zb_pdl_wait();
  __shared__ float red[8];
  const long long t = blockIdx.x;
  const int d = p.d;
  auto channel = [&](int i) { return VEC ? (threadIdx.x + 256 * (i >> 2)) * 4 + (i & 3) : threadIdx.x + 256 * i; };
  const float* xr = p.x + t * d;
  float v[NV];
#pragma unroll
  for (int i = 0; i < NV; i += VEC ? 4 : 1) {
    const int c = channel(i);
    if constexpr (VEC) {
      float4 f = make_float4(0.f, 0.f, 0.f, 0.f);
      if (c < d) {
        f = *reinterpret_cast<const float4*>(xr + c);
        f.x *= p.alpha; f.y *= p.alpha; f.z *= p.alpha; f.w *= p.alpha;
        if (p.y != nullptr && p.y_f32) {
          const float4 g = *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(p.y) + t * p.ldy + c);
          f.x += g.x; f.y += g.y; f.z += g.z; f.w += g.w;
        } else if (p.y != nullptr) {
          const uint2 g = *reinterpret_cast<const uint2*>(reinterpret_cast<const __nv_bfloat16*>(p.y) + t * p.ldy + c);
          const float2 lo = zb_unpack_bf16x2(g.x), hi = zb_unpack_bf16x2(g.y);
          f.x += lo.x; f.y += lo.y; f.z += hi.x; f.w += hi.y;
        }
      }
      v[i] = f.x; v[i + 1] = f.y; v[i + 2] = f.z; v[i + 3] = f.w;
    } else {
      v[i] = 0.f;
      if (c < d) {
        v[i] = p.alpha * xr[c];
        if (p.y != nullptr)
          v[i] += p.y_f32 ? reinterpret_cast<const float*>(p.y)[t * p.ldy + c]
                          : __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(p.y)[t * p.ldy + c]);
      }
    }
  }
  float sum = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) sum += v[i];
  const float mean = block_sum_256(sum, red) / static_cast<float>(d);
  float sq = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    if (channel(i) < d) {
      v[i] -= mean;
      sq += v[i] * v[i];
    }
  }
  const float inv = 1.f / sqrtf(block_sum_256(sq, red) / static_cast<float>(d) + p.eps);
#pragma unroll
  for (int i = 0; i < NV; i += VEC ? 4 : 1) {
    const int c = channel(i);
    if (c >= d) continue;
    if constexpr (VEC) {
      const float4 g = *reinterpret_cast<const float4*>(p.w + c);
      v[i] *= inv * g.x; v[i + 1] *= inv * g.y; v[i + 2] *= inv * g.z; v[i + 3] *= inv * g.w;
      if (p.x_out != nullptr) *reinterpret_cast<float4*>(p.x_out + t * d + c) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
      if (p.act != nullptr) {
        A* o = reinterpret_cast<A*>(p.act) + t * p.ld_act + c;
        if constexpr (sizeof(A) == 2) {
          if ((p.ld_act & 3) == 0) {
            *reinterpret_cast<uint2*>(o) = make_uint2(zb_pack_bf16x2(v[i], v[i + 1]), zb_pack_bf16x2(v[i + 2], v[i + 3]));
            continue;
          }
        }
#pragma unroll
        for (int e = 0; e < 4; ++e) zb_st_act(o + e, v[i + e]);
      }
    } else {
      v[i] *= inv * p.w[c];
      if (p.x_out != nullptr) p.x_out[t * d + c] = v[i];
      if (p.act != nullptr) zb_st_act(reinterpret_cast<A*>(p.act) + t * p.ld_act + c, v[i]);
    }
  }
  if (!p.conv) return;
  const int s = static_cast<int>(t);
  const int slot = a.slots[s];
  if (!ZB_BC_OK(slot, ZB_BC_STATE_SLOTS, kKernelStreamConv, 2)) return;
  const bool fresh = b.seq_lens[s] - 1 <= 0;
  float* st0 = a.state + static_cast<size_t>(slot) * a.rows * d;
  const int taps = a.taps;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = channel(i);
    if (c >= d) continue;
    float* st = st0 + c;
    float hist[kMaxTaps];                    // hist[j]: the j-th row of the state
#pragma unroll
    for (int j = 0; j < kMaxTaps; ++j) hist[j] = (j < a.rows && !fresh) ? st[static_cast<size_t>(j) * d] : 0.f;
    const int off = a.rows - (taps - 1);     // 1 when the state also reaches the previous token's first tap
    float h = 0.f, hp = 0.f;
#pragma unroll
    for (int j = 0; j < kMaxTaps; ++j) {
      if (j < taps) {
        const float w = a.w[static_cast<size_t>(j) * d + c];
        if (off == 1) hp += w * hist[j];
        float in = v[i];
        if (j < taps - 1) in = off == 1 ? hist[j + 1 < kMaxTaps ? j + 1 : j] : hist[j];
        h += w * in;
      }
    }
#pragma unroll
    for (int j = 0; j < kMaxTaps; ++j)
      if (off == 1 && j == taps - 1) hp += hist[j];
    emit_h<A>(a, t, c, v[i] + h, hp);
#pragma unroll
    for (int j = 0; j < kMaxTaps; ++j) {
      if (j < a.rows - 1) st[static_cast<size_t>(j) * d] = hist[j + 1 < kMaxTaps ? j + 1 : j];
      else if (j == a.rows - 1) st[static_cast<size_t>(j) * d] = v[i];
    }
  }
}

// The decode step's form of the above for d a multiple of 4: 512 threads, NG groups of four channels each.  Everything
// that the convolution reads is requested before the norm's reductions, the parameters even before the preceding kernel
// has finished; T >= taps.
template <int N>
ZB_DEVICE float block_sum_warps(float v, float* red) {
  v = zb_warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float tot = 0.f;
#pragma unroll
  for (int i = 0; i < N; ++i) tot += red[i];
  return tot;
}

template <typename A, int NG, int T, bool MIX>
__global__ void __launch_bounds__(512) zb_post_norm_conv_kernel(const PostNormArgs p, const ConvArgs a, const ZbVarlen b) {
  constexpr int R = MIX ? T : T - 1;                     // rows of state the window can need
  __shared__ float red[2][16];
  zb_pdl_launch();
  const int d = p.d, taps = a.taps, rows = a.rows;
  float w[NG][T][4], mu[NG][MIX ? kMaxMix : 1][4], nw[NG][4];
#pragma unroll
  for (int i = 0; i < NG; ++i) {
    const int c = (threadIdx.x + 512 * i) * 4;
    if (c >= d) continue;
    ld_vec<4>(nw[i], p.w + c);
#pragma unroll
    for (int j = 0; j < T; ++j) {                        // the last taps of the window count
      if (j >= T - taps) ld_vec<4>(w[i][j], a.w + static_cast<size_t>(j - (T - taps)) * d + c);
      else w[i][j][0] = w[i][j][1] = w[i][j][2] = w[i][j][3] = 0.f;
    }
    if constexpr (MIX) {
#pragma unroll
      for (int m = 0; m < kMaxMix; ++m)
        if (m < a.nmix) ld_vec<4>(mu[i][m], a.mu + static_cast<size_t>(m) * d + c);
    }
  }
  zb_pdl_wait();
  const int s = blockIdx.x;
  const long long t = s;
  const int slot = a.slots[s];
  const bool slot_ok = ZB_BC_OK(slot, ZB_BC_STATE_SLOTS, kKernelStreamConv, 2);
  const bool fresh = b.seq_lens[s] - 1 <= 0 || !slot_ok;
  float* st0 = a.state + static_cast<size_t>(slot_ok ? slot : 0) * rows * d;
  float v[NG][4], hist[NG][R > 0 ? R : 1][4];             // hist[R - 1]: the newest past input
#pragma unroll
  for (int i = 0; i < NG; ++i) {
    const int c = (threadIdx.x + 512 * i) * 4;
#pragma unroll
    for (int e = 0; e < 4; ++e) v[i][e] = 0.f;
    if (c >= d) continue;
    ld_vec<4>(v[i], p.x + t * d + c);
    float y[4] = {0.f, 0.f, 0.f, 0.f};
    if (p.y != nullptr && p.y_f32) {
      ld_vec<4>(y, reinterpret_cast<const float*>(p.y) + t * p.ldy + c);
    } else if (p.y != nullptr) {
      const uint2 g = *reinterpret_cast<const uint2*>(reinterpret_cast<const __nv_bfloat16*>(p.y) + t * p.ldy + c);
      const float2 lo = zb_unpack_bf16x2(g.x), hi = zb_unpack_bf16x2(g.y);
      y[0] = lo.x; y[1] = lo.y; y[2] = hi.x; y[3] = hi.y;
    }
#pragma unroll
    for (int j = 0; j < R; ++j) {
      if (j >= R - rows && !fresh) ld_vec<4>(hist[i][j], st0 + static_cast<size_t>(j - (R - rows)) * d + c);
      else hist[i][j][0] = hist[i][j][1] = hist[i][j][2] = hist[i][j][3] = 0.f;
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) v[i][e] = fmaf(p.alpha, v[i][e], y[e]);
  }
  float sum = 0.f;
#pragma unroll
  for (int i = 0; i < NG; ++i) sum += (v[i][0] + v[i][1]) + (v[i][2] + v[i][3]);
  const float mean = block_sum_warps<16>(sum, red[0]) / static_cast<float>(d);
  float sq = 0.f;
#pragma unroll
  for (int i = 0; i < NG; ++i) {
    if ((threadIdx.x + 512 * i) * 4 >= d) continue;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      v[i][e] -= mean;
      sq = fmaf(v[i][e], v[i][e], sq);
    }
  }
  const float inv = 1.f / sqrtf(block_sum_warps<16>(sq, red[1]) / static_cast<float>(d) + p.eps);
#pragma unroll
  for (int i = 0; i < NG; ++i) {
    const int c = (threadIdx.x + 512 * i) * 4;
    if (c >= d) continue;
    float h[4], hp[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      v[i][e] *= inv * nw[i][e];
      float acc = w[i][T - 1][e] * v[i][e], prev = 0.f;
#pragma unroll
      for (int j = 0; j + 1 < T; ++j) acc = fmaf(w[i][j][e], hist[i][j + R - (T - 1)][e], acc);
      if constexpr (MIX) {
#pragma unroll
        for (int j = 0; j < T; ++j) prev = fmaf(w[i][j][e], hist[i][j][e], prev);
        prev += hist[i][R - 1][e];
      }
      h[e] = v[i][e] + acc;
      hp[e] = prev;
    }
    if (p.x_out != nullptr) st_vec<float, 4>(p.x_out + t * d + c, v[i]);
    A* out = reinterpret_cast<A*>(a.out) + t * a.ld + c;
    if constexpr (MIX) {
#pragma unroll
      for (int m = 0; m < kMaxMix; ++m) {
        if (m >= a.nmix) break;
        float o[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) o[e] = fmaf(hp[e] - h[e], mu[i][m][e], h[e]);
        st_vec<A, 4>(out + m * a.plane, o);
      }
    } else {
      st_vec<A, 4>(out, h);
    }
    if (!slot_ok) continue;
#pragma unroll
    for (int j = 0; j < R; ++j) {
      if (j < R - rows) continue;
      float* dst = st0 + static_cast<size_t>(j - (R - rows)) * d + c;
      if (j + 1 < R) st_vec<float, 4>(dst, hist[i][j + 1 < R ? j + 1 : j]);
      else st_vec<float, 4>(dst, v[i]);
    }
  }
}

// ------------------------------------------------------------------------------------------ sandwich norm
struct SandwichArgs {
  const void* y;               // sublayer output [T, ldy], or expert rows [*, ldy] with pair_pos, or null: no residual sum
  long long ldy;
  const int32_t* pair_pos;     // [T, k]: row of y of every (token, chosen expert) pair, negative: held by another rank
  const float* pair_w;         // [T, k]
  int k;
  const float* x;              // [T, d]
  float mult;
  const float* w;              // [d]: norm behind the sublayer
  const float* w_next;         // [d] or null: no second norm
  float eps;
  float* x_out;                // [T, d] or null (may be x)
  void* act;                   // [T, ld_act]: columns d .. ld_act are zero
  long long ld_act;
  int d;
};

// Four values of a row at column c.
ZB_DEVICE void ld_row4(float (&v)[4], const float* p) { ld_vec<4>(v, p); }
ZB_DEVICE void ld_row4(float (&v)[4], const __nv_bfloat16* p) {
  const uint2 g = *reinterpret_cast<const uint2*>(p);
  const float2 lo = zb_unpack_bf16x2(g.x), hi = zb_unpack_bf16x2(g.y);
  v[0] = lo.x; v[1] = lo.y; v[2] = hi.x; v[3] = hi.y;
}

// Y: type of y, A: type of act.  NT threads, NG groups of V neighbouring channels per thread.
template <typename Y, typename A, int NT, int NG, int V>
__global__ void __launch_bounds__(NT) zb_sandwich_norm_kernel(const SandwichArgs p) {
  constexpr int kSlots = 32;                             // expert slots read through shared memory at a time
  __shared__ float red[2][NT / 32];
  __shared__ float sw[kSlots];
  __shared__ int spos[kSlots];
  zb_pdl_launch();
  const int d = p.d;
  float w[NG][V], wn[NG][V];                             // parameters: on their way before the input is there
#pragma unroll
  for (int i = 0; i < NG; ++i) {
    const int c = (threadIdx.x + NT * i) * V;
#pragma unroll
    for (int e = 0; e < V; ++e) w[i][e] = wn[i][e] = 0.f;
    if (c < d && p.y != nullptr) ld_vec<V>(w[i], p.w + c);
    if (c < d && p.w_next != nullptr) ld_vec<V>(wn[i], p.w_next + c);
  }
  zb_pdl_wait();
  const long long t = blockIdx.x;
  float x[NG][V], y[NG][V];
#pragma unroll
  for (int i = 0; i < NG; ++i) {
    const int c = (threadIdx.x + NT * i) * V;
#pragma unroll
    for (int e = 0; e < V; ++e) x[i][e] = y[i][e] = 0.f;
    if (c < d) ld_vec<V>(x[i], p.x + t * d + c);
  }
  if (p.y != nullptr) {
    const Y* ys = reinterpret_cast<const Y*>(p.y);
    auto add = [&](long long row, float wt) {
#pragma unroll
      for (int i = 0; i < NG; ++i) {
        const int c = (threadIdx.x + NT * i) * V;
        if (c >= d) continue;
        float v[V];
        if constexpr (V == 4) ld_row4(v, ys + row * p.ldy + c);
        else v[0] = zb_ld_act(ys + row * p.ldy + c);
#pragma unroll
        for (int e = 0; e < V; ++e) y[i][e] = fmaf(wt, v[e], y[i][e]);
      }
    };
    if (p.pair_pos == nullptr) {
      add(t, 1.f);
    } else {
      for (int j0 = 0; j0 < p.k; j0 += kSlots) {
        const int n = min(kSlots, p.k - j0);
        __syncthreads();
        if (threadIdx.x < n) {
          spos[threadIdx.x] = p.pair_pos[t * p.k + j0 + threadIdx.x];
          sw[threadIdx.x] = p.pair_w[t * p.k + j0 + threadIdx.x];
        }
        __syncthreads();
#pragma unroll 4
        for (int j = 0; j < n; ++j)
          if (spos[j] >= 0) add(spos[j], sw[j]);
      }
    }
    float sq = 0.f;
#pragma unroll
    for (int i = 0; i < NG; ++i)
#pragma unroll
      for (int e = 0; e < V; ++e) sq = fmaf(y[i][e], y[i][e], sq);
    const float inv = p.mult / sqrtf(block_sum_warps<NT / 32>(sq, red[0]) / static_cast<float>(d) + p.eps);
#pragma unroll
    for (int i = 0; i < NG; ++i) {
      const int c = (threadIdx.x + NT * i) * V;
      if (c >= d) continue;
#pragma unroll
      for (int e = 0; e < V; ++e) x[i][e] = fmaf(inv * y[i][e], w[i][e], x[i][e]);
      if (p.x_out != nullptr) st_vec<float, V>(p.x_out + t * d + c, x[i]);
    }
  }
  if (p.act == nullptr) return;
  float sq = 0.f;
#pragma unroll
  for (int i = 0; i < NG; ++i)
#pragma unroll
    for (int e = 0; e < V; ++e) sq = fmaf(x[i][e], x[i][e], sq);
  const float inv = 1.f / sqrtf(block_sum_warps<NT / 32>(sq, red[1]) / static_cast<float>(d) + p.eps);
  A* act = reinterpret_cast<A*>(p.act) + t * p.ld_act;
#pragma unroll
  for (int i = 0; i < NG; ++i) {
    const int c = (threadIdx.x + NT * i) * V;
    if (c >= p.ld_act) continue;
    float v[V];
#pragma unroll
    for (int e = 0; e < V; ++e) v[e] = inv * x[i][e] * wn[i][e];       // columns past d: zero
    st_vec<A, V>(act + c, v);
  }
}

template <typename Y, typename A, int V>
cudaError_t launch_sandwich(const SandwichArgs& p, int tokens, cudaStream_t s) {
  const long long groups = ((p.act != nullptr && p.ld_act > p.d ? p.ld_act : p.d) + V - 1) / V;
  if (groups <= 128) return zb_launch(zb_sandwich_norm_kernel<Y, A, 128, 1, V>, dim3(tokens), dim3(128), 0, s, p);
  if (groups <= 512) return zb_launch(zb_sandwich_norm_kernel<Y, A, 512, 1, V>, dim3(tokens), dim3(512), 0, s, p);
  if (groups <= 1024) return zb_launch(zb_sandwich_norm_kernel<Y, A, 512, 2, V>, dim3(tokens), dim3(512), 0, s, p);
  if (groups <= 4096) return zb_launch(zb_sandwich_norm_kernel<Y, A, 512, 8, V>, dim3(tokens), dim3(512), 0, s, p);
  return cudaErrorInvalidValue;
}
template <typename Y>
cudaError_t launch_sandwich(const SandwichArgs& p, int act_f32, int tokens, cudaStream_t s) {
  const bool vec = p.d % 4 == 0 && p.ld_act % 4 == 0 && p.ldy % 4 == 0 && (reinterpret_cast<uintptr_t>(p.y) & 15) == 0;
  if (act_f32) return vec ? launch_sandwich<Y, float, 4>(p, tokens, s) : launch_sandwich<Y, float, 1>(p, tokens, s);
  return vec ? launch_sandwich<Y, __nv_bfloat16, 4>(p, tokens, s) : launch_sandwich<Y, __nv_bfloat16, 1>(p, tokens, s);
}

// ------------------------------------------------------------------------------------------ residual sum and layer norm
struct AddNormArgs {
  const void* y;               // as SandwichArgs
  long long ldy;
  const int32_t* pair_pos;
  const float* pair_w;
  int k;
  const float* x;              // [T, d]
  float* x_out;                // [T, d] or null (may be x)
  const float* w;              // [d]: weight and bias of the norm; null: act is x_out itself
  const float* b;
  float eps;
  void* act;                   // [T, ld_act] or null: columns d .. ld_act are zero
  long long ld_act;
  int d;
};

// T > 0: one token per sequence, and the normed row goes on through the convolution `a` with a.taps <= T (its output is `act`).
template <typename Y, typename A, int NT, int NG, int V, int T>
__global__ void __launch_bounds__(NT) zb_add_norm_kernel(const AddNormArgs p, const ConvArgs a, const int32_t* __restrict__ seq_lens) {
  constexpr int kSlots = 32;                             // expert slots read through shared memory at a time
  constexpr int R = T > 1 ? T - 1 : 1;                   // rows of state the convolution can need
  __shared__ float red[2][NT / 32];
  __shared__ float sw[kSlots];
  __shared__ int spos[kSlots];
  zb_pdl_launch();
  const int d = p.d;
  float w[NG][V], b[NG][V], cw[NG][T > 0 ? T : 1][V];    // parameters: on their way before the input is there
#pragma unroll
  for (int i = 0; i < NG; ++i) {
    const int c = (threadIdx.x + NT * i) * V;
#pragma unroll
    for (int e = 0; e < V; ++e) w[i][e] = b[i][e] = 0.f;
    if (c < d && p.w != nullptr) {
      ld_vec<V>(w[i], p.w + c);
      ld_vec<V>(b[i], p.b + c);
    }
    if constexpr (T > 0) {
#pragma unroll
      for (int j = 0; j < T; ++j) {                      // the last taps of the window count
#pragma unroll
        for (int e = 0; e < V; ++e) cw[i][j][e] = 0.f;
        if (c < d && j >= T - a.taps) ld_vec<V>(cw[i][j], a.w + static_cast<size_t>(j - (T - a.taps)) * d + c);
      }
    }
  }
  zb_pdl_wait();
  const long long t = blockIdx.x;
  float x[NG][V], hist[NG][R][V];                        // hist[R - 1]: the newest past input
#pragma unroll
  for (int i = 0; i < NG; ++i) {
    const int c = (threadIdx.x + NT * i) * V;
#pragma unroll
    for (int e = 0; e < V; ++e) x[i][e] = 0.f;
    if (c < d) ld_vec<V>(x[i], p.x + t * d + c);
  }
  float* st0 = nullptr;
  const int rows = a.rows;
  if constexpr (T > 0) {
    const int slot = a.slots[t];
    const bool slot_ok = ZB_BC_OK(slot, ZB_BC_STATE_SLOTS, kKernelStreamConv, 3);
    if (slot_ok) st0 = a.state + static_cast<size_t>(slot) * rows * d;
    const bool fresh = !slot_ok || seq_lens[t] - 1 <= 0;
#pragma unroll
    for (int i = 0; i < NG; ++i) {
      const int c = (threadIdx.x + NT * i) * V;
#pragma unroll
      for (int j = 0; j < R; ++j) {
#pragma unroll
        for (int e = 0; e < V; ++e) hist[i][j][e] = 0.f;
        if (c < d && !fresh && j >= R - rows) ld_vec<V>(hist[i][j], st0 + static_cast<size_t>(j - (R - rows)) * d + c);
      }
    }
  }
  if (p.y != nullptr) {
    const Y* ys = reinterpret_cast<const Y*>(p.y);
    auto add = [&](long long row, float wt) {
#pragma unroll
      for (int i = 0; i < NG; ++i) {
        const int c = (threadIdx.x + NT * i) * V;
        if (c >= d) continue;
        float v[V];
        if constexpr (V == 4) ld_row4(v, ys + row * p.ldy + c);
        else v[0] = zb_ld_act(ys + row * p.ldy + c);
#pragma unroll
        for (int e = 0; e < V; ++e) x[i][e] = fmaf(wt, v[e], x[i][e]);
      }
    };
    if (p.pair_pos == nullptr) {
      add(t, 1.f);
    } else {
      for (int j0 = 0; j0 < p.k; j0 += kSlots) {
        const int n = min(kSlots, p.k - j0);
        __syncthreads();
        if (threadIdx.x < n) {
          spos[threadIdx.x] = p.pair_pos[t * p.k + j0 + threadIdx.x];
          sw[threadIdx.x] = p.pair_w[t * p.k + j0 + threadIdx.x];
        }
        __syncthreads();
#pragma unroll 4
        for (int j = 0; j < n; ++j)
          if (spos[j] >= 0) add(spos[j], sw[j]);
      }
    }
  }
  if (p.x_out != nullptr) {
#pragma unroll
    for (int i = 0; i < NG; ++i) {
      const int c = (threadIdx.x + NT * i) * V;
      if (c < d) st_vec<float, V>(p.x_out + t * d + c, x[i]);
    }
  }
  if (p.act == nullptr) return;
  if (p.w != nullptr) {
    float sum = 0.f, sq = 0.f;
#pragma unroll
    for (int i = 0; i < NG; ++i)
#pragma unroll
      for (int e = 0; e < V; ++e) sum += x[i][e];
    const float mean = block_sum_warps<NT / 32>(sum, red[0]) / static_cast<float>(d);
#pragma unroll
    for (int i = 0; i < NG; ++i) {
      if ((threadIdx.x + NT * i) * V >= d) continue;     // columns past d stay zero
#pragma unroll
      for (int e = 0; e < V; ++e) {
        x[i][e] -= mean;
        sq = fmaf(x[i][e], x[i][e], sq);
      }
    }
    const float inv = 1.f / sqrtf(block_sum_warps<NT / 32>(sq, red[1]) / static_cast<float>(d) + p.eps);
#pragma unroll
    for (int i = 0; i < NG; ++i)
#pragma unroll
      for (int e = 0; e < V; ++e) x[i][e] = fmaf(inv * x[i][e], w[i][e], b[i][e]);
  }
  A* act = reinterpret_cast<A*>(p.act) + t * p.ld_act;
#pragma unroll
  for (int i = 0; i < NG; ++i) {
    const int c = (threadIdx.x + NT * i) * V;
    if (c >= p.ld_act) continue;
    if constexpr (T > 0) {
      float h[V];
#pragma unroll
      for (int e = 0; e < V; ++e) {
        float acc = cw[i][T - 1][e] * x[i][e];
#pragma unroll
        for (int j = 0; j + 1 < T; ++j) acc = fmaf(cw[i][j][e], hist[i][j][e], acc);
        h[e] = x[i][e] + acc;
      }
      st_vec<A, V>(act + c, h);
      if (st0 == nullptr || c >= d) continue;
#pragma unroll
      for (int j = 0; j < R; ++j) {
        if (j < R - rows) continue;
        float* dst = st0 + static_cast<size_t>(j - (R - rows)) * d + c;
        if (j + 1 < R) st_vec<float, V>(dst, hist[i][j + 1 < R ? j + 1 : j]);
        else st_vec<float, V>(dst, x[i]);
      }
    } else {
      st_vec<A, V>(act + c, x[i]);
    }
  }
}

template <typename Y, typename A, int V, int T>
cudaError_t launch_add_norm(const AddNormArgs& p, const ConvArgs& a, const int32_t* seq_lens, int tokens, cudaStream_t s) {
  const long long groups = ((p.act != nullptr && p.ld_act > p.d ? p.ld_act : p.d) + V - 1) / V;
  if (groups <= 128) return zb_launch(zb_add_norm_kernel<Y, A, 128, 1, V, T>, dim3(tokens), dim3(128), 0, s, p, a, seq_lens);
  if (groups <= 512) return zb_launch(zb_add_norm_kernel<Y, A, 512, 1, V, T>, dim3(tokens), dim3(512), 0, s, p, a, seq_lens);
  if (groups <= 1024) return zb_launch(zb_add_norm_kernel<Y, A, 512, 2, V, T>, dim3(tokens), dim3(512), 0, s, p, a, seq_lens);
  if constexpr (T == 0)
    if (groups <= 4096) return zb_launch(zb_add_norm_kernel<Y, A, 512, 8, V, T>, dim3(tokens), dim3(512), 0, s, p, a, seq_lens);
  return cudaErrorInvalidValue;
}
template <typename Y, typename A, int V>
cudaError_t launch_add_norm(const AddNormArgs& p, const ConvArgs& a, const int32_t* seq_lens, int tokens, cudaStream_t s) {
  if (a.w == nullptr) return launch_add_norm<Y, A, V, 0>(p, a, seq_lens, tokens, s);
  if (a.taps <= 4) return launch_add_norm<Y, A, V, 4>(p, a, seq_lens, tokens, s);
  return launch_add_norm<Y, A, V, kMaxTaps>(p, a, seq_lens, tokens, s);
}
bool add_norm_vec(int d, long long ldy, const void* y) {
  return d % 4 == 0 && (y == nullptr || (ldy % 4 == 0 && (reinterpret_cast<uintptr_t>(y) & 15) == 0));
}
template <typename Y>
cudaError_t launch_add_norm(const AddNormArgs& p, const ConvArgs& a, const int32_t* seq_lens, int act_f32, int tokens, cudaStream_t s) {
  const bool vec = add_norm_vec(p.d, p.ldy, p.y) && (p.act == nullptr || p.ld_act % 4 == 0);
  if (act_f32) return vec ? launch_add_norm<Y, float, 4>(p, a, seq_lens, tokens, s) : launch_add_norm<Y, float, 1>(p, a, seq_lens, tokens, s);
  return vec ? launch_add_norm<Y, __nv_bfloat16, 4>(p, a, seq_lens, tokens, s) : launch_add_norm<Y, __nv_bfloat16, 1>(p, a, seq_lens, tokens, s);
}

// ------------------------------------------------------------------------------------------ hyper-connections
constexpr int kMaxStreams = 8;

struct HyperArgs {
  const void* y;               // sublayer output [T, ldy], or expert rows [*, ldy] with pair_pos, or null: nothing to add
  long long ldy;
  int y_f32;
  const int32_t* pair_pos;     // [T, k], as SandwichArgs
  const float* pair_w;
  int k;
  const float* x;              // [T, streams, d]
  int streams;
  const float* mix;            // [streams, streams]: from, to
  const float* out;            // [streams]
  const float* in;             // [streams] of what comes next, or null: no norm
  const float* w;              // [d]
  float eps;
  float* x_out;                // [T, streams, d] (may be x) or null
  void* act;                   // [T, ld_act]: columns d .. ld_act are zero
  long long ld_act;
  int act_f32;
  int d;
};

// S >= streams; NT threads, NG groups of V neighbouring channels per thread, all streams of a channel in one thread.
template <int S, int NT, int NG, int V>
__global__ void __launch_bounds__(NT) zb_hyper_norm_kernel(const HyperArgs p) {
  constexpr int kSlots = 32;                             // expert slots read through shared memory at a time
  __shared__ float red[NT / 32];
  __shared__ float sw[kSlots];
  __shared__ int spos[kSlots];
  __shared__ float s_mix[S][S], s_out[S], s_in[S];
  zb_pdl_launch();
  const int d = p.d, ns = p.streams;
  for (int i = threadIdx.x; i < S * S; i += NT) {        // coefficients of streams that do not exist are zero
    const int from = i / S, to = i % S;
    s_mix[from][to] = p.y != nullptr && from < ns && to < ns ? p.mix[from * ns + to] : 0.f;
    if (i < S) {
      s_out[i] = p.y != nullptr && i < ns ? p.out[i] : 0.f;
      s_in[i] = p.in != nullptr && i < ns ? p.in[i] : 0.f;
    }
  }
  float w[NG][V];
#pragma unroll
  for (int i = 0; i < NG; ++i) {
    const int c = (threadIdx.x + NT * i) * V;
#pragma unroll
    for (int e = 0; e < V; ++e) w[i][e] = 0.f;
    if (c < d && p.in != nullptr) ld_vec<V>(w[i], p.w + c);
  }
  __syncthreads();
  zb_pdl_wait();
  const long long t = blockIdx.x;
  float x[NG][S][V], y[NG][V];
#pragma unroll
  for (int i = 0; i < NG; ++i) {
    const int c = (threadIdx.x + NT * i) * V;
#pragma unroll
    for (int e = 0; e < V; ++e) y[i][e] = 0.f;
#pragma unroll
    for (int s = 0; s < S; ++s) {
#pragma unroll
      for (int e = 0; e < V; ++e) x[i][s][e] = 0.f;
      if (c < d && s < ns) ld_vec<V>(x[i][s], p.x + (t * ns + s) * d + c);
    }
  }
  if (p.y != nullptr) {
    auto add = [&](long long row, float wt) {
#pragma unroll
      for (int i = 0; i < NG; ++i) {
        const int c = (threadIdx.x + NT * i) * V;
        if (c >= d) continue;
        float v[V];
        if (p.y_f32) {
          ld_vec<V>(v, reinterpret_cast<const float*>(p.y) + row * p.ldy + c);
        } else {
          const __nv_bfloat16* src = reinterpret_cast<const __nv_bfloat16*>(p.y) + row * p.ldy + c;
          if constexpr (V == 4) ld_row4(v, src);
          else v[0] = zb_ld_act(src);
        }
#pragma unroll
        for (int e = 0; e < V; ++e) y[i][e] = fmaf(wt, v[e], y[i][e]);
      }
    };
    if (p.pair_pos == nullptr) {
      add(t, 1.f);
    } else {
      for (int j0 = 0; j0 < p.k; j0 += kSlots) {
        const int n = min(kSlots, p.k - j0);
        __syncthreads();
        if (threadIdx.x < n) {
          spos[threadIdx.x] = p.pair_pos[t * p.k + j0 + threadIdx.x];
          sw[threadIdx.x] = p.pair_w[t * p.k + j0 + threadIdx.x];
        }
        __syncthreads();
#pragma unroll 4
        for (int j = 0; j < n; ++j)
          if (spos[j] >= 0) add(spos[j], sw[j]);
      }
    }
#pragma unroll
    for (int i = 0; i < NG; ++i) {
      const int c = (threadIdx.x + NT * i) * V;
      float n[S][V];
#pragma unroll
      for (int to = 0; to < S; ++to) {
        const float o = s_out[to];
#pragma unroll
        for (int e = 0; e < V; ++e) n[to][e] = o * y[i][e];
#pragma unroll
        for (int from = 0; from < S; ++from) {
          const float f = s_mix[from][to];
#pragma unroll
          for (int e = 0; e < V; ++e) n[to][e] = fmaf(f, x[i][from][e], n[to][e]);
        }
      }
#pragma unroll
      for (int s = 0; s < S; ++s) {
#pragma unroll
        for (int e = 0; e < V; ++e) x[i][s][e] = n[s][e];
        if (p.x_out != nullptr && c < d && s < ns) st_vec<float, V>(p.x_out + (t * ns + s) * d + c, x[i][s]);
      }
    }
  }
  if (p.act == nullptr) return;
  float sq = 0.f;
#pragma unroll
  for (int i = 0; i < NG; ++i)
#pragma unroll
    for (int e = 0; e < V; ++e) {                        // the mix that the next sublayer reads, over y
      float u = 0.f;
#pragma unroll
      for (int s = 0; s < S; ++s) u = fmaf(s_in[s], x[i][s][e], u);
      y[i][e] = u;
      sq = fmaf(u, u, sq);
    }
  const float inv = 1.f / sqrtf(block_sum_warps<NT / 32>(sq, red) / static_cast<float>(d) + p.eps);
#pragma unroll
  for (int i = 0; i < NG; ++i) {
    const int c = (threadIdx.x + NT * i) * V;
    if (c >= p.ld_act) continue;
    float v[V];
#pragma unroll
    for (int e = 0; e < V; ++e) v[e] = inv * y[i][e] * w[i][e];        // columns past d: zero
    if (p.act_f32) st_vec<float, V>(reinterpret_cast<float*>(p.act) + t * p.ld_act + c, v);
    else st_vec<__nv_bfloat16, V>(reinterpret_cast<__nv_bfloat16*>(p.act) + t * p.ld_act + c, v);
  }
}

template <int S, int V>
cudaError_t launch_hyper(const HyperArgs& p, int tokens, cudaStream_t s) {
  const long long groups = ((p.act != nullptr && p.ld_act > p.d ? p.ld_act : p.d) + V - 1) / V;
  if (groups <= 128) return zb_launch(zb_hyper_norm_kernel<S, 128, 1, V>, dim3(tokens), dim3(128), 0, s, p);
  if (groups <= 512) return zb_launch(zb_hyper_norm_kernel<S, 512, 1, V>, dim3(tokens), dim3(512), 0, s, p);
  if (groups <= 1024) return zb_launch(zb_hyper_norm_kernel<S, 512, 2, V>, dim3(tokens), dim3(512), 0, s, p);
  if (groups <= 4096) return zb_launch(zb_hyper_norm_kernel<S, 512, 8, V>, dim3(tokens), dim3(512), 0, s, p);
  return cudaErrorInvalidValue;
}
template <int V>
cudaError_t launch_hyper(const HyperArgs& p, int tokens, cudaStream_t s) {
  if (p.streams <= 2) return launch_hyper<2, V>(p, tokens, s);
  if (p.streams <= 4) return launch_hyper<4, V>(p, tokens, s);
  return launch_hyper<kMaxStreams, V>(p, tokens, s);
}

template <typename A, int NG, bool MIX>
cudaError_t launch_post_norm_conv(const PostNormArgs& p, const ConvArgs& a, const ZbVarlen& b, int tokens, cudaStream_t s) {
  if (a.taps <= 4) return zb_launch(zb_post_norm_conv_kernel<A, NG, 4, MIX>, dim3(tokens), dim3(512), 0, s, p, a, b);
  return zb_launch(zb_post_norm_conv_kernel<A, NG, kMaxTaps, MIX>, dim3(tokens), dim3(512), 0, s, p, a, b);
}
template <typename A>
cudaError_t launch_post_norm_conv(const PostNormArgs& p, const ConvArgs& a, const ZbVarlen& b, int tokens, cudaStream_t s) {
  if (p.d <= 2048) return a.nmix > 0 ? launch_post_norm_conv<A, 1, true>(p, a, b, tokens, s) : launch_post_norm_conv<A, 1, false>(p, a, b, tokens, s);
  return a.nmix > 0 ? launch_post_norm_conv<A, 2, true>(p, a, b, tokens, s) : launch_post_norm_conv<A, 2, false>(p, a, b, tokens, s);
}

template <typename A, bool VEC>
int launch_post_norm(const PostNormArgs& p, const ConvArgs& a, const ZbVarlen& b, int tokens, cudaStream_t s) {
  const int per = (p.d + 255) / 256;
  cudaError_t e;
  if (per <= 4) e = zb_launch(zb_post_norm_kernel<A, 4, VEC>, dim3(tokens), dim3(256), 0, s, p, a, b);
  else if (per <= 8) e = zb_launch(zb_post_norm_kernel<A, 8, VEC>, dim3(tokens), dim3(256), 0, s, p, a, b);
  else if (per <= 16) e = zb_launch(zb_post_norm_kernel<A, 16, VEC>, dim3(tokens), dim3(256), 0, s, p, a, b);
  else if (per <= 32) e = zb_launch(zb_post_norm_kernel<A, 32, VEC>, dim3(tokens), dim3(256), 0, s, p, a, b);
  else if (per <= 64) e = zb_launch(zb_post_norm_kernel<A, 64, VEC>, dim3(tokens), dim3(256), 0, s, p, a, b);
  else return -70;
  zb_count_launch(1);
  return static_cast<int>(e != cudaSuccess ? e : cudaGetLastError());
}

ConvArgs conv_args(const float* w, float* state, const int32_t* slots, const float* mu, void* out, long long ld, long long plane,
                   int taps, int rows, int nmix, int d) {
  return ConvArgs{w, state, slots, mu, out, ld, plane, taps, rows, nmix, d};
}

bool conv_ok(int taps, int rows, int nmix) {
  return taps >= 1 && taps <= kMaxTaps && nmix >= 0 && nmix <= kMaxMix && rows == (nmix > 0 ? taps : taps - 1);
}
}  // namespace

extern "C" {

// out [tokens, copies, d].
int zb_embedding_f32(const int32_t* ids, const void* table, int table_f32, float* out, int tokens, int d, int vocab, float scale,
                     int copies, void* stream) {
  if (tokens <= 0) return 0;
  if (copies < 1) return -70;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const cudaError_t e =
      table_f32 ? zb_launch(zb_embedding_f32_kernel<float>, dim3(tokens), dim3(256), 0, s, ids, reinterpret_cast<const float*>(table), out, d, vocab, scale,
                            copies)
                : zb_launch(zb_embedding_f32_kernel<__nv_bfloat16>, dim3(tokens), dim3(256), 0, s, ids,
                            reinterpret_cast<const __nv_bfloat16*>(table), out, d, vocab, scale, copies);
  zb_count_launch(1);
  return static_cast<int>(e != cudaSuccess ? e : cudaGetLastError());
}

// h = x + conv(x) over a varlen batch; num_blocks >= sum over sequences of ceil(tokens / 32).
int zb_stream_conv(const float* x, const float* w, float* state, const int32_t* slots, const float* mu, void* out, int act_f32,
                   long long ld, long long plane, int taps, int rows, int nmix, int d, const int32_t* q_start,
                   const int32_t* seq_lens, int num_seqs, int num_blocks, void* stream) {
  if (num_seqs <= 0 || num_blocks <= 0) return 0;
  if (!conv_ok(taps, rows, nmix)) return -70;
  const ConvArgs a = conv_args(w, state, slots, mu, out, ld, plane, taps, rows, nmix, d);
  const ZbVarlen b = {q_start, seq_lens, num_seqs};
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const cudaError_t e = act_f32 ? launch_conv<float>(x, a, b, num_blocks, s) : launch_conv<__nv_bfloat16>(x, a, b, num_blocks, s);
  zb_count_launch(1);
  return static_cast<int>(e != cudaSuccess ? e : cudaGetLastError());
}

// x_out = layernorm(alpha * x + y) * w (row-wise); `conv_w` non-null: one token per sequence, and the row goes on
// through the convolution described by the remaining arguments (see zb_stream_conv).
int zb_post_norm(const void* y, long long ldy, int y_f32, const float* x, float alpha, const float* w, float eps, float* x_out,
                 void* act, long long ld_act, int act_f32, int tokens, int d, const float* conv_w, float* state,
                 const int32_t* slots, const float* mu, void* out, long long ld, long long plane, int taps, int rows, int nmix,
                 const int32_t* seq_lens, void* stream) {
  if (tokens <= 0) return 0;
  const PostNormArgs p = {y, ldy, y_f32, x, alpha, w, eps, x_out, act, ld_act, d, conv_w != nullptr ? 1 : 0};
  ConvArgs a = {};
  ZbVarlen b = {nullptr, seq_lens, tokens};
  if (conv_w != nullptr) {
    if (!conv_ok(taps, rows, nmix)) return -70;
    a = conv_args(conv_w, state, slots, mu, out, ld, plane, taps, rows, nmix, d);
  }
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const bool vec = d % 4 == 0 && (y == nullptr || ldy % 4 == 0) && (reinterpret_cast<uintptr_t>(y) & 15) == 0;
  if (conv_w != nullptr && vec && d <= 4096 && ld % 4 == 0 && plane % 4 == 0 && act == nullptr) {
    const cudaError_t e = act_f32 ? launch_post_norm_conv<float>(p, a, b, tokens, s) : launch_post_norm_conv<__nv_bfloat16>(p, a, b, tokens, s);
    zb_count_launch(1);
    return static_cast<int>(e != cudaSuccess ? e : cudaGetLastError());
  }
  if (act_f32) return vec ? launch_post_norm<float, true>(p, a, b, tokens, s) : launch_post_norm<float, false>(p, a, b, tokens, s);
  return vec ? launch_post_norm<__nv_bfloat16, true>(p, a, b, tokens, s) : launch_post_norm<__nv_bfloat16, false>(p, a, b, tokens, s);
}

// x_out = x + mult * rmsnorm(y) * w; act = rmsnorm(x_out) * w_next.  y null: act alone, of x.  pair_pos null: y [tokens, ldy];
// else y's rows are expert outputs and a token's value is sum_j pair_w[t, j] * y[pair_pos[t, j]].  d <= 4096 channels when
// it is not a multiple of 4, else 16384.
int zb_sandwich_norm(const void* y, long long ldy, int y_f32, const int32_t* pair_pos, const float* pair_w, int k, const float* x, float mult,
                     const float* w, const float* w_next, float eps, float* x_out, void* act, long long ld_act, int act_f32, int tokens,
                     int d, void* stream) {
  if (tokens <= 0) return 0;
  if (act != nullptr && (w_next == nullptr || ld_act < d)) return -70;
  const SandwichArgs p = {y, ldy, pair_pos, pair_w, k, x, mult, w, w_next, eps, x_out, act, ld_act, d};
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const cudaError_t e = y_f32 ? launch_sandwich<float>(p, act_f32, tokens, s) : launch_sandwich<__nv_bfloat16>(p, act_f32, tokens, s);
  zb_count_launch(1);
  return static_cast<int>(e != cudaSuccess ? e : cudaGetLastError());
}

// x [tokens, streams, d]: x_out[t] = sum_s mix[s, t] x[s] + out[t] * y, act = rmsnorm(sum_s in[s] x_out[s]) * w.  y as in
// zb_sandwich_norm; null: act alone, of x.  At most 8 streams; d as in zb_sandwich_norm.
int zb_hyper_norm(const void* y, long long ldy, int y_f32, const int32_t* pair_pos, const float* pair_w, int k, const float* x, int streams,
                  const float* mix, const float* out, const float* in, const float* w, float eps, float* x_out, void* act, long long ld_act,
                  int act_f32, int tokens, int d, void* stream) {
  if (tokens <= 0) return 0;
  if (streams < 1 || streams > kMaxStreams || (act != nullptr && (w == nullptr || in == nullptr || ld_act < d))) return -70;
  if (y != nullptr && (mix == nullptr || out == nullptr)) return -70;
  const HyperArgs p = {y, ldy, y_f32, pair_pos, pair_w, k, x, streams, mix, out, in, w, eps, x_out, act, ld_act, act_f32, d};
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const bool vec = d % 4 == 0 && (act == nullptr || ld_act % 4 == 0) && (y == nullptr || (ldy % 4 == 0 && (reinterpret_cast<uintptr_t>(y) & 15) == 0));
  const cudaError_t e = vec ? launch_hyper<4>(p, tokens, s) : launch_hyper<1>(p, tokens, s);
  zb_count_launch(1);
  return static_cast<int>(e != cudaSuccess ? e : cudaGetLastError());
}

// 1 when zb_add_norm takes a convolution for rows of d channels with these inputs: it holds a row in 512 threads.
int zb_add_norm_conv_supported(const void* y, long long ldy, int d, long long ld_act) {
  const int v = add_norm_vec(d, ldy, y) && ld_act % 4 == 0 ? 4 : 1;
  return (ld_act > d ? ld_act : d) <= 1024ll * v ? 1 : 0;
}

// x_out = x + y; act = layernorm(x_out) * w + b, or x_out itself without w.  y as in zb_sandwich_norm; null: nothing to add.
// `conv_w` non-null: one token per sequence, and act is what zb_stream_conv (without interpolations) makes of the normed rows.
// d as in zb_sandwich_norm.
int zb_add_norm(const void* y, long long ldy, int y_f32, const int32_t* pair_pos, const float* pair_w, int k, const float* x, float* x_out,
                const float* w, const float* b, float eps, void* act, long long ld_act, int act_f32, int tokens, int d, const float* conv_w,
                float* state, const int32_t* slots, int taps, const int32_t* seq_lens, void* stream) {
  if (tokens <= 0) return 0;
  if ((w == nullptr) != (b == nullptr) || (act != nullptr && ld_act < d)) return -70;
  const AddNormArgs p = {y, ldy, pair_pos, pair_w, k, x, x_out, w, b, eps, act, ld_act, d};
  ConvArgs a = {};
  if (conv_w != nullptr) {
    if (!conv_ok(taps, taps - 1, 0) || w == nullptr || act == nullptr || !zb_add_norm_conv_supported(y, ldy, d, ld_act)) return -70;
    a = conv_args(conv_w, state, slots, nullptr, act, ld_act, 0, taps, taps - 1, 0, d);
  }
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const cudaError_t e = y_f32 ? launch_add_norm<float>(p, a, seq_lens, act_f32, tokens, s)
                              : launch_add_norm<__nv_bfloat16>(p, a, seq_lens, act_f32, tokens, s);
  zb_count_launch(1);
  return static_cast<int>(e != cudaSuccess ? e : cudaGetLastError());
}

}  // extern "C"
