// Gated delta rule with one decay per key channel, over a varlen batch with the per-head state in registers.  Per head, with
// decay g, unit keys k and queries q, write gate beta:
//
//   S <- diag(g) S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q;   out = o / rms(o) * norm * sigmoid(gate)
//
// q, k and v come from a projection through a short causal convolution and silu; everything behind that is fp32.
//
//   zb_delta_prep_kernel    portions: convolutions, unit norms and decays of blocks of eight tokens, and what lets the scan
//                           work on a block at once.  With P_t the product of the decays of the block's tokens up to t and
//                           R_t the product of those behind t, the block's updates are, on the state S in front of it,
//                             a_t = S^T (P_t k_t),  b_t = S^T (P_t q_t)
//                             u_t = beta_t (v_t - a_t - sum_{j<t} L_tj u_j),  o_t = b_t + sum_{j<=t} Q_tj u_j
//                             S <- diag(P_7) S + sum_t (R_t k_t) u_t^T
//                           with L_tj = k_t^T diag(decays of j+1..t) k_j and Q_tj the same with q_t.  All factors are products
//                           of decays, none a quotient, so nothing overflows however fast a channel forgets
//   zb_delta_scan_kernel    walks the blocks of a (sequence, head): a warp owns eight columns of S (value channels), bulk
//                           copies bring the blocks in through a ring of stages
//   zb_delta_finish_kernel  norm and gate, and the convolution inputs that later tokens need
//   zb_delta_step_kernel    one token per sequence: everything above in one launch, the whole state of the head requested
//                           before anything else
//
// State pools: S as [slots, H, value, key padded to 4] fp32; the convolution's inputs as a ring [slots, taps, channels] in
// which position p has row p % taps (a step reads the taps - 1 rows of earlier positions and writes the remaining one, so
// heads that share key channels do not disturb each other).
#include "act.cuh"
#include "host_api.h"

namespace {
constexpr uint32_t kKernelDelta = 36;
constexpr int kB = 8;                       // tokens per block
constexpr int kMaxTaps = 8;                 // at most kB: only a sequence's first block reaches back into the ring
constexpr int kColsPerCta = 32;
constexpr int kScanStages = 3;

struct DeltaArgs {
  const void* in;            // [T, ld_in]: q (G dk) | k (G dk) | v (H dv) at 0, write-gate logits (H) at beta_off
  long long ld_in;
  int beta_off;
  const float* low;          // [T, ld_low]: decay pre-activation (H dk) | output-gate logits (H dv)
  long long ld_low;
  const float* conv_w;       // [taps, 2 G dk + H dv], the last tap on the current token
  int taps;
  const float* a_log;        // [H]
  const float* dt_bias;      // [H dk]
  const float* norm;         // [dv]
  float eps;
  void* ring;                // [slots, taps, 2 G dk + H dv]
  float* state;              // [slots, H, dv, dk4]
  const int32_t* slots;
  float* blocks;             // scratch of the portion path: see BlockLayout
  float* o;                  // scratch [T, H dv]
  void* out;                 // [T, ld_out]
  long long ld_out;
  int H, G, dk, dv, dk4;
};

// One (block of tokens, head) as the scan reads it, in floats: key-side part, then the values in groups of kColsPerCta
// columns, [group][token][column].
struct BlockLayout {
  int DK, groups;            // padded key channels, groups of value columns
  __host__ __device__ int pk() const { return 0; }                       // P_t k_t   [8][DK]
  __host__ __device__ int pq() const { return kB * DK; }                 // P_t q_t   [8][DK]
  __host__ __device__ int rk() const { return 2 * kB * DK; }             // R_t k_t   [8][DK]
  __host__ __device__ int p7() const { return 3 * kB * DK; }             // P_7       [DK]
  __host__ __device__ int bl() const { return p7() + DK; }               // beta_t L  [8][8]
  __host__ __device__ int ql() const { return bl() + kB * kB; }          // Q         [8][8]
  __host__ __device__ int beta() const { return ql() + kB * kB; }        // beta      [8]
  __host__ __device__ int head() const { return beta() + kB; }           // floats of the key-side part
  __host__ __device__ int vals(int group) const { return head() + group * kB * kColsPerCta; }
  __host__ __device__ int total() const { return vals(groups); }
};

// A: the activation type.  fp32 models take CUDA's accurate functions; with bf16 inputs a few units in the last place of the
// fast ones do not count, except where a decay close to one acts over many tokens: there the exponential and the logarithm
// are short series (arguments below 2^-6, fourth order: 2^-26 relative).
template <typename A>
ZB_DEVICE float sigmoid(float z) {
  if constexpr (sizeof(A) == 2) return __fdividef(1.f, 1.f + __expf(-z));
  return 1.f / (1.f + expf(-z));
}
template <typename A>
ZB_DEVICE float silu(float z) {
  if constexpr (sizeof(A) == 2) return __fdividef(z, 1.f + __expf(-z));
  return z / (1.f + expf(-z));
}
// exp(-rate * softplus(z)), rate = exp(a_log).
template <typename A>
ZB_DEVICE float decay_of(float rate, float z) {
  if constexpr (sizeof(A) == 2) {
    const float e = __expf(z);
    const float sp = z > 20.f ? z : e < 0.015625f ? e * (1.f + e * (-0.5f + e * (1.f / 3.f - 0.25f * e))) : __logf(1.f + e);
    const float x = -rate * sp;
    return x > -0.015625f ? 1.f + x * (1.f + x * (0.5f + x * (1.f / 6.f + x * (1.f / 24.f)))) : __expf(x);
  }
  const float x = -rate * (z > 20.f ? z : log1pf(expf(z)));
  return x > -0.5f ? 1.f + expm1f(x) : expf(x);             // 1 + expm1 is correctly rounded near one, expf is not
}

// Sums N values over the G lanes of a group; lane kl of the group ends up with values kl * N / G .. in v[0 .. N / G - 1].
template <int N, int G>
ZB_DEVICE void reduce_scatter(float (&v)[N], int kl) {
  int n = N;
#pragma unroll
  for (int m = G / 2; m > 0; m >>= 1) {
    n >>= 1;
    const bool up = kl & m;
#pragma unroll
    for (int i = 0; i < N / 2; ++i) {
      if (i >= n) break;
      const float give = up ? v[i] : v[i + n], keep = up ? v[i + n] : v[i];
      v[i] = keep + __shfl_xor_sync(0xffffffffu, give, m);
    }
  }
}

// ------------------------------------------------------------------------------------------ portions: blocks
// One CTA per (block of tokens, head).  The head's query, key and value channels and its decays are dealt over the threads,
// one channel's eight tokens each; T bounds the taps, KI = DK / 32.
template <typename A, int KI, int T>
__global__ void __launch_bounds__(512, 2) zb_delta_prep_kernel(const DeltaArgs p, const BlockLayout bl, const ZbVarlen b) {
  constexpr int DK = KI * 32;
  __shared__ float sk[kB][DK], sq[kB][DK], sg[kB][DK];
  __shared__ float sinv[2 * kB], sbeta[kB];
  zb_pdl_launch();
  zb_pdl_wait();
  const int h = blockIdx.y, g = h / (p.H / p.G), tid = threadIdx.x, NT = blockDim.x, warps = NT / 32, warp = tid >> 5, lane = tid & 31;
  int s, blk;
  if (!zb_find_block_warp(b, kB, blockIdx.x, s, blk)) return;
  const int t0 = b.q_start[s], n = b.q_start[s + 1] - t0, i0 = blk * kB, cn = min(kB, n - i0);
  const int pos0 = b.seq_lens[s] - n;
  const int slot = p.slots[s];
  if (!ZB_BC_OK(slot, ZB_BC_STATE_SLOTS, kKernelDelta, 1)) return;
  const int C = 2 * p.G * p.dk + p.H * p.dv, vals = bl.groups * kColsPerCta;
  const A* in = reinterpret_cast<const A*>(p.in) + (t0 + i0) * p.ld_in;
  float* blob = p.blocks + (static_cast<long long>(blockIdx.x) * p.H + h) * bl.total();
  const float rate = expf(p.a_log[h]);
  if (tid < kB) {
    const float beta = tid < cn ? sigmoid<A>(zb_ld_act(in + tid * p.ld_in + p.beta_off + h)) : 0.f;
    sbeta[tid] = beta;
    blob[bl.beta() + tid] = beta;
  }
  for (int item = tid; item < 3 * DK + vals; item += NT) {
    if (item < DK) {                                         // decays; a token past the end leaves the state as it is
      float z[kB];
      const int c = min(item, p.dk - 1);
#pragma unroll
      for (int t = 0; t < kB; ++t) z[t] = p.low[(t0 + i0 + min(t, cn - 1)) * p.ld_low + h * p.dk + c];
      const float bias = p.dt_bias[h * p.dk + c];
#pragma unroll
      for (int t = 0; t < kB; ++t) sg[t][item] = t < cn && item < p.dk ? decay_of<A>(rate, z[t] + bias) : 1.f;
      continue;
    }
    const int part = item < 2 * DK ? 0 : item < 3 * DK ? 1 : 2;           // q, k, v
    const int c = item - (part + 1) * DK, width = part < 2 ? p.dk : p.dv;
    const bool live = c < width;
    const int col = (part < 2 ? (part * p.G + g) * p.dk : 2 * p.G * p.dk + h * p.dv) + min(c, width - 1);
    A x[T - 1 + kB];                                         // raw inputs; all requested at once
    if (i0 > 0) {
#pragma unroll
      for (int e = 0; e < T - 1; ++e) x[e] = in[(e - (T - 1)) * p.ld_in + col];
    } else {
      const A* ring = reinterpret_cast<const A*>(p.ring) + static_cast<long long>(slot) * p.taps * C + col;
#pragma unroll
      for (int e = 0; e < T - 1; ++e) x[e] = ring[static_cast<long long>(max(pos0 + e - (T - 1), 0) % p.taps) * C];
    }
#pragma unroll
    for (int t = 0; t < kB; ++t) x[T - 1 + t] = in[min(t, cn - 1) * p.ld_in + col];
    float w[T], y[kB];                                       // w[d]: the tap on the input d tokens back
#pragma unroll
    for (int d = 0; d < T; ++d) w[d] = d < p.taps ? p.conv_w[static_cast<long long>(p.taps - 1 - d) * C + col] : 0.f;
    float f[T - 1 + kB];
#pragma unroll
    for (int e = 0; e < T - 1 + kB; ++e) {
      const int back = T - 1 - e;                            // what lies before the start, or further back than the taps, counts nothing
      f[e] = back > 0 && (back >= p.taps || pos0 + i0 < back) ? 0.f : zb_ld_act(&x[e]);
    }
#pragma unroll
    for (int t = 0; t < kB; ++t) {
      float acc = 0.f;
#pragma unroll
      for (int d = 0; d < T; ++d) acc = fmaf(w[d], f[T - 1 + t - d], acc);
      y[t] = live && t < cn ? silu<A>(acc) : 0.f;
    }
    if (part < 2) {
#pragma unroll
      for (int t = 0; t < kB; ++t) (part == 0 ? sq : sk)[t][c] = y[t];
    } else {
      float* dst = blob + bl.vals(c / kColsPerCta) + c % kColsPerCta;
#pragma unroll
      for (int t = 0; t < kB; ++t) dst[t * kColsPerCta] = y[t];
    }
  }
  __syncthreads();
  for (int j = warp; j < 2 * kB; j += warps) {               // unit norms
    const float* v = j < kB ? sq[j] : sk[j - kB];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < KI; ++i) ss = fmaf(v[lane + 32 * i], v[lane + 32 * i], ss);
    ss = zb_warp_sum(ss);
    if (lane == 0) sinv[j] = (j < kB ? 1.f / sqrtf(static_cast<float>(p.dk)) : 1.f) / sqrtf(ss + 1e-6f);
  }
  __syncthreads();
  for (int item = tid; item < 3 * DK; item += NT) {
    const int part = item / DK, c = item % DK;
    float prod = 1.f;
    if (part < 2) {
      const float (*v)[DK] = part == 0 ? sk : sq;
      float* dst = blob + (part == 0 ? bl.pk() : bl.pq()) + c;
#pragma unroll
      for (int t = 0; t < kB; ++t) {
        prod *= sg[t][c];
        dst[t * DK] = prod * v[t][c] * sinv[part == 0 ? kB + t : t];
      }
      if (part == 0) blob[bl.p7() + c] = prod;
    } else {
#pragma unroll
      for (int t = kB - 1; t >= 0; --t) {
        blob[bl.rk() + t * DK + c] = prod * sk[t][c] * sinv[kB + t];
        prod *= sg[t][c];
      }
    }
  }
  // L and Q: a warp per column j of one of them
  for (int jj = warp; jj < 2 * kB; jj += warps) {
    const int j = jj % kB;
    const bool is_q = jj >= kB;
    const float (*other)[DK] = is_q ? sq : sk;
    float kp[KI], sum[kB];
#pragma unroll
    for (int i = 0; i < KI; ++i) kp[i] = sk[j][lane + 32 * i];
#pragma unroll
    for (int t = 0; t < kB; ++t) {
      sum[t] = 0.f;
      if (t < j) continue;
#pragma unroll
      for (int i = 0; i < KI; ++i) {
        const int c = lane + 32 * i;
        if (t > j) kp[i] *= sg[t][c];
        sum[t] = fmaf(kp[i], other[t][c], sum[t]);
      }
    }
    reduce_scatter<kB, 8>(sum, lane & 7);                    // lane l: token l % 8, over the eight lanes that share l / 8
    float v = sum[0];
    v += __shfl_xor_sync(0xffffffffu, v, 8);
    v += __shfl_xor_sync(0xffffffffu, v, 16);
    if (lane < kB) {
      const int t = lane;
      v *= sinv[kB + j] * sinv[is_q ? t : kB + t];
      if (is_q) blob[bl.ql() + t * kB + j] = t >= j ? v : 0.f;
      else blob[bl.bl() + t * kB + j] = t > j ? sbeta[t] * v : 0.f;
    }
  }
}

// ------------------------------------------------------------------------------------------ portions: scan
// N consecutive floats of shared memory that start on a multiple of N.
template <int N>
ZB_DEVICE void ld_floats(float (&v)[N], const float* p) {
  if constexpr (N % 4 == 0) {
#pragma unroll
    for (int i = 0; i < N; i += 4) {
      const float4 f = *reinterpret_cast<const float4*>(p + i);
      v[i] = f.x; v[i + 1] = f.y; v[i + 2] = f.z; v[i + 3] = f.w;
    }
  } else if constexpr (N == 2) {
    const float2 f = *reinterpret_cast<const float2*>(p);
    v[0] = f.x; v[1] = f.y;
  } else {
    v[0] = *p;
  }
}

constexpr int kScanColumns = 8;              // per warp
constexpr int kScanWarps = kColsPerCta / kScanColumns;

// G lanes share a column, each with KT key channels (float4 number i at channel (i G + lane) 4); C columns per lane; TB
// tokens are summed over the lanes at a time.
template <int G, int KT, int C, int TB>
__global__ void __launch_bounds__(32 * (kScanWarps + 1)) zb_delta_scan_kernel(const DeltaArgs p, const BlockLayout bl, const ZbVarlen b,
                                                                              ZbStatus* status) {
  constexpr int DK = G * KT;
  constexpr int CW = kScanColumns;
  constexpr int R = 32 / CW;                                 // lanes that solve for the same column
  static_assert(32 / G * C == CW && kB % TB == 0 && kB % R == 0, "");
  extern __shared__ __align__(128) float delta_smem[];
  __shared__ uint64_t full_bar[kScanStages], empty_bar[kScanStages];
  __shared__ uint32_t abort_word;
  __shared__ __align__(16) float sa[kScanWarps][kB][CW], sb[kScanWarps][kB][CW], su[kScanWarps][kB][CW];
  volatile uint32_t* abort_flag = &abort_word;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.x, s = blockIdx.y, group = blockIdx.z;
  const int stage_floats = bl.head() + kB * kColsPerCta;
  if (threadIdx.x == 0) {
    for (int i = 0; i < kScanStages; ++i) {
      zb_mbar_init(&full_bar[i], 1);
      zb_mbar_init(&empty_bar[i], kScanWarps);
    }
    abort_word = 0u;
    zb_mbar_fence_init();
  }
  __syncthreads();
  zb_pdl_launch();
  zb_pdl_wait();
  const int t0 = b.q_start[s], n = b.q_start[s + 1] - t0;
  const int slot = p.slots[s];
  if (n <= 0 || !ZB_BC_OK(slot, ZB_BC_STATE_SLOTS, kKernelDelta, 2)) return;          // uniform over the block
  const int first = zb_blocks_before(b, kB, s);
  const int nblk = (n + kB - 1) / kB;
  if (warp == kScanWarps) {
    if (lane == 0) {
      uint32_t stage = 0, phase = 0;
      const uint32_t head_bytes = bl.head() * 4, val_bytes = kB * kColsPerCta * 4;
      for (int i = 0; i < nblk; ++i) {
        if (!zb_mbar_wait(&empty_bar[stage], phase ^ 1u, abort_flag)) break;
        const float* src = p.blocks + (static_cast<long long>(first + i) * p.H + h) * bl.total();
        float* dst = delta_smem + stage * stage_floats;
        zb_mbar_expect_tx(&full_bar[stage], head_bytes + val_bytes);
        zb_bulk_load(dst, src, head_bytes, &full_bar[stage]);
        zb_bulk_load(dst + bl.head(), src + bl.vals(group), val_bytes, &full_bar[stage]);
        if (++stage == kScanStages) {
          stage = 0;
          phase ^= 1u;
        }
      }
    }
  } else {
    const int kl = lane % G, grp = lane / G, cw = lane % CW, r = lane / CW;
    const int col_w = group * kColsPerCta + warp * CW;              // the warp's first column
    const bool fresh = b.seq_lens[s] - n <= 0;
    float* st = p.state + ((static_cast<long long>(slot) * p.H + h) * p.dv + col_w + grp * C) * p.dk4;
    ZbF2 S[C][KT / 2];
#pragma unroll
    for (int c = 0; c < C; ++c)
#pragma unroll
      for (int i = 0; i < KT / 4; ++i) {
        const int key = (i * G + kl) * 4;
        float4 f = make_float4(0.f, 0.f, 0.f, 0.f);
        if (!fresh && key < p.dk4 && col_w + grp * C + c < p.dv) f = *reinterpret_cast<const float4*>(st + c * p.dk4 + key);
        S[c][2 * i] = zb_pack2(f.x, f.y);
        S[c][2 * i + 1] = zb_pack2(f.z, f.w);
      }
    uint32_t stage = 0, phase = 0;
    for (int blk = 0; blk < nblk; ++blk) {
      if (!__all_sync(0xffffffffu, zb_mbar_wait(&full_bar[stage], phase, abort_flag))) break;
      const float* d = delta_smem + stage * stage_floats;
      auto keys = [&](const float* row, ZbF2 (&v)[KT / 2]) {
#pragma unroll
        for (int i = 0; i < KT / 4; ++i) {
          const ulonglong2 x = *reinterpret_cast<const ulonglong2*>(row + (i * G + kl) * 4);
          v[2 * i] = x.x;
          v[2 * i + 1] = x.y;
        }
      };
#pragma unroll
      for (int tb = 0; tb < kB; tb += TB) {
        float part[2 * TB * C];
#pragma unroll
        for (int t = 0; t < TB; ++t)
#pragma unroll
          for (int ab = 0; ab < 2; ++ab) {
            ZbF2 v[KT / 2];
            keys(d + (ab == 0 ? bl.pk() : bl.pq()) + (tb + t) * DK, v);
#pragma unroll
            for (int c = 0; c < C; ++c) {
              ZbF2 acc = zb_mul2(v[0], S[c][0]);
#pragma unroll
              for (int i = 1; i < KT / 2; ++i) acc = zb_fma2(v[i], S[c][i], acc);
              part[(t * 2 + ab) * C + c] = zb_sum2(acc);
            }
          }
        reduce_scatter<2 * TB * C, G>(part, kl);
#pragma unroll
        for (int i = 0; i < 2 * TB * C / G; ++i) {
          const int idx = kl * (2 * TB * C / G) + i, c = idx % C, ab = idx / C % 2, t = idx / (2 * C);
          (ab == 0 ? sa : sb)[warp][tb + t][grp * C + c] = part[i];
        }
      }
      __syncwarp();
      // every lane solves for the block's u of column cw; the R lanes of a column then take every R-th output
      float u[kB], lo[kB][kB], beta[kB];
      const float* vals = d + bl.head() + warp * CW + cw;
      ld_floats<kB>(beta, d + bl.beta());
#pragma unroll
      for (int t = 0; t < kB; ++t) {
        if (t > 0) ld_floats<4>(reinterpret_cast<float (&)[4]>(lo[t][0]), d + bl.bl() + t * kB);
        if (t > 4) ld_floats<4>(reinterpret_cast<float (&)[4]>(lo[t][4]), d + bl.bl() + t * kB + 4);
        u[t] = beta[t] * (vals[t * kColsPerCta] - sa[warp][t][cw]);
      }
#pragma unroll
      for (int j = 0; j < kB; ++j) {
#pragma unroll
        for (int t = j + 1; t < kB; ++t) u[t] = fmaf(-lo[t][j], u[j], u[t]);
        if (j % R == r) su[warp][j][cw] = u[j];
      }
#pragma unroll
      for (int e = 0; e < kB / R; ++e) {
        const int t = r + R * e, i = blk * kB + t;
        float ql[kB], o = sb[warp][t][cw];
        ld_floats<kB>(ql, d + bl.ql() + t * kB);
#pragma unroll
        for (int j = 0; j < kB; ++j) o = fmaf(ql[j], u[j], o);
        if (i < n && col_w + cw < p.dv) p.o[static_cast<long long>(t0 + i) * p.H * p.dv + h * p.dv + col_w + cw] = o;
      }
      __syncwarp();
      ZbF2 v[KT / 2];
      keys(d + bl.p7(), v);
#pragma unroll
      for (int c = 0; c < C; ++c)
#pragma unroll
        for (int i = 0; i < KT / 2; ++i) S[c][i] = zb_mul2(S[c][i], v[i]);
#pragma unroll
      for (int t = 0; t < kB; ++t) {
        float uc[C];
        ld_floats<C>(uc, &su[warp][t][grp * C]);
        keys(d + bl.rk() + t * DK, v);
#pragma unroll
        for (int c = 0; c < C; ++c) {
          const ZbF2 uu = zb_pack2(uc[c], uc[c]);
#pragma unroll
          for (int i = 0; i < KT / 2; ++i) S[c][i] = zb_fma2(v[i], uu, S[c][i]);
        }
      }
      __syncwarp();
      if (lane == 0) zb_mbar_arrive(&empty_bar[stage]);
      if (++stage == kScanStages) {
        stage = 0;
        phase ^= 1u;
      }
    }
#pragma unroll
    for (int c = 0; c < C; ++c)
#pragma unroll
      for (int i = 0; i < KT / 4; ++i) {
        const int key = (i * G + kl) * 4;
        if (key < p.dk4 && col_w + grp * C + c < p.dv)
          *reinterpret_cast<ulonglong2*>(st + c * p.dk4 + key) = make_ulonglong2(S[c][2 * i], S[c][2 * i + 1]);
      }
  }
  __syncthreads();
  if (*abort_flag != 0u) {
    if (threadIdx.x == 0) zb_record_error(status, ZB_ERR_MBAR_TIMEOUT, kKernelDelta, 2u, blockIdx.x);
    const uint64_t w0 = zb_globaltimer();            // copies still in flight must land before the shared memory is reused
    while (zb_globaltimer() - w0 < 200000ull) {
    }
    __syncthreads();
  }
}

// out = o / rms(o) * norm * sigmoid(gate), one warp per (token, head); the last tokens of a sequence leave their convolution
// inputs in the ring.
template <typename A>
__global__ void __launch_bounds__(256) zb_delta_finish_kernel(const DeltaArgs p, const ZbVarlen b, long long rows) {
  zb_pdl_launch();
  zb_pdl_wait();
  const int lane = threadIdx.x & 31;
  const long long row = blockIdx.x * 8ll + (threadIdx.x >> 5);
  if (row >= rows) return;
  const int t = static_cast<int>(row / p.H), h = static_cast<int>(row % p.H);
  const float* o = p.o + row * p.dv;
  const float* gate = p.low + t * p.ld_low + p.H * p.dk + h * p.dv;
  A* out = reinterpret_cast<A*>(p.out) + t * p.ld_out + h * p.dv;
  float ss = 0.f;
  constexpr int kHeld = 4;                                   // values per lane that stay in registers
  float ov[kHeld], gv[kHeld];
#pragma unroll
  for (int i = 0; i < kHeld; ++i) {
    const int c = lane + 32 * i;
    ov[i] = c < p.dv ? o[c] : 0.f;
    gv[i] = c < p.dv ? gate[c] : 0.f;
    ss = fmaf(ov[i], ov[i], ss);
  }
  for (int c = lane + 32 * kHeld; c < p.dv; c += 32) ss = fmaf(o[c], o[c], ss);
  const float inv = 1.f / sqrtf(zb_warp_sum(ss) / static_cast<float>(p.dv) + p.eps);
#pragma unroll
  for (int i = 0; i < kHeld; ++i) {
    const int c = lane + 32 * i;
    if (c < p.dv) zb_st_act(out + c, ov[i] * inv * p.norm[c] * sigmoid<A>(gv[i]));
  }
  for (int c = lane + 32 * kHeld; c < p.dv; c += 32) zb_st_act(out + c, o[c] * inv * p.norm[c] * sigmoid<A>(gate[c]));
  const int s = zb_sequence_of(b, t);
  const int n = b.q_start[s + 1] - b.q_start[s], left = b.q_start[s + 1] - t;      // left: tokens from here to the portion's end
  if (left > p.taps || left <= 0) return;
  const int slot = p.slots[s], pos = b.seq_lens[s] - left;
  if (!ZB_BC_OK(slot, ZB_BC_STATE_SLOTS, kKernelDelta, 3) || n <= 0) return;
  const int C = 2 * p.G * p.dk + p.H * p.dv, rep = p.H / p.G, g = h / rep;
  const A* in = reinterpret_cast<const A*>(p.in) + t * p.ld_in;
  A* ring = reinterpret_cast<A*>(p.ring) + (static_cast<long long>(slot) * p.taps + pos % p.taps) * C;
  for (int c = lane; c < p.dv; c += 32) ring[2 * p.G * p.dk + h * p.dv + c] = in[2 * p.G * p.dk + h * p.dv + c];
  if (h % rep == 0)
    for (int c = lane; c < p.dk; c += 32) {
      ring[g * p.dk + c] = in[g * p.dk + c];
      ring[(p.G + g) * p.dk + c] = in[(p.G + g) * p.dk + c];
    }
}

// ------------------------------------------------------------------------------------------ one token
// SG lanes share a column, KT key channels each; the columns of a head in passes of NT / SG.  The head's query, key and value
// channels and its decays are dealt over the threads, a channel each; T bounds the taps.
template <typename A, int KT, int SG, int T>
__global__ void __launch_bounds__(512, 2) zb_delta_step_kernel(const DeltaArgs p, const ZbVarlen b) {
  constexpr int DP = KT * SG;
  __shared__ __align__(16) float s_q[DP], s_k[DP], s_g[DP], s_gk[DP];
  extern __shared__ float sy[];                              // [dv] values, then outputs
  __shared__ float red[4][16];
  zb_pdl_launch();
  const int h = blockIdx.x, s = blockIdx.y, tid = threadIdx.x, NT = blockDim.x, warps = NT / 32;
  const int kg = tid % SG, rep = p.H / p.G, g = h / rep;
  const int C = 2 * p.G * p.dk + p.H * p.dv, items = 3 * p.dk + p.dv;
  // item: the head's query | key | value channels, then its decays; the first one's parameters do not wait for the input
  auto column = [&](int item) {
    return item < p.dk ? g * p.dk + item : item < 2 * p.dk ? p.G * p.dk + g * p.dk + item - p.dk : 2 * p.G * p.dk + h * p.dv + item - 2 * p.dk;
  };
  float w[T];                                                // w[d]: the tap on the input d tokens back
  auto parameters = [&](int item) {
    const bool decay = item >= 2 * p.dk + p.dv;
    const int col = decay ? 0 : column(item);
#pragma unroll
    for (int d = 0; d < T; ++d) w[d] = !decay && d < p.taps ? p.conv_w[static_cast<long long>(p.taps - 1 - d) * C + col] : 0.f;
    if (decay) w[0] = p.dt_bias[h * p.dk + item - 2 * p.dk - p.dv];
  };
  if (tid < items) parameters(tid);
  const float rate = expf(p.a_log[h]);
  zb_pdl_wait();
  const int t = b.q_start[s];
  if (b.q_start[s + 1] <= t) return;
  const int slot = p.slots[s];
  if (!ZB_BC_OK(slot, ZB_BC_STATE_SLOTS, kKernelDelta, 4)) return;
  const int pos = max(0, b.seq_lens[s] - 1), row = pos % p.taps;
  float* st0 = p.state + (static_cast<long long>(slot) * p.H + h) * p.dv * p.dk4;
  ZbF2 S[KT / 2];
  auto load = [&](int col) {
#pragma unroll
    for (int i = 0; i < KT / 4; ++i) {
      const int key = (i * SG + kg) * 4;
      ulonglong2 f = make_ulonglong2(0ull, 0ull);
      if (pos > 0 && key < p.dk4 && col < p.dv) f = *reinterpret_cast<const ulonglong2*>(st0 + static_cast<long long>(col) * p.dk4 + key);
      S[2 * i] = f.x;
      S[2 * i + 1] = f.y;
    }
  };
  load(tid / SG);
  const A* in = reinterpret_cast<const A*>(p.in) + t * p.ld_in;
  A* ring = reinterpret_cast<A*>(p.ring) + static_cast<long long>(slot) * p.taps * C;
  const float beta_logit = zb_ld_act(in + p.beta_off + h);
  for (int item = tid; item < items; item += NT) {
    if (item >= NT) parameters(item);
    if (item >= 2 * p.dk + p.dv) {
      const int c = item - 2 * p.dk - p.dv;
      s_g[c] = decay_of<A>(rate, p.low[t * p.ld_low + h * p.dk + c] + w[0]);
      continue;
    }
    const int col = column(item);
    A x[T];
    x[0] = in[col];
#pragma unroll
    for (int d = 1; d < T; ++d) {                            // all requested at once; what lies before the start counts nothing
      const int r = row - d < 0 ? row - d + p.taps : row - d;
      x[d] = ring[static_cast<long long>(d < p.taps ? r : row) * C + col];
    }
    float acc = w[0] * zb_ld_act(&x[0]);
#pragma unroll
    for (int d = 1; d < T; ++d) acc = d < p.taps && d <= pos ? fmaf(w[d], zb_ld_act(&x[d]), acc) : acc;
    if (item >= 2 * p.dk || h % rep == 0) ring[static_cast<long long>(row) * C + col] = x[0];
    const float y = silu<A>(acc);
    if (item < p.dk) s_q[item] = y;
    else if (item < 2 * p.dk) s_k[item - p.dk] = y;
    else sy[item - 2 * p.dk] = y;
  }
  for (int c = p.dk + tid; c < DP; c += NT) {
    s_q[c] = s_k[c] = 0.f;
    s_g[c] = 1.f;
  }
  __syncthreads();
  float qq = 0.f, kk = 0.f, qk = 0.f;
  for (int c = tid; c < DP; c += NT) {
    const float q = s_q[c], k = s_k[c];
    qq = fmaf(q, q, qq);
    kk = fmaf(k, k, kk);
    qk = fmaf(q, k, qk);
  }
  qq = zb_warp_sum(qq);
  kk = zb_warp_sum(kk);
  qk = zb_warp_sum(qk);
  if ((tid & 31) == 0) {
    red[0][tid >> 5] = qq;
    red[1][tid >> 5] = kk;
    red[2][tid >> 5] = qk;
  }
  __syncthreads();
  const float beta = sigmoid<A>(beta_logit);
  qq = kk = qk = 0.f;
  for (int i = 0; i < min(warps, (DP + 31) / 32); ++i) {     // warps past the channels have nothing to add
    qq += red[0][i];
    kk += red[1][i];
    qk += red[2][i];
  }
  const float qi = 1.f / (sqrtf(qq + 1e-6f) * sqrtf(static_cast<float>(p.dk))), ki = 1.f / sqrtf(kk + 1e-6f);
  qk *= qi * ki;
  for (int c = tid; c < DP; c += NT) {
    const float k = s_k[c] * ki, dec = s_g[c];
    s_k[c] = k;
    s_gk[c] = dec * k;
    s_q[c] *= dec * qi;
  }
  __syncthreads();
  float ss = 0.f;
  for (int c0 = 0; c0 < p.dv; c0 += NT / SG) {
    const int col = c0 + tid / SG;
    if (c0 > 0) load(col);
    const float v = col < p.dv ? sy[col] : 0.f;
    ZbF2 a2 = 0ull, b2 = 0ull;
#pragma unroll
    for (int i = 0; i < KT / 4; ++i) {
      const ulonglong2 x = *reinterpret_cast<const ulonglong2*>(s_gk + (i * SG + kg) * 4), y = *reinterpret_cast<const ulonglong2*>(s_q + (i * SG + kg) * 4);
      a2 = zb_fma2(S[2 * i], x.x, a2);
      b2 = zb_fma2(S[2 * i], y.x, b2);
      a2 = zb_fma2(S[2 * i + 1], x.y, a2);
      b2 = zb_fma2(S[2 * i + 1], y.y, b2);
    }
    float a = zb_sum2(a2), o = zb_sum2(b2);
#pragma unroll
    for (int m = 1; m < SG; m <<= 1) {
      a += __shfl_xor_sync(0xffffffffu, a, m);
      o += __shfl_xor_sync(0xffffffffu, o, m);
    }
    const float u = beta * (v - a);
    o = fmaf(qk, u, o);
    const ZbF2 uu = zb_pack2(u, u);
    if (col < p.dv) {
#pragma unroll
      for (int i = 0; i < KT / 4; ++i) {
        const int key = (i * SG + kg) * 4;
        const ulonglong2 gg = *reinterpret_cast<const ulonglong2*>(s_g + key), k = *reinterpret_cast<const ulonglong2*>(s_k + key);
        S[2 * i] = zb_fma2(S[2 * i], gg.x, zb_mul2(k.x, uu));
        S[2 * i + 1] = zb_fma2(S[2 * i + 1], gg.y, zb_mul2(k.y, uu));
        if (key < p.dk4) *reinterpret_cast<ulonglong2*>(st0 + static_cast<long long>(col) * p.dk4 + key) = make_ulonglong2(S[2 * i], S[2 * i + 1]);
      }
      if (kg == 0) {
        sy[col] = o;                                         // this thread and its SG - 1 neighbours alone have read it
        ss = fmaf(o, o, ss);
      }
    }
  }
  ss = zb_warp_sum(ss);
  if ((tid & 31) == 0) red[3][tid >> 5] = ss;
  __syncthreads();
  ss = 0.f;
  for (int i = 0; i < warps; ++i) ss += red[3][i];
  const float inv = 1.f / sqrtf(ss / static_cast<float>(p.dv) + p.eps);
  const float* gate = p.low + t * p.ld_low + p.H * p.dk + h * p.dv;
  A* out = reinterpret_cast<A*>(p.out) + t * p.ld_out + h * p.dv;
  for (int c = tid; c < p.dv; c += NT) zb_st_act(out + c, sy[c] * inv * p.norm[c] * sigmoid<A>(gate[c]));
}

// ------------------------------------------------------------------------------------------ launches
template <typename A, int KI>
cudaError_t launch_prep(const DeltaArgs& p, const BlockLayout& bl, const ZbVarlen& b, int num_blocks, cudaStream_t s) {
  int threads = (3 * bl.DK + bl.groups * kColsPerCta + 127) / 128 * 128;
  if (threads > 512) threads = 512;
  const dim3 grid(num_blocks, p.H);
  if (p.taps <= 4) return zb_launch(zb_delta_prep_kernel<A, KI, 4>, grid, dim3(threads), 0, s, p, bl, b);
  return zb_launch(zb_delta_prep_kernel<A, KI, kMaxTaps>, grid, dim3(threads), 0, s, p, bl, b);
}
template <typename A>
cudaError_t launch_prep(const DeltaArgs& p, const BlockLayout& bl, const ZbVarlen& b, int num_blocks, cudaStream_t s) {
  if (bl.DK == 32) return launch_prep<A, 1>(p, bl, b, num_blocks, s);
  if (bl.DK == 64) return launch_prep<A, 2>(p, bl, b, num_blocks, s);
  if (bl.DK == 128) return launch_prep<A, 4>(p, bl, b, num_blocks, s);
  return launch_prep<A, 8>(p, bl, b, num_blocks, s);
}
template <int G, int KT, int C, int TB>
int launch_scan(const DeltaArgs& p, const BlockLayout& bl, const ZbVarlen& b, ZbStatus* status, cudaStream_t s) {
  const int smem = kScanStages * (bl.head() + kB * kColsPerCta) * 4;
  static bool configured[16] = {};
  if (const int rc = zb_config_smem_once(zb_delta_scan_kernel<G, KT, C, TB>, smem, configured)) return rc;
  const cudaError_t e = zb_launch(zb_delta_scan_kernel<G, KT, C, TB>, dim3(p.H, b.num_seqs, bl.groups), dim3(32 * (kScanWarps + 1)), smem, s, p, bl, b, status);
  return static_cast<int>(e);
}
int launch_scan(const DeltaArgs& p, const BlockLayout& bl, const ZbVarlen& b, ZbStatus* status, cudaStream_t s) {
  if (bl.DK == 32) return launch_scan<8, 4, 2, 8>(p, bl, b, status, s);
  if (bl.DK == 64) return launch_scan<16, 4, 4, 8>(p, bl, b, status, s);
  if (bl.DK == 128) return launch_scan<16, 8, 4, 8>(p, bl, b, status, s);
  return launch_scan<32, 8, 8, 4>(p, bl, b, status, s);
}
template <typename A, int KT, int SG>
cudaError_t launch_step(const DeltaArgs& p, const ZbVarlen& b, cudaStream_t s) {
  int threads = (p.dv * SG + 31) / 32 * 32;
  if (threads > 512) threads = 512;
  const dim3 grid(p.H, b.num_seqs);
  if (p.taps <= 4) return zb_launch(zb_delta_step_kernel<A, KT, SG, 4>, grid, dim3(threads), p.dv * sizeof(float), s, p, b);
  return zb_launch(zb_delta_step_kernel<A, KT, SG, kMaxTaps>, grid, dim3(threads), p.dv * sizeof(float), s, p, b);
}
template <typename A>
cudaError_t launch_step(const DeltaArgs& p, const ZbVarlen& b, cudaStream_t s) {
  if (p.dk <= 32) return launch_step<A, 8, 4>(p, b, s);
  if (p.dk <= 64) return launch_step<A, 16, 4>(p, b, s);
  if (p.dk <= 128) return launch_step<A, 32, 4>(p, b, s);
  return launch_step<A, 32, 8>(p, b, s);
}
BlockLayout layout_of(int dk, int dv) {
  return BlockLayout{dk <= 32 ? 32 : dk <= 64 ? 64 : dk <= 128 ? 128 : 256, (dv + kColsPerCta - 1) / kColsPerCta};
}
}  // namespace

extern "C" {

// Floats of the portion path's block scratch per (block of eight tokens, head).
int zb_channel_delta_block_floats(int dk, int dv) { return layout_of(dk, dv).total(); }

// The mixer behind its input projections over a varlen batch; see the top of the file.  `blocks` null: one token per
// sequence; else scratch for num_blocks >= sum of ceil(tokens / 8) blocks x H heads, and `o` scratch [tokens, H dv].
// dk <= 256, dv <= 4096, taps <= 8.
int zb_channel_delta(const void* in, long long ld_in, int beta_off, const float* low, long long ld_low, const float* conv_w, int taps,
                     const float* a_log, const float* dt_bias, const float* norm, float eps, void* ring, float* state, const int32_t* slots,
                     float* blocks, float* o, void* out, long long ld_out, int H, int G, int dk, int dv, int act_f32, const int32_t* q_start,
                     const int32_t* seq_lens, int num_seqs, int tokens, int num_blocks, void* stream) {
  if (num_seqs <= 0 || tokens <= 0) return 0;
  if (G <= 0 || H % G != 0 || taps < 1 || taps > kMaxTaps) return -71;
  if (dk > 256 || dv > 4096) return -72;
  const DeltaArgs p = {in, ld_in, beta_off, low, ld_low, conv_w, taps, a_log, dt_bias, norm, eps, ring, state, slots, blocks, o, out, ld_out,
                       H, G, dk, dv, (dk + 3) / 4 * 4};
  const ZbVarlen b = {q_start, seq_lens, num_seqs};
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (blocks == nullptr) {
    if (tokens > num_seqs) return -73;
    const cudaError_t e = act_f32 ? launch_step<float>(p, b, s) : launch_step<__nv_bfloat16>(p, b, s);
    zb_count_launch(1);
    return static_cast<int>(e != cudaSuccess ? e : cudaGetLastError());
  }
  ZbDeviceState* st = zb_device_state();
  if (!st) return -20;
  const BlockLayout bl = layout_of(dk, dv);
  cudaError_t e = act_f32 ? launch_prep<float>(p, bl, b, num_blocks, s) : launch_prep<__nv_bfloat16>(p, bl, b, num_blocks, s);
  if (e != cudaSuccess) return static_cast<int>(e);
  if (const int rc = launch_scan(p, bl, b, st->status, s)) return rc;
  const long long rows = static_cast<long long>(tokens) * H;
  const dim3 grid(static_cast<unsigned>((rows + 7) / 8));
  e = act_f32 ? zb_launch(zb_delta_finish_kernel<float>, grid, dim3(256), 0, s, p, b, rows)
              : zb_launch(zb_delta_finish_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, p, b, rows);
  zb_count_launch(3);
  return static_cast<int>(e != cudaSuccess ? e : cudaGetLastError());
}

}  // extern "C"
