// WKV recurrence (the token mixing of RWKV models) over a varlen batch with the per-head state in registers:
//
//   o_t = (S_{t-1} + diag(u) k_t v_t^T)^T r_t,   S_t = diag(w_t) S_{t-1} + k_t v_t^T,   w_t = exp(-exp(z_t + w0))
//
// followed by out = o / rms(o) * norm * silu(gate) per head.  All of it is fp32; r, k, v and the gate come from
// projections (bf16 or fp32), z from a projection with fp32 output.
//
//   zb_wkv_scan_kernel    portions: the columns of S (value channels) are independent until the norm, so a CTA owns `CB`
//                         columns of one (sequence, head) and few long sequences still occupy all SMs; eight lanes share
//                         a column, and zb_wkv_finish_kernel normalises afterwards
//   zb_wkv_step_kernel    one token per sequence: one CTA per (sequence, head), four lanes per column, the whole state of
//                         the head requested before anything else; norm and gate in the same launch
// The state pool is [slots, H, value, key], so that the lanes of a column read and write it with consecutive 16-byte
// accesses.
#include "act.cuh"
#include "host_api.h"

namespace {
constexpr uint32_t kKernelWkv = 31;
constexpr int kKG = 8;                  // lanes per column

struct WkvArgs {
  const void* r;                        // [T, ld] each: H * dim columns
  const void* k;
  const void* v;
  const void* g;
  long long ld;
  const float* z;                       // [T, ldz]
  long long ldz;
  const float* w0;                      // [H * dim]
  const float* u;                       // [H * dim]
  const float* norm;                    // [H * dim]
  float eps;
  float* state;                         // [slots, H, dim, dim]
  const int32_t* slots;
  void* out;                            // [T, ld_out]
  long long ld_out;
  float* o;                             // [T, H * dim] fp32 when the norm runs in a launch of its own
  int heads, dim;
};

// Lane kg of the G lanes of a column holds key channels (i * G + kg) * 4 .. + 3 in S[4 i .. 4 i + 3].
template <int KT, int G>
ZB_DEVICE void load_state(float (&S)[KT], const float* st, int kg, int D, bool vec, bool valid) {
#pragma unroll
  for (int i = 0; i < KT / 4; ++i) {
    const int key = (i * G + kg) * 4;
    float4 f = make_float4(0.f, 0.f, 0.f, 0.f);
    if (valid) {
      if (vec) {
        if (key < D) f = *reinterpret_cast<const float4*>(st + key);
      } else {
        if (key < D) f.x = st[key];
        if (key + 1 < D) f.y = st[key + 1];
        if (key + 2 < D) f.z = st[key + 2];
        if (key + 3 < D) f.w = st[key + 3];
      }
    }
    S[4 * i] = f.x; S[4 * i + 1] = f.y; S[4 * i + 2] = f.z; S[4 * i + 3] = f.w;
  }
}
template <int KT, int G>
ZB_DEVICE void store_state(const float (&S)[KT], float* st, int kg, int D, bool vec) {
#pragma unroll
  for (int i = 0; i < KT / 4; ++i) {
    const int key = (i * G + kg) * 4;
    if (vec) {
      if (key < D) *reinterpret_cast<float4*>(st + key) = make_float4(S[4 * i], S[4 * i + 1], S[4 * i + 2], S[4 * i + 3]);
    } else {
      if (key < D) st[key] = S[4 * i];
      if (key + 1 < D) st[key + 1] = S[4 * i + 1];
      if (key + 2 < D) st[key + 2] = S[4 * i + 2];
      if (key + 3 < D) st[key + 3] = S[4 * i + 3];
    }
  }
}

// exp(-exp(x)): the fp32 path takes the accurate functions
template <typename A>
ZB_DEVICE float decay_of(float x) {
  if constexpr (sizeof(A) == 2) return __expf(-__expf(x));
  return expf(-expf(x));
}

// DP = 8 * KT padded key channels; CH tokens are staged in shared memory at a time, the next ones are requested into
// registers (as they are, so that nothing waits for them) before the current ones are worked on.
template <typename A, int KT, int CB, int CH>
__global__ void __launch_bounds__(CB * kKG) zb_wkv_scan_kernel(const WkvArgs p, const ZbVarlen b) {
  constexpr int DP = KT * kKG;
  constexpr int NT = CB * kKG;
  constexpr int NI = (CH * DP + NT - 1) / NT;      // staged (token, key) pairs per thread
  constexpr int NV = (CH * CB + NT - 1) / NT;
  constexpr int TB = 8;                             // tokens whose outputs are summed over the lanes together
  static_assert(CH % TB == 0, "");
  extern __shared__ __align__(16) float wkv_smem[];
  float* sr = wkv_smem;                             // [CH][DP]
  float* sk = sr + CH * DP;
  float* sw = sk + CH * DP;
  float* sv = sw + CH * DP;                         // [CH][CB]
  float* sy = sv + CH * CB;                         // [CH][CB]
  float* sru = sy + CH * CB;                        // [CH]: sum_k r u k
  float* su = sru + CH;                             // [DP]
  float* sw0 = su + DP;                             // [DP]
  zb_pdl_launch();
  zb_pdl_wait();
  const int h = blockIdx.x, s = blockIdx.y, c0 = blockIdx.z * CB;
  const int tid = threadIdx.x, kg = tid & (kKG - 1), col = tid / kKG;
  const int warp = tid >> 5, lane = tid & 31;
  const int D = p.dim;
  const int t0 = b.q_start[s], n = b.q_start[s + 1] - t0;
  if (n <= 0) return;
  const int slot = p.slots[s];
  if (!ZB_BC_OK(slot, ZB_BC_STATE_SLOTS, kKernelWkv, 1)) return;
  const bool fresh = b.seq_lens[s] - n <= 0;
  const bool mine = c0 + col < D;
  float* st = p.state + ((static_cast<long long>(slot) * p.heads + h) * D + c0 + col) * D;
  const bool vec = (D & 3) == 0;
  float S[KT];
  load_state<KT, kKG>(S, st, kg, D, vec, !fresh && mine);
  const long long hb = static_cast<long long>(h) * D;
  const A* gr = reinterpret_cast<const A*>(p.r) + t0 * p.ld + hb;
  const A* gk = reinterpret_cast<const A*>(p.k) + t0 * p.ld + hb;
  const A* gv = reinterpret_cast<const A*>(p.v) + t0 * p.ld + hb;
  const float* gz = p.z + t0 * p.ldz + hb;
  for (int i = tid; i < DP; i += NT) {
    su[i] = i < D ? p.u[hb + i] : 0.f;
    sw0[i] = i < D ? p.w0[hb + i] : 0.f;
  }

  A nr[NI], nk[NI], nv[NV];
  float nz[NI];
  auto fetch = [&](int base) {                      // past the end: some valid element, masked when it is staged
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int e = tid + i * NT, tt = min(base + e / DP, n - 1), kk = min(e % DP, D - 1);
      nr[i] = gr[tt * p.ld + kk];
      nk[i] = gk[tt * p.ld + kk];
      nz[i] = gz[tt * p.ldz + kk];
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int e = tid + i * NT, tt = min(base + e / CB, n - 1), cc = min(c0 + e % CB, D - 1);
      nv[i] = gv[tt * p.ld + cc];
    }
  };
  fetch(0);
  __syncthreads();
  for (int base = 0; base < n; base += CH) {
    const int cn = min(CH, n - base);
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int e = tid + i * NT, tt = e / DP, kk = e % DP;
      if (CH * DP % NT != 0 && e >= CH * DP) continue;
      const bool in = tt < cn && kk < D;            // a token past the end leaves the state as it is: r = k = 0, w = 1
      sr[e] = in ? zb_ld_act(&nr[i]) : 0.f;
      sk[e] = in ? zb_ld_act(&nk[i]) : 0.f;
      sw[e] = in ? decay_of<A>(nz[i] + sw0[kk]) : 1.f;
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int e = tid + i * NT;
      if (CH * CB % NT == 0 || e < CH * CB) sv[e] = zb_ld_act(&nv[i]);
    }
    __syncthreads();
    if (base + CH < n) fetch(base + CH);
    for (int tt = warp; tt < cn; tt += NT / 32) {
      float d = 0.f;
#pragma unroll
      for (int kk = lane; kk < DP; kk += 32) d = fmaf(sr[tt * DP + kk] * su[kk], sk[tt * DP + kk], d);
      d = zb_warp_sum(d);
      if (lane == 0) sru[tt] = d;
    }
    __syncthreads();
    for (int tb = 0; tb < cn; tb += TB) {
      float y[TB];
#pragma unroll
      for (int j = 0; j < TB; ++j) {
        const int tt = tb + j;
        const float v = sv[tt * CB + col];
        const float4* r4 = reinterpret_cast<const float4*>(sr + tt * DP);
        const float4* k4 = reinterpret_cast<const float4*>(sk + tt * DP);
        const float4* w4 = reinterpret_cast<const float4*>(sw + tt * DP);
        float y0 = 0.f, y1 = 0.f;
#pragma unroll
        for (int i = 0; i < KT / 4; ++i) {
          const float4 r = r4[i * kKG + kg], k = k4[i * kKG + kg], w = w4[i * kKG + kg];
          y0 = fmaf(S[4 * i], r.x, y0);
          y1 = fmaf(S[4 * i + 1], r.y, y1);
          y0 = fmaf(S[4 * i + 2], r.z, y0);
          y1 = fmaf(S[4 * i + 3], r.w, y1);
          S[4 * i] = fmaf(S[4 * i], w.x, k.x * v);
          S[4 * i + 1] = fmaf(S[4 * i + 1], w.y, k.y * v);
          S[4 * i + 2] = fmaf(S[4 * i + 2], w.z, k.z * v);
          S[4 * i + 3] = fmaf(S[4 * i + 3], w.w, k.w * v);
        }
        y[j] = y0 + y1;
      }
      // eight sums over eight lanes: halve the tokens a lane is responsible for at every exchange, so that lane kg ends
      // up with the sum of token tb + kg
      const bool up4 = kg & 4, up2 = kg & 2, up1 = kg & 1;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float give = up4 ? y[j] : y[j + 4], keep = up4 ? y[j + 4] : y[j];
        y[j] = keep + __shfl_xor_sync(0xffffffffu, give, 4);
      }
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const float give = up2 ? y[j] : y[j + 2], keep = up2 ? y[j + 2] : y[j];
        y[j] = keep + __shfl_xor_sync(0xffffffffu, give, 2);
      }
      const float give = up1 ? y[0] : y[1], keep = up1 ? y[1] : y[0];
      const float sum = keep + __shfl_xor_sync(0xffffffffu, give, 1);
      const int tt = tb + kg;
      if (tt < cn) sy[tt * CB + col] = fmaf(sv[tt * CB + col], sru[tt], sum);
    }
    __syncthreads();
    for (int e = tid; e < cn * CB; e += NT) {
      const int tt = e / CB, cc = e % CB;
      if (c0 + cc < D) p.o[(t0 + base + tt) * (static_cast<long long>(p.heads) * D) + hb + c0 + cc] = sy[e];
    }
    // no barrier here: the next pass writes sr / sk / sw / sv, whose last readers are behind the barrier above, and
    // sy is written again only after the next pass's barriers
  }
  if (mine) store_state<KT, kKG>(S, st, kg, D, vec);
}

// One token per sequence: four lanes per column.
constexpr int kSG = 4;

template <typename A, int KT>
__global__ void __launch_bounds__(KT * kSG * kSG) zb_wkv_step_kernel(const WkvArgs p, const ZbVarlen b) {
  constexpr int DP = KT * kSG;
  constexpr int NT = DP * kSG;
  __shared__ __align__(16) float sr[DP], sk[DP], sw[DP], sv[DP], sy[DP];
  __shared__ float red[2][NT / 32];
  zb_pdl_launch();
  zb_pdl_wait();
  const int h = blockIdx.x, s = blockIdx.y, tid = threadIdx.x, kg = tid & (kSG - 1), col = tid / kSG;
  const int D = p.dim;
  const int t = b.q_start[s];
  if (b.q_start[s + 1] <= t) return;
  const int slot = p.slots[s];
  if (!ZB_BC_OK(slot, ZB_BC_STATE_SLOTS, kKernelWkv, 2)) return;
  const bool fresh = b.seq_lens[s] - 1 <= 0;
  const bool mine = col < D, vec = (D & 3) == 0;
  float* st = p.state + ((static_cast<long long>(slot) * p.heads + h) * D + col) * D;
  float S[KT];
  load_state<KT, kSG>(S, st, kg, D, vec, !fresh && mine);
  const long long hb = static_cast<long long>(h) * D, in = t * p.ld + hb;
  float d = 0.f;
  if (tid < DP) {
    float r = 0.f, k = 0.f, v = 0.f, w = 0.f;
    if (tid < D) {
      r = zb_ld_act(reinterpret_cast<const A*>(p.r) + in + tid);
      k = zb_ld_act(reinterpret_cast<const A*>(p.k) + in + tid);
      v = zb_ld_act(reinterpret_cast<const A*>(p.v) + in + tid);
      w = decay_of<A>(p.z[t * p.ldz + hb + tid] + p.w0[hb + tid]);
      d = r * p.u[hb + tid] * k;
    }
    sr[tid] = r;
    sk[tid] = k;
    sv[tid] = v;
    sw[tid] = w;
  }
  d = zb_warp_sum(d);
  if ((tid & 31) == 0) red[0][tid >> 5] = d;
  __syncthreads();
  d = 0.f;
#pragma unroll
  for (int i = 0; i < NT / 32; ++i) d += red[0][i];
  const float v = sv[col];
  float y = 0.f;
#pragma unroll
  for (int i = 0; i < KT / 4; ++i) {
    const float4 r = reinterpret_cast<const float4*>(sr)[i * kSG + kg], k = reinterpret_cast<const float4*>(sk)[i * kSG + kg];
    const float4 w = reinterpret_cast<const float4*>(sw)[i * kSG + kg];
    y = fmaf(S[4 * i], r.x, y);
    y = fmaf(S[4 * i + 1], r.y, y);
    y = fmaf(S[4 * i + 2], r.z, y);
    y = fmaf(S[4 * i + 3], r.w, y);
    S[4 * i] = fmaf(S[4 * i], w.x, k.x * v);
    S[4 * i + 1] = fmaf(S[4 * i + 1], w.y, k.y * v);
    S[4 * i + 2] = fmaf(S[4 * i + 2], w.z, k.z * v);
    S[4 * i + 3] = fmaf(S[4 * i + 3], w.w, k.w * v);
  }
  if (mine) store_state<KT, kSG>(S, st, kg, D, vec);
  y += __shfl_xor_sync(0xffffffffu, y, 1);
  y += __shfl_xor_sync(0xffffffffu, y, 2);
  y = mine ? fmaf(v, d, y) : 0.f;
  if (kg == 0) sy[col] = y;
  float ss = zb_warp_sum(kg == 0 ? y * y : 0.f);
  if ((tid & 31) == 0) red[1][tid >> 5] = ss;
  __syncthreads();
  ss = 0.f;
#pragma unroll
  for (int i = 0; i < NT / 32; ++i) ss += red[1][i];
  const float inv = 1.f / sqrtf(ss / static_cast<float>(D) + p.eps);
  if (tid < D) {
    const float z = zb_ld_act(reinterpret_cast<const A*>(p.g) + in + tid);
    zb_st_act(reinterpret_cast<A*>(p.out) + t * p.ld_out + hb + tid, sy[tid] * inv * p.norm[hb + tid] * (z / (1.f + expf(-z))));
  }
}

// out = o / rms(o) * norm * silu(gate), one warp per (token, head).
template <typename A>
__global__ void __launch_bounds__(256) zb_wkv_finish_kernel(const WkvArgs p, long long rows) {
  zb_pdl_launch();
  zb_pdl_wait();
  const int lane = threadIdx.x & 31, D = p.dim;
  const long long row = blockIdx.x * 8ll + (threadIdx.x >> 5);
  if (row >= rows) return;
  const long long t = row / p.heads, hb = (row % p.heads) * D;
  const float* o = p.o + row * D;
  float ss = 0.f;
  for (int c = lane; c < D; c += 32) ss += o[c] * o[c];
  ss = zb_warp_sum(ss);
  const float inv = 1.f / sqrtf(ss / static_cast<float>(D) + p.eps);
  for (int c = lane; c < D; c += 32) {
    const float z = zb_ld_act(reinterpret_cast<const A*>(p.g) + t * p.ld + hb + c);
    zb_st_act(reinterpret_cast<A*>(p.out) + t * p.ld_out + hb + c, o[c] * inv * p.norm[hb + c] * (z / (1.f + expf(-z))));
  }
}

// out[t, n] = sum_r tanh(a[t, r]) * w[r, n], fp32 sums: the second half of a low-rank pre-activation for few tokens.
// One CTA: eight tokens, 64 outputs.
constexpr int kTlTokens = 8;

template <typename W>
__global__ void __launch_bounds__(64) zb_tanh_linear_kernel(const float* __restrict__ a, long long lda, const W* __restrict__ w, long long ldw,
                                                            float* __restrict__ out, long long ldo, int tokens, int n, int rank) {
  constexpr int kFirst = 64;
  zb_pdl_launch();
  const int c = blockIdx.x * 64 + threadIdx.x;
  W first[kFirst];                                        // the weights are parameters: on their way before the input is there
#pragma unroll
  for (int r = 0; r < kFirst; ++r) first[r] = w[min(r, rank - 1) * ldw + min(c, n - 1)];
  zb_pdl_wait();
  extern __shared__ __align__(16) float tl_smem[];        // [rank][kTlTokens]
  const int t0 = blockIdx.y * kTlTokens, nt = min(kTlTokens, tokens - t0);
  for (int i = threadIdx.x; i < rank * kTlTokens; i += 64) {
    const int t = i / rank, r = i - t * rank;
    tl_smem[r * kTlTokens + t] = t < nt ? tanhf(a[(t0 + t) * lda + r]) : 0.f;
  }
  __syncthreads();
  if (c >= n) return;
  float acc[kTlTokens] = {};
  auto add = [&](int r, float wv) {
    const float4 lo = *reinterpret_cast<const float4*>(tl_smem + r * kTlTokens), hi = *reinterpret_cast<const float4*>(tl_smem + r * kTlTokens + 4);
    acc[0] = fmaf(lo.x, wv, acc[0]);
    acc[1] = fmaf(lo.y, wv, acc[1]);
    acc[2] = fmaf(lo.z, wv, acc[2]);
    acc[3] = fmaf(lo.w, wv, acc[3]);
    acc[4] = fmaf(hi.x, wv, acc[4]);
    acc[5] = fmaf(hi.y, wv, acc[5]);
    acc[6] = fmaf(hi.z, wv, acc[6]);
    acc[7] = fmaf(hi.w, wv, acc[7]);
  };
#pragma unroll
  for (int r = 0; r < kFirst; ++r)
    if (r < rank) add(r, zb_ld_act(&first[r]));
#pragma unroll 8
  for (int r = kFirst; r < rank; ++r) add(r, zb_ld_act(w + r * ldw + c));
#pragma unroll
  for (int t = 0; t < kTlTokens; ++t)
    if (t < nt) out[(t0 + t) * ldo + c] = acc[t];
}

// tanh(a) as two bf16 pieces, [hi | lo] side by side: a bf16 product with the weights repeated twice along K then has
// 16 significant bits of the activation.  Columns rank .. half are zero.
__global__ void __launch_bounds__(256) zb_tanh_split_kernel(const float* __restrict__ a, long long lda, __nv_bfloat16* __restrict__ out, int half,
                                                            int rank, long long total) {
  zb_pdl_launch();
  zb_pdl_wait();
  for (long long idx = blockIdx.x * 256ll + threadIdx.x; idx < total; idx += gridDim.x * 256ll) {
    const long long t = idx / half;
    const int i = static_cast<int>(idx - t * half);
    const float v = i < rank ? tanhf(a[t * lda + i]) : 0.f;
    const __nv_bfloat16 hi = __float2bfloat16(v);
    out[t * 2 * half + i] = hi;
    out[t * 2 * half + half + i] = __float2bfloat16(v - __bfloat162float(hi));
  }
}

template <typename A, int KT, int CB, int CH>
int launch_scan(const WkvArgs& p, const ZbVarlen& b, cudaStream_t s) {
  constexpr int kSmem = (3 * CH * KT * kKG + 2 * CH * CB + CH + 2 * KT * kKG) * 4;
  static bool configured[16] = {};
  if (const int rc = zb_config_smem_once(zb_wkv_scan_kernel<A, KT, CB, CH>, kSmem, configured)) return rc;
  const cudaError_t e = zb_launch(zb_wkv_scan_kernel<A, KT, CB, CH>, dim3(p.heads, b.num_seqs, (p.dim + CB - 1) / CB), dim3(CB * kKG), kSmem, s, p, b);
  zb_count_launch(1);
  return static_cast<int>(e != cudaSuccess ? e : cudaGetLastError());
}

template <typename A, int KT>
int launch_step(const WkvArgs& p, const ZbVarlen& b, cudaStream_t s) {
  const cudaError_t e = zb_launch(zb_wkv_step_kernel<A, KT>, dim3(p.heads, b.num_seqs), dim3(KT * kSG * kSG), 0, s, p, b);
  zb_count_launch(1);
  return static_cast<int>(e != cudaSuccess ? e : cudaGetLastError());
}

template <typename A>
int scan(const WkvArgs& p, const ZbVarlen& b, cudaStream_t s) {
  const int D = p.dim;
  // wider CTAs stage less per column, narrower ones spread a few heads over more SMs
  const bool wide = D > 16 && static_cast<long long>(p.heads) * b.num_seqs * ((D + 31) / 32) >= 2 * 148;
  if (D <= 32) return wide ? launch_scan<A, 4, 32, 16>(p, b, s) : launch_scan<A, 4, 16, 16>(p, b, s);
  if (D <= 64) return wide ? launch_scan<A, 8, 32, 16>(p, b, s) : launch_scan<A, 8, 16, 16>(p, b, s);
  if (D <= 96) return wide ? launch_scan<A, 12, 32, 16>(p, b, s) : launch_scan<A, 12, 16, 16>(p, b, s);
  if (D <= 128) return wide ? launch_scan<A, 16, 32, 16>(p, b, s) : launch_scan<A, 16, 16, 16>(p, b, s);
  if (D <= 192) return launch_scan<A, 24, 16, 8>(p, b, s);
  if (D <= 256) return launch_scan<A, 32, 16, 8>(p, b, s);
  return -72;
}

template <typename A>
int step(const WkvArgs& p, const ZbVarlen& b, cudaStream_t s) {
  if (p.dim <= 32) return launch_step<A, 8>(p, b, s);
  if (p.dim <= 64) return launch_step<A, 16>(p, b, s);
  if (p.dim <= 96) return launch_step<A, 24>(p, b, s);
  if (p.dim <= 128) return launch_step<A, 32>(p, b, s);
  return -72;
}
}  // namespace

extern "C" {

// 1 when the one-token kernel takes this head size.
int zb_wkv_step_supported(int dim) { return dim <= 128 ? 1 : 0; }

// The recurrence over a varlen batch.  `o` null: one token per sequence (dim <= 128), norm and gate in the same launch;
// else o is scratch [T, H * dim] fp32 and a second launch finishes.  dim <= 256.
int zb_wkv_scan(const void* r, const void* k, const void* v, const void* g, long long ld, const float* z, long long ldz, const float* w0,
                const float* u, const float* norm, float eps, float* state, const int32_t* slots, void* out, long long ld_out, float* o,
                int act_f32, int heads, int dim, const int32_t* q_start, const int32_t* seq_lens, int num_seqs, int tokens, void* stream) {
  if (num_seqs <= 0 || tokens <= 0) return 0;
  const WkvArgs p = {r, k, v, g, ld, z, ldz, w0, u, norm, eps, state, slots, out, ld_out, o, heads, dim};
  const ZbVarlen b = {q_start, seq_lens, num_seqs};
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (o == nullptr) return tokens > num_seqs ? -73 : (act_f32 ? step<float>(p, b, s) : step<__nv_bfloat16>(p, b, s));
  const int rc = act_f32 ? scan<float>(p, b, s) : scan<__nv_bfloat16>(p, b, s);
  if (rc != 0) return rc;
  const long long rows = static_cast<long long>(tokens) * heads;
  const dim3 grid(static_cast<unsigned>((rows + 7) / 8));
  const cudaError_t e = act_f32 ? zb_launch(zb_wkv_finish_kernel<float>, grid, dim3(256), 0, s, p, rows)
                                : zb_launch(zb_wkv_finish_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, p, rows);
  zb_count_launch(1);
  return static_cast<int>(e != cudaSuccess ? e : cudaGetLastError());
}

int zb_tanh_linear(const float* a, long long lda, const void* w, long long ldw, int w_f32, float* out, long long ldo, int tokens, int n,
                   int rank, void* stream) {
  if (tokens <= 0 || n <= 0) return 0;
  const size_t smem = static_cast<size_t>(rank) * kTlTokens * sizeof(float);
  if (smem > 48 * 1024 || tokens > 65535 * kTlTokens) return -70;
  const dim3 grid((n + 63) / 64, (tokens + kTlTokens - 1) / kTlTokens);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const cudaError_t e =
      w_f32 ? zb_launch(zb_tanh_linear_kernel<float>, grid, dim3(64), smem, s, a, lda, reinterpret_cast<const float*>(w), ldw, out, ldo, tokens, n, rank)
            : zb_launch(zb_tanh_linear_kernel<__nv_bfloat16>, grid, dim3(64), smem, s, a, lda, reinterpret_cast<const __nv_bfloat16*>(w), ldw, out,
                        ldo, tokens, n, rank);
  zb_count_launch(1);
  return static_cast<int>(e != cudaSuccess ? e : cudaGetLastError());
}

int zb_tanh_split(const float* a, long long lda, void* out, int half, int rank, int tokens, void* stream) {
  if (tokens <= 0) return 0;
  const long long total = static_cast<long long>(tokens) * half;
  long long blocks = (total + 255) / 256;
  if (blocks > 148 * 8) blocks = 148 * 8;
  const cudaError_t e = zb_launch(zb_tanh_split_kernel, dim3(static_cast<unsigned>(blocks)), dim3(256), 0, reinterpret_cast<cudaStream_t>(stream), a,
                                  lda, reinterpret_cast<__nv_bfloat16*>(out), half, rank, total);
  zb_count_launch(1);
  return static_cast<int>(e != cudaSuccess ? e : cudaGetLastError());
}

}  // extern "C"
