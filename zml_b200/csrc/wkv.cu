// WKV recurrence (RWKV-style time mixing) over a varlen batch with the per-head state in registers:
//
//   o_t = (S_{t-1} + diag(u) k_t v_t^T)^T r_t,   S_t = diag(w_t) S_{t-1} + k_t v_t^T,   w_t = exp(-exp(z_t + w0))
//
// followed by out = o / rms(o) * norm * silu(gate) per head.  All of it is fp32; r, k, v and the gate come from
// projections (bf16 or fp32), z from a projection with fp32 output.
//
// The columns of S (value channels) are independent until the norm, so a CTA owns `CB` columns of one (sequence, head):
// eight lanes share a column, each holding every eighth group of four key channels.  With CB = the whole head the norm
// and the gate run in the same launch (decode, or enough heads to fill the GPU); with CB = 16 a few long sequences
// still occupy all SMs, and zb_wkv_finish normalises afterwards.  The state pool is [slots, H, value, key], so that the
// eight lanes of a column read and write it with consecutive 16-byte accesses.
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

// DP = 8 * KT padded key channels; CH tokens are staged in shared memory at a time, the next ones prefetched into
// registers meanwhile.  FUSED: CB covers the head, norm + gate in this launch.
template <typename A, int KT, int CB, int CH, bool FUSED>
__global__ void __launch_bounds__(CB * kKG) zb_wkv_scan_kernel(const WkvArgs p, const ZbVarlen b) {
  constexpr int DP = KT * kKG;
  constexpr int NT = CB * kKG;
  constexpr int NI = (CH * DP + NT - 1) / NT;      // staged (token, key) pairs per thread
  constexpr int NV = (CH * CB + NT - 1) / NT;
  extern __shared__ __align__(16) float wkv_smem[];
  float* sr = wkv_smem;                             // [CH][DP]
  float* sk = sr + CH * DP;
  float* sw = sk + CH * DP;
  float* sv = sw + CH * DP;                         // [CH][CB]
  float* sy = sv + CH * CB;                         // [CH][CB]
  float* sru = sy + CH * CB;                        // [CH]: sum_k r u k
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
#pragma unroll
  for (int i = 0; i < KT / 4; ++i) {
    const int key = (i * kKG + kg) * 4;
    float4 f = make_float4(0.f, 0.f, 0.f, 0.f);
    if (!fresh && mine) {
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
  const long long hb = static_cast<long long>(h) * D;
  const A* gr = reinterpret_cast<const A*>(p.r) + hb;
  const A* gk = reinterpret_cast<const A*>(p.k) + hb;
  const A* gv = reinterpret_cast<const A*>(p.v) + hb + c0;
  const float* gz = p.z + hb;

  float nr[NI], nk[NI], nw[NI], nv[NV];
  auto fetch = [&](int base) {
    const int cn = min(CH, n - base);
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int e = tid + i * NT, tt = e / DP, kk = e % DP;
      nr[i] = nk[i] = 0.f;
      nw[i] = 0.f;
      if (tt < cn && kk < D) {
        const long long t = t0 + base + tt;
        nr[i] = zb_ld_act(gr + t * p.ld + kk);
        nk[i] = zb_ld_act(gk + t * p.ld + kk);
        nw[i] = gz[t * p.ldz + kk];
      }
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int e = tid + i * NT, tt = e / CB, cc = e % CB;
      nv[i] = 0.f;
      if (tt < cn && c0 + cc < D) nv[i] = zb_ld_act(gv + (t0 + base + tt) * p.ld + cc);
    }
  };
  fetch(0);
  for (int base = 0; base < n; base += CH) {
    const int cn = min(CH, n - base);
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int e = tid + i * NT, kk = e % DP;
      if (e < CH * DP) {
        sr[e] = nr[i];
        sk[e] = nk[i];
        sw[e] = kk < D ? expf(-expf(nw[i] + p.w0[hb + kk])) : 0.f;
      }
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int e = tid + i * NT;
      if (e < CH * CB) sv[e] = nv[i];
    }
    __syncthreads();
    if (base + CH < n) fetch(base + CH);
    for (int tt = warp; tt < cn; tt += NT / 32) {
      float d = 0.f;
      for (int kk = lane; kk < D; kk += 32) d = fmaf(sr[tt * DP + kk] * p.u[hb + kk], sk[tt * DP + kk], d);
      d = zb_warp_sum(d);
      if (lane == 0) sru[tt] = d;
    }
    __syncthreads();
#pragma unroll 2
    for (int tt = 0; tt < cn; ++tt) {
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
      float y = y0 + y1;
      y += __shfl_xor_sync(0xffffffffu, y, 1);
      y += __shfl_xor_sync(0xffffffffu, y, 2);
      y += __shfl_xor_sync(0xffffffffu, y, 4);
      if (kg == 0) sy[tt * CB + col] = fmaf(v, sru[tt], y);
    }
    __syncthreads();
    if constexpr (FUSED) {
      for (int tt = warp; tt < cn; tt += NT / 32) {
        float ss = 0.f;
        for (int c = lane; c < D; c += 32) ss += sy[tt * CB + c] * sy[tt * CB + c];
        ss = zb_warp_sum(ss);
        const float inv = 1.f / sqrtf(ss / static_cast<float>(D) + p.eps);
        const long long t = t0 + base + tt;
        for (int c = lane; c < D; c += 32) {
          const float z = zb_ld_act(reinterpret_cast<const A*>(p.g) + t * p.ld + hb + c);
          zb_st_act(reinterpret_cast<A*>(p.out) + t * p.ld_out + hb + c, sy[tt * CB + c] * inv * p.norm[hb + c] * (z / (1.f + expf(-z))));
        }
      }
    } else {
      for (int e = tid; e < cn * CB; e += NT) {
        const int tt = e / CB, cc = e % CB;
        if (c0 + cc < D) p.o[(t0 + base + tt) * (static_cast<long long>(p.heads) * D) + hb + c0 + cc] = sy[e];
      }
    }
    // no barrier here: the next pass writes sr / sk / sw / sv, whose last readers are behind the barrier above, and
    // sy is written again only after the next pass's barriers
  }
  if (!mine) return;
#pragma unroll
  for (int i = 0; i < KT / 4; ++i) {
    const int key = (i * kKG + kg) * 4;
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

// out[t, n] = sum_r tanh(a[t, r]) * w[n, r], fp32 sums: the second half of a low-rank pre-activation for few tokens.
// One CTA: one token, 256 outputs.
template <typename W>
__global__ void __launch_bounds__(256) zb_tanh_linear_kernel(const float* __restrict__ a, long long lda, const W* __restrict__ w, long long ldw,
                                                             float* __restrict__ out, long long ldo, int n, int rank) {
  zb_pdl_launch();
  zb_pdl_wait();
  extern __shared__ float tl_smem[];
  const long long t = blockIdx.y;
  for (int i = threadIdx.x; i < rank; i += 256) tl_smem[i] = tanhf(a[t * lda + i]);
  __syncthreads();
  const int c = blockIdx.x * 256 + threadIdx.x;
  if (c >= n) return;
  const W* row = w + c * ldw;
  float acc = 0.f;
  for (int i = 0; i < rank; ++i) acc = fmaf(tl_smem[i], zb_ld_act(row + i), acc);
  out[t * ldo + c] = acc;
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

template <typename A, int KT, int CB, int CH, bool FUSED>
int launch_scan(const WkvArgs& p, const ZbVarlen& b, cudaStream_t s) {
  constexpr int kSmem = (3 * CH * KT * kKG + 2 * CH * CB + CH) * 4;
  static bool configured[16] = {};
  if (const int rc = zb_config_smem_once(zb_wkv_scan_kernel<A, KT, CB, CH, FUSED>, kSmem, configured)) return rc;
  const cudaError_t e = zb_launch(zb_wkv_scan_kernel<A, KT, CB, CH, FUSED>, dim3(p.heads, b.num_seqs, (p.dim + CB - 1) / CB), dim3(CB * kKG),
                                  kSmem, s, p, b);
  zb_count_launch(1);
  return static_cast<int>(e != cudaSuccess ? e : cudaGetLastError());
}

template <typename A>
int scan(const WkvArgs& p, const ZbVarlen& b, bool fused, cudaStream_t s) {
  const int D = p.dim;
  if (fused) {
    if (D <= 32) return launch_scan<A, 4, 32, 16, true>(p, b, s);
    if (D <= 64) return launch_scan<A, 8, 64, 16, true>(p, b, s);
    if (D <= 96) return launch_scan<A, 12, 96, 16, true>(p, b, s);
    if (D <= 128) return launch_scan<A, 16, 128, 16, true>(p, b, s);
    return -72;
  }
  if (D <= 32) return launch_scan<A, 4, 16, 16, false>(p, b, s);
  if (D <= 64) return launch_scan<A, 8, 16, 16, false>(p, b, s);
  if (D <= 96) return launch_scan<A, 12, 16, 16, false>(p, b, s);
  if (D <= 128) return launch_scan<A, 16, 16, 16, false>(p, b, s);
  if (D <= 192) return launch_scan<A, 24, 16, 8, false>(p, b, s);
  if (D <= 256) return launch_scan<A, 32, 16, 8, false>(p, b, s);
  return -72;
}
}  // namespace

extern "C" {

// 1 when a launch with the norm inside is possible for this head size.
int zb_wkv_can_fuse(int dim) { return dim <= 128 ? 1 : 0; }

// The recurrence over a varlen batch.  `o` null: norm and gate in the same launch (dim <= 128); else o is scratch
// [T, H * dim] fp32 and a second launch finishes.  dim <= 256.
int zb_wkv_scan(const void* r, const void* k, const void* v, const void* g, long long ld, const float* z, long long ldz, const float* w0,
                const float* u, const float* norm, float eps, float* state, const int32_t* slots, void* out, long long ld_out, float* o,
                int act_f32, int heads, int dim, const int32_t* q_start, const int32_t* seq_lens, int num_seqs, int tokens, void* stream) {
  if (num_seqs <= 0 || tokens <= 0) return 0;
  const WkvArgs p = {r, k, v, g, ld, z, ldz, w0, u, norm, eps, state, slots, out, ld_out, o, heads, dim};
  const ZbVarlen b = {q_start, seq_lens, num_seqs};
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const int rc = act_f32 ? scan<float>(p, b, o == nullptr, s) : scan<__nv_bfloat16>(p, b, o == nullptr, s);
  if (rc != 0 || o == nullptr) return rc;
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
  if (rank > 8192 || tokens > 65535) return -70;
  const dim3 grid((n + 255) / 256, tokens);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const size_t smem = static_cast<size_t>(rank) * sizeof(float);
  const cudaError_t e = w_f32 ? zb_launch(zb_tanh_linear_kernel<float>, grid, dim3(256), smem, s, a, lda, reinterpret_cast<const float*>(w), ldw, out, ldo, n, rank)
                              : zb_launch(zb_tanh_linear_kernel<__nv_bfloat16>, grid, dim3(256), smem, s, a, lda,
                                          reinterpret_cast<const __nv_bfloat16*>(w), ldw, out, ldo, n, rank);
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
