// Grouped-query attention whose heads are normalised, partly rotated, soft-capped, windowed with kept first tokens, sunk and
// gated (any of these may be off), with key and value sizes of their own, bf16 or fp32:
//
//   zb_gqa_prep     per head RMS norm of q and k, rotation of the first `rot` dimensions (pairs (i, i + rot / 2)), cache write
//                   of k and v.  Heads are written with a padded stride (zeros behind their elements), so that the
//                   tensor-core kernels of attention.cu / attention_tc.cu take any size up to theirs
//   zb_gqa_attend   attention over the paged cache for any sizes: the fp32 path and the fall-back for sizes the tensor-core
//                   kernels do not take
//
// Position i sees j when j <= i and (i - j < window or j < keep).  score = q . k * scale, then cap * tanh(score / cap); with
// a sink the softmax denominator has an additional exp(0).  Norms, angles, scores and softmax are fp32.
#include "act.cuh"
#include "host_api.h"

namespace {
constexpr uint32_t kKernelGqaPrep = 34;
constexpr uint32_t kKernelGqaAttend = 35;

struct GqaPrepArgs {
  const void* in;            // [T, ld_in]: q heads | k heads | v heads
  long long ld_in;
  const float* q_norm;       // [dk]
  const float* k_norm;       // [dk]
  const float* inv_freq;     // [rot / 2]
  const int32_t* positions;
  const int32_t* slots;      // cache row of every token, negative: no write
  void* q;                   // [T, hq, ldq]
  void* k_cache;             // [rows, hkv, ldk]
  void* v_cache;             // [rows, hkv, ldv]
  long long num_rows;
  float eps;
  int hq, hkv, dk, dv, rot;
  int ldq, ldk, ldv;         // elements per head where it is written
};

template <int V>
ZB_DEVICE void ld_elems(float (&v)[V], const __nv_bfloat16* p) {
  if constexpr (V == 4) {
    const uint2 g = *reinterpret_cast<const uint2*>(p);
    const float2 lo = zb_unpack_bf16x2(g.x), hi = zb_unpack_bf16x2(g.y);
    v[0] = lo.x; v[1] = lo.y; v[2] = hi.x; v[3] = hi.y;
  } else {
    v[0] = zb_ld_act(p);
  }
}
template <int V>
ZB_DEVICE void ld_elems(float (&v)[V], const float* p) {
  if constexpr (V == 4) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
  } else {
    v[0] = *p;
  }
}
template <int V>
ZB_DEVICE void st_elems(__nv_bfloat16* p, const float (&v)[V]) {
  if constexpr (V == 4) *reinterpret_cast<uint2*>(p) = make_uint2(zb_pack_bf16x2(v[0], v[1]), zb_pack_bf16x2(v[2], v[3]));
  else zb_st_act(p, v[0]);
}
template <int V>
ZB_DEVICE void st_elems(float* p, const float (&v)[V]) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  else *p = v[0];
}

// One CTA per token, one warp per head; NR groups of V neighbouring elements per lane.
constexpr int kPrepThreads = 256;

template <typename A, int NR, int V>
__global__ void __launch_bounds__(kPrepThreads) zb_gqa_prep_kernel(const GqaPrepArgs p) {
  extern __shared__ __align__(16) float prep_smem[];      // [rot / 2] (cos, sin) | [warps][rot] the rotated part's elements
  zb_pdl_launch();
  zb_pdl_wait();
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, half = p.rot / 2;
  float2* cs = reinterpret_cast<float2*>(prep_smem);
  float* row = prep_smem + p.rot + warp * p.rot;
  const float pos = static_cast<float>(p.positions[t]);
  for (int i = threadIdx.x; i < half; i += kPrepThreads) {
    float sn, c;
    sincosf(pos * p.inv_freq[i], &sn, &c);
    cs[i] = make_float2(c, sn);
  }
  __syncthreads();
  const long long slot = p.slots[t];
  if (slot >= p.num_rows) (void)ZB_BC_OK(slot, p.num_rows, kKernelGqaPrep, 1);
  const bool slot_ok = slot >= 0 && slot < p.num_rows;
  const A* in = reinterpret_cast<const A*>(p.in) + t * p.ld_in;
  const int heads = p.hq + 2 * p.hkv;
  for (int h = warp; h < heads; h += kPrepThreads / 32) {
    const bool is_q = h < p.hq, is_v = h >= p.hq + p.hkv;
    if (!is_q && !slot_ok) continue;
    const int g = is_q ? h : (is_v ? h - p.hq - p.hkv : h - p.hq);
    const int n = is_v ? p.dv : p.dk, ld = is_q ? p.ldq : (is_v ? p.ldv : p.ldk);
    const A* src = in + (is_v ? (p.hq + p.hkv) * p.dk + g * p.dv : h * p.dk);
    A* dst = is_q ? reinterpret_cast<A*>(p.q) + (static_cast<long long>(t) * p.hq + g) * ld
                  : reinterpret_cast<A*>(is_v ? p.v_cache : p.k_cache) + (slot * p.hkv + g) * ld;
    float v[NR][V];
    float ss = 0.f;
#pragma unroll
    for (int r = 0; r < NR; ++r) {
      const int i = (lane + 32 * r) * V;
#pragma unroll
      for (int e = 0; e < V; ++e) v[r][e] = 0.f;
      if (i < n) ld_elems<V>(v[r], src + i);
#pragma unroll
      for (int e = 0; e < V; ++e) ss = fmaf(v[r][e], v[r][e], ss);
    }
    if (!is_v) {
      const float inv = 1.f / sqrtf(zb_warp_sum(ss) / static_cast<float>(n) + p.eps);
      const float* nw = is_q ? p.q_norm : p.k_norm;
      __syncwarp();
#pragma unroll
      for (int r = 0; r < NR; ++r) {
        const int i = (lane + 32 * r) * V;
        if (i >= n) continue;
#pragma unroll
        for (int e = 0; e < V; ++e) {
          v[r][e] *= inv * nw[i + e];
          if (i + e < p.rot) row[i + e] = v[r][e];
        }
      }
      __syncwarp();
#pragma unroll
      for (int r = 0; r < NR; ++r) {
        const int i = (lane + 32 * r) * V;
#pragma unroll
        for (int e = 0; e < V; ++e) {
          const int j = i + e;
          if (j >= p.rot) continue;
          const bool low = j < half;
          const float2 f = cs[low ? j : j - half];
          const float other = row[low ? j + half : j - half];
          v[r][e] = low ? v[r][e] * f.x - other * f.y : v[r][e] * f.x + other * f.y;
        }
      }
    }
#pragma unroll
    for (int r = 0; r < NR; ++r) {
      const int i = (lane + 32 * r) * V;
      if (i < ld) st_elems<V>(dst + i, v[r]);             // elements n .. ld are zero
    }
  }
}

template <typename A, int V>
cudaError_t launch_prep(const GqaPrepArgs& p, int tokens, cudaStream_t s) {
  const int widest = max(max(p.ldq, p.ldk), p.ldv);
  const size_t smem = static_cast<size_t>(p.rot) * (1 + kPrepThreads / 32) * sizeof(float);
  if (smem > 48 * 1024) return cudaErrorInvalidValue;
  const int nr = (widest + 32 * V - 1) / (32 * V);
  if (nr <= 1) return zb_launch(zb_gqa_prep_kernel<A, 1, V>, dim3(tokens), dim3(kPrepThreads), smem, s, p);
  if (nr <= 2) return zb_launch(zb_gqa_prep_kernel<A, 2, V>, dim3(tokens), dim3(kPrepThreads), smem, s, p);
  if (nr <= 8) return zb_launch(zb_gqa_prep_kernel<A, 8, V>, dim3(tokens), dim3(kPrepThreads), smem, s, p);
  if (nr <= 32) return zb_launch(zb_gqa_prep_kernel<A, 32, V>, dim3(tokens), dim3(kPrepThreads), smem, s, p);
  return cudaErrorInvalidValue;
}
template <typename A>
cudaError_t launch_prep(const GqaPrepArgs& p, int tokens, cudaStream_t s) {
  const bool vec = p.dk % 4 == 0 && p.dv % 4 == 0 && p.ld_in % 4 == 0 && p.ldq % 4 == 0 && p.ldk % 4 == 0 && p.ldv % 4 == 0 &&
                   (reinterpret_cast<uintptr_t>(p.in) & (4 * sizeof(A) - 1)) == 0;
  return vec ? launch_prep<A, 4>(p, tokens, s) : launch_prep<A, 1>(p, tokens, s);
}

// ------------------------------------------------------------------------------------------ attention, any sizes
struct GqaArgs {
  const void* q;             // [T, hq, ldq]
  const void* k_cache;       // [rows, hkv, ldk]
  const void* v_cache;       // [rows, hkv, ldv]
  int ldq, ldk, ldv;
  const void* gate;          // [T, ld_gate]: hq * dv columns, or null
  long long ld_gate;
  void* out;                 // [T, ld_out]: hq * dv columns
  long long ld_out;
  const int32_t* block_table;
  int max_pages, page_size;
  int hq, hkv, dk, dv;
  int window, keep;
  float scale, cap;          // cap 0: none
  int sink;
};

constexpr int kGqaKeys = 64;

template <typename A, int RC>      // RC: value columns per thread
__global__ void __launch_bounds__(128) zb_gqa_attend_kernel(const GqaArgs p, const ZbVarlen b) {
  zb_pdl_launch();
  zb_pdl_wait();
  extern __shared__ float gqa_smem[];                // [dk] the query
  __shared__ float sc[kGqaKeys];
  __shared__ long long srow[kGqaKeys];
  const int t = blockIdx.x, h = blockIdx.y, g = h / (p.hq / p.hkv);
  int s = 0;
  while (s + 1 < b.num_seqs && b.q_start[s + 1] <= t) ++s;
  const int n = b.q_start[s + 1] - b.q_start[s];
  const int pos = b.seq_lens[s] - n + (t - b.q_start[s]);
  A* out = reinterpret_cast<A*>(p.out) + t * p.ld_out + static_cast<long long>(h) * p.dv;
  if (pos < 0) {                                     // a padding row of a decode batch: no key
    for (int c = threadIdx.x; c < p.dv; c += 128) zb_st_act(out + c, 0.f);
    return;
  }
  const int first = p.window > 0 ? max(0, pos - p.window + 1) : 0;      // seen: [0, kept) and [first, pos]
  const int kept = min(p.keep, first);
  const A* q = reinterpret_cast<const A*>(p.q) + (static_cast<long long>(t) * p.hq + h) * p.ldq;
  for (int i = threadIdx.x; i < p.dk; i += 128) gqa_smem[i] = zb_ld_act(q + i);
  const int32_t* bt = p.block_table + static_cast<long long>(s) * p.max_pages;
  const A* kc = reinterpret_cast<const A*>(p.k_cache) + static_cast<long long>(g) * p.ldk;
  const A* vc = reinterpret_cast<const A*>(p.v_cache) + static_cast<long long>(g) * p.ldv;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float m = p.sink ? 0.f : -INFINITY, l = p.sink ? 1.f : 0.f, acc[RC];
#pragma unroll
  for (int i = 0; i < RC; ++i) acc[i] = 0.f;
  const int total = kept + pos + 1 - first;
  for (int k0 = 0; k0 < total; k0 += kGqaKeys) {
    const int nk = min(kGqaKeys, total - k0);
    __syncthreads();
    if (threadIdx.x < nk) {
      const int i = k0 + threadIdx.x, key = i < kept ? i : first + i - kept;
      int page = bt[key / p.page_size];
      if (!ZB_BC_OK(page, ZB_BC_PAGES, kKernelGqaAttend, 1)) page = 0;
      srow[threadIdx.x] = (static_cast<long long>(page) * p.page_size + key % p.page_size) * p.hkv;
    }
    __syncthreads();
    for (int j = warp; j < nk; j += 4) {
      const A* row = kc + srow[j] * p.ldk;
      float d = 0.f;
      for (int i = lane; i < p.dk; i += 32) d = fmaf(gqa_smem[i], zb_ld_act(row + i), d);
      d = zb_warp_sum(d) * p.scale;
      if (p.cap > 0.f) d = p.cap * tanhf(d / p.cap);
      if (lane == 0) sc[j] = d;
    }
    __syncthreads();
    float mx = m;
    for (int j = 0; j < nk; ++j) mx = fmaxf(mx, sc[j]);
    const float corr = m == -INFINITY ? 0.f : expf(m - mx);
    m = mx;
    l *= corr;
#pragma unroll
    for (int i = 0; i < RC; ++i) acc[i] *= corr;
    for (int j = 0; j < nk; ++j) {
      const float pj = expf(sc[j] - m);
      l += pj;
      const A* row = vc + srow[j] * p.ldv;
#pragma unroll
      for (int i = 0; i < RC; ++i) {
        const int c = threadIdx.x + 128 * i;
        if (c < p.dv) acc[i] = fmaf(pj, zb_ld_act(row + c), acc[i]);
      }
    }
  }
  const float inv = 1.f / l;
  const A* gate = p.gate != nullptr ? reinterpret_cast<const A*>(p.gate) + t * p.ld_gate + static_cast<long long>(h) * p.dv : nullptr;
#pragma unroll
  for (int i = 0; i < RC; ++i) {
    const int c = threadIdx.x + 128 * i;
    if (c >= p.dv) continue;
    float o = acc[i] * inv;
    if (gate != nullptr) o *= 1.f / (1.f + expf(-zb_ld_act(gate + c)));
    zb_st_act(out + c, o);
  }
}

template <typename A>
cudaError_t launch_attend(const GqaArgs& p, const ZbVarlen& b, int tokens, cudaStream_t s) {
  const size_t smem = static_cast<size_t>(p.dk) * sizeof(float);
  const dim3 grid(tokens, p.hq);
  if (smem > 40 * 1024) return cudaErrorInvalidValue;
  if (p.dv <= 128) return zb_launch(zb_gqa_attend_kernel<A, 1>, grid, dim3(128), smem, s, p, b);
  if (p.dv <= 256) return zb_launch(zb_gqa_attend_kernel<A, 2>, grid, dim3(128), smem, s, p, b);
  if (p.dv <= 1024) return zb_launch(zb_gqa_attend_kernel<A, 8>, grid, dim3(128), smem, s, p, b);
  return cudaErrorInvalidValue;
}
}  // namespace

extern "C" {

int zb_gqa_prep(const void* in, long long ld_in, const float* q_norm, const float* k_norm, const float* inv_freq, const int32_t* positions,
                const int32_t* slots, void* q, void* k_cache, void* v_cache, long long num_rows, float eps, int hq, int hkv, int dk, int dv,
                int rot, int ldq, int ldk, int ldv, int act_f32, int tokens, void* stream) {
  if (tokens <= 0) return 0;
  if (rot % 2 != 0 || rot > dk || ldq < dk || ldk < dk || ldv < dv) return -70;
  const GqaPrepArgs p = {in, ld_in, q_norm, k_norm, inv_freq, positions, slots, q, k_cache, v_cache, num_rows, eps, hq, hkv, dk, dv, rot, ldq, ldk, ldv};
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const cudaError_t e = act_f32 ? launch_prep<float>(p, tokens, s) : launch_prep<__nv_bfloat16>(p, tokens, s);
  zb_count_launch(1);
  return static_cast<int>(e != cudaSuccess ? e : cudaGetLastError());
}

int zb_gqa_attend(const void* q, int ldq, const void* k_cache, int ldk, const void* v_cache, int ldv, const void* gate, long long ld_gate, void* out,
                  long long ld_out, const int32_t* block_table, int max_pages, int page_size, int hq, int hkv, int dk, int dv, int window, int keep,
                  float scale, float cap, int sink, const int32_t* q_start, const int32_t* seq_lens, int num_seqs, int tokens, int act_f32,
                  void* stream) {
  if (tokens <= 0) return 0;
  if (hkv <= 0 || hq % hkv != 0) return -30;
  const GqaArgs p = {q, k_cache, v_cache, ldq, ldk, ldv, gate, ld_gate, out, ld_out, block_table, max_pages, page_size,
                     hq, hkv, dk, dv, window, keep, scale, cap, sink};
  const ZbVarlen b = {q_start, seq_lens, num_seqs};
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const cudaError_t e = act_f32 ? launch_attend<float>(p, b, tokens, s) : launch_attend<__nv_bfloat16>(p, b, tokens, s);
  zb_count_launch(1);
  return static_cast<int>(e != cudaSuccess ? e : cudaGetLastError());
}

}  // extern "C"
