// Grouped-query attention whose heads are normalised, partly rotated, soft-capped, windowed with kept first tokens or chunked,
// sunk and gated (any of these may be off), with key and value sizes of their own and one or two maps per head, bf16 or fp32:
//
//   zb_gqa_prep     RMS norm of q and k (per head, or over all heads of a projection at once), rotation of the first `rot` dimensions (pairs (i, i + rot / 2)), cache write
//                   of k and v.  Heads are written with a padded stride (zeros behind their elements), so that the
//                   tensor-core kernels of attention.cu / attention_tc.cu take any size up to theirs.  With two maps a cached
//                   key is [map 1 | map 2], and a head has two query rows, each zero where the other map's keys are
//   zb_gqa_attend   attention over the paged cache for any sizes: the fp32 path and the fall-back for sizes the tensor-core
//                   kernels do not take
//   zb_gqa_pool     pooled blocks of a windowed cache: the mean of the cached keys and values of every `pool` positions whose last
//                   one is new (for decode steps zb_gqa_prep does it behind its cache write)
//   zb_pair_combine differential attention: the two maps' results a1, a2 of every head -> a1 - lambda a2 at unit root mean
//                   square, times a constant (the kernels of attention.cu and attention_tc.cu do it as they store)
//
// Position i sees j when j <= i and (i - j < window or j < keep), or with chunks when floor(i / chunk) = floor(j / chunk); with
// pooled blocks also the mean key and value of every block in front of its window.  score = q . k * scale, then cap * tanh(score / cap); with
// a sink the softmax denominator has an additional exp(0).  Norms, angles, scores and softmax are fp32.
#include "act.cuh"
#include "attention_tiles.cuh"
#include "host_api.h"

namespace {
constexpr uint32_t kKernelGqaPrep = 34;
constexpr uint32_t kKernelGqaAttend = 35;
constexpr uint32_t kKernelGqaPool = 37;

// Pooled blocks of a cache (ZbAttnExt.pool).
struct PoolArgs {
  int pool;                  // positions per block, 0: none
  int rows;                  // blocks per page at most
  void* k;                   // [pages, rows, hkv, ldk]
  void* v;                   // [pages, rows, hkv, ldv]
  const int32_t* block_table;
  int max_pages, page_size;
};

struct GqaPrepArgs {
  const void* in;            // [T, ld_in]: q heads | k heads | v heads
  long long ld_in;
  const float* q_norm;       // [dk], or null: no norm
  const float* k_norm;
  const float* inv_freq;     // [rot / 2]
  const int32_t* positions;
  const int32_t* slots;      // cache row of every token, negative: no write
  void* q;                   // [T, hq, ldq]
  void* k_cache;             // [rows, hkv, ldk]
  void* v_cache;             // [rows, hkv, ldv]
  long long num_rows;
  float eps;
  int hq, hkv, dk, dv, rot;  // hq: query rows, maps of a head counted one by one; hkv 0: queries only
  int maps;
  int ldq, ldk, ldv;         // elements per row where it is written
  int whole;                 // 1: one norm over all query rows and one over all keys, weights [hq dk] and [hkv dk]
  const float* sumsq;        // whole: [T, 2] sums of squares of q and k over all ranks, or null: those of `in`
  int total_q, total_k;      // whole: elements that the sums cover
  float amp;                 // factor on cosines and sines
  PoolArgs pool;             // one token per sequence: blocks that the token completes are pooled
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

// Mean key and value of block b of sequence s: V elements per thread of a row of CTAs.
template <typename A, int V>
ZB_DEVICE void pool_block(const PoolArgs& p, const A* kc, const A* vc, int hkv, int ldk, int ldv, int s, int b) {
  const int32_t* bt = p.block_table + static_cast<long long>(s) * p.max_pages;
  const int index = min(zb_pool_page_index(b, p.pool, p.page_size), p.max_pages - 1);
  int page = bt[index];
  if (!ZB_BC_OK(page, ZB_BC_PAGES, kKernelGqaPool, 1)) page = 0;
  const long long row = zb_pool_row(page, index, b, p.pool, p.page_size, p.rows);
  const float scale = 1.f / static_cast<float>(p.pool);
  const int nk = hkv * ldk, n = nk + hkv * ldv;
  const int i = (blockIdx.y * blockDim.x + threadIdx.x) * V;
  if (i < n) {
    const bool is_k = i < nk;
    const int c = is_k ? i : i - nk, ld = is_k ? nk : n - nk;
    const A* src = (is_k ? kc : vc) + c;
    float acc[V];
#pragma unroll
    for (int e = 0; e < V; ++e) acc[e] = 0.f;
#pragma unroll 8
    for (int j = 0; j < p.pool; ++j) {
      const int tok = b * p.pool + j;
      int pg = bt[min(tok / p.page_size, p.max_pages - 1)];
      if (!ZB_BC_OK(pg, ZB_BC_PAGES, kKernelGqaPool, 2)) pg = 0;
      float v[V];
      ld_elems<V>(v, src + (static_cast<long long>(pg) * p.page_size + tok % p.page_size) * ld);
#pragma unroll
      for (int e = 0; e < V; ++e) acc[e] += v[e];
    }
#pragma unroll
    for (int e = 0; e < V; ++e) acc[e] *= scale;
    st_elems<V>((is_k ? reinterpret_cast<A*>(p.k) : reinterpret_cast<A*>(p.v)) + row * ld + c, acc);
  }
}

// One CTA per token (STEP: several, which share its heads, and blocks are pooled), L lanes (a warp or half of one) per head; NR groups of V neighbouring elements per lane.
constexpr int kPrepThreads = 256;

template <typename A, int NR, int V, int L, bool STEP>
__global__ void __launch_bounds__(kPrepThreads) zb_gqa_prep_kernel(const GqaPrepArgs p) {
  extern __shared__ __align__(16) float prep_smem[];      // [rot / 2] (cos, sin) | [warps][rot] the rotated part's elements
  zb_pdl_launch();
  zb_pdl_wait();
  const int t = blockIdx.x, team = threadIdx.x / L, lane = threadIdx.x % L, half = p.rot / 2;
  const uint32_t members = L == 32 ? 0xffffffffu : 0xffffu << (threadIdx.x & 16);
  float2* cs = reinterpret_cast<float2*>(prep_smem);
  float* row = prep_smem + p.rot + team * p.rot;
  const float pos = static_cast<float>(p.positions[t]);
  for (int i = threadIdx.x; i < half; i += kPrepThreads) {
    float sn, c;
    sincosf(pos * p.inv_freq[i], &sn, &c);
    cs[i] = make_float2(c * p.amp, sn * p.amp);
  }
  const A* in = reinterpret_cast<const A*>(p.in) + t * p.ld_in;
  __shared__ float whole_part[2][kPrepThreads / 32];
  float whole_q = 1.f, whole_k = 1.f;
  if (p.whole) {
    float sq = 0.f, sk = 0.f;
    if (p.sumsq != nullptr) {
      sq = p.sumsq[2 * t];
      sk = p.sumsq[2 * t + 1];
      __syncthreads();
    } else {
      const int nq = p.hq * p.dk, nk = p.hkv * p.dk;
#pragma unroll 4
      for (int i = threadIdx.x * V; i < nq + nk; i += kPrepThreads * V) {
        float v[V], s2 = 0.f;
        ld_elems<V>(v, in + i);
#pragma unroll
        for (int e = 0; e < V; ++e) s2 = fmaf(v[e], v[e], s2);
        if (i < nq) sq += s2;
        else sk += s2;
      }
      sq = zb_warp_sum(sq);
      sk = zb_warp_sum(sk);
      if ((threadIdx.x & 31) == 0) {
        whole_part[0][threadIdx.x >> 5] = sq;
        whole_part[1][threadIdx.x >> 5] = sk;
      }
      __syncthreads();
      sq = sk = 0.f;
#pragma unroll
      for (int i = 0; i < kPrepThreads / 32; ++i) {
        sq += whole_part[0][i];
        sk += whole_part[1][i];
      }
    }
    whole_q = 1.f / sqrtf(sq / static_cast<float>(p.total_q) + p.eps);
    whole_k = 1.f / sqrtf(sk / static_cast<float>(p.total_k) + p.eps);
  } else {
    __syncthreads();
  }
  const long long slot = p.slots[t];
  if (slot >= p.num_rows) (void)ZB_BC_OK(slot, p.num_rows, kKernelGqaPrep, 1);
  const bool slot_ok = slot >= 0 && slot < p.num_rows;
  const int keys = p.hkv * p.maps, heads = p.hq + keys + p.hkv;
  const int done = STEP && p.pool.pool > 0 && slot_ok ? p.positions[t] + 1 : 0;
  const bool pool_now = STEP && done > 0 && done % p.pool.pool == 0;     // this token completes a block
  for (int h = team + (STEP ? kPrepThreads / L * blockIdx.y : 0); h < heads; h += kPrepThreads / L * (STEP ? gridDim.y : 1)) {
    const bool is_q = h < p.hq, is_v = h >= p.hq + keys;
    if (!is_q && !slot_ok) continue;
    const int u = is_q ? h : (is_v ? h - p.hq - keys : h - p.hq);        // row among its kind
    const int map = is_v ? 0 : u % p.maps;
    const int n = is_v ? p.dv : p.dk, ld = is_v ? p.ldv : (is_q ? p.ldq : p.ldk) / p.maps;
    const A* src = in + (is_v ? (p.hq + keys) * p.dk + u * p.dv : h * p.dk);
    A* dst = is_q ? reinterpret_cast<A*>(p.q) + (static_cast<long long>(t) * p.hq + u) * p.ldq + map * ld
                  : (is_v ? reinterpret_cast<A*>(p.v_cache) + (slot * p.hkv + u) * p.ldv
                          : reinterpret_cast<A*>(p.k_cache) + (slot * p.hkv + u / p.maps) * p.ldk + map * ld);
    float v[NR][V];
    float ss = 0.f;
#pragma unroll
    for (int r = 0; r < NR; ++r) {
      const int i = (lane + L * r) * V;
#pragma unroll
      for (int e = 0; e < V; ++e) v[r][e] = 0.f;
      if (i < n) ld_elems<V>(v[r], src + i);
#pragma unroll
      for (int e = 0; e < V; ++e) ss = fmaf(v[r][e], v[r][e], ss);
    }
    if (!is_v) {
      const float* nw = is_q ? p.q_norm : p.k_norm;
      float inv = is_q ? whole_q : whole_k;
      if (p.whole) {
        nw += u * p.dk;
      } else if (nw != nullptr) {
#pragma unroll
        for (int o = L / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(members, ss, o);
        inv = 1.f / sqrtf(ss / static_cast<float>(n) + p.eps);
      }
      __syncwarp(members);
#pragma unroll
      for (int r = 0; r < NR; ++r) {
        const int i = (lane + L * r) * V;
        if (i >= n) continue;
#pragma unroll
        for (int e = 0; e < V; ++e) {
          if (nw != nullptr) v[r][e] *= inv * nw[i + e];
          if (i + e < p.rot) row[i + e] = v[r][e];
        }
      }
      __syncwarp(members);
#pragma unroll
      for (int r = 0; r < NR; ++r) {
        const int i = (lane + L * r) * V;
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
      const int i = (lane + L * r) * V;
      if (i >= ld) continue;
      st_elems<V>(dst + i, v[r]);                          // elements n .. ld are zero
      if (is_q && p.maps == 2) {
        const float zero[V] = {};
        st_elems<V>(dst + i + (map == 0 ? ld : -ld), zero);
      }
    }
    if (STEP && pool_now && !is_q) {                               // every lane averages the elements that it has written
      const A* cache = reinterpret_cast<const A*>(is_v ? p.v_cache : p.k_cache) + static_cast<long long>(u) * ld;
      const long long step = static_cast<long long>(p.hkv) * ld;
      const int32_t* bt = p.pool.block_table + static_cast<long long>(t) * p.pool.max_pages;
#pragma unroll
      for (int r = 0; r < NR; ++r)
#pragma unroll
        for (int e = 0; e < V; ++e) v[r][e] = 0.f;
      auto page_of = [&](int index) {
        const int page = bt[min(index, p.pool.max_pages - 1)];
        return ZB_BC_OK(page, ZB_BC_PAGES, kKernelGqaPool, 3) ? page : 0;
      };
#pragma unroll 8
      for (int j = 0; j < p.pool.pool; ++j) {
        const int tok = done - p.pool.pool + j;
        const A* row_j = cache + (static_cast<long long>(page_of(tok / p.pool.page_size)) * p.pool.page_size + tok % p.pool.page_size) * step;
#pragma unroll
        for (int r = 0; r < NR; ++r) {
          const int i = (lane + L * r) * V;
          float w[V];
#pragma unroll
          for (int e = 0; e < V; ++e) w[e] = 0.f;
          if (i < ld) ld_elems<V>(w, row_j + i);
#pragma unroll
          for (int e = 0; e < V; ++e) v[r][e] += w[e];
        }
      }
      const int b = done / p.pool.pool - 1, index = min(zb_pool_page_index(b, p.pool.pool, p.pool.page_size), p.pool.max_pages - 1);
      A* out = reinterpret_cast<A*>(is_v ? p.pool.v : p.pool.k) +
               zb_pool_row(page_of(index), index, b, p.pool.pool, p.pool.page_size, p.pool.rows) * step + static_cast<long long>(u) * ld;
      const float scale = 1.f / static_cast<float>(p.pool.pool);
#pragma unroll
      for (int r = 0; r < NR; ++r) {
        const int i = (lane + L * r) * V;
#pragma unroll
        for (int e = 0; e < V; ++e) v[r][e] *= scale;
        if (i < ld) st_elems<V>(out + i, v[r]);
      }
    }
  }
}

// The blocks that a varlen batch completes, a row of CTAs each.
template <typename A, int V>
__global__ void __launch_bounds__(128) zb_gqa_pool_kernel(const PoolArgs p, const void* k_cache, const void* v_cache, int hkv, int ldk, int ldv,
                                                          const ZbVarlen b) {
  zb_pdl_launch();
  zb_pdl_wait();
  int idx = blockIdx.x;
  for (int s = 0; s < b.num_seqs; ++s) {
    const int len = b.seq_lens[s], first = (len - (b.q_start[s + 1] - b.q_start[s])) / p.pool, n = len / p.pool - first;
    if (idx < n) {
      pool_block<A, V>(p, reinterpret_cast<const A*>(k_cache), reinterpret_cast<const A*>(v_cache), hkv, ldk, ldv, s, first + idx);
      return;
    }
    idx -= n;
  }
}

template <typename A, int V, bool STEP>
cudaError_t launch_prep(const GqaPrepArgs& p, int tokens, cudaStream_t s) {
  const int widest = max(max(p.ldq, p.hkv > 0 ? p.ldk : 0) / p.maps, p.hkv > 0 ? p.ldv : 0);
  const bool narrow = max(p.dk, p.hkv > 0 ? p.ldk / p.maps : 0) <= 16 * V && widest <= 32 * V;      // keys in half a warp, values in two rounds
  const size_t smem = static_cast<size_t>(p.rot) * (1 + kPrepThreads / (narrow ? 16 : 32)) * sizeof(float);
  if (smem > 48 * 1024) return cudaErrorInvalidValue;
  // few tokens: several CTAs per token, so that a decode step does not wait for one CTA to walk over all heads
  const int teams = kPrepThreads / (narrow ? 16 : 32), heads = p.hq + p.hkv * (p.maps + 1);
  const dim3 grid(tokens, STEP ? min((heads + teams - 1) / teams, 8) : 1);
  const int nr = (widest + 32 * V - 1) / (32 * V);
  if (narrow) return zb_launch(zb_gqa_prep_kernel<A, 2, V, 16, STEP>, grid, dim3(kPrepThreads), smem, s, p);
  if (nr <= 1) return zb_launch(zb_gqa_prep_kernel<A, 1, V, 32, STEP>, grid, dim3(kPrepThreads), smem, s, p);
  if (nr <= 2) return zb_launch(zb_gqa_prep_kernel<A, 2, V, 32, STEP>, grid, dim3(kPrepThreads), smem, s, p);
  if (nr <= 8) return zb_launch(zb_gqa_prep_kernel<A, 8, V, 32, STEP>, grid, dim3(kPrepThreads), smem, s, p);
  if (nr <= 32) return zb_launch(zb_gqa_prep_kernel<A, 32, V, 32, STEP>, grid, dim3(kPrepThreads), smem, s, p);
  return cudaErrorInvalidValue;
}
template <typename A>
cudaError_t launch_prep(const GqaPrepArgs& p, int tokens, cudaStream_t s) {
  const bool vec = p.dk % 4 == 0 && p.dv % 4 == 0 && p.ld_in % 4 == 0 && p.ldq / p.maps % 4 == 0 && p.ldk / p.maps % 4 == 0 && p.ldv % 4 == 0 &&
                   (reinterpret_cast<uintptr_t>(p.in) & (4 * sizeof(A) - 1)) == 0;
  if (p.pool.pool > 0 || tokens <= 128) return vec ? launch_prep<A, 4, true>(p, tokens, s) : launch_prep<A, 1, true>(p, tokens, s);
  return vec ? launch_prep<A, 4, false>(p, tokens, s) : launch_prep<A, 1, false>(p, tokens, s);
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
  int out_f32;
  const int32_t* block_table;
  int max_pages, page_size;
  int hq, hkv, dk, dv;
  int window, keep, chunk;
  float scale, cap;          // cap 0: none
  int sink;
  PoolArgs pool;             // block_table and page size as above
  float out_scale;
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
  const long long out_at = t * p.ld_out + static_cast<long long>(h) * p.dv;
  auto store = [&](int c, float v) {
    if (p.out_f32) reinterpret_cast<float*>(p.out)[out_at + c] = v;
    else zb_st_act(reinterpret_cast<A*>(p.out) + out_at + c, v);
  };
  if (pos < 0) {                                     // a padding row of a decode batch: no key
    for (int c = threadIdx.x; c < p.dv; c += 128) store(c, 0.f);
    return;
  }
  // seen: [0, kept) and [first, pos]
  const int first = p.chunk > 0 ? pos / p.chunk * p.chunk : (p.window > 0 ? max(0, pos - p.window + 1) : 0);
  const int kept = min(p.keep, first);
  const A* q = reinterpret_cast<const A*>(p.q) + (static_cast<long long>(t) * p.hq + h) * p.ldq;
  for (int i = threadIdx.x; i < p.dk; i += 128) gqa_smem[i] = zb_ld_act(q + i);
  const int pooled = p.pool.pool > 0 ? zb_pooled_visible(pos, p.window, p.pool.pool) : 0;      // first in the list of keys
  const int32_t* bt = p.block_table + static_cast<long long>(s) * p.max_pages;
  const A* kc = reinterpret_cast<const A*>(p.k_cache) + static_cast<long long>(g) * p.ldk;
  const A* vc = reinterpret_cast<const A*>(p.v_cache) + static_cast<long long>(g) * p.ldv;
  const A* pk = reinterpret_cast<const A*>(p.pool.k) + static_cast<long long>(g) * p.ldk;
  const A* pv = reinterpret_cast<const A*>(p.pool.v) + static_cast<long long>(g) * p.ldv;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float m = p.sink ? 0.f : -INFINITY, l = p.sink ? 1.f : 0.f, acc[RC];
#pragma unroll
  for (int i = 0; i < RC; ++i) acc[i] = 0.f;
  const int total = pooled + kept + pos + 1 - first;
  for (int k0 = 0; k0 < total; k0 += kGqaKeys) {
    const int nk = min(kGqaKeys, total - k0);
    __syncthreads();
    if (threadIdx.x < nk) {
      const int at = k0 + threadIdx.x, i = at - pooled, key = i < kept ? i : first + i - kept;
      const int index = i < 0 ? zb_pool_page_index(at, p.pool.pool, p.page_size) : key / p.page_size;
      int page = bt[index];
      if (!ZB_BC_OK(page, ZB_BC_PAGES, kKernelGqaAttend, 1)) page = 0;
      srow[threadIdx.x] = (i < 0 ? zb_pool_row(page, index, at, p.pool.pool, p.page_size, p.pool.rows)
                                 : static_cast<long long>(page) * p.page_size + key % p.page_size) * p.hkv;
    }
    __syncthreads();
    for (int j = warp; j < nk; j += 4) {
      const A* row = (k0 + j < pooled ? pk : kc) + srow[j] * p.ldk;
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
      const A* row = (k0 + j < pooled ? pv : vc) + srow[j] * p.ldv;
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
    store(c, o * p.out_scale);
  }
}

// One warp per (token, head); a [T, 2 heads, dv].
template <typename A>
__global__ void __launch_bounds__(256) zb_pair_combine_kernel(const float* __restrict__ a, A* __restrict__ out, long long ld_out, int rows, int heads,
                                                              int dv, float lambda, float scale, float eps) {
  zb_pdl_launch();
  zb_pdl_wait();
  const int row = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (row >= rows) return;
  const float* a1 = a + static_cast<long long>(row) * 2 * dv;
  float ss = 0.f;
  for (int c = lane; c < dv; c += 32) {
    const float o = a1[c] - lambda * a1[dv + c];
    ss = fmaf(o, o, ss);
  }
  const float f = scale / sqrtf(zb_warp_sum(ss) / static_cast<float>(dv) + eps);
  A* dst = out + row / heads * ld_out + static_cast<long long>(row % heads) * dv;
  for (int c = lane; c < dv; c += 32) zb_st_act(dst + c, (a1[c] - lambda * a1[dv + c]) * f);
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
                int rot, int maps, int ldq, int ldk, int ldv, int whole, const float* sumsq, int total_q, int total_k, float amp, int pool, int pool_rows,
                void* pool_k, void* pool_v, const int32_t* block_table, int max_pages, int page_size, int act_f32, int tokens, void* stream) {
  if (tokens <= 0) return 0;
  if (whole && (maps != 1 || q_norm == nullptr || k_norm == nullptr || total_q < 1 || total_k < 1)) return -70;
  if (pool < 0 || (pool > 0 && (hkv < 1 || pool_rows * pool < page_size || pool_k == nullptr || pool_v == nullptr || block_table == nullptr))) return -70;
  if ((maps != 1 && maps != 2) || hq % maps != 0 || ldq % maps != 0 || ldk % maps != 0) return -70;
  if (rot % 2 != 0 || rot > dk || ldq < maps * dk || (hkv > 0 && (ldk < maps * dk || ldv < dv))) return -70;
  const GqaPrepArgs p = {in, ld_in, q_norm, k_norm, inv_freq, positions, slots, q, k_cache, v_cache, num_rows, eps,
                         hq, hkv, dk, dv, rot, maps, ldq, ldk, ldv, whole, sumsq, total_q, total_k, amp,
                         {pool, pool_rows, pool_k, pool_v, block_table, max_pages, page_size}};
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const cudaError_t e = act_f32 ? launch_prep<float>(p, tokens, s) : launch_prep<__nv_bfloat16>(p, tokens, s);
  zb_count_launch(1);
  return static_cast<int>(e != cudaSuccess ? e : cudaGetLastError());
}

// Pools the blocks that a varlen batch completes; num_blocks >= their number.
int zb_gqa_pool(const void* k_cache, const void* v_cache, void* pool_k, void* pool_v, int pool, int pool_rows, const int32_t* block_table, int max_pages,
                int page_size, int hkv, int ldk, int ldv, const int32_t* q_start, const int32_t* seq_lens, int num_seqs, int num_blocks, int act_f32,
                void* stream) {
  if (num_seqs <= 0 || num_blocks <= 0) return 0;
  if (pool < 1 || hkv < 1 || pool_rows * pool < page_size) return -70;
  const PoolArgs p = {pool, pool_rows, pool_k, pool_v, block_table, max_pages, page_size};
  const ZbVarlen b = {q_start, seq_lens, num_seqs};
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const bool vec = ldk % 4 == 0 && ldv % 4 == 0;
  const auto kernel = act_f32 ? (vec ? zb_gqa_pool_kernel<float, 4> : zb_gqa_pool_kernel<float, 1>)
                              : (vec ? zb_gqa_pool_kernel<__nv_bfloat16, 4> : zb_gqa_pool_kernel<__nv_bfloat16, 1>);
  const int threads = (hkv * (ldk + ldv) + (vec ? 3 : 0)) / (vec ? 4 : 1);
  const cudaError_t e = zb_launch(kernel, dim3(num_blocks, (threads + 127) / 128), dim3(128), 0, s, p, k_cache, v_cache, hkv, ldk, ldv, b);
  zb_count_launch(1);
  return static_cast<int>(e != cudaSuccess ? e : cudaGetLastError());
}

int zb_gqa_attend(const void* q, int ldq, const void* k_cache, int ldk, const void* v_cache, int ldv, const void* gate, long long ld_gate, void* out,
                  long long ld_out, int out_f32, const int32_t* block_table, int max_pages, int page_size, int hq, int hkv, int dk, int dv,
                  int window, int keep, int chunk, float scale, float cap, int sink, int pool, int pool_rows, const void* pool_k, const void* pool_v,
                  float out_scale, const int32_t* q_start, const int32_t* seq_lens, int num_seqs, int tokens, int act_f32, void* stream) {
  if (tokens <= 0) return 0;
  if (pool < 0 || (pool > 0 && (window <= 0 || chunk != 0 || pool_rows * pool < page_size || pool_k == nullptr || pool_v == nullptr))) return -70;
  if (hkv <= 0 || hq % hkv != 0) return -30;
  const GqaArgs p = {q, k_cache, v_cache, ldq, ldk, ldv, gate, ld_gate, out, ld_out, out_f32, block_table, max_pages, page_size,
                     hq, hkv, dk, dv, window, keep, chunk, scale, cap, sink,
                     {pool, pool_rows, const_cast<void*>(pool_k), const_cast<void*>(pool_v), block_table, max_pages, page_size}, out_scale};
  const ZbVarlen b = {q_start, seq_lens, num_seqs};
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const cudaError_t e = act_f32 ? launch_attend<float>(p, b, tokens, s) : launch_attend<__nv_bfloat16>(p, b, tokens, s);
  zb_count_launch(1);
  return static_cast<int>(e != cudaSuccess ? e : cudaGetLastError());
}

// a fp32 [tokens, 2 heads, dv] -> out [tokens, ld_out] with heads * dv columns (fp32 or bf16).
int zb_pair_combine(const float* a, void* out, long long ld_out, int tokens, int heads, int dv, float lambda, float scale, float eps, int act_f32,
                    void* stream) {
  if (tokens <= 0) return 0;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const int rows = tokens * heads;
  const dim3 grid((rows + 7) / 8);
  const cudaError_t e =
      act_f32 ? zb_launch(zb_pair_combine_kernel<float>, grid, dim3(256), 0, s, a, reinterpret_cast<float*>(out), ld_out, rows, heads, dv, lambda, scale, eps)
              : zb_launch(zb_pair_combine_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, a, reinterpret_cast<__nv_bfloat16*>(out), ld_out, rows, heads, dv,
                          lambda, scale, eps);
  zb_count_launch(1);
  return static_cast<int>(e != cudaSuccess ? e : cudaGetLastError());
}

}  // extern "C"
