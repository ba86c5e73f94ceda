// Latent attention (multi-head attention whose keys and values are projections of one low-rank latent per token), as
// Dopurax and Sodotar layers use it: the paged cache holds, per token, the normalised latent c [rank] and one rotated key part
// [rot] for every head.  A cache row is [c | pad | rotated part | pad] with both parts padded to 16 elements.
//
//   zb_latent_prep     one token per CTA: RMS norm of the query latent (where there is one), RMS norm of c, rotation of the
//                      shared key part, cache write
//   zb_latent_absorb   per head out[t, h] = a[t, h] * W[h]^T for the small per-head matrices: queries into the latent
//                      space (together with the rotation of their rotated part) and attention results out of it
//                      (together with the sigmoid output gate, where there is one)
//   zb_latent_attend   attention in the latent space (one key vector per token for all heads), any sizes, bf16 or fp32:
//                      the fp32 path and the fall-back for sizes the tensor-core kernels do not take
//   zb_latent_gather   visible cache rows of a batch -> contiguous rows, for the prefill path that expands keys and values
//   zb_latent_q_pack   queries [T, H, dim + rot] -> zero-padded rows with the rotated part rotated, for the prefill kernel
//
// Rotated parts are turned in neighbouring pairs; a design that pairs i with i + rot / 2 has its projections' rows permuted at
// load.  A sink (one number per head, or none) is a term exp(sink) of the softmax denominator: a running maximum of `sink` and a
// running sum of 1 before the first key.  Scores, softmax, norms and angles are fp32.
#include "act.cuh"
#include "host_api.h"

namespace {
constexpr uint32_t kKernelPrep = 28;
constexpr uint32_t kKernelAttend = 29;
constexpr uint32_t kKernelGather = 30;

// ------------------------------------------------------------------------------------------ prep
struct PrepArgs {
  const void* in;            // [T, ld_in]: query latent | c | shared key part
  long long ld_in;
  const float* q_norm;       // [q_rank]
  const float* c_norm;       // [rank]
  const float* inv_freq;     // [rot / 2]
  const int32_t* positions;
  const int32_t* slots;      // cache row of every token, negative: no write
  void* cq;                  // [T, ld_cq]
  long long ld_cq;
  void* cache;               // [rows, ld_cache]
  long long ld_cache;
  long long num_rows;
  float eps;
  int q_rank, rank, rot, rot_off;
};

// NV values per thread; the input row is read once, and both norms are reduced together.
template <typename A, int NV>
__global__ void __launch_bounds__(256) zb_latent_prep_kernel(const PrepArgs p) {
  __shared__ float red[2][8];
  __shared__ float rot_s[2048];
  zb_pdl_launch();
  const int cols = p.q_rank + p.rank + p.rot;
  float w[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) {                 // the norm weights are parameters
    const int c = threadIdx.x + 256 * i;
    w[i] = c < p.q_rank ? p.q_norm[c] : (c < p.q_rank + p.rank ? p.c_norm[c - p.q_rank] : 0.f);
  }
  zb_pdl_wait();
  const long long t = blockIdx.x;
  const A* in = reinterpret_cast<const A*>(p.in) + t * p.ld_in;
  const long long slot = p.slots[t];
  const float pos = static_cast<float>(p.positions[t]);
  A raw[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) raw[i] = in[min(threadIdx.x + 256 * i, cols - 1)];
  float v[NV], sq = 0.f, sc = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = threadIdx.x + 256 * i;
    v[i] = zb_ld_act(&raw[i]);
    if (c < p.q_rank) sq = fmaf(v[i], v[i], sq);
    else if (c < p.q_rank + p.rank) sc = fmaf(v[i], v[i], sc);
    else if (c < cols) rot_s[c - p.q_rank - p.rank] = v[i];
  }
  sq = zb_warp_sum(sq);
  sc = zb_warp_sum(sc);
  if ((threadIdx.x & 31) == 0) {
    red[0][threadIdx.x >> 5] = sq;
    red[1][threadIdx.x >> 5] = sc;
  }
  __syncthreads();
  sq = sc = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    sq += red[0][i];
    sc += red[1][i];
  }
  const float iq = 1.f / sqrtf(sq / static_cast<float>(max(p.q_rank, 1)) + p.eps), ic = 1.f / sqrtf(sc / static_cast<float>(p.rank) + p.eps);
  if (slot >= p.num_rows) (void)ZB_BC_OK(slot, p.num_rows, kKernelPrep, 1);
  const bool write = slot >= 0 && slot < p.num_rows;
  A* cq = reinterpret_cast<A*>(p.cq) + t * p.ld_cq;
  A* row = reinterpret_cast<A*>(p.cache) + (write ? slot : 0) * p.ld_cache;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = threadIdx.x + 256 * i;
    if (c < p.q_rank) zb_st_act(cq + c, v[i] * iq * w[i]);
    else if (c < p.q_rank + p.rank && write) zb_st_act(row + c - p.q_rank, v[i] * ic * w[i]);
  }
  if (!write) return;
  for (int i = threadIdx.x; i < p.rot / 2; i += 256) {
    float sn, cs;
    sincosf(pos * p.inv_freq[i], &sn, &cs);
    const float u = rot_s[2 * i], x = rot_s[2 * i + 1];
    zb_st_act(row + p.rot_off + 2 * i, u * cs - x * sn);
    zb_st_act(row + p.rot_off + 2 * i + 1, x * cs + u * sn);
  }
}

template <typename A>
cudaError_t launch_prep(const PrepArgs& p, int tokens, cudaStream_t s) {
  const int per = (p.q_rank + p.rank + p.rot + 255) / 256;
  if (per <= 2) return zb_launch(zb_latent_prep_kernel<A, 2>, dim3(tokens), dim3(256), 0, s, p);
  if (per <= 4) return zb_launch(zb_latent_prep_kernel<A, 4>, dim3(tokens), dim3(256), 0, s, p);
  if (per <= 9) return zb_launch(zb_latent_prep_kernel<A, 9>, dim3(tokens), dim3(256), 0, s, p);
  return zb_launch(zb_latent_prep_kernel<A, 32>, dim3(tokens), dim3(256), 0, s, p);
}

// ------------------------------------------------------------------------------------------ per-head products
struct AbsorbArgs {
  const void* a;             // a[t * lda + h * ha + k]
  long long lda, ha;
  const void* w;             // [H, N, ldw]
  long long ldw;
  void* out;                 // out[t * ldo + h * ho + n]
  long long ldo, ho;
  const void* gate;          // gate[t * ldg + h * N + n] or null: out *= sigmoid(gate)
  long long ldg;
  const float* inv_freq;     // non-null: also rotate a[.., rot_src ..] into out[.., rot_dst ..]
  const int32_t* positions;
  int rot, rot_src, rot_dst;
  int tokens, heads, n, k;
};

template <typename A>
ZB_DEVICE void absorb_rotate(const AbsorbArgs& p, int h, int t_begin, int t_end) {
  const int half = p.rot / 2;
  for (int idx = threadIdx.x; idx < (t_end - t_begin) * half; idx += blockDim.x) {
    const int t = t_begin + idx / half, i = idx % half;
    float sn, cs;
    sincosf(static_cast<float>(p.positions[t]) * p.inv_freq[i], &sn, &cs);
    const A* src = reinterpret_cast<const A*>(p.a) + t * p.lda + h * p.ha + p.rot_src + 2 * i;
    A* dst = reinterpret_cast<A*>(p.out) + t * p.ldo + h * p.ho + p.rot_dst + 2 * i;
    const float u = zb_ld_act(src), v = zb_ld_act(src + 1);
    zb_st_act(dst, u * cs - v * sn);
    zb_st_act(dst + 1, v * cs + u * sn);
  }
}

// Any sizes: 8 tokens x 64 outputs of one head per CTA.
template <typename A>
__global__ void __launch_bounds__(64) zb_latent_absorb_simple_kernel(const AbsorbArgs p) {
  zb_pdl_launch();
  zb_pdl_wait();
  const int h = blockIdx.y, t0 = blockIdx.z * 8, n = blockIdx.x * 64 + threadIdx.x;
  const int nt = min(8, p.tokens - t0);
  if (p.inv_freq != nullptr && blockIdx.x == 0) absorb_rotate<A>(p, h, t0, t0 + nt);
  if (n >= p.n) return;
  const A* a = reinterpret_cast<const A*>(p.a) + t0 * p.lda + h * p.ha;
  const A* w = reinterpret_cast<const A*>(p.w) + (static_cast<long long>(h) * p.n + n) * p.ldw;
  float acc[8] = {};
  for (int k = 0; k < p.k; ++k) {
    const float wv = zb_ld_act(w + k);
#pragma unroll
    for (int i = 0; i < 8; ++i)
      if (i < nt) acc[i] = fmaf(zb_ld_act(a + i * p.lda + k), wv, acc[i]);
  }
  for (int i = 0; i < nt; ++i) {
    float v = acc[i];
    if (p.gate != nullptr) {
      const float g = zb_ld_act(reinterpret_cast<const A*>(p.gate) + (t0 + i) * p.ldg + static_cast<long long>(h) * p.n + n);
      v *= 1.f / (1.f + expf(-g));
    }
    zb_st_act(reinterpret_cast<A*>(p.out) + (t0 + i) * p.ldo + h * p.ho + n, v);
  }
}

ZB_DEVICE void mma16816(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

// bf16, decode-sized: 16 outputs of one head for up to 16 * MT tokens per CTA; the four warps cut K among them.  The
// products are weight streams, so fragments come straight from memory with 16-byte loads: in a block of 32 values of
// K, lane quad position q holds values 8 q .. 8 q + 7 of its row, for both operands, which is a permutation of K that
// the sum does not see.
template <int MT>
__global__ void __launch_bounds__(128) zb_latent_absorb_kernel(const AbsorbArgs p) {
  __shared__ float part[4][MT * 16][17];
  zb_pdl_launch();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, q = lane & 3;
  const int h = blockIdx.y, t0 = blockIdx.z * (16 * MT), n0 = blockIdx.x * 16;
  const int nt = min(16 * MT, p.tokens - t0);
  const int blocks = (p.k + 31) / 32, per = (blocks + 3) / 4;
  const int b0 = warp * per, b1 = min(blocks, b0 + per);
  const __nv_bfloat16* a = reinterpret_cast<const __nv_bfloat16*>(p.a) + h * p.ha;
  const __nv_bfloat16* w = reinterpret_cast<const __nv_bfloat16*>(p.w) + static_cast<long long>(h) * p.n * p.ldw;
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  float acc[MT][2][4] = {};
  zb_pdl_wait();
  if (p.inv_freq != nullptr && blockIdx.x == 0) absorb_rotate<__nv_bfloat16>(p, h, t0, t0 + nt);
#pragma unroll 2
  for (int b = b0; b < b1; ++b) {
    const int k = b * 32 + q * 8;
    const bool kin = k < p.k;                     // K is a multiple of 8: a piece of 8 is inside or outside
    uint4 wf[2], af[MT][2];
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int n = n0 + j * 8 + g;
      wf[j] = kin && n < p.n ? *reinterpret_cast<const uint4*>(w + n * p.ldw + k) : zero;
    }
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int t = m * 16 + i * 8 + g;
        af[m][i] = kin && t < nt ? *reinterpret_cast<const uint4*>(a + (t0 + t) * p.lda + k) : zero;
      }
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        mma16816(acc[m][j], af[m][0].x, af[m][1].x, af[m][0].y, af[m][1].y, wf[j].x, wf[j].y);
        mma16816(acc[m][j], af[m][0].z, af[m][1].z, af[m][0].w, af[m][1].w, wf[j].z, wf[j].w);
      }
  }
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) part[warp][m * 16 + g + 8 * (e >> 1)][j * 8 + 2 * q + (e & 1)] = acc[m][j][e];
  __syncthreads();
  for (int idx = threadIdx.x; idx < nt * 16; idx += 128) {
    const int t = idx >> 4, c = idx & 15, n = n0 + c;
    if (n >= p.n) continue;
    float v = part[0][t][c] + part[1][t][c] + part[2][t][c] + part[3][t][c];
    if (p.gate != nullptr) {
      const float gt = __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(p.gate)[(t0 + t) * p.ldg + static_cast<long long>(h) * p.n + n]);
      v *= 1.f / (1.f + __expf(-gt));
    }
    reinterpret_cast<__nv_bfloat16*>(p.out)[(t0 + t) * p.ldo + h * p.ho + n] = __float2bfloat16(v);
  }
}

// ------------------------------------------------------------------------------------------ attention, any sizes
struct AttendArgs {
  const void* q;             // [T, H, ld_cache]: latent part at 0, rotated part at rot_off
  const void* cache;         // [rows, ld_cache]
  long long ld_cache;
  void* out;                 // [T, H, ld_out]
  long long ld_out;
  const int32_t* block_table;
  int max_pages, page_size;
  int heads, rank, rot, rot_off;
  int window;
  float scale;
  const float* sink;         // [heads] or null
};

constexpr int kAttendKeys = 64;

template <typename A, int RC>      // RC: latent columns per thread
__global__ void __launch_bounds__(128) zb_latent_attend_kernel(const AttendArgs p, const ZbVarlen b) {
  zb_pdl_launch();
  zb_pdl_wait();
  extern __shared__ float attend_smem[];
  __shared__ float sc[kAttendKeys];
  __shared__ long long srow[kAttendKeys];
  const int t = blockIdx.x, h = blockIdx.y;
  int s = 0;
  while (s + 1 < b.num_seqs && b.q_start[s + 1] <= t) ++s;
  const int n = b.q_start[s + 1] - b.q_start[s];
  const int pos = b.seq_lens[s] - n + (t - b.q_start[s]);
  A* out = reinterpret_cast<A*>(p.out) + (static_cast<long long>(t) * p.heads + h) * p.ld_out;
  if (pos < 0) {                                    // a padding row of a decode batch: no key
    for (int r = threadIdx.x; r < p.rank; r += 128) zb_st_act(out + r, 0.f);
    return;
  }
  const int first = p.window > 0 ? max(0, pos - p.window + 1) : 0;
  float* sq = attend_smem;                          // [rot_off + rot]
  const A* q = reinterpret_cast<const A*>(p.q) + (static_cast<long long>(t) * p.heads + h) * p.ld_cache;
  const int cols = p.rot_off + p.rot;
  for (int i = threadIdx.x; i < cols; i += 128) sq[i] = (i < p.rank || i >= p.rot_off) ? zb_ld_act(q + i) : 0.f;
  const int32_t* bt = p.block_table + static_cast<long long>(s) * p.max_pages;
  const A* cache = reinterpret_cast<const A*>(p.cache);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float m = p.sink != nullptr ? p.sink[h] : -INFINITY, l = p.sink != nullptr ? 1.f : 0.f, acc[RC];
#pragma unroll
  for (int i = 0; i < RC; ++i) acc[i] = 0.f;
  for (int k0 = first; k0 <= pos; k0 += kAttendKeys) {
    const int nk = min(kAttendKeys, pos + 1 - k0);
    __syncthreads();
    if (threadIdx.x < nk) {
      const int key = k0 + threadIdx.x;
      int page = bt[key / p.page_size];
      if (!ZB_BC_OK(page, ZB_BC_PAGES, kKernelAttend, 1)) page = 0;
      srow[threadIdx.x] = (static_cast<long long>(page) * p.page_size + key % p.page_size) * p.ld_cache;
    }
    __syncthreads();
    for (int j = warp; j < nk; j += 4) {
      const A* row = cache + srow[j];
      float d = 0.f;
      for (int i = lane; i < p.rank; i += 32) d = fmaf(sq[i], zb_ld_act(row + i), d);
      for (int i = p.rot_off + lane; i < cols; i += 32) d = fmaf(sq[i], zb_ld_act(row + i), d);
      d = zb_warp_sum(d);
      if (lane == 0) sc[j] = d * p.scale;
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
      const A* row = cache + srow[j];
#pragma unroll
      for (int i = 0; i < RC; ++i) {
        const int r = threadIdx.x + 128 * i;
        if (r < p.rank) acc[i] = fmaf(pj, zb_ld_act(row + r), acc[i]);
      }
    }
  }
  const float inv = 1.f / l;
#pragma unroll
  for (int i = 0; i < RC; ++i) {
    const int r = threadIdx.x + 128 * i;
    if (r < p.rank) zb_st_act(out + r, acc[i] * inv);
  }
}

// ------------------------------------------------------------------------------------------ gather / pack
__global__ void __launch_bounds__(256) zb_latent_gather_kernel(const __nv_bfloat16* __restrict__ cache, long long ld_cache,
                                                               const int32_t* __restrict__ block_table, int max_pages, int page_size,
                                                               const int32_t* __restrict__ key_start, const int32_t* __restrict__ first_key,
                                                               int num_seqs, __nv_bfloat16* __restrict__ out, long long ld_out, int rows,
                                                               int rank, int rot, int rot_off, int rot_out) {
  zb_pdl_launch();
  zb_pdl_wait();
  // one warp per row
  const int row = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (row >= rows) return;
  int s = 0;
  while (s + 1 < num_seqs && key_start[s + 1] <= row) ++s;
  const int key = first_key[s] + row - key_start[s];
  int page = block_table[static_cast<long long>(s) * max_pages + key / page_size];
  if (!ZB_BC_OK(page, ZB_BC_PAGES, kKernelGather, 1)) page = 0;
  const __nv_bfloat16* src = cache + (static_cast<long long>(page) * page_size + key % page_size) * ld_cache;
  __nv_bfloat16* dst = out + row * ld_out;
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  // both parts of a cache row are zero-padded to 16 elements, the destination to more
  for (int c = lane * 8; c < rot_out; c += 256) *reinterpret_cast<uint4*>(dst + c) = c < rot_off ? *reinterpret_cast<const uint4*>(src + c) : zero;
  for (int c = lane * 8; c < ld_out - rot_out; c += 256)
    *reinterpret_cast<uint4*>(dst + rot_out + c) = c < rot ? *reinterpret_cast<const uint4*>(src + rot_off + c) : zero;
}

__global__ void __launch_bounds__(256) zb_latent_q_pack_kernel(const __nv_bfloat16* __restrict__ q, long long ldq, __nv_bfloat16* __restrict__ out,
                                                               const float* __restrict__ inv_freq, const int32_t* __restrict__ positions,
                                                               int tokens, int heads, int dim, int rot, int dim_p, int rot_p) {
  zb_pdl_launch();
  zb_pdl_wait();
  extern __shared__ float2 pack_cs[];               // [rot / 2] (cos, sin) of this token
  const int t = blockIdx.x;
  const float pos = static_cast<float>(positions[t]);
  for (int i = threadIdx.x; i < rot / 2; i += 256) {
    float sn, cs;
    sincosf(pos * inv_freq[i], &sn, &cs);
    pack_cs[i] = make_float2(cs, sn);
  }
  __syncthreads();
  const int width = dim_p + rot_p;
  // pieces of 8 elements (dim and rot are multiples of 8)
  for (int idx = threadIdx.x; idx < heads * (width / 8); idx += 256) {
    const int h = idx / (width / 8), c = (idx - h * (width / 8)) * 8;
    const __nv_bfloat16* src = q + t * ldq + static_cast<long long>(h) * (dim + rot);
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (c < dim_p) {
      if (c < dim) v = *reinterpret_cast<const uint4*>(src + c);
    } else if (c - dim_p < rot) {
      v = *reinterpret_cast<const uint4*>(src + dim + c - dim_p);
      uint32_t* w = reinterpret_cast<uint32_t*>(&v);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float2 f = zb_unpack_bf16x2(w[j]), e = pack_cs[(c - dim_p) / 2 + j];
        w[j] = zb_pack_bf16x2(f.x * e.x - f.y * e.y, f.y * e.x + f.x * e.y);
      }
    }
    *reinterpret_cast<uint4*>(out + (static_cast<long long>(t) * heads + h) * width + c) = v;
  }
}

template <typename A>
int launch_attend(const AttendArgs& p, const ZbVarlen& b, int tokens, cudaStream_t s) {
  const size_t smem = static_cast<size_t>(p.rot_off + p.rot) * sizeof(float);
  if (smem > 40 * 1024) return -71;
  const dim3 grid(tokens, p.heads);
  const int rc = (p.rank + 127) / 128;
  cudaError_t e;
  if (rc <= 1) e = zb_launch(zb_latent_attend_kernel<A, 1>, grid, dim3(128), smem, s, p, b);
  else if (rc <= 2) e = zb_launch(zb_latent_attend_kernel<A, 2>, grid, dim3(128), smem, s, p, b);
  else if (rc <= 4) e = zb_launch(zb_latent_attend_kernel<A, 4>, grid, dim3(128), smem, s, p, b);
  else if (rc <= 16) e = zb_launch(zb_latent_attend_kernel<A, 16>, grid, dim3(128), smem, s, p, b);
  else return -72;
  zb_count_launch(1);
  return static_cast<int>(e != cudaSuccess ? e : cudaGetLastError());
}
}  // namespace

extern "C" {

int zb_latent_prep(const void* in, long long ld_in, const float* q_norm, const float* c_norm, const float* inv_freq,
                   const int32_t* positions, const int32_t* slots, void* cq, long long ld_cq, void* cache, long long ld_cache,
                   long long num_rows, float eps, int q_rank, int rank, int rot, int rot_off, int act_f32, int tokens, void* stream) {
  if (tokens <= 0) return 0;
  if (rot % 2 != 0 || rot_off < rank || rot_off + rot > ld_cache || rot > 2048 || q_rank + rank + rot > 32 * 256) return -70;
  const PrepArgs p = {in, ld_in, q_norm, c_norm, inv_freq, positions, slots, cq, ld_cq, cache, ld_cache, num_rows, eps, q_rank, rank, rot, rot_off};
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const cudaError_t e = act_f32 ? launch_prep<float>(p, tokens, s) : launch_prep<__nv_bfloat16>(p, tokens, s);
  zb_count_launch(1);
  return static_cast<int>(e != cudaSuccess ? e : cudaGetLastError());
}

int zb_latent_absorb(const void* a, long long lda, long long ha, const void* w, long long ldw, void* out, long long ldo, long long ho,
                     const void* gate, long long ldg, const float* inv_freq, const int32_t* positions, int rot, int rot_src, int rot_dst,
                     int tokens, int heads, int n, int k, int act_f32, void* stream) {
  if (tokens <= 0) return 0;
  const AbsorbArgs p = {a, lda, ha, w, ldw, out, ldo, ho, gate, ldg, inv_freq, positions, rot, rot_src, rot_dst, tokens, heads, n, k};
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  cudaError_t e;
  const bool fast = !act_f32 && k % 8 == 0 && lda % 8 == 0 && ha % 8 == 0 && ldw % 8 == 0 && (reinterpret_cast<uintptr_t>(a) & 15) == 0 &&
                    (reinterpret_cast<uintptr_t>(w) & 15) == 0;
  if (fast) {
    const dim3 grid((n + 15) / 16, heads, (tokens + 63) / 64);
    if (tokens <= 16) e = zb_launch(zb_latent_absorb_kernel<1>, grid, dim3(128), 0, s, p);
    else if (tokens <= 32) e = zb_launch(zb_latent_absorb_kernel<2>, grid, dim3(128), 0, s, p);
    else e = zb_launch(zb_latent_absorb_kernel<4>, grid, dim3(128), 0, s, p);
  } else {
    const dim3 grid((n + 63) / 64, heads, (tokens + 7) / 8);
    e = act_f32 ? zb_launch(zb_latent_absorb_simple_kernel<float>, grid, dim3(64), 0, s, p)
                : zb_launch(zb_latent_absorb_simple_kernel<__nv_bfloat16>, grid, dim3(64), 0, s, p);
  }
  zb_count_launch(1);
  return static_cast<int>(e != cudaSuccess ? e : cudaGetLastError());
}

int zb_latent_attend(const void* q, const void* cache, long long ld_cache, void* out, long long ld_out, const int32_t* block_table,
                     int max_pages, int page_size, int heads, int rank, int rot, int rot_off, int window, float scale, const float* sink,
                     const int32_t* q_start, const int32_t* seq_lens, int num_seqs, int tokens, int act_f32, void* stream) {
  if (tokens <= 0) return 0;
  const AttendArgs p = {q, cache, ld_cache, out, ld_out, block_table, max_pages, page_size, heads, rank, rot, rot_off, window, scale, sink};
  const ZbVarlen b = {q_start, seq_lens, num_seqs};
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  return act_f32 ? launch_attend<float>(p, b, tokens, s) : launch_attend<__nv_bfloat16>(p, b, tokens, s);
}

int zb_latent_gather(const void* cache, long long ld_cache, const int32_t* block_table, int max_pages, int page_size,
                     const int32_t* key_start, const int32_t* first_key, int num_seqs, void* out, long long ld_out, int rows, int rank,
                     int rot, int rot_off, int rot_out, void* stream) {
  if (rows <= 0) return 0;
  if (ld_cache % 8 != 0 || ld_out % 8 != 0 || rot_off % 8 != 0 || rot_out % 8 != 0) return -70;
  const cudaError_t e = zb_launch(zb_latent_gather_kernel, dim3((rows + 7) / 8), dim3(256), 0, reinterpret_cast<cudaStream_t>(stream),
                                  reinterpret_cast<const __nv_bfloat16*>(cache), ld_cache, block_table, max_pages, page_size, key_start,
                                  first_key, num_seqs, reinterpret_cast<__nv_bfloat16*>(out), ld_out, rows, rank, rot, rot_off, rot_out);
  zb_count_launch(1);
  return static_cast<int>(e != cudaSuccess ? e : cudaGetLastError());
}

int zb_latent_q_pack(const void* q, long long ldq, void* out, const float* inv_freq, const int32_t* positions, int tokens, int heads,
                     int dim, int rot, int dim_p, int rot_p, void* stream) {
  if (tokens <= 0) return 0;
  if (dim % 8 != 0 || rot % 8 != 0 || dim_p % 8 != 0 || rot_p % 8 != 0 || ldq % 8 != 0 || rot > 4096) return -70;
  const cudaError_t e = zb_launch(zb_latent_q_pack_kernel, dim3(tokens), dim3(256), static_cast<size_t>(rot / 2) * sizeof(float2),
                                  reinterpret_cast<cudaStream_t>(stream), reinterpret_cast<const __nv_bfloat16*>(q), ldq,
                                  reinterpret_cast<__nv_bfloat16*>(out), inv_freq, positions, tokens, heads, dim, rot, dim_p, rot_p);
  zb_count_launch(1);
  return static_cast<int>(e != cudaSuccess ? e : cudaGetLastError());
}

}  // extern "C"
