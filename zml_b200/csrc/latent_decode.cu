// Decode of latent attention in the latent space (bf16, mma.sync): one query token per sequence, all heads share one key
// vector [c | rotated part] per cached token, whose first `rank` elements are the value as well.
//
// A CTA takes up to 16 * MT heads of one sequence and a chunk of its visible tokens.  A producer warp brings 32 cache
// rows at a time into a ring of padded shared-memory rows (one bulk copy per row, mbarrier completion); small tiles keep
// the ring deep enough for the copies to run without gaps.  Eight consumer warps compute
//   scores   warp (key group, K quarter): 16 keys x all heads over a quarter of the row, added by the softmax
//   softmax  fp32, rows spread over the 256 threads, running maximum and sum in registers
//   values   warp w owns 8 * NT latent columns of the output accumulator for all heads
// Every cache row is read once per group of heads.  A sequence's chunks leave partial results in scratch for a second
// launch to merge (with all SMs: a partial is as large as 57 cache rows).  Every wait is bounded.
#include "act.cuh"
#include "host_api.h"

namespace {
constexpr uint32_t kKernelId = 33;
constexpr int kKeys = 32;
constexpr int kConsumers = 256;
constexpr int kThreads = kConsumers + 32;
constexpr int kScoreLd = kKeys + 4;               // fp32 score rows
constexpr int kProbLd = kKeys + 8;                // bf16 probability rows: an odd number of 16-byte chunks
constexpr int kMaxStages = 6;
constexpr int kQuarters = 4;                      // K pieces of the score products
constexpr int kMaxSplits = 64;

struct DecodeParams {
  const __nv_bfloat16* q;       // [B, H, row]
  const __nv_bfloat16* cache;   // [pages * page_size, row]
  __nv_bfloat16* out;           // [B, H, ld_out]
  long long ld_out;
  const int32_t* block_table;
  const int32_t* seq_lens;
  float* part_o;                // [B, groups, splits, 16 * MT, rank_p]
  float* part_ml;               // [B, groups, splits, 16 * MT, 2]
  int max_pages, page_size, heads, row, rank_p, window, num_splits, stages;
  float scale_log2;
  const float* sink;            // [heads] or null: the first chunk of a sequence starts with it as its running maximum
  ZbStatus* status;
};

ZB_DEVICE void ldsm_x4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
ZB_DEVICE void ldsm_x4_t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
ZB_DEVICE void mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
ZB_DEVICE void consumer_sync() { asm volatile("bar.sync 1, 256;" ::: "memory"); }
// Barrier of the consumer warps that also tells all of them whether every one is still fine.
ZB_DEVICE bool consumer_sync_and(bool ok) {
  uint32_t r;
  asm volatile(
      "{\n\t.reg .pred p, q;\n\tsetp.ne.u32 p, %1, 0;\n\tbarrier.cta.red.and.pred q, 1, 256, p;\n\tselp.u32 %0, 1, 0, q;\n\t}\n"
      : "=r"(r) : "r"(ok ? 1u : 0u) : "memory");
  return r != 0u;
}

template <int MT, int NT>
__global__ void __launch_bounds__(kThreads, 1) zb_latent_decode_kernel(const DecodeParams p) {
  constexpr int kRows = 16 * MT;                  // heads of this CTA
  constexpr int kTpr = kConsumers / kRows;        // softmax threads per row
  constexpr int kKpt = kKeys / kTpr;              // keys per softmax thread
  extern __shared__ __align__(16) uint8_t smem[];
  const int row_bytes = p.row * 2, ld = row_bytes + 16;      // 16-byte chunks per padded row: odd, so ldmatrix has no conflicts
  uint8_t* q_s = smem;                                       // [kRows][ld]
  uint8_t* kv_s = q_s + kRows * ld;                          // [stages][kKeys][ld]
  float* s_s = reinterpret_cast<float*>(kv_s + p.stages * kKeys * ld);      // [kQuarters][kRows][kScoreLd]
  __nv_bfloat16* p_s = reinterpret_cast<__nv_bfloat16*>(s_s + kQuarters * kRows * kScoreLd);      // [kRows][kProbLd]
  float* corr_s = reinterpret_cast<float*>(p_s + kRows * kProbLd);          // [kRows]
  float* ml_s = corr_s + kRows;                              // [kRows][2]
  __shared__ uint64_t full_bar[kMaxStages], empty_bar[kMaxStages];
  __shared__ uint32_t abort_word;
  volatile uint32_t* abort_flag = &abort_word;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, tid = threadIdx.x;
  if (tid == 0) {
    for (int s = 0; s < p.stages; ++s) {
      zb_mbar_init(&full_bar[s], 1);
      zb_mbar_init(&empty_bar[s], 8);
    }
    abort_word = 0u;
    zb_mbar_fence_init();
  }
  __syncthreads();
  zb_pdl_launch();
  zb_pdl_wait();
  const int split = blockIdx.x, grp = blockIdx.y, seq = blockIdx.z;
  const int h0 = grp * kRows, nh = min(kRows, p.heads - h0);
  const int len = p.seq_lens[seq];
  const int first = p.window > 0 ? max(0, len - p.window) : 0;
  const int tile_lo = first / kKeys, tile_hi = (max(len, 0) + kKeys - 1) / kKeys;
  const int per = max(1, (tile_hi - tile_lo + p.num_splits - 1) / p.num_splits);
  const int my_splits = max(1, (tile_hi - tile_lo + per - 1) / per);
  if (split >= my_splits) return;
  const int tile0 = tile_lo + split * per, tile1 = min(tile_hi, tile0 + per);

  float acc[MT][NT][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < NT; ++n) acc[m][n][0] = acc[m][n][1] = acc[m][n][2] = acc[m][n][3] = 0.f;

  if (warp == 8) {
    // ------------------------------------------------------------------ producer: 32 rows per tile, one per lane
    const int32_t* bt = p.block_table + static_cast<long long>(seq) * p.max_pages;
    uint32_t stage = 0, phase = 0;
    for (int t = tile0; t < tile1; ++t) {
      const int key = min(t * kKeys + lane, len - 1);        // past the end: a visible row again, masked by the softmax
      int page = bt[key / p.page_size];
      if (!ZB_BC_OK(page, ZB_BC_PAGES, kKernelId, 1)) page = 0;
      const __nv_bfloat16* src = p.cache + (static_cast<long long>(page) * p.page_size + key % p.page_size) * p.row;
      if (t - tile0 >= p.stages) {
        const bool ok = zb_mbar_wait(&empty_bar[stage], phase ^ 1u, abort_flag);
        if (!__all_sync(0xffffffffu, ok)) break;
      }
      if (lane == 0) zb_mbar_expect_tx(&full_bar[stage], static_cast<uint32_t>(kKeys * row_bytes));
      __syncwarp();
      zb_bulk_load(kv_s + (stage * kKeys + lane) * ld, src, row_bytes, &full_bar[stage]);
      if (++stage == static_cast<uint32_t>(p.stages)) {
        stage = 0;
        phase ^= 1u;
      }
    }
  } else {
    // ------------------------------------------------------------------ consumers
    for (int i = tid; i < kRows * (p.row / 8); i += kConsumers) {
      const int r = i / (p.row / 8), c = i % (p.row / 8);
      uint4 v = make_uint4(0u, 0u, 0u, 0u);
      if (r < nh) v = *reinterpret_cast<const uint4*>(p.q + (static_cast<long long>(seq) * p.heads + h0 + r) * p.row + c * 8);
      *reinterpret_cast<uint4*>(q_s + r * ld + c * 16) = v;
    }
    consumer_sync();
    const int kgrp = warp & 1, kq = warp >> 1;
    const int steps = p.row / 16, quarter = (steps + kQuarters - 1) / kQuarters;
    const int st0 = kq * quarter, st1 = min(steps, st0 + quarter);
    const int srow = tid / kTpr, scol = (tid % kTpr) * kKpt;
    const int g = lane >> 2, tq = lane & 3;
    // lane's row and 16-byte half for the three kinds of ldmatrix tiles
    const uint32_t a_off = static_cast<uint32_t>((lane & 15) * ld + (lane >> 4) * 16);                               // 16 x 16, row-major A
    const uint32_t b_off = static_cast<uint32_t>((kgrp * 16 + ((lane >> 4) << 3) + (lane & 7)) * ld + ((lane >> 3) & 1) * 16);      // 16 keys x 16 of K
    const uint32_t v_off = static_cast<uint32_t>((lane & 15) * ld + (lane >> 4) * 16);                               // 16 keys x 16 columns, transposed
    const uint32_t p_off = static_cast<uint32_t>((lane & 15) * (kProbLd * 2) + (lane >> 4) * 16);
    const uint32_t qa = zb_smem_u32(q_s), ka = zb_smem_u32(kv_s), pa = zb_smem_u32(p_s);
    const int col0 = warp * 8 * NT;
    float m_run = -INFINITY, l_run = 0.f;
    if (p.sink != nullptr && split == 0 && srow < nh) {
      m_run = p.sink[h0 + srow] * 1.4426950408889634f;
      l_run = 1.f;
    }
    bool fine = true;
    uint32_t stage = 0, phase = 0;
    for (int t = tile0; t < tile1; ++t) {
      const bool here = zb_mbar_wait(&full_bar[stage], phase, abort_flag);
      const bool ok = __all_sync(0xffffffffu, here);
      const uint32_t tile = ka + stage * kKeys * ld;
      float sc[MT][2][4];
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int n = 0; n < 2; ++n) sc[m][n][0] = sc[m][n][1] = sc[m][n][2] = sc[m][n][3] = 0.f;
      if (ok) {
#pragma unroll 3
        for (int s = st0; s < st1; ++s) {
          uint32_t b[4];
          ldsm_x4(b, tile + b_off + s * 32);
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            uint32_t a[4];
            ldsm_x4(a, qa + a_off + m * 16 * ld + s * 32);
            mma(sc[m][0], a, b[0], b[1]);
            mma(sc[m][1], a, b[2], b[3]);
          }
        }
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
          for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int e = 0; e < 2; ++e)
              *reinterpret_cast<float2*>(s_s + (kq * kRows + m * 16 + g + 8 * e) * kScoreLd + kgrp * 16 + n * 8 + 2 * tq) =
                  make_float2(sc[m][n][2 * e], sc[m][n][2 * e + 1]);
      }
      if (!consumer_sync_and(ok)) {
        fine = false;
        break;
      }
      {
        const float* r0 = s_s + srow * kScoreLd + scol;
        const int key0 = t * kKeys + scol;
        float v[kKpt], mx = m_run;
#pragma unroll
        for (int i = 0; i < kKpt; ++i) {
          v[i] = ((r0[i] + r0[i + kRows * kScoreLd]) + (r0[i + 2 * kRows * kScoreLd] + r0[i + 3 * kRows * kScoreLd])) * p.scale_log2;
          if (key0 + i < first || key0 + i >= len) v[i] = -INFINITY;
          mx = fmaxf(mx, v[i]);
        }
#pragma unroll
        for (int o = kTpr / 2; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
        const float use = mx == -INFINITY ? 0.f : mx;
        const float corr = m_run == -INFINITY ? 0.f : zb_ex2(m_run - use);
        m_run = mx;
        float sum = 0.f;
        __nv_bfloat16* pr = p_s + srow * kProbLd + scol;
#pragma unroll
        for (int i = 0; i < kKpt; i += 2) {
          const float a = zb_ex2(v[i] - use), b = zb_ex2(v[i + 1] - use);
          sum += a + b;
          *reinterpret_cast<uint32_t*>(pr + i) = zb_pack_bf16x2(a, b);
        }
#pragma unroll
        for (int o = kTpr / 2; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
        l_run = l_run * corr + sum;
        if (tid % kTpr == 0) corr_s[srow] = corr;
      }
      consumer_sync();
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        const float c0 = corr_s[m * 16 + g], c1 = corr_s[m * 16 + g + 8];
#pragma unroll
        for (int n = 0; n < NT; ++n) {
          acc[m][n][0] *= c0;
          acc[m][n][1] *= c0;
          acc[m][n][2] *= c1;
          acc[m][n][3] *= c1;
        }
      }
#pragma unroll
      for (int s = 0; s < kKeys / 16; ++s) {
        uint32_t a[MT][4];
#pragma unroll
        for (int m = 0; m < MT; ++m) ldsm_x4(a[m], pa + p_off + m * 16 * (kProbLd * 2) + s * 32);
#pragma unroll
        for (int n = 0; n < NT; n += 2) {
          if (col0 + n * 8 >= p.rank_p) continue;            // uniform over the warp; rank_p is a multiple of 16
          uint32_t b[4];
          ldsm_x4_t(b, tile + v_off + s * 16 * ld + (col0 + n * 8) * 2);
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            mma(acc[m][n], a[m], b[0], b[1]);
            mma(acc[m][n + 1], a[m], b[2], b[3]);
          }
        }
      }
      __syncwarp();
      if (lane == 0) zb_mbar_arrive(&empty_bar[stage]);
      if (++stage == static_cast<uint32_t>(p.stages)) {
        stage = 0;
        phase ^= 1u;
      }
    }
    if (tid % kTpr == 0) {
      ml_s[srow * 2] = m_run;
      ml_s[srow * 2 + 1] = l_run;
    }
    if (!fine && tid == 0) zb_record_error(p.status, ZB_ERR_MBAR_TIMEOUT, kKernelId, 1u, blockIdx.z);
    consumer_sync();
    // ------------------------------------------------------------------ result of this chunk
    const long long cell = (static_cast<long long>(seq) * gridDim.y + grp) * p.num_splits + split;
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int r = m * 16 + g + 8 * e;
        if (r >= nh) continue;
        const float l = ml_s[r * 2 + 1], inv = l > 0.f ? 1.f / l : 0.f;
#pragma unroll
        for (int n = 0; n < NT; ++n) {
          const int c = col0 + n * 8 + 2 * tq;
          if (c >= p.rank_p) continue;
          if (my_splits == 1)
            *reinterpret_cast<uint32_t*>(p.out + (static_cast<long long>(seq) * p.heads + h0 + r) * p.ld_out + c) =
                zb_pack_bf16x2(acc[m][n][2 * e] * inv, acc[m][n][2 * e + 1] * inv);
          else
            *reinterpret_cast<float2*>(p.part_o + (cell * kRows + r) * p.rank_p + c) = make_float2(acc[m][n][2 * e], acc[m][n][2 * e + 1]);
        }
      }
    if (my_splits > 1 && tid < kRows) {
      p.part_ml[(cell * kRows + tid) * 2] = ml_s[tid * 2];
      p.part_ml[(cell * kRows + tid) * 2 + 1] = ml_s[tid * 2 + 1];
    }
  }

  if (*abort_flag != 0u) {                                   // copies still in flight must land before the shared memory is reused
    const uint64_t t0 = zb_globaltimer();
    while (zb_globaltimer() - t0 < 200000ull) {
    }
  }
}

// Merges the chunks of a sequence: one CTA per (head, sequence).
template <int ROWS>
__global__ void __launch_bounds__(128) zb_latent_merge_kernel(const DecodeParams p) {
  zb_pdl_launch();
  zb_pdl_wait();
  __shared__ float f_s[kMaxSplits];
  __shared__ float inv_s;
  const int seq = blockIdx.y, head = blockIdx.x, r = head % ROWS;
  const int len = p.seq_lens[seq];
  const int first = p.window > 0 ? max(0, len - p.window) : 0;
  const int tiles = (max(len, 0) + kKeys - 1) / kKeys - first / kKeys;
  const int per = max(1, (tiles + p.num_splits - 1) / p.num_splits);
  const int n = max(1, (tiles + per - 1) / per);
  if (n == 1) return;                                        // written by the chunk itself
  const long long base = (static_cast<long long>(seq) * ((p.heads + ROWS - 1) / ROWS) + head / ROWS) * p.num_splits;
  if (threadIdx.x < 32) {
    float m[kMaxSplits / 32], l[kMaxSplits / 32], mm = -INFINITY, ll = 0.f;
#pragma unroll
    for (int i = 0; i < kMaxSplits / 32; ++i) {
      const int s = threadIdx.x + 32 * i;
      m[i] = s < n ? p.part_ml[((base + s) * ROWS + r) * 2] : -INFINITY;
      l[i] = s < n ? p.part_ml[((base + s) * ROWS + r) * 2 + 1] : 0.f;
      mm = fmaxf(mm, m[i]);
    }
    mm = zb_warp_max(mm);
    const float use = mm == -INFINITY ? 0.f : mm;
#pragma unroll
    for (int i = 0; i < kMaxSplits / 32; ++i) {
      const float f = exp2f(m[i] - use);
      f_s[threadIdx.x + 32 * i] = f;
      ll += f * l[i];
    }
    ll = zb_warp_sum(ll);
    if (threadIdx.x == 0) inv_s = ll > 0.f ? 1.f / ll : 0.f;
  }
  __syncthreads();
  const float inv = inv_s;
  for (int c = threadIdx.x * 4; c < p.rank_p; c += 512) {
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
    for (int s = 0; s < n; ++s) {
      const float4 v = *reinterpret_cast<const float4*>(p.part_o + ((base + s) * ROWS + r) * p.rank_p + c);
      const float f = f_s[s];
      o.x = fmaf(f, v.x, o.x);
      o.y = fmaf(f, v.y, o.y);
      o.z = fmaf(f, v.z, o.z);
      o.w = fmaf(f, v.w, o.w);
    }
    *reinterpret_cast<uint2*>(p.out + (static_cast<long long>(seq) * p.heads + head) * p.ld_out + c) =
        make_uint2(zb_pack_bf16x2(o.x * inv, o.y * inv), zb_pack_bf16x2(o.z * inv, o.w * inv));
  }
}

constexpr int kMaxSmem = 232448 - 1024;           // static shared memory and the reserved kilobyte stay outside

int smem_bytes(int rows, int row, int stages) {
  const int ld = row * 2 + 16;
  return rows * ld + stages * kKeys * ld + kQuarters * rows * kScoreLd * 4 + rows * kProbLd * 2 + rows * 4 + rows * 8;
}
int pick_stages(int rows, int row) {
  for (int s = kMaxStages; s >= 2; --s)
    if (smem_bytes(rows, row, s) <= kMaxSmem) return s;
  return 0;
}
int rows_for(int heads) { return heads <= 16 ? 16 : 32; }

template <int MT, int NT>
int launch(const DecodeParams& p, int batch, int groups, cudaStream_t s) {
  static bool configured[16] = {};
  if (const int rc = zb_config_smem_once(zb_latent_decode_kernel<MT, NT>, kMaxSmem, configured)) return rc;
  const cudaError_t e = zb_launch(zb_latent_decode_kernel<MT, NT>, dim3(p.num_splits, groups, batch), dim3(kThreads),
                                  smem_bytes(16 * MT, p.row, p.stages), s, p);
  zb_count_launch(1);
  if (e != cudaSuccess || p.num_splits == 1) return static_cast<int>(e != cudaSuccess ? e : cudaGetLastError());
  const cudaError_t m = zb_launch(zb_latent_merge_kernel<16 * MT>, dim3(p.heads, batch), dim3(128), 0, s, p);
  zb_count_launch(1);
  return static_cast<int>(m != cudaSuccess ? m : cudaGetLastError());
}
}  // namespace

extern "C" {

// 1 when the kernel takes the sizes (rank_p and row: multiples of 16, at most 512 latent columns).
int zb_latent_decode_supported(int row, int rank_p) {
  return row % 16 == 0 && rank_p % 16 == 0 && rank_p > 0 && rank_p <= 512 && rank_p <= row && pick_stages(32, row) >= 2 ? 1 : 0;
}

// Head groups (CTAs) a sequence is cut into, besides its chunks of tokens.
int zb_latent_decode_groups(int heads) { return (heads + rows_for(heads) - 1) / rows_for(heads); }

int zb_latent_decode(const void* q, const void* cache, int row, void* out, long long ld_out, const int32_t* block_table, int max_pages,
                     int page_size, const int32_t* seq_lens, int batch, int heads, int rank_p, int window, float scale, const float* sink,
                     int num_splits, void* stream) {
  if (batch <= 0) return 0;
  if (!zb_latent_decode_supported(row, rank_p) || ld_out % 4 != 0) return -32;
  ZbDeviceState* st = zb_device_state();
  if (!st) return -20;
  const int rows = rows_for(heads), groups = zb_latent_decode_groups(heads);
  if (num_splits < 1) num_splits = 1;
  if (num_splits > kMaxSplits) num_splits = kMaxSplits;
  const size_t cells = static_cast<size_t>(batch) * groups;
  const size_t per_split = cells * rows * (static_cast<size_t>(rank_p) + 2) * sizeof(float);
  while (num_splits > 1 && per_split * num_splits > st->attn_scratch_bytes) --num_splits;
  DecodeParams p = {};
  p.q = reinterpret_cast<const __nv_bfloat16*>(q);
  p.cache = reinterpret_cast<const __nv_bfloat16*>(cache);
  p.out = reinterpret_cast<__nv_bfloat16*>(out);
  p.ld_out = ld_out;
  p.block_table = block_table;
  p.seq_lens = seq_lens;
  p.part_o = st->attn_scratch;
  p.part_ml = st->attn_scratch + cells * num_splits * rows * rank_p;
  p.max_pages = max_pages;
  p.page_size = page_size;
  p.heads = heads;
  p.row = row;
  p.rank_p = rank_p;
  p.window = window;
  p.num_splits = num_splits;
  p.stages = pick_stages(rows, row);
  p.scale_log2 = scale * 1.4426950408889634f;
  p.sink = sink;
  p.status = st->status;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const int nt = rank_p <= 128 ? 2 : (rank_p <= 256 ? 4 : 8);
  switch ((rows == 16 ? 0 : 3) + (nt == 2 ? 0 : (nt == 4 ? 1 : 2))) {
    case 0: return launch<1, 2>(p, batch, groups, s);
    case 1: return launch<1, 4>(p, batch, groups, s);
    case 2: return launch<1, 8>(p, batch, groups, s);
    case 3: return launch<2, 2>(p, batch, groups, s);
    case 4: return launch<2, 4>(p, batch, groups, s);
    default: return launch<2, 8>(p, batch, groups, s);
  }
}

}  // extern "C"
