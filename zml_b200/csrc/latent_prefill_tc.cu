// Prefill of latent attention on the 5th-generation tensor cores (tcgen05 / TMEM / TMA): varlen, causal, windowed, every
// head with its own keys and values, query / key vectors made of an unrotated part per head and a rotated key part that
// all heads share.
//
// The operands are contiguous: the visible latents of the batch have been gathered and projected, so a key row of
// head h is [kv[row, h * dim ...] | shared[row, rot_out ...]] and a value row kv[row, H * dim + h * vdim ...].  Tiles are
// made of 64-column sub-tiles; where dim, rot or vdim is not a multiple of 64 a sub-tile reaches into the neighbouring
// columns, which the zero padding of the packed queries (scores) or the store (outputs) drops.
//
// One CTA works on 256 query rows of one head as two softmax pipelines of 128 rows that share every K / V tile:
//   warps 0-3 / 4-7 : softmax and epilogue of rows 0-127 / 128-255 (one thread per query row)
//   warp  8         : TMA producer (Q once, then K and V of one 64-key tile per step through a ring)
//   warp  9         : MMA issuer (one thread)
// Each pipeline only touches the tiles between its own window edge and diagonal.  S, P and O live in tensor memory:
// S_0 0-63 | S_1 64-127 | P_0 128-159 | P_1 160-191 | O_0 192.. | O_1 behind it.  The structure of a step (scores -> running
// maximum -> lazy rescale of O -> P back into tensor memory -> O += P V) is that of attention_tc.cu.  A sink is the running
// maximum, with a running sum of 1, in front of the first tile.  The epilogue normalises and applies the sigmoid output gate
// (either may be absent).  Every wait is bounded.
#include <cuda.h>

#include "act.cuh"
#include "host_api.h"

int zb_make_tmap_bf16_2d(CUtensorMap* out, const void* base, int rows, int k, int ld, int box_rows);

namespace {

constexpr int kQRows = 128;
constexpr int kKeys = 64;
constexpr int kThreads = 320;
constexpr uint32_t kKernelId = 32;
constexpr uint32_t kTmemCols = 512;
constexpr uint32_t kColS = 0, kColP = 128, kColO = 192;
constexpr int kQSub = kQRows * 128;              // one 64-column sub-tile of 128 query rows
constexpr int kKvSub = kKeys * 128;              // one 64-column sub-tile of 64 keys

struct LatentPrefillParams {
  __nv_bfloat16* out;           // [T, ld_out]
  const __nv_bfloat16* gate;    // [T, ld_gate] or null
  long long ld_out, ld_gate;
  ZbVarlen b;
  const int32_t* key_start;     // [num_seqs + 1] first gathered row of every sequence
  const int32_t* first_key;     // [num_seqs] position of that row's token
  int heads, dim, vdim;
  int nn;                       // sub-tiles of the unrotated part; the others are the shared part
  int rot_out;                  // its first column in the gathered rows
  int window;
  float scale_log2;
  const float* sink;            // [heads] or null
  ZbStatus* status;
};

template <int NQ, int NV, int STAGES>
__global__ void __launch_bounds__(kThreads, 1)
zb_latent_prefill_tc_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_kv,
                            const __grid_constant__ CUtensorMap tmap_shared, const LatentPrefillParams p) {
  zb_pdl_wait();
  constexpr int kQBytes = NQ * kQSub;
  constexpr int kKBytes = NQ * kKvSub, kVBytes = NV * kKvSub;
  constexpr int kOCols = NV * 64;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  uint8_t* q_s = smem;                               // [2][NQ sub-tiles]
  uint8_t* k_s = q_s + 2 * kQBytes;                  // [STAGES][NQ sub-tiles]
  uint8_t* v_s = k_s + STAGES * kKBytes;             // [STAGES][NV sub-tiles]
  uint64_t* bars = reinterpret_cast<uint64_t*>(v_s + STAGES * kVBytes);
  uint64_t* q_full = bars;
  uint64_t* k_full = bars + 1;
  uint64_t* v_full = k_full + STAGES;
  uint64_t* kv_empty = v_full + STAGES;
  uint64_t* s_full = kv_empty + STAGES;              // 2
  uint64_t* p_full = s_full + 2;                     // 2 (128 arrivals)
  uint64_t* o_ready = p_full + 2;                    // 2
  uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(o_ready + 2);
  volatile uint32_t* abort_flag = tmem_holder + 1;
  volatile uint32_t* abort_where = tmem_holder + 2;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int head = blockIdx.y;
  int seq, qb;
  // blocks are handed out from the end of the batch backwards: long (late) blocks of a sequence first
  if (!zb_find_block(p.b, 2 * kQRows, static_cast<int>(gridDim.x) - 1 - static_cast<int>(blockIdx.x), seq, qb)) return;
  const int q_len = p.b.q_start[seq + 1] - p.b.q_start[seq];
  const int first = p.first_key[seq];
  const int row0 = p.key_start[seq];
  const int len = p.b.seq_lens[seq] - first;         // keys and positions below are relative to the first gathered one
  const int ctx = len - q_len;
  const int row_base = qb * 2 * kQRows;
  const int tok_base = p.b.q_start[seq] + row_base;
  const int rows_valid = min(2 * kQRows, q_len - row_base);
  const int n_pipe = rows_valid > kQRows ? 2 : 1;
  int t_begin[2], t_end[2];                          // tiles of each pipeline
#pragma unroll
  for (int w = 0; w < 2; ++w) {
    const int base = ctx + row_base + w * kQRows;
    t_begin[w] = p.window > 0 ? max(0, base - p.window + 1) / kKeys : 0;
    t_end[w] = (min(len, base + kQRows) + kKeys - 1) / kKeys;
  }
  const int tile0 = t_begin[0], tile1 = t_end[n_pipe - 1];

  if (threadIdx.x == 0) {
    zb_mbar_init(q_full, 1);
    for (int s = 0; s < STAGES; ++s) {
      zb_mbar_init(&k_full[s], 1);
      zb_mbar_init(&v_full[s], 1);
      zb_mbar_init(&kv_empty[s], 1);
    }
    for (int w = 0; w < 2; ++w) {
      zb_mbar_init(&s_full[w], 1);
      zb_mbar_init(&p_full[w], 128);
      zb_mbar_init(&o_ready[w], 1);
    }
    *abort_flag = 0u;
    *abort_where = 0u;
    zb_mbar_fence_init();
    zb_tma_prefetch_desc(&tmap_q);
    zb_tma_prefetch_desc(&tmap_kv);
    zb_tma_prefetch_desc(&tmap_shared);
  }
  if (warp == 9) {
    zb_tmem_alloc(tmem_holder, kTmemCols);
    zb_tmem_relinquish();
  }
  zb_tc_fence_before();
  __syncthreads();
  zb_tc_fence_after();
  const uint32_t tmem_base = *tmem_holder;
  zb_pdl_launch();       // only now: a dependent CTA that allocated its tensor memory first would block this one for good

  if (warp == 8) {
    // ------------------------------------------------------------------ TMA producer
    if (lane == 0) {
      zb_mbar_expect_tx(q_full, n_pipe * kQBytes);
      for (int w = 0; w < n_pipe; ++w)
        for (int c = 0; c < NQ; ++c)
          zb_tma_load_2d(q_s + w * kQBytes + c * kQSub, &tmap_q, q_full, (head * NQ + c) * 64, tok_base + w * kQRows);
      uint32_t stage = 0, phase = 0;
      for (int j = tile0; j < tile1; ++j) {
        if (j - tile0 >= STAGES) {
          if (!zb_mbar_wait(&kv_empty[stage], phase ^ 1u, abort_flag)) {
            *abort_where = 1u;
            break;
          }
        }
        const int row = row0 + j * kKeys;
        zb_mbar_expect_tx(&k_full[stage], kKBytes);
        for (int c = 0; c < NQ; ++c) {
          uint8_t* dst = k_s + stage * kKBytes + c * kKvSub;
          if (c < p.nn) zb_tma_load_2d(dst, &tmap_kv, &k_full[stage], head * p.dim + c * 64, row);
          else zb_tma_load_2d(dst, &tmap_shared, &k_full[stage], p.rot_out + (c - p.nn) * 64, row);
        }
        zb_mbar_expect_tx(&v_full[stage], kVBytes);
        for (int c = 0; c < NV; ++c)
          zb_tma_load_2d(v_s + stage * kVBytes + c * kKvSub, &tmap_kv, &v_full[stage], p.heads * p.dim + head * p.vdim + c * 64, row);
        if (++stage == STAGES) {
          stage = 0;
          phase ^= 1u;
        }
      }
    }
  } else if (warp == 9) {
    // ------------------------------------------------------------------ MMA issuer
    if (lane == 0) {
      constexpr uint32_t kIdescS = zb_make_idesc_bf16(kQRows, kKeys);
      constexpr uint32_t kIdescO = zb_make_idesc_bf16(kQRows, kOCols) | (1u << 16);    // B (= V) is MN-major
      bool ok = zb_mbar_wait(q_full, 0u, abort_flag);
      if (!ok) *abort_where = 2u;
      auto mma_s = [&](int w, uint32_t st) {
        const uint32_t qa = zb_smem_u32(q_s + w * kQBytes), ka = zb_smem_u32(k_s + st * kKBytes);
#pragma unroll
        for (int c = 0; c < NQ; ++c) {
          const uint64_t dq = zb_make_desc_sw128(qa + c * kQSub), dk = zb_make_desc_sw128(ka + c * kKvSub);
#pragma unroll
          for (int kk = 0; kk < 4; ++kk)
            zb_umma_f16(tmem_base + kColS + w * kKeys, dq + 2 * kk, dk + 2 * kk, kIdescS, (c > 0 || kk > 0) ? 1u : 0u);
        }
        zb_umma_commit(&s_full[w]);
      };
      uint32_t stage = 0, phase = 0;
      if (ok && tile0 < tile1) {
        ok = zb_mbar_wait(&k_full[0], 0u, abort_flag);
        if (!ok) *abort_where = 3u;
        if (ok) {
          zb_tc_fence_after();
          for (int w = 0; w < n_pipe; ++w)
            if (t_begin[w] == tile0) mma_s(w, 0);
        }
      }
      uint32_t done[2] = {0u, 0u};
      for (int j = tile0; ok && j < tile1; ++j) {
        uint32_t nstage = stage + 1, nphase = phase;
        if (nstage == STAGES) {
          nstage = 0;
          nphase ^= 1u;
        }
        if (!zb_mbar_wait(&v_full[stage], phase, abort_flag)) {
          *abort_where = 4u;
          break;
        }
        bool k_next = false;
        for (int w = 0; w < n_pipe && ok; ++w) {
          if (j >= t_begin[w] && j < t_end[w]) {
            if (!zb_mbar_wait(&p_full[w], done[w] & 1u, abort_flag)) {
              *abort_where = 5u + w;
              ok = false;
              break;
            }
            zb_tc_fence_after();
            const uint32_t va = zb_smem_u32(v_s + stage * kVBytes);
#pragma unroll
            for (int k = 0; k < 4; ++k) {
              const uint64_t dv = zb_make_desc_sw128_mn(va + k * (16 * 128), kKvSub, 1024u);
              zb_umma_f16_ts(tmem_base + kColO + w * kOCols, tmem_base + kColP + w * 32 + 8 * k, dv, kIdescO, (done[w] > 0u || k > 0) ? 1u : 0u);
            }
            zb_umma_commit(&o_ready[w]);
            ++done[w];
          }
          if (j + 1 >= t_begin[w] && j + 1 < t_end[w]) {
            if (!k_next) {
              if (!zb_mbar_wait(&k_full[nstage], nphase, abort_flag)) {
                *abort_where = 7u;
                ok = false;
                break;
              }
              zb_tc_fence_after();
              k_next = true;
            }
            mma_s(w, nstage);                        // the softmax warps of w have read S_w (they published P_w)
          }
        }
        if (!ok) break;
        zb_umma_commit(&kv_empty[stage]);
        stage = nstage;
        phase = nphase;
      }
    }
  } else if ((warp >> 2) < n_pipe) {
    // ------------------------------------------------------------------ softmax + epilogue (one row per thread)
    const int w = warp >> 2;
    const int quad = warp & 3;
    const int r = quad * 32 + lane;
    const int base = ctx + row_base + w * kQRows;    // position of this pipeline's first row
    const int qpos = base + r;
    const uint32_t lane_off = static_cast<uint32_t>(quad * 32) << 16;
    const uint32_t t_s = tmem_base + kColS + w * kKeys + lane_off;
    const uint32_t t_p = tmem_base + kColP + w * 32 + lane_off;
    const uint32_t t_o = tmem_base + kColO + w * kOCols + lane_off;
    const int jb = t_begin[w], je = t_end[w];
    float m = p.sink != nullptr ? p.sink[head] * 1.4426950408889634f : -INFINITY, l = p.sink != nullptr ? 1.f : 0.f;
    bool ok = true;
    for (int j = jb; j < je; ++j) {
      const uint32_t jj = static_cast<uint32_t>(j - jb);
      if (!zb_mbar_wait(&s_full[w], jj & 1u, abort_flag)) {
        *abort_where = 10u + w;
        ok = false;
        break;
      }
      zb_tc_fence_after();
      uint32_t sr[64];
      zb_tmem_ld32(t_s, reinterpret_cast<uint32_t(&)[32]>(sr[0]));
      zb_tmem_ld32(t_s + 32, reinterpret_cast<uint32_t(&)[32]>(sr[32]));
      zb_tmem_ld_wait();
      const int key0 = j * kKeys;
      const bool full = (key0 + kKeys - 1 <= base) && (key0 + kKeys <= len) && (p.window <= 0 || key0 > base + kQRows - 1 - p.window);
      float mx_raw = -INFINITY;
      if (full) {
#pragma unroll
        for (int i = 0; i < 64; ++i) mx_raw = fmaxf(mx_raw, __uint_as_float(sr[i]));
      } else {
        const int hi = min(qpos, len - 1) - key0, lo = p.window > 0 ? qpos - p.window - key0 : -1;     // visible: lo < i <= hi
#pragma unroll
        for (int i = 0; i < 64; ++i) {
          if (i > hi || i <= lo) sr[i] = 0xff800000u;
          mx_raw = fmaxf(mx_raw, __uint_as_float(sr[i]));
        }
      }
      const float mx = fmaxf(m, mx_raw * p.scale_log2);
      const float m_use = mx == -INFINITY ? 0.f : mx;
      {
        const float alpha = m == -INFINITY ? 1.f : zb_ex2(m - m_use);
        const bool moved = alpha != 1.f;
        if (jj > 0 && __any_sync(0xffffffffu, moved)) {
          if (!zb_mbar_wait(&o_ready[w], (jj - 1u) & 1u, abort_flag)) {
            *abort_where = 12u + w;
            ok = false;
            break;
          }
          zb_tc_fence_after();
#pragma unroll 1
          for (int c0 = 0; c0 < kOCols; c0 += 32) {
            uint32_t o[32];
            zb_tmem_ld32(t_o + c0, o);
            zb_tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * alpha);
            zb_tmem_st16(t_o + c0, o);
            zb_tmem_st16(t_o + c0 + 16, o + 16);
          }
          zb_tmem_st_wait();
        }
        l *= alpha;
      }
      m = mx;
      const float neg_m = -m_use;
      uint32_t pw[32];
      float sum0 = 0.f, sum1 = 0.f;
#pragma unroll
      for (int i = 0; i < 32; ++i) {
        const float p0 = zb_ex2(fmaf(__uint_as_float(sr[2 * i]), p.scale_log2, neg_m));
        const float p1 = zb_ex2(fmaf(__uint_as_float(sr[2 * i + 1]), p.scale_log2, neg_m));
        pw[i] = zb_pack_bf16x2(p0, p1);
        sum0 += p0;
        sum1 += p1;
      }
      l += sum0 + sum1;
      zb_tmem_st16(t_p, pw);
      zb_tmem_st16(t_p + 16, pw + 16);
      zb_tmem_st_wait();
      zb_tc_fence_before();
      zb_mbar_arrive(&p_full[w]);
    }
    if (ok && jb < je) {
      const uint32_t last = static_cast<uint32_t>(je - 1 - jb);
      if (zb_mbar_wait(&o_ready[w], last & 1u, abort_flag)) {
        zb_tc_fence_after();
        const float inv = l > 0.f ? 1.f / l : 0.f;
        const int row = w * kQRows + r;
        const long long t = tok_base + row;
        __nv_bfloat16* orow = p.out + t * p.ld_out + static_cast<long long>(head) * p.vdim;
        const __nv_bfloat16* grow = p.gate != nullptr ? p.gate + t * p.ld_gate + static_cast<long long>(head) * p.vdim : nullptr;
#pragma unroll 1
        for (int c0 = 0; c0 < kOCols; c0 += 32) {
          uint32_t o[32];
          zb_tmem_ld32(t_o + c0, o);
          zb_tmem_ld_wait();
          if (row >= rows_valid) continue;
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const int c = c0 + 8 * i;
            if (c >= p.vdim) continue;
            uint32_t wd[4];
            if (grow == nullptr) {
#pragma unroll
              for (int q = 0; q < 4; ++q)
                wd[q] = zb_pack_bf16x2(__uint_as_float(o[8 * i + 2 * q]) * inv, __uint_as_float(o[8 * i + 2 * q + 1]) * inv);
            } else {
              const uint4 gv = *reinterpret_cast<const uint4*>(grow + c);
              const uint32_t gu[4] = {gv.x, gv.y, gv.z, gv.w};
#pragma unroll
              for (int q = 0; q < 4; ++q) {
                const float2 g = zb_unpack_bf16x2(gu[q]);
                wd[q] = zb_pack_bf16x2(__uint_as_float(o[8 * i + 2 * q]) * inv / (1.f + __expf(-g.x)),
                                       __uint_as_float(o[8 * i + 2 * q + 1]) * inv / (1.f + __expf(-g.y)));
              }
            }
            *reinterpret_cast<uint4*>(orow + c) = make_uint4(wd[0], wd[1], wd[2], wd[3]);
          }
        }
      } else {
        *abort_where = 14u + w;
      }
    }
  }

  // ------------------------------------------------------------------ common exit
  zb_tc_fence_before();
  __syncthreads();
  if (*abort_flag != 0u) {
    if (threadIdx.x == 0) zb_record_error(p.status, ZB_ERR_MBAR_TIMEOUT, kKernelId, *abort_where, blockIdx.x);
    const uint64_t t0 = zb_globaltimer();            // copies still in flight must land before the shared memory is reused
    while (zb_globaltimer() - t0 < 200000ull) {
    }
    __syncthreads();
  }
  if (warp == 9) {
    zb_tc_fence_after();
    zb_tmem_dealloc(tmem_base, kTmemCols);
  }
}

template <int NQ, int NV, int STAGES>
int launch(const CUtensorMap& tq, const CUtensorMap& tkv, const CUtensorMap& ts, const LatentPrefillParams& p, int blocks, cudaStream_t s) {
  constexpr int kSmem = 2 * NQ * kQSub + STAGES * (NQ + NV) * kKvSub + 1024 + 256;
  static_assert(kSmem <= 232448, "shared memory");
  static bool configured[16] = {};
  if (const int rc = zb_config_smem_once(zb_latent_prefill_tc_kernel<NQ, NV, STAGES>, kSmem, configured)) return rc;
  const cudaError_t e = zb_launch(zb_latent_prefill_tc_kernel<NQ, NV, STAGES>, dim3(blocks, p.heads), dim3(kThreads), kSmem, s, tq, tkv, ts, p);
  zb_count_launch(1);
  return static_cast<int>(e != cudaSuccess ? e : cudaGetLastError());
}

}  // namespace

extern "C" {

// 1 when the kernel takes the sizes: parts in multiples of 8 (16-byte copies), at most 256 padded query columns and 128
// value columns.
int zb_latent_prefill_tc_supported(int dim, int rot, int vdim, int rank) {
  if (dim % 8 != 0 || rot % 8 != 0 || vdim % 8 != 0 || rank % 8 != 0 || dim <= 0 || vdim <= 0 || vdim > 128) return 0;
  const int nq = (dim + 63) / 64 + (rot + 63) / 64;
  return nq >= 1 && nq <= 4;
}

// q [T, H, 64 * nq] packed (zb_latent_q_pack), kv [rows, ld_kv] with H * dim + H * vdim columns, shared [rows, ld_shared]
// with the rotated key part at column rot_out (zero-padded to 64); blocks >= sum over sequences of ceil(tokens / 256).
int zb_latent_prefill_tc(const void* q, const void* kv, long long ld_kv, const void* shared, long long ld_shared, int rot_out, void* out,
                         long long ld_out, const void* gate, long long ld_gate, const int32_t* q_start, const int32_t* seq_lens,
                         int num_seqs, const int32_t* key_start, const int32_t* first_key, int tokens, int rows, int blocks, int heads,
                         int dim, int rot, int vdim, int window, float scale, const float* sink, void* stream) {
  if (tokens <= 0 || blocks <= 0) return 0;
  if (!zb_latent_prefill_tc_supported(dim, rot, vdim, 8)) return -32;
  if (ld_kv % 8 != 0 || ld_shared % 8 != 0 || ld_out % 8 != 0 || ld_gate % 8 != 0 || rot_out % 8 != 0 ||
      (reinterpret_cast<uintptr_t>(gate) & 15) != 0 || (reinterpret_cast<uintptr_t>(out) & 15) != 0)
    return -33;
  ZbDeviceState* st = zb_device_state();
  if (!st) return -20;
  LatentPrefillParams p = {};
  p.nn = (dim + 63) / 64;
  const int nq = p.nn + (rot + 63) / 64, nv = (vdim + 63) / 64;
  CUtensorMap tq, tkv, ts;
  int rc = zb_make_tmap_bf16_2d(&tq, q, tokens, heads * nq * 64, heads * nq * 64, kQRows);
  if (rc != 0) return rc;
  rc = zb_make_tmap_bf16_2d(&tkv, kv, rows, heads * (dim + vdim), static_cast<int>(ld_kv), kKeys);
  if (rc != 0) return rc;
  rc = zb_make_tmap_bf16_2d(&ts, shared, rows, static_cast<int>(ld_shared), static_cast<int>(ld_shared), kKeys);
  if (rc != 0) return rc;
  p.out = reinterpret_cast<__nv_bfloat16*>(out);
  p.gate = reinterpret_cast<const __nv_bfloat16*>(gate);
  p.ld_out = ld_out;
  p.ld_gate = ld_gate;
  p.b = ZbVarlen{q_start, seq_lens, num_seqs};
  p.key_start = key_start;
  p.first_key = first_key;
  p.heads = heads;
  p.dim = dim;
  p.vdim = vdim;
  p.rot_out = rot_out;
  p.window = window;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.sink = sink;
  p.status = st->status;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  switch (nq * 2 + nv) {
    case 3: return launch<1, 1, 4>(tq, tkv, ts, p, blocks, s);
    case 4: return launch<1, 2, 4>(tq, tkv, ts, p, blocks, s);
    case 5: return launch<2, 1, 3>(tq, tkv, ts, p, blocks, s);
    case 6: return launch<2, 2, 3>(tq, tkv, ts, p, blocks, s);
    case 7: return launch<3, 1, 3>(tq, tkv, ts, p, blocks, s);
    case 8: return launch<3, 2, 3>(tq, tkv, ts, p, blocks, s);
    case 9: return launch<4, 1, 2>(tq, tkv, ts, p, blocks, s);
    case 10: return launch<4, 2, 2>(tq, tkv, ts, p, blocks, s);
  }
  return -32;
}

}  // extern "C"
