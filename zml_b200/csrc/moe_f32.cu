// fp32 grouped GEMM over the experts on the FMA pipes, with the token gather in its loads and the gate in its epilogue: the
// counterpart of the bf16 grouped GEMM of moe.cu for models that run in fp32.
//
//   out[rows of expert e, :] = x[source of the row, :K] * w[e][N, K]^T,  or the gated unit of interleaved gate / up rows
#include "act.cuh"
#include "host_api.h"

namespace {
constexpr int kT = 64, kK = 16;

struct GroupedF32 {
  const float* x;
  long long ldx;
  const int32_t* pair;      // row -> (token, choice) pair: the row's source is x[pair / per]; null: row itself
  int per;
  const float* w;           // [E][N][K]
  float* out;
  long long ldo;
  const int32_t* offsets;   // [E + 1]
  int n, k;
  int act;                  // ZbMoeAct; gated: rows of w in blocks of [64 gate | 64 up]
  const float* limits;      // [E] of ZB_ACT_CLIPPED_GLU
};

template <bool GATED>
__global__ void __launch_bounds__(256) zb_moe_grouped_f32_kernel(const GroupedF32 p) {
  __shared__ float sx[kK][kT + 4], sw[GATED ? 2 : 1][kK][kT + 4];
  zb_pdl_launch();
  zb_pdl_wait();
  const int e = blockIdx.z, r0 = p.offsets[e] + blockIdx.y * kT, end = p.offsets[e + 1];
  if (r0 >= end) return;
  const int n0 = blockIdx.x * kT * (GATED ? 2 : 1);            // first weight row of the tile
  const float* w = p.w + static_cast<long long>(e) * p.n * p.k;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const float* src[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int row = r0 + ((threadIdx.x + 256 * i) >> 4);
    src[i] = row < end ? p.x + (p.pair != nullptr ? p.pair[row] / p.per : row) * p.ldx : nullptr;
  }
  float acc[GATED ? 2 : 1][4][4] = {};
  for (int k0 = 0; k0 < p.k; k0 += kK) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int idx = threadIdx.x + 256 * i, row = idx >> 4, kk = idx & 15;
      const bool in = k0 + kk < p.k;
      sx[kk][row] = in && src[i] != nullptr ? src[i][k0 + kk] : 0.f;
#pragma unroll
      for (int g = 0; g < (GATED ? 2 : 1); ++g) {
        const int wr = n0 + g * kT + row;
        sw[g][kk][row] = in && wr < p.n ? w[static_cast<long long>(wr) * p.k + k0 + kk] : 0.f;
      }
    }
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < kK; ++kk) {
      const float4 xv = *reinterpret_cast<const float4*>(&sx[kk][ty * 4]);
      const float xr[4] = {xv.x, xv.y, xv.z, xv.w};
#pragma unroll
      for (int g = 0; g < (GATED ? 2 : 1); ++g) {
        const float4 wv = *reinterpret_cast<const float4*>(&sw[g][kk][tx * 4]);
        const float wr[4] = {wv.x, wv.y, wv.z, wv.w};
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) acc[g][i][j] = fmaf(xr[i], wr[j], acc[g][i][j]);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int row = r0 + ty * 4 + i;
    if (row >= end) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int c = tx * 4 + j;
      if constexpr (GATED) {
        const float g = acc[0][i][j], u = acc[1][i][j];
        float v;
        if (p.act == ZB_ACT_CLIPPED_GLU) v = zb_clipped_glu<true>(g, u, p.limits[e]);
        else v = (p.act == ZB_ACT_SWIGLU ? g / (1.f + expf(-g)) : zb_gate_act(g, p.act)) * u;
        p.out[row * p.ldo + blockIdx.x * kT + c] = v;
      } else if (n0 + c < p.n) {
        p.out[row * p.ldo + n0 + c] = zb_plain_act(acc[0][i][j], p.act);
      }
    }
  }
}
}  // namespace

// max_rows: an upper bound of the rows of one expert.  act and limits as zb_moe_grouped_gemm's (gated: n a multiple of 128).
extern "C" int zb_moe_grouped_f32(const float* x, long long ldx, const int32_t* pair, int per, const float* w, float* out, long long ldo,
                                  const int32_t* offsets, int experts, int n, int k, int max_rows, int act, const float* limits,
                                  void* stream) {
  if (max_rows <= 0 || experts <= 0) return 0;
  if (act < 0 || act > ZB_ACT_CLIPPED_GLU || (act == ZB_ACT_CLIPPED_GLU && limits == nullptr)) return -67;
  const bool gated = zb_act_is_gated(act);
  if (gated && n % (2 * kT) != 0) return -64;
  const int rows = (max_rows + kT - 1) / kT;
  if (rows > 65535 || experts > 65535) return -61;
  const GroupedF32 p = {x, ldx, pair, per, w, out, ldo, offsets, n, k, act, limits};
  const dim3 grid(gated ? n / (2 * kT) : (n + kT - 1) / kT, rows, experts);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const cudaError_t e = gated ? zb_launch(zb_moe_grouped_f32_kernel<true>, grid, dim3(256), 0, s, p)
                              : zb_launch(zb_moe_grouped_f32_kernel<false>, grid, dim3(256), 0, s, p);
  zb_count_launch(1);
  return static_cast<int>(e != cudaSuccess ? e : cudaGetLastError());
}
