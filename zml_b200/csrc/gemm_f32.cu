// fp32 GEMM on the FMA pipes: out[M,N] = act(A[M,K] * W[N,K]^T (+ bias)), every product and sum in IEEE fp32 (no TF32,
// no split accumulation order that depends on M).  It serves models that run in fp32 for verification; the bf16 GEMMs
// on the tensor cores are the serving path.  Any M, N, K and any leading dimensions.
#include "act.cuh"
#include "host_api.h"

namespace {
constexpr int kB = 64, kK = 16;

__global__ void __launch_bounds__(256) zb_gemm_f32_kernel(const float* __restrict__ a, long long lda, const float* __restrict__ w,
                                                          long long ldw, const float* __restrict__ bias, float* __restrict__ out,
                                                          long long ldo, int m, int n, int k, int act) {
  zb_pdl_launch();
  zb_pdl_wait();
  __shared__ float sa[kK][kB + 4], sw[kK][kB + 4];
  const int n0 = blockIdx.x * kB, m0 = blockIdx.y * kB;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < k; k0 += kK) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int idx = threadIdx.x + 256 * i, row = idx >> 4, kk = idx & 15;
      sa[kk][row] = (m0 + row < m && k0 + kk < k) ? a[(m0 + row) * lda + k0 + kk] : 0.f;
      sw[kk][row] = (n0 + row < n && k0 + kk < k) ? w[(n0 + row) * ldw + k0 + kk] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < kK; ++kk) {
      const float4 av = *reinterpret_cast<const float4*>(&sa[kk][ty * 4]), wv = *reinterpret_cast<const float4*>(&sw[kk][tx * 4]);
      const float ar[4] = {av.x, av.y, av.z, av.w}, wr[4] = {wv.x, wv.y, wv.z, wv.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(ar[i], wr[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int r = m0 + ty * 4 + i;
    if (r >= m) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int c = n0 + tx * 4 + j;
      if (c >= n) continue;
      float v = acc[i][j];
      if (bias != nullptr) v += bias[c];
      out[r * ldo + c] = zb_plain_act(v, act);
    }
  }
}
}  // namespace

extern "C" int zb_gemm_f32(const float* a, long long lda, const float* w, long long ldw, const float* bias, float* out, long long ldo,
                           int m, int n, int k, int act, void* stream) {
  if (m <= 0 || n <= 0) return 0;
  if (act != ZB_ACT_NONE && act != ZB_ACT_RELU2) return -16;
  const cudaError_t e = zb_launch(zb_gemm_f32_kernel, dim3((n + kB - 1) / kB, (m + kB - 1) / kB), dim3(256), 0,
                                  reinterpret_cast<cudaStream_t>(stream), a, lda, w, ldw, bias, out, ldo, m, n, k, act);
  zb_count_launch(1);
  return static_cast<int>(e != cudaSuccess ? e : cudaGetLastError());
}
