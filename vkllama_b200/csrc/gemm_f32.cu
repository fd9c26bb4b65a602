// Many tokens in true 32-bit: Y[M,N] = A[M,K] . W[N,K]^T on the FMA units, A fp32, W bf16 widened exactly,
// the sum over K in order. The layer-list decoders' 32-bit mode runs its prompts through it; segments,
// grouping by expert and epilogues are those of the bfloat16 tensor-core GEMM.
#include "rows.cuh"

namespace vkl {
namespace {

constexpr uint32_t TM = 64, TN = 64, TK = 16;

// 128 threads: thread = (row of the tile, half of its columns), 32 accumulators = one chunk of the epilogue.
__global__ void __launch_bounds__(128) gemm_f32_kernel(const GemmRows p) {
  __shared__ float as[TK][TM + 1];
  __shared__ __align__(16) float wsm[TK][TN + 4];
  const uint32_t tid = threadIdx.x, m0 = blockIdx.x * TM, n0 = blockIdx.y * TN, row = tid % TM, half = tid / TM;
  size_t w0 = n0;
  if (p.tile_expert) {
    const int32_t e = p.tile_expert[m0 / 128];
    if (e < 0) return;
    w0 += (size_t)e * p.N;
  }
  const float *a = static_cast<const float *>(p.a) + (p.n2 && n0 >= p.n2 ? (size_t)p.M * p.K : 0);
  float acc[32];
#pragma unroll
  for (int i = 0; i < 32; ++i) acc[i] = 0.f;
  for (uint32_t k = 0; k < p.K; k += TK) {
    for (uint32_t i = tid; i < TM * TK; i += 128) {
      const uint32_t r = i / TK, c = i % TK;
      as[c][r] = m0 + r < p.M ? a[(size_t)(m0 + r) * p.K + k + c] : 0.f;
      wsm[c][r] = n0 + r < p.N ? __bfloat162float(p.w[(w0 + r) * p.K + k + c]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (uint32_t c = 0; c < TK; ++c) {
      const float x = as[c][row];
      const float4 *w = reinterpret_cast<const float4 *>(&wsm[c][half * 32]);
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const float4 v = w[i];
        acc[4 * i] = fmaf(x, v.x, acc[4 * i]);
        acc[4 * i + 1] = fmaf(x, v.y, acc[4 * i + 1]);
        acc[4 * i + 2] = fmaf(x, v.z, acc[4 * i + 2]);
        acc[4 * i + 3] = fmaf(x, v.w, acc[4 * i + 3]);
      }
    }
    __syncthreads();
  }
  const uint32_t m = m0 + row, n = n0 + half * 32;
  if (m < p.M && n < p.N) rows_chunk<float>(p.out, m, n, acc);
}

}  // namespace

cudaError_t launch_gemm_rows_f32(const GemmRows &p, cudaStream_t s) {
  if (!p.M || !p.N || p.N % 32 || p.K % 64 || p.n2 % kInputAlign) return cudaErrorInvalidValue;
  gemm_f32_kernel<<<dim3((p.M + TM - 1) / TM, (p.N + TN - 1) / TN), 128, 0, s>>>(p);
  return cudaGetLastError();
}

}  // namespace vkl
