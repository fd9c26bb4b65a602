// Routing of tokens to experts by a table over token ids, and the row-wise helpers of the layer-list
// decoders: gather, combine, embedding, weight placement.
#include <algorithm>

#include "rows.cuh"

namespace vkl {
namespace {

// One CTA per routed layer: count the tokens of every expert, give each expert whole 128-row tiles, place every
// (token, choice). The order inside an expert does not matter: a row's result depends on that row alone.
constexpr uint32_t kMaxLayersPerLaunch = 32;
struct RouteArgs {
  RouteTable l[kMaxLayersPerLaunch];
};
__global__ void __launch_bounds__(1024) route_kernel(const RouteArgs args, const uint32_t *toks, uint32_t T) {
  extern __shared__ int32_t sm[];
  const RouteTable &r = args.l[blockIdx.x];
  int32_t *count = sm, *at = sm + r.experts;
  const uint32_t n = T * r.top, used = n < r.experts ? n : r.experts, tiles = n / 128 + used;
  for (uint32_t e = threadIdx.x; e < r.experts; e += blockDim.x) count[e] = 0;
  for (uint32_t i = threadIdx.x; i < tiles * 128; i += blockDim.x) r.token[i] = -1;
  for (uint32_t i = threadIdx.x; i < tiles; i += blockDim.x) r.tile_expert[i] = -1;
  __syncthreads();
  for (uint32_t i = threadIdx.x; i < n; i += blockDim.x) atomicAdd(&count[r.table[(size_t)toks[i / r.top] * r.top + i % r.top]], 1);
  __syncthreads();
  if (threadIdx.x == 0) {
    int32_t t = 0;
    for (uint32_t e = 0; e < r.experts; ++e) {
      at[e] = t * 128;
      for (int32_t k = (count[e] + 127) / 128; k > 0; --k) r.tile_expert[t++] = (int32_t)e;
    }
  }
  __syncthreads();
  for (uint32_t i = threadIdx.x; i < n; i += blockDim.x) {
    const int32_t row = atomicAdd(&at[r.table[(size_t)toks[i / r.top] * r.top + i % r.top]], 1);
    r.slot[i] = row;
    r.token[row] = (int32_t)(i / r.top);
  }
}

__global__ void gather_rows_kernel(const uint4 *__restrict__ src, const int32_t *__restrict__ rows, uint32_t vecs, uint4 *__restrict__ dst) {
  const int32_t r = rows[blockIdx.x];
  if (r < 0) return;
  for (uint32_t i = threadIdx.x; i < vecs; i += blockDim.x) dst[(size_t)blockIdx.x * vecs + i] = src[(size_t)r * vecs + i];
}

template <class T> __global__ void combine_kernel(const float *__restrict__ y, uint32_t y_ld, const int32_t *__restrict__ slot, uint32_t top, const Residual r) {
  const uint32_t m = blockIdx.x;
  for (uint32_t n = threadIdx.x; n < r.ldw; n += blockDim.x) {
    float v = 0.f;
    for (uint32_t j = 0; j < top; ++j) v += y[(size_t)slot[m * top + j] * y_ld + n];
    finish_residual<T>(r, m, n, r.x[(size_t)m * r.ldw + n] + r.mult * v);
  }
}

template <class T> __global__ void embed_rows_kernel(const bf16 *__restrict__ emb, const uint32_t *__restrict__ toks, float scale, const Residual r) {
  const uint32_t m = blockIdx.x;
  const bf16 *e = emb + (size_t)toks[m] * r.ldw;
  for (uint32_t n = threadIdx.x; n < r.ldw; n += blockDim.x) finish_residual<T>(r, m, n, __bfloat162float(e[n]) * scale);
}

__global__ void pack_rows_kernel(const bf16 *__restrict__ src, uint32_t rows, uint32_t cols, bf16 *__restrict__ dst, uint32_t ld, const PackMap m) {
  const uint64_t n = (uint64_t)rows * cols;
  for (uint64_t i = (uint64_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (uint64_t)gridDim.x * blockDim.x) {
    const uint32_t r = (uint32_t)(i / cols), c = (uint32_t)(i % cols);
    dst[(size_t)((r / m.ra) * m.rb + r % m.ra + m.r0) * ld + (c / m.ca) * m.cb + c % m.ca + m.c0] = src[i];
  }
}

}  // namespace

cudaError_t launch_route(const RouteTable *layers, uint32_t n, uint32_t max_experts, const uint32_t *toks, uint32_t T, cudaStream_t s) {
  const size_t smem = (size_t)max_experts * 2 * sizeof(int32_t);
  if (smem > 48 * 1024) return cudaErrorInvalidValue;
  for (uint32_t i = 0; i < n; i += kMaxLayersPerLaunch) {
    RouteArgs a;
    const uint32_t k = std::min(n - i, kMaxLayersPerLaunch);
    std::copy(layers + i, layers + i + k, a.l);
    route_kernel<<<k, 1024, smem, s>>>(a, toks, T);
    if (cudaError_t e = cudaGetLastError()) return e;
  }
  return cudaSuccess;
}
cudaError_t launch_gather_rows(const void *src, const int32_t *rows, uint32_t n, uint32_t row_bytes, void *dst, cudaStream_t s) {
  if (row_bytes % 16) return cudaErrorInvalidValue;
  if (!n) return cudaSuccess;
  gather_rows_kernel<<<n, 128, 0, s>>>(static_cast<const uint4 *>(src), rows, row_bytes / 16, static_cast<uint4 *>(dst));
  return cudaGetLastError();
}
cudaError_t launch_combine(const float *y, uint32_t y_ld, const int32_t *slot, uint32_t top, uint32_t T, const Residual &r, bool f32, cudaStream_t s) {
  if (f32) combine_kernel<float><<<T, 256, 0, s>>>(y, y_ld, slot, top, r);
  else combine_kernel<bf16><<<T, 256, 0, s>>>(y, y_ld, slot, top, r);
  return cudaGetLastError();
}
cudaError_t launch_embed_rows(const bf16 *emb, const uint32_t *toks, uint32_t T, float scale, const Residual &r, bool f32, cudaStream_t s) {
  if (f32) embed_rows_kernel<float><<<T, 256, 0, s>>>(emb, toks, scale, r);
  else embed_rows_kernel<bf16><<<T, 256, 0, s>>>(emb, toks, scale, r);
  return cudaGetLastError();
}
cudaError_t launch_pack_rows(const bf16 *src, uint32_t rows, uint32_t cols, bf16 *dst, uint32_t ld, const PackMap &m, cudaStream_t s) {
  const uint64_t n = (uint64_t)rows * cols;
  if (!n) return cudaSuccess;
  pack_rows_kernel<<<(unsigned)std::min<uint64_t>((n + 255) / 256, 148 * 32), 256, 0, s>>>(src, rows, cols, dst, ld, m);
  return cudaGetLastError();
}

}  // namespace vkl
