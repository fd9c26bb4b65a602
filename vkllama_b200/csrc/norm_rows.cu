// Norms with statistics and rotation for the layer-list decoder designs: the RMS norm of the residual stream (for
// one or two weights at once: parallel sublayers with norms of their own share the statistic), and what happens to
// query and key rows between projection and attention. Everything is fp32 inside; inputs and outputs of the query
// step are in the compute type. One CTA per token.
#include "rows.cuh"

namespace vkl {
namespace {

constexpr int kThreads = 256, kWarps = kThreads / 32;

// Sums of two numbers over the CTA, the same order every time.
__device__ __forceinline__ float2 block_sum2(float a, float b) {
  __shared__ float2 part[kWarps];
  a = warp_sum(a);
  b = warp_sum(b);
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = make_float2(a, b);
  __syncthreads();
  float2 r = part[0];
#pragma unroll
  for (int w = 1; w < kWarps; ++w) {
    r.x += part[w].x;
    r.y += part[w].y;
  }
  return r;
}

template <class T> __global__ void __launch_bounds__(kThreads) rms_rows_kernel(const RmsRows p) {
  if (p.use_pdl) asm volatile("griddepcontrol.wait;" ::: "memory");
  const float *x = p.x + (size_t)blockIdx.x * p.ldw;
  const size_t o = (size_t)blockIdx.x * p.ldw;
  float ss = 0.f;
  for (uint32_t n = threadIdx.x * 8; n < p.ldw; n += kThreads * 8) {
    float v[8];
    load8(x + n, v);
#pragma unroll
    for (int i = 0; i < 8; ++i) ss = fmaf(v[i], v[i], ss);
  }
  ss = block_sum2(ss, 0.f).x;
  const float r = 1.0f / sqrtf(ss / (float)p.width + p.eps);
  for (uint32_t n = threadIdx.x * 8; n < p.ldw; n += kThreads * 8) {
    float v[8], w[8], y[8];
    load8(x + n, v);
    load8(p.w + n, w);
#pragma unroll
    for (int i = 0; i < 8; ++i) y[i] = v[i] * r * w[i];
    store8(static_cast<T *>(p.h) + o + n, y);
    if (p.w2) {
      load8(p.w2 + n, w);
#pragma unroll
      for (int i = 0; i < 8; ++i) y[i] = v[i] * r * w[i];
      store8(static_cast<T *>(p.h2) + o + n, y);
    }
  }
  if (p.use_pdl) asm volatile("griddepcontrol.launch_dependents;");
}

constexpr uint32_t kMaxPairs = 128;  // head width at most 256

template <class T> __global__ void __launch_bounds__(kThreads) qk_rows_kernel(const QkRows p) {
  __shared__ float2 turn[kMaxPairs];
  if (p.use_pdl) asm volatile("griddepcontrol.wait;" ::: "memory");
  const uint32_t m = blockIdx.x, pos = *p.pos + m, tid = threadIdx.x;
  const uint32_t nq = p.heads * p.dp, nk = p.kcache ? p.kv_heads * p.dp : 0u;
  T *q = static_cast<T *>(p.q) + (size_t)m * p.q_ld, *k = q + p.k_col;
  if (tid < p.pairs) {
    float s, c;
    sincosf((float)pos * p.freq[tid], &s, &c);
    turn[tid] = make_float2(c, s);
  }
  float sq = 0.f, sk = 0.f;
  for (uint32_t n = tid * 8; n < nq; n += kThreads * 8) {  // padded columns are zero
    float v[8];
    load8(q + n, v);
#pragma unroll
    for (int i = 0; i < 8; ++i) sq = fmaf(v[i], v[i], sq);
  }
  for (uint32_t n = tid * 8; n < nk; n += kThreads * 8) {
    float v[8];
    load8(k + n, v);
#pragma unroll
    for (int i = 0; i < 8; ++i) sk = fmaf(v[i], v[i], sk);
  }
  const float2 ss = block_sum2(sq, sk);  // also: every thread's angles are in place
  const float rq = p.qw ? 1.0f / sqrtf(ss.x / (float)(p.heads * p.dim) + p.eps) : 1.f;
  const float rk = p.kw ? 1.0f / sqrtf(ss.y / (float)(p.kv_heads * p.dim) + p.eps) : 1.f;
  for (uint32_t n = tid * 8; n < nq + nk; n += kThreads * 8) {
    const bool key = n >= nq;
    const uint32_t c = key ? n - nq : n, d = c % p.dp;
    const float *w = key ? p.kw : p.qw;
    float v[8];
    load8(key ? k + c : q + c, v);
    const float r = key ? rk : rq;
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] *= w ? r * w[c + i] : 1.f;
#pragma unroll
    for (int i = 0; i < 8; i += 2) {
      if ((d + i) / 2 < p.pairs) {
        const float2 t = turn[(d + i) / 2];
        const float a = v[i], b = v[i + 1];
        v[i] = a * t.x - b * t.y;
        v[i + 1] = b * t.x + a * t.y;
      }
    }
    store8(key ? cache_slot<T>(p.kcache, p.dp, p.maxlen, pos, c) : q + c, v);
  }
  if (p.use_pdl) asm volatile("griddepcontrol.launch_dependents;");
}

template <class P> cudaError_t launch(void (*kern)(const P), const P &p, cudaStream_t s) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(p.T);
  cfg.blockDim = dim3(kThreads);
  cfg.stream = s;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = p.use_pdl ? 1 : 0;
  return cudaLaunchKernelEx(&cfg, kern, p);
}

}  // namespace

cudaError_t launch_rms_rows(const RmsRows &p, bool f32, cudaStream_t s) {
  if (!p.T || !p.width || p.ldw % 8) return cudaErrorInvalidValue;
  return f32 ? launch(rms_rows_kernel<float>, p, s) : launch(rms_rows_kernel<bf16>, p, s);
}

cudaError_t launch_qk_rows(const QkRows &p, bool f32, cudaStream_t s) {
  if (!p.T || p.dp % 16 || p.pairs > kMaxPairs || 2 * p.pairs > p.dim || p.k_col % 8 || p.q_ld % 8) return cudaErrorInvalidValue;
  return f32 ? launch(qk_rows_kernel<float>, p, s) : launch(qk_rows_kernel<bf16>, p, s);
}

}  // namespace vkl
