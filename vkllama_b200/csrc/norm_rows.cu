// Norms with statistics and rotation for the layer-list decoder designs: the RMS norm of the residual stream (for
// one or two weights at once: parallel sublayers with norms of their own share the statistic), and what happens to
// query and key rows between projection and attention. Everything is fp32 inside; inputs and outputs of the query
// step are in the compute type. One CTA per token.
#include "rows.cuh"

namespace vkl {
namespace {

constexpr int kThreads = 256, kWarps = kThreads / 32;

template <class T> __global__ void __launch_bounds__(kThreads) rms_rows_kernel(const RmsRows p) {
  if (p.use_pdl) asm volatile("griddepcontrol.wait;" ::: "memory");
  const size_t o = (size_t)blockIdx.x * p.ldw;
  rms_row<T, kWarps>(p, p.x + o, static_cast<T *>(p.h) + o, static_cast<T *>(p.h2) + o);
  if (p.use_pdl) asm volatile("griddepcontrol.launch_dependents;");
}

template <class T> __global__ void __launch_bounds__(kThreads) qk_rows_kernel(const QkRows p) {
  __shared__ float2 turn[kMaxPairs];
  if (p.use_pdl) asm volatile("griddepcontrol.wait;" ::: "memory");
  const uint32_t m = blockIdx.x, pos = *p.pos + m, tid = threadIdx.x;
  const uint32_t nq = p.heads * p.dp, nk = p.kcache ? p.kv_heads * p.dp : 0u;
  T *q = static_cast<T *>(p.q) + (size_t)m * p.q_ld, *k = q + p.k_col;
  if (tid < p.pairs) turn[tid] = turn_of(pos, p.freq[tid]);
  float sq = 0.f, sk = 0.f, v[8];
  for (uint32_t n = tid * 8; n < nq; n += kThreads * 8) {  // padded columns are zero
    load8(q + n, v);
    sq = square_sum8(v, sq);
  }
  for (uint32_t n = tid * 8; n < nk; n += kThreads * 8) {
    load8(k + n, v);
    sk = square_sum8(v, sk);
  }
  const float2 ss = block_sum2<kWarps>(sq, sk);  // also: every thread's angles are in place
  const float rq = 1.0f / sqrtf(ss.x / (float)(p.heads * p.dim) + p.eps), rk = 1.0f / sqrtf(ss.y / (float)(p.kv_heads * p.dim) + p.eps);
  for (uint32_t n = tid * 8; n < nq + nk; n += kThreads * 8) {
    const bool key = n >= nq;
    const uint32_t c = key ? n - nq : n;
    const float *w = key ? p.kw : p.qw;
    load8(key ? k + c : q + c, v);
    norm_and_turn(v, w ? w + c : nullptr, key ? rk : rq, c % p.dp, turn, p.pairs);
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
