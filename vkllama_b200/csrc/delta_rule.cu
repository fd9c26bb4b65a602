// Gated delta rule with a decay per head and key channel, for prompts and portions of any length: the steps between
// the in-projection and the out-projection. Everything is fp32 except the projections that come in and the rows
// that go out.
//
//   prepare     a warp per token and row (query, key or value head): short causal convolution over time, SiLU, unit
//               norm of queries and keys. Tokens before the call come from the ring of past projections.
//   recurrence  the columns of a state do not depend on each other: a CTA owns 16 columns of a head in registers,
//               eight lanes per column, and walks over the tokens. Queries, keys, decays and values travel through a
//               ring of shared-memory stages. A column's arithmetic is the same however a prompt is cut.
//   finish      a warp per token and head: RMS norm of the head's outputs, gate; and the call's last projections
//               go to the ring.
#include <algorithm>

#include "rows.cuh"

namespace vkl {
namespace {

constexpr int kThreads = 256, kWarps = kThreads / 32;
constexpr float kUnitEps = 1e-6f;

__device__ __forceinline__ float load1(const bf16 *p) { return __bfloat162float(*p); }
__device__ __forceinline__ float load1(const float *p) { return *p; }
__device__ __forceinline__ float silu_f(float z) { return z * sigmoid_f(z); }

// Channel c of token m after convolution and SiLU; pos0: position of token 0.
template <class T> __device__ __forceinline__ float convolved(const DeltaRows &p, uint32_t m, uint32_t pos0, uint32_t c) {
  const float *w = p.taps + (size_t)c * p.ntaps;
  float a = 0.f;
  for (uint32_t j = 0; j < p.ntaps; ++j) {
    const uint32_t back = p.ntaps - 1 - j;
    if (back > pos0 + m) continue;  // before the sequence's start
    const T *x = back <= m ? static_cast<const T *>(p.raw) + (size_t)(m - back) * p.raw_ld : static_cast<const T *>(p.ring) + (size_t)((pos0 + m - back) % p.ntaps) * p.raw_ld;
    a = fmaf(load1(x + c), w[j], a);
  }
  return silu_f(a);
}

template <class T> __global__ void __launch_bounds__(kThreads) delta_prepare_kernel(const DeltaRows p) {
  if (p.use_pdl) asm volatile("griddepcontrol.wait;" ::: "memory");
  const uint32_t m = blockIdx.x, lane = threadIdx.x & 31, unit = blockIdx.y * kWarps + (threadIdx.x >> 5);
  const uint32_t pos0 = *p.pos;
  if (unit >= 2 * p.kv_heads + p.heads) return;
  if (unit >= 2 * p.kv_heads) {
    const uint32_t h = unit - 2 * p.kv_heads;
    float *v = p.v + ((size_t)m * p.heads + h) * p.vp;
    for (uint32_t d = lane; d < p.vp; d += 32) v[d] = convolved<T>(p, m, pos0, p.v_col + h * p.vp + d);
    return;
  }
  const bool key = unit >= p.kv_heads;
  const uint32_t g = key ? unit - p.kv_heads : unit;
  float y[8], ss = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const uint32_t d = i * 32 + lane;
    y[i] = d < p.dp ? convolved<T>(p, m, pos0, (key ? p.k_col : 0u) + g * p.dp + d) : 0.f;
    ss = fmaf(y[i], y[i], ss);
  }
  ss = warp_sum(ss);
  const float r = 1.0f / sqrtf(ss + kUnitEps) * (key ? 1.f : 1.0f / sqrtf((float)p.dim));
  float *o = (key ? p.k : p.q) + ((size_t)m * p.kv_heads + g) * p.dp;
#pragma unroll
  for (int i = 0; i < 8; ++i)
    if (i * 32 < p.dp) o[i * 32 + lane] = y[i] * r;
}

__device__ __forceinline__ void copy16(void *dst, const void *src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

constexpr uint32_t kCols = 16, kLanes = 8, kRecThreads = kCols * kLanes;
constexpr uint32_t kStageTokens = 8, kStages = 3;
// A stage: [token][q | k | g | v | beta], floats.
__host__ __device__ constexpr uint32_t rec_token_floats(uint32_t E) { return 3 * E * 32 + kCols + 4; }

// E: 32-element steps of the key width. Lane l of a column holds elements 32 i + 4 l .. + 3, i < E.
template <int E> __global__ void __launch_bounds__(kRecThreads) delta_recurrence_kernel(const DeltaRows p) {
  constexpr uint32_t DP = E * 32, TF = rec_token_floats(E);
  extern __shared__ __align__(16) float stage_mem[];
  if (p.use_pdl) asm volatile("griddepcontrol.wait;" ::: "memory");
  const uint32_t h = blockIdx.x, c0 = blockIdx.y * kCols, tid = threadIdx.x, col = tid / kLanes, l = tid % kLanes;
  const uint32_t kv = h / (p.heads / p.kv_heads), T = p.T;
  float *state = p.state + ((size_t)h * p.vp + c0 + col) * DP + l * 4;
  float S[E * 4];
  if (*p.pos == 0) {
#pragma unroll
    for (int i = 0; i < E * 4; ++i) S[i] = 0.f;
  } else {
#pragma unroll
    for (int i = 0; i < E; ++i) {
      const float4 v = *reinterpret_cast<const float4 *>(state + i * 32);
      S[4 * i] = v.x; S[4 * i + 1] = v.y; S[4 * i + 2] = v.z; S[4 * i + 3] = v.w;
    }
  }
  auto fetch = [&](uint32_t tile) {
    float *st = stage_mem + (tile % kStages) * kStageTokens * TF;
    const uint32_t t0 = tile * kStageTokens;
    constexpr uint32_t V = DP / 4, PER = 3 * V + kCols / 4;  // 16-byte pieces of a token
    for (uint32_t i = tid; i < kStageTokens * PER; i += kRecThreads) {
      const uint32_t t = i / PER, x = i % PER, at = t0 + t;
      if (at >= T) break;
      float *dst = st + t * TF + x * 4;
      const float *src;
      if (x < V) src = p.q + ((size_t)at * p.kv_heads + kv) * DP + x * 4;
      else if (x < 2 * V) src = p.k + ((size_t)at * p.kv_heads + kv) * DP + (x - V) * 4;
      else if (x < 3 * V) src = p.g + (size_t)at * p.g_ld + h * DP + (x - 2 * V) * 4;
      else src = p.v + ((size_t)at * p.heads + h) * p.vp + c0 + (x - 3 * V) * 4;
      copy16(dst, src);
    }
    if (tid < kStageTokens && t0 + tid < T) {
      const uint32_t dst = (uint32_t)__cvta_generic_to_shared(st + tid * TF + 3 * DP + kCols);
      asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(dst), "l"(p.beta + (size_t)(t0 + tid) * p.beta_ld + h) : "memory");
    }
  };
  const uint32_t tiles = (T + kStageTokens - 1) / kStageTokens;
  for (uint32_t i = 0; i < kStages - 1; ++i) {
    if (i < tiles) fetch(i);
    asm volatile("cp.async.commit_group;" ::: "memory");
  }
  for (uint32_t tile = 0; tile < tiles; ++tile) {
    asm volatile("cp.async.wait_group %0;" ::"n"(kStages - 2) : "memory");
    __syncthreads();  // this stage has landed for everyone, the one before is consumed
    if (tile + kStages - 1 < tiles) fetch(tile + kStages - 1);
    asm volatile("cp.async.commit_group;" ::: "memory");
    const float *st = stage_mem + (tile % kStages) * kStageTokens * TF;
    const uint32_t n = min(kStageTokens, T - tile * kStageTokens);
    for (uint32_t t = 0; t < n; ++t, st += TF) {
      float k[E * 4], a = 0.f, b = 0.f;
#pragma unroll
      for (int i = 0; i < E; ++i) {
        const float4 kk = *reinterpret_cast<const float4 *>(st + DP + i * 32 + l * 4), g = *reinterpret_cast<const float4 *>(st + 2 * DP + i * 32 + l * 4);
        k[4 * i] = kk.x; k[4 * i + 1] = kk.y; k[4 * i + 2] = kk.z; k[4 * i + 3] = kk.w;
        S[4 * i] *= g.x; S[4 * i + 1] *= g.y; S[4 * i + 2] *= g.z; S[4 * i + 3] *= g.w;
        a = fmaf(S[4 * i], kk.x, a);
        b = fmaf(S[4 * i + 1], kk.y, b);
        a = fmaf(S[4 * i + 2], kk.z, a);
        b = fmaf(S[4 * i + 3], kk.w, b);
      }
      a += b;
#pragma unroll
      for (uint32_t o = 1; o < kLanes; o <<= 1) a += __shfl_xor_sync(0xffffffffu, a, o);
      const float u = st[3 * DP + kCols] * (st[3 * DP + col] - a);
      float y = 0.f, z = 0.f;
#pragma unroll
      for (int i = 0; i < E; ++i) {
        const float4 q = *reinterpret_cast<const float4 *>(st + i * 32 + l * 4);
        S[4 * i] = fmaf(k[4 * i], u, S[4 * i]);
        S[4 * i + 1] = fmaf(k[4 * i + 1], u, S[4 * i + 1]);
        S[4 * i + 2] = fmaf(k[4 * i + 2], u, S[4 * i + 2]);
        S[4 * i + 3] = fmaf(k[4 * i + 3], u, S[4 * i + 3]);
        y = fmaf(S[4 * i], q.x, y);
        z = fmaf(S[4 * i + 1], q.y, z);
        y = fmaf(S[4 * i + 2], q.z, y);
        z = fmaf(S[4 * i + 3], q.w, z);
      }
      y += z;
#pragma unroll
      for (uint32_t o = 1; o < kLanes; o <<= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
      if (l == 0) p.v[((size_t)(tile * kStageTokens + t) * p.heads + h) * p.vp + c0 + col] = y;
    }
  }
#pragma unroll
  for (int i = 0; i < E; ++i) *reinterpret_cast<float4 *>(state + i * 32) = make_float4(S[4 * i], S[4 * i + 1], S[4 * i + 2], S[4 * i + 3]);
  if (p.use_pdl) asm volatile("griddepcontrol.launch_dependents;");
}

template <class T> __global__ void __launch_bounds__(kThreads) delta_finish_kernel(const DeltaRows p) {
  if (p.use_pdl) asm volatile("griddepcontrol.wait;" ::: "memory");
  const uint32_t m = blockIdx.x, lane = threadIdx.x & 31, h = blockIdx.y * kWarps + (threadIdx.x >> 5);
  if (m + p.ntaps >= p.T) {  // one of the last ntaps tokens: later ones look back at it
    const T *src = static_cast<const T *>(p.raw) + (size_t)m * p.raw_ld;
    T *dst = static_cast<T *>(p.ring) + (size_t)((*p.pos + m) % p.ntaps) * p.raw_ld;
    for (uint32_t c = blockIdx.y * kThreads + threadIdx.x; c < p.raw_ld; c += gridDim.y * kThreads) dst[c] = src[c];
  }
  if (h >= p.heads) return;
  const float *o = p.v + ((size_t)m * p.heads + h) * p.vp;
  float y[8], ss = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const uint32_t d = i * 32 + lane;
    y[i] = d < p.vp ? o[d] : 0.f;  // padded columns are zero
    ss = fmaf(y[i], y[i], ss);
  }
  ss = warp_sum(ss);
  const float r = 1.0f / sqrtf(ss / (float)p.vdim + p.eps);
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const uint32_t d = i * 32 + lane;
    if (d < p.vp) store1(static_cast<T *>(p.out) + (size_t)m * p.out_ld + h * p.vp + d, y[i] * r * p.norm[d] * p.gate[(size_t)m * p.gate_ld + h * p.vp + d]);
  }
}

cudaError_t launch(void (*kern)(const DeltaRows), const DeltaRows &p, dim3 grid, uint32_t threads, size_t smem, cudaStream_t s) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = dim3(threads);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = s;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = p.use_pdl ? 1 : 0;
  return cudaLaunchKernelEx(&cfg, kern, p);
}

template <int E> cudaError_t launch_recurrence(const DeltaRows &p, cudaStream_t s) {
  constexpr size_t smem = (size_t)kStages * kStageTokens * rec_token_floats(E) * sizeof(float);
  if (cudaError_t e = cudaFuncSetAttribute(delta_recurrence_kernel<E>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)) return e;
  return launch(delta_recurrence_kernel<E>, p, dim3(p.heads, p.vp / kCols), kRecThreads, smem, s);
}

bool sane(const DeltaRows &p) {
  return p.T && p.heads && p.kv_heads && p.heads % p.kv_heads == 0 && p.ntaps && p.dp % 32 == 0 && p.dp <= 256 && p.vp % kCols == 0 && p.vp <= 256 && p.g_ld % 4 == 0;
}

}  // namespace

cudaError_t launch_delta_prepare(const DeltaRows &p, bool f32, cudaStream_t s) {
  if (!sane(p)) return cudaErrorInvalidValue;
  const dim3 grid(p.T, (2 * p.kv_heads + p.heads + kWarps - 1) / kWarps);
  return launch(f32 ? delta_prepare_kernel<float> : delta_prepare_kernel<bf16>, p, grid, kThreads, 0, s);
}

cudaError_t launch_delta_recurrence(const DeltaRows &p, cudaStream_t s) {
  if (!sane(p)) return cudaErrorInvalidValue;
  switch (p.dp / 32) {
    case 1: return launch_recurrence<1>(p, s);
    case 2: return launch_recurrence<2>(p, s);
    case 3: return launch_recurrence<3>(p, s);
    case 4: return launch_recurrence<4>(p, s);
    case 5: return launch_recurrence<5>(p, s);
    case 6: return launch_recurrence<6>(p, s);
    case 7: return launch_recurrence<7>(p, s);
    default: return launch_recurrence<8>(p, s);
  }
}

cudaError_t launch_delta_finish(const DeltaRows &p, bool f32, cudaStream_t s) {
  if (!sane(p)) return cudaErrorInvalidValue;
  const dim3 grid(p.T, (p.heads + kWarps - 1) / kWarps);
  return launch(f32 ? delta_finish_kernel<float> : delta_finish_kernel<bf16>, p, grid, kThreads, 0, s);
}

}  // namespace vkl
