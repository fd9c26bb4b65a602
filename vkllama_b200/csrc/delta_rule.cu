// Gated delta rule with a decay per head and key channel: everything between the in-projection and the out-projection
// of a recurrent layer. All arithmetic is fp32 except the projections that come in and the rows that go out.
//
// Many tokens, in blocks of eight. Inside a block the recurrence is unrolled: with P_t the product of the block's decays
// up to token t, and S the state before the block,
//   w_t = v_t - S^T (P_t k_t)                          how far the state is from each value,
//   u   = M w, M = (1 + beta A)^-1 beta                A_ts = k_t . (decays s+1 .. t) k_s for s < t, the writes' overlap,
//   o_t = S^T (P_t q_t) + (N w)_t, N = B M             B_ts = q_t . (decays s+1 .. t) k_s for s <= t,
//   S  <- P_8 S + sum_s (decays s+1 .. 8) k_s u_s^T.
// Decays only ever multiply (no quotient of products), so nothing overflows and a decay of zero is exact.
//   blocks      a CTA per head and block: convolution, SiLU, unit norms, decays, and from them the rows P k, P q,
//               (later decays) k, the product of the decays, M and N. Depends on no state: all blocks at once.
//   scan        the columns of a state do not depend on each other: 16 or 32 lanes hold four columns in registers and
//               walk over the blocks, whose rows travel through a ring of shared-memory stages. A column's arithmetic within
//               a block is all independent dot products.
//   finish      a warp per token and head: RMS norm of the head's outputs, gate; and the call's last projections go to
//               the ring of past projections.
// One token: a cluster of CTAs per head, 32 columns each, does all of it in one kernel; what does not depend on the
// kernel before (weights, state) is requested before waiting for it, and the norm's sum crosses the cluster.
#include <cooperative_groups.h>

#include <algorithm>
#include <type_traits>

#include "rows.cuh"

namespace vkl {
namespace {

namespace cg = cooperative_groups;

constexpr float kUnitEps = 1e-6f;
constexpr uint32_t kBlock = 8, kPairsA = 28, kPairs = 64;  // token pairs s < t, and those plus s <= t

__device__ __forceinline__ float load1(const bf16 *p) { return __bfloat162float(*p); }
__device__ __forceinline__ float load1(const float *p) { return *p; }

// Projection c of token m, which may lie before the call's first token (position pos0) or the sequence's.
template <class T> __device__ __forceinline__ float projection(const DeltaRows &p, int m, uint32_t pos0, uint32_t c) {
  if (m >= 0) return load1(static_cast<const T *>(p.raw) + (size_t)m * p.raw_ld + c);
  const int at = (int)pos0 + m;
  return at < 0 ? 0.f : load1(static_cast<const T *>(p.ring) + (size_t)((uint32_t)at % p.ntaps) * p.raw_ld + c);
}

__device__ __forceinline__ float fast_sigmoid(float z) { return __fdividef(1.0f, 1.0f + expf(-z)); }

// Projection c of tokens t0 - (TAPS - 1) .. t0 + 7; 0 from token t0 + n on.
template <class T, int TAPS> __device__ __forceinline__ void load_window(const DeltaRows &p, uint32_t t0, uint32_t n, uint32_t pos0, uint32_t c, float (&x)[kBlock + TAPS - 1]) {
  constexpr int BACK = TAPS - 1;
  if (n == kBlock && t0 >= (uint32_t)BACK) {
    const T *r = static_cast<const T *>(p.raw) + (size_t)(t0 - BACK) * p.raw_ld + c;
#pragma unroll
    for (int i = 0; i < (int)kBlock + BACK; ++i) x[i] = load1(r + (size_t)i * p.raw_ld);
  } else {
#pragma unroll
    for (int i = 0; i < (int)kBlock + BACK; ++i) x[i] = (int)n > i - BACK ? projection<T>(p, (int)t0 + i - BACK, pos0, c) : 0.f;
  }
}
// Convolution and SiLU of a window; 0 from token n on.
template <int TAPS> __device__ __forceinline__ void convolve8(const DeltaRows &p, uint32_t n, uint32_t c, const float (&x)[kBlock + TAPS - 1], float (&y)[kBlock]) {
  float w[TAPS];
#pragma unroll
  for (int j = 0; j < TAPS; ++j) w[j] = p.taps[(size_t)c * TAPS + j];
#pragma unroll
  for (int t = 0; t < (int)kBlock; ++t) {
    float a = 0.f;
#pragma unroll
    for (int j = 0; j < TAPS; ++j) a = fmaf(x[t + j], w[j], a);
    y[t] = t < (int)n ? a * fast_sigmoid(a) : 0.f;
  }
}
// The same for any number of taps, one token after the other.
template <class T> __device__ __forceinline__ void convolve8_any(const DeltaRows &p, uint32_t t0, uint32_t n, uint32_t pos0, uint32_t c, float (&y)[kBlock]) {
  const float *w = p.taps + (size_t)c * p.ntaps;
#pragma unroll
  for (int t = 0; t < (int)kBlock; ++t) {
    float a = 0.f;
    if (t < (int)n)
      for (uint32_t j = 0; j < p.ntaps; ++j) a = fmaf(projection<T>(p, (int)(t0 + t + j) - (int)(p.ntaps - 1), pos0, c), w[j], a);
    y[t] = a * fast_sigmoid(a);
  }
}

// Sums N values over the warp; lane i ends with the sums of values (i * N / 32) ... (N >= 32), or of value i / (32 / N).
template <int N, int BIT> __device__ __forceinline__ void scatter_sum(float *v, uint32_t lane) {
  if constexpr (BIT > 0) {
    const bool up = lane & BIT;
    if constexpr (N > 1) {
#pragma unroll
      for (int i = 0; i < N / 2; ++i) {
        const float send = up ? v[i] : v[N / 2 + i], keep = up ? v[N / 2 + i] : v[i];
        v[i] = keep + __shfl_xor_sync(0xffffffffu, send, BIT);
      }
      scatter_sum<N / 2, BIT / 2>(v, lane);
    } else {
      v[0] += __shfl_xor_sync(0xffffffffu, v[0], BIT);
      scatter_sum<1, BIT / 2>(v, lane);
    }
  }
}

// A block's record, in floats: P k [8][dp], P q [8][dp], (later decays) k [8][dp], P_8 [dp], M [8][8], N [8][8].
__host__ __device__ constexpr uint32_t block_floats(uint32_t dp) { return 25 * dp + 128; }
__device__ __forceinline__ uint32_t pair_a(uint32_t t, uint32_t s) { return s * 7 - s * (s - 1) / 2 + t - s - 1; }   // s < t
__device__ __forceinline__ uint32_t pair_b(uint32_t t, uint32_t s) { return kPairsA + s * 8 - s * (s - 1) / 2 + t - s; }  // s <= t

// NT threads, one per key channel and one per value channel. first: token of block 0 of this launch.
template <class T, int TAPS, int NT> __global__ void __launch_bounds__(NT, 768 / NT) delta_blocks_kernel(const DeltaRows p, uint32_t first) {
  constexpr int NW = NT / 32;
  __shared__ float sums[NW][2 * kBlock], pairs[NW][kPairs], ab[kPairs], minv[kBlock][kBlock], beta_s[kBlock], scale_s[2 * kBlock];
  const uint32_t h = blockIdx.x, t0 = first + blockIdx.y * kBlock, n = min(kBlock, p.T - t0), tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const uint32_t kv = h / (p.heads / p.kv_heads), pos0 = *p.pos;
  float *rec = p.blocks + ((size_t)blockIdx.y * p.heads + h) * block_floats(p.dp);
  if (tid < kBlock) beta_s[tid] = tid < n ? p.beta[(size_t)(t0 + tid) * p.beta_ld + h] : 0.f;
  const bool on = tid < p.dp, von = tid < p.vp;
  const uint32_t cq = kv * p.dp + tid, ck = p.k_col + cq, cv = p.v_col + h * p.vp + tid, cg = h * p.dp + tid;
  float q[kBlock], k[kBlock], g[kBlock], v[kBlock];
#pragma unroll
  for (uint32_t t = 0; t < kBlock; ++t) {
    q[t] = k[t] = 0.f;
    g[t] = on && t < n ? p.z[(size_t)(t0 + t) * p.z_ld + cg] : 0.f;
  }
  if constexpr (TAPS > 0) {
    float xq[kBlock + TAPS - 1], xk[kBlock + TAPS - 1], xv[kBlock + TAPS - 1];
    if (on) {
      load_window<T, TAPS>(p, t0, n, pos0, cq, xq);
      load_window<T, TAPS>(p, t0, n, pos0, ck, xk);
    }
    if (von) {
      load_window<T, TAPS>(p, t0, n, pos0, cv, xv);
      convolve8<TAPS>(p, n, cv, xv, v);
    }
    if (on) {
      convolve8<TAPS>(p, n, cq, xq, q);
      convolve8<TAPS>(p, n, ck, xk, k);
    }
  } else {
    if (on) {
      convolve8_any<T>(p, t0, n, pos0, cq, q);
      convolve8_any<T>(p, t0, n, pos0, ck, k);
    }
    if (von) convolve8_any<T>(p, t0, n, pos0, cv, v);
  }
  if (von) {
#pragma unroll
    for (uint32_t t = 0; t < kBlock; ++t)
      if (t < n) p.v[((size_t)(t0 + t) * p.heads + h) * p.vp + tid] = v[t];
  }
  const float rate = on ? p.rate[cg] : 0.f, bias = on ? p.bias[cg] : 0.f;
#pragma unroll
  for (uint32_t t = 0; t < kBlock; ++t) g[t] = t < n ? expf(-rate * softplus_f(g[t] + bias)) : 1.f;
  float ss[2 * kBlock];
#pragma unroll
  for (uint32_t t = 0; t < kBlock; ++t) {
    ss[t] = q[t] * q[t];
    ss[kBlock + t] = k[t] * k[t];
  }
  scatter_sum<2 * kBlock, 16>(ss, lane);  // lane: value lane / 2
  if (!(lane & 1)) sums[warp][lane >> 1] = ss[0];
  __syncthreads();
  if (tid < 2 * kBlock) {
    float a = 0.f;
#pragma unroll
    for (int w = 0; w < NW; ++w) a += sums[w][tid];
    scale_s[tid] = 1.0f / sqrtf(a + kUnitEps) * (tid < kBlock ? 1.0f / sqrtf((float)p.dim) : 1.0f);
  }
  __syncthreads();
#pragma unroll
  for (uint32_t t = 0; t < kBlock; ++t) {
    q[t] *= scale_s[t];
    k[t] *= scale_s[kBlock + t];
  }
  if (on) {
    float d = 1.f;
#pragma unroll
    for (uint32_t t = 0; t < kBlock; ++t) {
      d *= g[t];
      rec[t * p.dp + tid] = d * k[t];
      rec[(kBlock + t) * p.dp + tid] = d * q[t];
    }
    rec[3 * kBlock * p.dp + tid] = d;
    d = 1.f;
#pragma unroll
    for (int t = kBlock - 1; t >= 0; --t) {
      rec[(2 * kBlock + t) * p.dp + tid] = d * k[t];
      d *= g[t];
    }
  }
  float pr[kPairs];
  int ia = 0, ib = kPairsA;
#pragma unroll
  for (int s = 0; s < (int)kBlock; ++s) {
    float d = k[s];
    pr[ib++] = d * q[s];
#pragma unroll
    for (int t = s + 1; t < (int)kBlock; ++t) {
      d *= g[t];
      pr[ia++] = d * k[t];
      pr[ib++] = d * q[t];
    }
  }
  scatter_sum<kPairs, 16>(pr, lane);  // lane: values 2 lane, 2 lane + 1
  pairs[warp][2 * lane] = pr[0];
  pairs[warp][2 * lane + 1] = pr[1];
  __syncthreads();
  if (tid < kPairs) {
    float a = 0.f;
#pragma unroll
    for (int w = 0; w < NW; ++w) a += pairs[w][tid];
    ab[tid] = a;
  }
  __syncthreads();
  float *mn = rec + 25 * p.dp;
  if (tid < kBlock) {  // column tid of M
    float m[kBlock];
#pragma unroll
    for (int t = 0; t < (int)kBlock; ++t) {
      float a = t == (int)tid ? 1.f : 0.f;
#pragma unroll
      for (int s = 0; s < t; ++s) a = fmaf(-ab[pair_a(t, s)], m[s], a);
      m[t] = beta_s[t] * a;
      minv[t][tid] = m[t];
      mn[t * kBlock + tid] = m[t];
    }
  }
  __syncthreads();
  if (tid < kBlock * kBlock) {
    const uint32_t t = tid / kBlock, j = tid % kBlock;
    float a = 0.f;
    for (uint32_t s = 0; s <= t; ++s) a = fmaf(ab[pair_b(t, s)], minv[s][j], a);
    mn[kBlock * kBlock + tid] = a;
  }
}

__device__ __forceinline__ uint32_t smem_at(const void *p) { return (uint32_t)__cvta_generic_to_shared(p); }
constexpr uint32_t kWaitLimit = 1u << 22;
__device__ __forceinline__ bool wait_bounded(uint64_t *bar, uint32_t parity) {
  for (uint32_t i = 0; i < kWaitLimit; ++i) {
    uint32_t ok;
    asm volatile("{\n .reg .pred p;\n mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n selp.u32 %0, 1, 0, p;\n}" : "=r"(ok) : "r"(smem_at(bar)), "r"(parity) : "memory");
    if (ok) return true;
  }
  return false;
}
// Two fp32 numbers in one register pair.
using f2 = unsigned long long;
__device__ __forceinline__ f2 fma2(f2 a, f2 b, f2 c) {
  f2 d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ f2 mul2(f2 a, f2 b) {
  f2 d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ f2 both(float v) {
  f2 d;
  asm("mov.b64 %0, {%1, %1};" : "=l"(d) : "f"(v));
  return d;
}
__device__ __forceinline__ float add_halves(f2 a) {
  float lo, hi;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(a));
  return lo + hi;
}
// N consecutive pairs, N = 1 or 2.
template <int N> __device__ __forceinline__ void load_pairs(const float *p, f2 *o) {
  if constexpr (N == 2) {
    const ulonglong2 v = *reinterpret_cast<const ulonglong2 *>(p);
    o[0] = v.x;
    o[1] = v.y;
  } else {
    o[0] = *reinterpret_cast<const f2 *>(p);
  }
}
template <int N> __device__ __forceinline__ void store_pairs(float *p, const f2 *o) {
  if constexpr (N == 2) *reinterpret_cast<ulonglong2 *>(p) = make_ulonglong2(o[0], o[1]);
  else *reinterpret_cast<f2 *>(p) = o[0];
}

constexpr uint32_t kScanCols = 4, kScanThreads = 128, kStages = 3;  // and a warp that requests the records
__host__ __device__ constexpr uint32_t cta_cols(uint32_t lp) { return kScanThreads / lp * kScanCols; }

// E: 32-element steps of the key width. LP lanes share four columns; lane l holds elements (LP i + l) V .. + V - 1 of
// each, and ends up with the sums of token tok = l / (LP / 8) for CP of the columns. So that the sums can be exchanged
// without choosing registers by lane, slot t of a lane's sums is token t ^ tok and slot c column c ^ cmask.
template <int E, int LP> __global__ void __launch_bounds__(kScanThreads + 32, 1) delta_scan_kernel(const DeltaRows p, uint32_t first, uint32_t count) {
  constexpr uint32_t DP = E * 32, RF = block_floats(DP);
  constexpr int PER = DP / LP, V = PER % 4 ? 2 : 4, NV = PER / V, NP = V / 2, CG = LP / 8, CP = kScanCols / CG;
  static_assert(PER % 2 == 0 && (CG == 2 || CG == 4), "pairs of elements, two or four lanes per token");
  extern __shared__ __align__(16) float stage_mem[];
  __shared__ __align__(8) uint64_t landed[kStages], consumed[kStages];
  const uint32_t h = blockIdx.x, tid = threadIdx.x, l = tid % LP, tok = l / CG, cg = l % CG, cmask = cg * CP;
  const uint32_t c0 = blockIdx.y * cta_cols(LP) + tid / LP * kScanCols, blocks = (count + kBlock - 1) / kBlock;
  if (tid == 0) {
    const uint32_t cols = min(cta_cols(LP), p.vp - blockIdx.y * cta_cols(LP)), warps = cols * LP / (32 * kScanCols);
    for (uint32_t i = 0; i < kStages; ++i) {
      asm volatile("mbarrier.init.shared::cta.b64 [%0], 1;" ::"r"(smem_at(&landed[i])) : "memory");
      asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(smem_at(&consumed[i])), "r"(warps) : "memory");
    }
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  __syncthreads();
  if (tid >= kScanThreads) {  // a record is one piece of memory: one lane requests them, a ring of stages ahead
    if (tid > kScanThreads) return;
    const float *recs = p.blocks + (size_t)h * RF;
    uint32_t b = 0;
    for (; b < blocks; ++b) {
      const uint32_t s = b % kStages, bar = smem_at(&landed[s]);
      if (b >= kStages && !wait_bounded(&consumed[s], (b / kStages - 1) & 1)) break;
      asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(bar), "r"(RF * 4u) : "memory");
      asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(smem_at(stage_mem + s * RF)),
                   "l"(recs + (size_t)b * p.heads * RF), "r"(RF * 4u), "r"(bar)
                   : "memory");
    }
    if (b < blocks) {  // given up: what is still on its way lands before the CTA's memory is given back
      *p.error = 4;
      for (uint32_t i = b - kStages; i < b; ++i) wait_bounded(&landed[i % kStages], i / kStages & 1);
    }
    return;
  }
  if (c0 >= p.vp) return;  // a whole warp: vp is a multiple of 16
  float *state = p.state + ((size_t)h * p.vp + c0) * DP;
  auto state_at = [&](uint32_t c, int i) { return state + (size_t)(c ^ cmask) * DP + (i * LP + l) * V; };
  f2 S[kScanCols][NV * NP];
  const bool fresh = first == 0 && *p.pos == 0;
#pragma unroll
  for (int c = 0; c < (int)kScanCols; ++c)
#pragma unroll
    for (int i = 0; i < NV; ++i) {
#pragma unroll
      for (int j = 0; j < NP; ++j) S[c][i * NP + j] = 0;
      if (!fresh) load_pairs<NP>(state_at(c, i), &S[c][i * NP]);
    }
  float *vrow = p.v + ((size_t)(first + tok) * p.heads + h) * p.vp + c0 + cmask;
  const size_t vstep = (size_t)kBlock * p.heads * p.vp;
  float vnext[CP];
  auto next_values = [&](uint32_t b) {
    const bool have = b * kBlock + tok < count;
#pragma unroll
    for (int c = 0; c < CP; ++c) vnext[c] = have ? vrow[b * vstep + c] : 0.f;
  };
  next_values(0);
  for (uint32_t b = 0; b < blocks; ++b) {
    float w[CP], o[CP], u[CP];
#pragma unroll
    for (int c = 0; c < CP; ++c) w[c] = vnext[c];
    if (b + 1 < blocks) next_values(b + 1);
    if (!__all_sync(0xffffffffu, wait_bounded(&landed[b % kStages], b / kStages & 1))) {
      *p.error = 4;
      return;
    }
    const float *st = stage_mem + (b % kStages) * RF, *mn = st + 25 * DP + tok * kBlock;
    f2 acc[2][kBlock][kScanCols];
#pragma unroll
    for (int r = 0; r < 2; ++r)
#pragma unroll
      for (int t = 0; t < (int)kBlock; ++t)
#pragma unroll
        for (int c = 0; c < (int)kScanCols; ++c) acc[r][t][c] = 0;
#pragma unroll
    for (int i = 0; i < NV; ++i)
#pragma unroll
      for (int t = 0; t < (int)kBlock; ++t)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          f2 x[NP];
          load_pairs<NP>(st + (r * kBlock + (t ^ tok)) * DP + (i * LP + l) * V, x);
#pragma unroll
          for (int j = 0; j < NP; ++j)
#pragma unroll
            for (int c = 0; c < (int)kScanCols; ++c) acc[r][t][c] = fma2(S[c][i * NP + j], x[j], acc[r][t][c]);
        }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      f2 x[NP];
      load_pairs<NP>(st + 3 * kBlock * DP + (i * LP + l) * V, x);
#pragma unroll
      for (int j = 0; j < NP; ++j)
#pragma unroll
        for (int c = 0; c < (int)kScanCols; ++c) S[c][i * NP + j] = mul2(S[c][i * NP + j], x[j]);
    }
    float sum[2][kBlock][kScanCols];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
#pragma unroll
      for (int t = 0; t < (int)kBlock; ++t)
#pragma unroll
        for (int c = 0; c < (int)kScanCols; ++c) sum[r][t][c] = add_halves(acc[r][t][c]);
#pragma unroll
      for (int bit = kBlock / 2; bit; bit /= 2)
#pragma unroll
        for (int t = 0; t < bit; ++t)
#pragma unroll
          for (int c = 0; c < (int)kScanCols; ++c) sum[r][t][c] += __shfl_xor_sync(0xffffffffu, sum[r][t + bit][c], bit * CG);
#pragma unroll
      for (int n = kScanCols / 2, x = CG / 2; x; n /= 2, x /= 2)
#pragma unroll
        for (int c = 0; c < n; ++c) sum[r][0][c] += __shfl_xor_sync(0xffffffffu, sum[r][0][c + n], x);
    }
#pragma unroll
    for (int c = 0; c < CP; ++c) {
      w[c] -= sum[0][0][c];
      o[c] = sum[1][0][c];
      u[c] = 0.f;
    }
#pragma unroll
    for (int s = 0; s < (int)kBlock; ++s) {
      const float m = mn[s], n = mn[kBlock * kBlock + s];
#pragma unroll
      for (int c = 0; c < CP; ++c) {
        const float x = __shfl_sync(0xffffffffu, w[c], s * CG + cg, LP);
        u[c] = fmaf(m, x, u[c]);
        o[c] = fmaf(n, x, o[c]);
      }
    }
    if (b * kBlock + tok < count) {
#pragma unroll
      for (int c = 0; c < CP; ++c) vrow[b * vstep + c] = o[c];
    }
    f2 us[kBlock][kScanCols];  // column c ^ cmask is with the lane of its group
#pragma unroll
    for (int s = 0; s < (int)kBlock; ++s)
#pragma unroll
      for (int c = 0; c < (int)kScanCols; ++c) us[s][c] = both(__shfl_sync(0xffffffffu, u[c % CP], s * CG + ((c / CP) ^ cg), LP));
#pragma unroll
    for (int s = 0; s < (int)kBlock; ++s)
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        f2 x[NP];
        load_pairs<NP>(st + (2 * kBlock + s) * DP + (i * LP + l) * V, x);
#pragma unroll
        for (int j = 0; j < NP; ++j)
#pragma unroll
          for (int c = 0; c < (int)kScanCols; ++c) S[c][i * NP + j] = fma2(x[j], us[s][c], S[c][i * NP + j]);
      }
    __syncwarp();
    if ((tid & 31) == 0) asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(smem_at(&consumed[b % kStages])) : "memory");
  }
#pragma unroll
  for (int c = 0; c < (int)kScanCols; ++c)
#pragma unroll
    for (int i = 0; i < NV; ++i) store_pairs<NP>(state_at(c, i), &S[c][i * NP]);
}

constexpr int kFinishThreads = 256;
template <class T> __global__ void __launch_bounds__(kFinishThreads) delta_finish_kernel(const DeltaRows p) {
  const uint32_t m = blockIdx.x, lane = threadIdx.x & 31, h = blockIdx.y * (kFinishThreads / 32) + (threadIdx.x >> 5);
  if (m + p.ntaps >= p.T) {  // one of the last ntaps tokens: later ones look back at it
    const uint32_t pieces = p.raw_ld * sizeof(T) / 16;
    const uint4 *src = static_cast<const uint4 *>(p.raw) + (size_t)m * pieces;
    uint4 *dst = static_cast<uint4 *>(p.ring) + (size_t)((*p.pos + m) % p.ntaps) * pieces;
    for (uint32_t c = blockIdx.y * kFinishThreads + threadIdx.x; c < pieces; c += gridDim.y * kFinishThreads) dst[c] = src[c];
  }
  if (h >= p.heads || lane * 8 >= p.vp) return;  // a lane holds eight columns
  const uint32_t lanes = 0xffffffffu >> (32 - p.vp / 8);
  float y[8], z[8], w[8], ss = 0.f;
  load8(p.v + ((size_t)m * p.heads + h) * p.vp + lane * 8, y);  // padded columns are zero
  load8(p.z + (size_t)m * p.z_ld + p.z_gate + h * p.vp + lane * 8, z);
  load8(p.norm + lane * 8, w);
#pragma unroll
  for (int i = 0; i < 8; ++i) ss = fmaf(y[i], y[i], ss);
  float tot = 0.f;
  for (uint32_t i = 0; i < p.vp / 8; ++i) tot += __shfl_sync(lanes, ss, i);
  const float r = 1.0f / sqrtf(tot / (float)p.vdim + p.eps);
#pragma unroll
  for (int i = 0; i < 8; ++i) y[i] *= r * w[i] * fast_sigmoid(z[i]);
  store8(static_cast<T *>(p.out) + (size_t)m * p.out_ld + h * p.vp + lane * 8, y);
}

// ---- one token ----
constexpr uint32_t kStepThreads = 256, kStepCols = 32, kStepLanes = 8, kRowGroups = kStepThreads / 8, kAhead = 10;

// grid: heads x cluster; a cluster is a head, a CTA 32 of its columns. E: 32-element steps of the key width.
template <class T, int E> __global__ void __launch_bounds__(kStepThreads) delta_step_kernel(const DeltaRows p, uint32_t cluster) {
  constexpr uint32_t DP = E * 32;
  __shared__ float q_s[DP], k_s[DP], g_s[DP], v_s[kStepCols], gate_s[kStepCols], part[kStepThreads / 32], peers[8];
  const uint32_t h = blockIdx.x / cluster, rank = blockIdx.x % cluster, tid = threadIdx.x, lane = tid & 31, col = tid / kStepLanes, l = tid % kStepLanes;
  const uint32_t kv = h / (p.heads / p.kv_heads), c0 = rank * kStepCols, cols = c0 < p.vp ? min(kStepCols, p.vp - c0) : 0u;
  const bool active = col < cols;
  if (cluster > 1) asm volatile("barrier.cluster.arrive.relaxed.aligned;" ::: "memory");  // waited for before another CTA's memory is touched
  // Rows of the projections' second steps, 8 lanes each: DP decays, then this CTA's gates. The first ones, and the
  // state, do not depend on the kernel before.
  const uint32_t rows = DP + cols, steps = p.low_ld / 64, items = (rows + kRowGroups - 1) / kRowGroups * steps;
  auto item_row = [&](uint32_t i) { return i / steps * kRowGroups + col; };
  auto item_weights = [&](uint32_t i, uint32_t row) {
    const size_t r = row < DP ? (size_t)h * DP + row : (size_t)p.z_gate + h * p.vp + c0 + row - DP;
    return p.wl + r * p.low_ld + i % steps * 64 + l * 8;
  };
  uint4 wa[kAhead];
#pragma unroll
  for (uint32_t i = 0; i < kAhead; ++i) {
    wa[i] = make_uint4(0, 0, 0, 0);
    if (i < items && item_row(i) < rows) wa[i] = ldg_stream(item_weights(i, item_row(i)));
  }
  float4 S[E];
  float *state = p.state + ((size_t)h * p.vp + c0 + col) * DP + l * 4;
  const uint32_t pos = *p.pos;
#pragma unroll
  for (int i = 0; i < E; ++i) S[i] = active && pos ? *reinterpret_cast<const float4 *>(state + i * 32) : make_float4(0.f, 0.f, 0.f, 0.f);
  // convolution: query and key channels, this CTA's value channels; the past tokens' part
  constexpr int ROUNDS = (2 * DP + kStepCols + kStepThreads - 1) / kStepThreads;
  uint32_t chan[ROUNDS];
  float past[ROUNDS], last[ROUNDS];
#pragma unroll
  for (int r = 0; r < ROUNDS; ++r) {
    const uint32_t i = r * kStepThreads + tid;
    past[r] = last[r] = 0.f;
    chan[r] = i < DP ? kv * DP + i : i < 2 * DP ? p.k_col + kv * DP + i - DP : p.v_col + h * p.vp + c0 + i - 2 * DP;
    if (i >= 2 * DP + cols) continue;
    const float *w = p.taps + (size_t)chan[r] * p.ntaps;
    last[r] = w[p.ntaps - 1];
    const uint32_t back = min(p.ntaps - 1, pos);
    uint32_t slot = (pos - back) % p.ntaps;
#pragma unroll 4
    for (uint32_t j = p.ntaps - 1 - back; j < p.ntaps - 1; ++j) {
      past[r] = fmaf(load1(static_cast<const T *>(p.ring) + (size_t)slot * p.raw_ld + chan[r]), w[j], past[r]);
      slot = slot + 1 == p.ntaps ? 0u : slot + 1;
    }
  }
  if (p.use_pdl) {
    asm volatile("griddepcontrol.launch_dependents;");
    asm volatile("griddepcontrol.wait;" ::: "memory");
  }
#pragma unroll
  for (int r = 0; r < ROUNDS; ++r) {
    const uint32_t i = r * kStepThreads + tid;
    if (i >= 2 * DP + cols) continue;
    const T x = static_cast<const T *>(p.raw)[chan[r]];
    float a = fmaf(load1(&x), last[r], past[r]);
    a *= fast_sigmoid(a);
    if (i < DP) q_s[i] = a;
    else if (i < 2 * DP) k_s[i - DP] = a;
    else v_s[i - 2 * DP] = a;
    // the slot of this position is read by no one in this step; heads that share a key head write the same number
    static_cast<T *>(p.ring)[(size_t)(pos % p.ntaps) * p.raw_ld + chan[r]] = x;
  }
  auto finish_row = [&](uint32_t row, float z) {
#pragma unroll
    for (uint32_t o = 1; o < 8; o <<= 1) z += __shfl_xor_sync(0xffffffffu, z, o);
    if (l || row >= rows) return;
    if (row < DP) g_s[row] = expf(-p.rate[h * DP + row] * softplus_f(z + p.bias[h * DP + row]));
    else gate_s[row - DP] = sigmoid_f(z);
  };
  auto dot8 = [&](uint32_t i, uint32_t row, const uint4 &w) {
    float wf[8], x[8], a = 0.f;
    unpack8(w, wf);
    load8(static_cast<const T *>(p.low) + (row < DP ? 0u : p.low_ld) + i % steps * 64 + l * 8, x);
#pragma unroll
    for (int e = 0; e < 8; ++e) a = fmaf(wf[e], x[e], a);
    return a;
  };
  float z = 0.f;
#pragma unroll
  for (uint32_t i = 0; i < kAhead; ++i) {
    if (i >= items) break;
    const uint32_t row = item_row(i);
    if (row < rows) z += dot8(i, row, wa[i]);
    if (i % steps == steps - 1) {
      finish_row(row, z);
      z = 0.f;
    }
  }
  for (uint32_t i = kAhead; i < items; ++i) {
    const uint32_t row = item_row(i);
    if (row < rows) z += dot8(i, row, ldg_stream(item_weights(i, row)));
    if (i % steps == steps - 1) {
      finish_row(row, z);
      z = 0.f;
    }
  }
  __syncthreads();
  float qq = 0.f, kk = 0.f;  // every warp for itself
#pragma unroll
  for (int i = 0; i < E; ++i) {
    qq = fmaf(q_s[i * 32 + lane], q_s[i * 32 + lane], qq);
    kk = fmaf(k_s[i * 32 + lane], k_s[i * 32 + lane], kk);
  }
  const float rq = 1.0f / sqrtf(warp_sum(qq) + kUnitEps) / sqrtf((float)p.dim), rk = 1.0f / sqrtf(warp_sum(kk) + kUnitEps);
  float a = 0.f, o = 0.f;
  float4 k[E];
#pragma unroll
  for (int i = 0; i < E; ++i) {
    const float4 g = *reinterpret_cast<const float4 *>(g_s + i * 32 + l * 4), x = *reinterpret_cast<const float4 *>(k_s + i * 32 + l * 4);
    k[i] = make_float4(x.x * rk, x.y * rk, x.z * rk, x.w * rk);
    S[i] = make_float4(S[i].x * g.x, S[i].y * g.y, S[i].z * g.z, S[i].w * g.w);
    a = fmaf(S[i].x, k[i].x, fmaf(S[i].y, k[i].y, fmaf(S[i].z, k[i].z, fmaf(S[i].w, k[i].w, a))));
  }
#pragma unroll
  for (uint32_t x = 1; x < kStepLanes; x <<= 1) a += __shfl_xor_sync(0xffffffffu, a, x);
  const float u = active ? p.beta[h] * (v_s[col] - a) : 0.f;
#pragma unroll
  for (int i = 0; i < E; ++i) {
    const float4 x = *reinterpret_cast<const float4 *>(q_s + i * 32 + l * 4);
    S[i] = make_float4(fmaf(k[i].x, u, S[i].x), fmaf(k[i].y, u, S[i].y), fmaf(k[i].z, u, S[i].z), fmaf(k[i].w, u, S[i].w));
    o = fmaf(S[i].x, x.x, fmaf(S[i].y, x.y, fmaf(S[i].z, x.z, fmaf(S[i].w, x.w, o))));
    if (active) *reinterpret_cast<float4 *>(state + i * 32) = S[i];
  }
#pragma unroll
  for (uint32_t x = 1; x < kStepLanes; x <<= 1) o += __shfl_xor_sync(0xffffffffu, o, x);
  o *= rq;
  const float ss = warp_sum(active && l == 0 ? o * o : 0.f);
  if (lane == 0) part[tid >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
#pragma unroll
  for (uint32_t w = 0; w < kStepThreads / 32; ++w) tot += part[w];
  if (cluster > 1) {
    cg::cluster_group cl = cg::this_cluster();
    asm volatile("barrier.cluster.wait.aligned;" ::: "memory");
    if (tid < cluster) *cl.map_shared_rank(&peers[rank], tid) = tot;
    cl.sync();
    tot = 0.f;
    for (uint32_t i = 0; i < cluster; ++i) tot += peers[i];
  }
  if (active && l == 0) {
    const float y = o / sqrtf(tot / (float)p.vdim + p.eps) * p.norm[c0 + col] * gate_s[col];
    store1(static_cast<T *>(p.out) + h * p.vp + c0 + col, y);
  }
}

bool sane(const DeltaRows &p) {
  return p.T && p.heads && p.kv_heads && p.heads % p.kv_heads == 0 && p.ntaps && p.dp % 32 == 0 && p.dp && p.dp <= 256 && p.vp % 16 == 0 && p.vp && p.vp <= 256;
}

template <class T, int TAPS> cudaError_t launch_blocks(const DeltaRows &p, uint32_t first, uint32_t count, cudaStream_t s) {
  const dim3 grid(p.heads, (count + kBlock - 1) / kBlock);
  if (std::max(p.dp, p.vp) <= 128) delta_blocks_kernel<T, TAPS, 128><<<grid, 128, 0, s>>>(p, first);
  else delta_blocks_kernel<T, TAPS, 256><<<grid, 256, 0, s>>>(p, first);
  return cudaGetLastError();
}
template <int E, int LP> cudaError_t launch_scan(const DeltaRows &p, uint32_t first, uint32_t count, cudaStream_t s) {
  constexpr size_t smem = (size_t)kStages * block_floats(E * 32) * sizeof(float);
  if (cudaError_t e = cudaFuncSetAttribute(delta_scan_kernel<E, LP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)) return e;
  delta_scan_kernel<E, LP><<<dim3(p.heads, (p.vp + cta_cols(LP) - 1) / cta_cols(LP)), kScanThreads + 32, smem, s>>>(p, first, count);
  return cudaGetLastError();
}
// f<E>() for a key width of 32 E.
template <class F> cudaError_t by_width(uint32_t dp, F f) {
  switch (dp / 32) {
    case 1: return f(std::integral_constant<int, 1>());
    case 2: return f(std::integral_constant<int, 2>());
    case 3: return f(std::integral_constant<int, 3>());
    case 4: return f(std::integral_constant<int, 4>());
    case 5: return f(std::integral_constant<int, 5>());
    case 6: return f(std::integral_constant<int, 6>());
    case 7: return f(std::integral_constant<int, 7>());
    default: return f(std::integral_constant<int, 8>());
  }
}
template <class T, int E> cudaError_t launch_step(const DeltaRows &p, cudaStream_t s) {
  uint32_t cluster = 1;
  while (cluster * kStepCols < p.vp) cluster *= 2;  // at most 8
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(p.heads * cluster);
  cfg.blockDim = dim3(kStepThreads);
  cfg.stream = s;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = cluster;
  attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = p.use_pdl ? 2 : 1;
  return cudaLaunchKernelEx(&cfg, delta_step_kernel<T, E>, p, cluster);
}

}  // namespace

size_t delta_block_floats(uint32_t T, uint32_t heads, uint32_t dp) {
  return (size_t)((std::min(T, kDeltaSlice) + kBlock - 1) / kBlock) * heads * block_floats(dp);
}

cudaError_t launch_delta_rows(const DeltaRows &p, bool f32, cudaStream_t s) {
  if (!sane(p) || p.z_ld % 8 || p.z_gate % 8) return cudaErrorInvalidValue;
  for (uint32_t first = 0; first < p.T; first += kDeltaSlice) {
    const uint32_t count = std::min(kDeltaSlice, p.T - first);
    cudaError_t e = f32 ? (p.ntaps == 4 ? launch_blocks<float, 4>(p, first, count, s) : launch_blocks<float, 0>(p, first, count, s))
                        : (p.ntaps == 4 ? launch_blocks<bf16, 4>(p, first, count, s) : launch_blocks<bf16, 0>(p, first, count, s));
    if (e == cudaSuccess) e = by_width(p.dp, [&](auto w) {
      constexpr int E = decltype(w)::value;
      if constexpr (E % 2 == 0)  // few heads: more SMs, with fewer columns each
        if (p.heads * (p.vp / 16) <= (uint32_t)p.sms) return launch_scan<E, 32>(p, first, count, s);
      return launch_scan<E, 16>(p, first, count, s);
    });
    if (e != cudaSuccess) return e;
  }
  const dim3 grid(p.T, (p.heads + kFinishThreads / 32 - 1) / (kFinishThreads / 32));
  if (f32) delta_finish_kernel<float><<<grid, kFinishThreads, 0, s>>>(p);
  else delta_finish_kernel<bf16><<<grid, kFinishThreads, 0, s>>>(p);
  return cudaGetLastError();
}

cudaError_t launch_delta_step(const DeltaRows &p, bool f32, cudaStream_t s) {
  if (!sane(p) || p.T != 1 || p.low_ld % 64) return cudaErrorInvalidValue;
  return by_width(p.dp, [&](auto w) { return f32 ? launch_step<float, decltype(w)::value>(p, s) : launch_step<bf16, decltype(w)::value>(p, s); });
}

}  // namespace vkl
