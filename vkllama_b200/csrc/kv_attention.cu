// Causal attention over a cache with grouped queries, of keys and values or of rows that are both, optionally only
// over the last `window` positions. A position may also enter as a temperature of its query and as a bias by
// distance (rotations are in the cache already); a head may have a sink in its denominator and a gate on its
// output. Scores, softmax and accumulation are fp32 (scores in units of log2).
//
// row kernel   one token (decode), few tokens, and every call of the 32-bit mode. A CTA takes a query row, a
//              key head and a range of the cache, and up to four of the head's query heads: every cache row is
//              read once (where the keys are the values, the registers that held a row for the score are added
//              to the outputs). Ranges are merged by the CTA that finishes last.
// tile kernel  64 query rows of a head per CTA on mma.sync m16n8k16 (bf16, fp32 accumulate): a 64-row cache tile
//              is copied to shared memory once (cp.async, double buffered) and serves Q.K^T directly; it, or the
//              value tile beside it, serves P.V through transposing loads. The 127 biases that a tile pair can need travel with the tile.
#include <algorithm>

#include "rows.cuh"

namespace vkl {
namespace {

constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ float query_scale(const KvAttn &p, uint32_t pos) {
  float s = p.scale;
  if (p.temp_coef != 0.f) s *= 1.0f + p.temp_coef * logf(floorf((float)(pos + 1) / p.temp_every) + 1.0f);
  return s * kLog2e;
}
__device__ __forceinline__ float bias_at(const KvAttn &p, uint32_t h, uint32_t n) {
  return p.bias ? p.bias[(size_t)h * p.bias_n + min(n, p.bias_n - 1)] : 0.f;
}

// First position that a query at `pos` sees.
__device__ __forceinline__ uint32_t first_seen(const KvAttn &p, uint32_t pos) { return p.window && pos >= p.window ? pos + 1 - p.window : 0u; }
__device__ __forceinline__ float sink_log2(const KvAttn &p, uint32_t h) { return p.sink ? p.sink[h] * kLog2e : -INFINITY; }

constexpr int kRowThreads = 128;
constexpr uint32_t kMaxSplits = 32, kSplitRows = 64;  // a split holds about this many cache rows: a short cache uses fewer splits

template <class T> struct Raw8;
template <> struct Raw8<bf16> {
  uint4 u = make_uint4(0, 0, 0, 0);
  __device__ __forceinline__ void load(const bf16 *p) { u = *reinterpret_cast<const uint4 *>(p); }
  __device__ __forceinline__ void get(float (&v)[8]) const { unpack8(u, v); }
};
template <> struct Raw8<float> {
  float4 a = make_float4(0.f, 0.f, 0.f, 0.f), b = make_float4(0.f, 0.f, 0.f, 0.f);
  __device__ __forceinline__ void load(const float *p) {
    a = *reinterpret_cast<const float4 *>(p);
    b = *reinterpret_cast<const float4 *>(p + 4);
  }
  __device__ __forceinline__ void get(float (&v)[8]) const {
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
  }
};

// LPR lanes hold one cache row (8 values each), NQ query heads per CTA, SEP: values in a cache of their own.
// grid (kv heads x head groups, rows, splits)
template <class T, int LPR, int NQ, bool SEP> __global__ void __launch_bounds__(kRowThreads) kv_row_kernel(const KvAttn p) {
  constexpr uint32_t NS = kRowThreads / LPR, U = SEP && sizeof(T) == 4 ? 2 : 4, DMAX = LPR * 8;
  __shared__ float sm_o[kRowThreads / 32][NQ][DMAX], sm_m[kRowThreads / 32][NQ], sm_l[kRowThreads / 32][NQ];
  __shared__ float sm_pm[kMaxSplits][NQ], sm_pl[kMaxSplits][NQ];
  __shared__ uint32_t last_s;
  __shared__ float2 turn_s[kMaxPairs];
  const uint32_t per = p.heads / p.kv_heads, groups = (per + NQ - 1) / NQ;
  const uint32_t g = blockIdx.x / groups, hg = blockIdx.x % groups, h0 = g * per + hg * NQ, nh = min((uint32_t)NQ, per - hg * NQ);
  const uint32_t m = blockIdx.y, split = blockIdx.z, tid = threadIdx.x, sub = tid / LPR, l = tid % LPR, e0 = l * 8, warp = tid >> 5;
  const bool ev = e0 < p.dp, vv = SEP && e0 < p.vp;
  if (p.use_pdl) {
    asm volatile("griddepcontrol.launch_dependents;");  // the out-projection asks for its weights meanwhile
    asm volatile("griddepcontrol.wait;" ::: "memory");
  }
  const uint32_t pos = *p.pos + m, vis = pos + 1, lo = first_seen(p, pos);
  const uint32_t splits = min(p.splits, (vis - lo + kSplitRows - 1) / kSplitRows);
  if (split >= splits) return;
  uint32_t chunk = (vis - lo + splits - 1) / splits;
  chunk = (chunk + 31) & ~31u;
  const uint32_t c0 = min(lo + split * chunk, vis), c1 = min(c0 + chunk, vis);
  const float qs = query_scale(p, pos);
  float rq = 1.f;
  if (p.qk.q) {  // one raw token: every CTA norms and turns its queries, the ones that see the token itself its key
    const bool newest = c0 < vis && c1 == vis && p.qk.kcache;
    const T *qr = static_cast<const T *>(p.qk.q), *kr = qr + p.qk.k_col;
    if (tid < p.qk.pairs) turn_s[tid] = turn_of(pos, p.qk.freq[tid]);
    float sq = 0.f, sk = 0.f, v[8];
    for (uint32_t n = tid * 8; n < p.heads * p.dp; n += kRowThreads * 8) {
      load8(qr + n, v);
      sq = square_sum8(v, sq);
    }
    for (uint32_t n = tid * 8; newest && n < p.kv_heads * p.dp; n += kRowThreads * 8) {
      load8(kr + n, v);
      sk = square_sum8(v, sk);
    }
    const float2 ss = block_sum2<kRowThreads / 32>(sq, sk);  // also: the angles are in place
    rq = 1.0f / sqrtf(ss.x / (float)(p.heads * p.qk.dim) + p.qk.eps);
    if (newest && tid < p.dp / 8) {
      const uint32_t c = g * p.dp + tid * 8;
      load8(kr + c, v);
      norm_and_turn(v, p.qk.kw ? p.qk.kw + c : nullptr, 1.0f / sqrtf(ss.y / (float)(p.kv_heads * p.qk.dim) + p.qk.eps), tid * 8, turn_s, p.qk.pairs);
      store8(cache_slot<T>(p.qk.kcache, p.dp, p.maxlen, pos, c), v);
    }
    __syncthreads();
  }

  float q[NQ][8], acc[NQ][8], mx[NQ], sum[NQ];
#pragma unroll
  for (int i = 0; i < NQ; ++i) {
    Raw8<T> r;
    if (ev && i < nh) r.load(static_cast<const T *>(p.q) + (size_t)m * p.q_ld + (size_t)(h0 + i) * p.dp + e0);
    r.get(q[i]);
    if (p.qk.q && ev && i < nh) norm_and_turn(q[i], p.qk.qw ? p.qk.qw + (size_t)(h0 + i) * p.dp + e0 : nullptr, rq, e0, turn_s, p.qk.pairs);
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      q[i][e] *= qs;
      acc[i][e] = 0.f;
    }
    mx[i] = -INFINITY;
    sum[i] = 0.f;
  }
  const T *base = static_cast<const T *>(p.cache) + (size_t)g * p.maxlen * p.dp + e0;
  const T *vbase = SEP ? static_cast<const T *>(p.vcache) + (size_t)g * p.maxlen * p.vp + e0 : nullptr;
  for (uint32_t jb = c0; jb < c1; jb += NS * U) {  // the same trip count for every thread
    Raw8<T> kr[U], vr[SEP ? U : 1];
    float s[U][NQ];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const uint32_t j = jb + u * NS + sub;
      if (ev && j < c1) kr[u].load(base + (size_t)j * p.dp);
      if constexpr (SEP) {
        if (vv && j < c1) vr[u].load(vbase + (size_t)j * p.vp);
      }
#pragma unroll
      for (int i = 0; i < NQ; ++i) s[u][i] = (j < c1 && i < nh) ? bias_at(p, h0 + i, pos - j) : -INFINITY;
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      float k[8];
      kr[u].get(k);
#pragma unroll
      for (int i = 0; i < NQ; ++i) {
        float d = 0.f;
#pragma unroll
        for (int e = 0; e < 8; ++e) d = fmaf(q[i][e], k[e], d);
#pragma unroll
        for (int o = LPR / 2; o > 0; o >>= 1) d += __shfl_xor_sync(0xffffffffu, d, o);
        s[u][i] += d;
      }
    }
#pragma unroll
    for (int i = 0; i < NQ; ++i) {
      float mn = mx[i];
#pragma unroll
      for (int u = 0; u < U; ++u) mn = fmaxf(mn, s[u][i]);
      const float ref = mn == -INFINITY ? 0.f : mn, corr = exp2f(mx[i] - ref);
      mx[i] = mn;
      sum[i] *= corr;
#pragma unroll
      for (int e = 0; e < 8; ++e) acc[i][e] *= corr;
#pragma unroll
      for (int u = 0; u < U; ++u) {
        s[u][i] = exp2f(s[u][i] - ref);
        sum[i] += s[u][i];
      }
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      float v[8];
      if constexpr (SEP) vr[u].get(v);
      else kr[u].get(v);
#pragma unroll
      for (int i = 0; i < NQ; ++i)
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[i][e] = fmaf(s[u][i], v[e], acc[i][e]);
    }
  }
  // merge the warp's row streams, then the warps, in a fixed order
#pragma unroll
  for (int i = 0; i < NQ; ++i) {
#pragma unroll
    for (int o = LPR; o < 32; o <<= 1) {
      const float om = __shfl_xor_sync(0xffffffffu, mx[i], o), os = __shfl_xor_sync(0xffffffffu, sum[i], o);
      const float M = fmaxf(mx[i], om), ref = M == -INFINITY ? 0.f : M, ca = exp2f(mx[i] - ref), cb = exp2f(om - ref);
      mx[i] = M;
      sum[i] = sum[i] * ca + os * cb;
#pragma unroll
      for (int e = 0; e < 8; ++e) acc[i][e] = acc[i][e] * ca + __shfl_xor_sync(0xffffffffu, acc[i][e], o) * cb;
    }
    if ((tid & 31) < LPR) {
#pragma unroll
      for (int e = 0; e < 8; ++e) sm_o[warp][i][e0 + e] = acc[i][e];
      if (l == 0) {
        sm_m[warp][i] = mx[i];
        sm_l[warp][i] = sum[i];
      }
    }
  }
  __syncthreads();
  const size_t unit = (size_t)m * gridDim.x + blockIdx.x;
  const uint32_t rec = p.vp + 4;
  float *part = p.scratch + unit * p.splits * NQ * rec;  // [split][NQ][vp + 4]: output, max, sum
  auto write = [&](uint32_t i, uint32_t d, float v) {
    if (p.gate) v *= p.gate[(size_t)m * p.gate_ld + h0 + i];
    store1(static_cast<T *>(p.out) + (size_t)m * p.out_ld + (size_t)(h0 + i) * p.vp + d, v);
  };
  for (uint32_t x = tid; x < nh * p.vp; x += kRowThreads) {
    const uint32_t i = x / p.vp, d = x % p.vp;
    const float sink = splits == 1 ? sink_log2(p, h0 + i) : -INFINITY;  // counts once: here, or in the merge
    float M = sink;
#pragma unroll
    for (int w = 0; w < kRowThreads / 32; ++w) M = fmaxf(M, sm_m[w][i]);
    const float ref = M == -INFINITY ? 0.f : M;
    float num = 0.f, den = exp2f(sink - ref);
#pragma unroll
    for (int w = 0; w < kRowThreads / 32; ++w) {
      const float c = exp2f(sm_m[w][i] - ref);
      num += c * sm_o[w][i][d];
      den += c * sm_l[w][i];
    }
    if (splits == 1) {
      write(i, d, num / den);
    } else {
      float *r = part + ((size_t)split * NQ + i) * rec;
      r[d] = num;
      if (d == 0) {
        r[p.vp] = M;
        r[p.vp + 1] = den;
      }
    }
  }
  if (splits == 1) return;
  __threadfence();
  __syncthreads();
  if (tid == 0) last_s = atomicAdd(&p.counters[unit], 1u) == splits - 1;
  __syncthreads();
  if (!last_s) return;
  __threadfence();
  for (uint32_t x = tid; x < splits * nh; x += kRowThreads) {
    const float *r = part + ((size_t)(x / nh) * NQ + x % nh) * rec + p.vp;
    sm_pm[x / nh][x % nh] = __ldcg(r);
    sm_pl[x / nh][x % nh] = __ldcg(r + 1);
  }
  __syncthreads();
  for (uint32_t x = tid; x < nh * (p.vp / 4); x += kRowThreads) {
    const uint32_t i = x / (p.vp / 4), d = x % (p.vp / 4) * 4;
    const float sink = sink_log2(p, h0 + i);
    float M = sink;  // split 0 is never empty: M becomes finite
    for (uint32_t s = 0; s < splits; ++s) M = fmaxf(M, sm_pm[s][i]);
    float4 num = make_float4(0.f, 0.f, 0.f, 0.f);
    float den = exp2f(sink - M);
#pragma unroll 8
    for (uint32_t s = 0; s < splits; ++s) {
      const float c = exp2f(sm_pm[s][i] - M);
      const float4 v = __ldcg(reinterpret_cast<const float4 *>(part + ((size_t)s * NQ + i) * rec + d));
      num.x = fmaf(c, v.x, num.x);
      num.y = fmaf(c, v.y, num.y);
      num.z = fmaf(c, v.z, num.z);
      num.w = fmaf(c, v.w, num.w);
      den = fmaf(c, sm_pl[s][i], den);
    }
    write(i, d, num.x / den);
    write(i, d + 1, num.y / den);
    write(i, d + 2, num.z / den);
    write(i, d + 3, num.w / den);
  }
  if (tid == 0) p.counters[unit] = 0;
}

template <class T, int LPR, bool SEP> cudaError_t launch_row(const KvAttn &p, cudaStream_t s) {
  const uint32_t per = p.heads / p.kv_heads;
  auto kern = per >= 3 ? kv_row_kernel<T, LPR, 4, SEP> : per == 2 ? kv_row_kernel<T, LPR, 2, SEP> : kv_row_kernel<T, LPR, 1, SEP>;
  const uint32_t nq = per >= 3 ? 4 : per;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(p.kv_heads * ((per + nq - 1) / nq), p.T, p.splits);
  cfg.blockDim = dim3(kRowThreads);
  cfg.stream = s;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = p.use_pdl ? 1 : 0;
  return cudaLaunchKernelEx(&cfg, kern, p);
}
template <class T, bool SEP> cudaError_t launch_row_d(const KvAttn &p, cudaStream_t s) {
  const uint32_t d = std::max(p.dp, p.vp);
  if (d <= 64) return launch_row<T, 8, SEP>(p, s);
  if (d <= 128) return launch_row<T, 16, SEP>(p, s);
  return launch_row<T, 32, SEP>(p, s);
}

// ------------------------------------------------------------------------------------------ tiles
__device__ __forceinline__ void mma_bf16(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void cp_async16(void *dst, const void *src, bool valid) {  // zero-fills when not valid
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src), "r"(valid ? 16u : 0u) : "memory");
}
__device__ __forceinline__ void cp_async4(void *dst, const void *src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

constexpr int QT = 64, KT = 64;
template <int D, bool SEP> struct TileSmem {
  static constexpr int LD = D + 8;  // padded rows: conflict-free fragment loads
  bf16 q[QT * LD];
  bf16 k[2][KT * LD];
  bf16 v[SEP ? 2 : 1][SEP ? KT * LD : 8];
  float bias[2][128];
};

// D: the wider of key and value rounded up to what is instantiated; dp, vp the widths in memory.
template <int D, bool SEP> __global__ void __launch_bounds__(128) kv_tile_kernel(const KvAttn p) {
  constexpr int LD = TileSmem<D, SEP>::LD;
  extern __shared__ __align__(16) unsigned char raw[];
  TileSmem<D, SEP> &sm = *reinterpret_cast<TileSmem<D, SEP> *>(raw);
  const uint32_t h = blockIdx.x, g = h / (p.heads / p.kv_heads), tiles = gridDim.y, m0 = (tiles - 1 - blockIdx.y) * QT;  // longest rows first
  const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, gq = lane >> 2, t = lane & 3;
  const uint32_t T = p.T, pos0 = *p.pos, vecs = p.dp / 8;
  const bf16 *cache = static_cast<const bf16 *>(p.cache) + (size_t)g * p.maxlen * p.dp;
  const uint32_t jmax = pos0 + min(m0 + QT, T), jmin = first_seen(p, pos0 + m0) / KT * KT;  // cache rows that some row of the tile sees
  auto fetch = [&](uint32_t j0, uint32_t b) {
    for (uint32_t i = tid; i < KT * (D / 8); i += 128) {
      const uint32_t r = i / (D / 8), c = i % (D / 8);
      const bool ok = j0 + r < jmax && c < vecs;
      cp_async16(&sm.k[b][r * LD + c * 8], cache + (ok ? (size_t)(j0 + r) * p.dp + c * 8 : 0), ok);
    }
    if constexpr (SEP) {
      const bf16 *vc = static_cast<const bf16 *>(p.vcache) + (size_t)g * p.maxlen * p.vp;
      for (uint32_t i = tid; i < KT * (D / 8); i += 128) {
        const uint32_t r = i / (D / 8), c = i % (D / 8);
        const bool ok = j0 + r < jmax && c < p.vp / 8;
        cp_async16(&sm.v[b][r * LD + c * 8], vc + (ok ? (size_t)(j0 + r) * p.vp + c * 8 : 0), ok);
      }
    }
    if (p.bias && tid < 127) {  // distance of (row r, column c): pos0 + m0 + r - j0 - c = entry r - c + 63
      const int n = (int)(pos0 + m0) - (int)j0 + (int)tid - 63;
      cp_async4(&sm.bias[b][tid], p.bias + (size_t)h * p.bias_n + min((uint32_t)max(n, 0), p.bias_n - 1));
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  for (uint32_t i = tid; i < QT * (D / 8); i += 128) {
    const uint32_t r = i / (D / 8), c = i % (D / 8);
    const bool ok = m0 + r < T && c < vecs;
    cp_async16(&sm.q[r * LD + c * 8], static_cast<const bf16 *>(p.q) + (ok ? (size_t)(m0 + r) * p.q_ld + (size_t)h * p.dp + c * 8 : 0), ok);
  }
  if (!p.bias)
    for (uint32_t i = tid; i < 256; i += 128) sm.bias[i >> 7][i & 127] = 0.f;
  fetch(jmin, 0);
  const uint32_t rl = warp * 16 + gq, rh = rl + 8;                                       // rows in the tile
  const uint32_t vis_lo = m0 + rl < T ? pos0 + m0 + rl + 1 : 0u, vis_hi = m0 + rh < T ? pos0 + m0 + rh + 1 : 0u;
  const uint32_t see_lo = first_seen(p, pos0 + m0 + rl), see_hi = first_seen(p, pos0 + m0 + rh);
  const float qs_lo = query_scale(p, pos0 + m0 + rl), qs_hi = query_scale(p, pos0 + m0 + rh);
  float o[D / 8][4];
#pragma unroll
  for (int i = 0; i < D / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float mx_lo = -INFINITY, mx_hi = -INFINITY, l_lo = 0.f, l_hi = 0.f;
  const bf16 *qw = sm.q + rl * LD + 2 * t;
  uint32_t b = 0;
  for (uint32_t j0 = jmin; j0 < jmax; j0 += KT, b ^= 1) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();  // tile b has landed for everyone, tile b ^ 1 is consumed
    if (j0 + KT < jmax) fetch(j0 + KT, b ^ 1);
    const bf16 *ks = sm.k[b];
    const float *bs = sm.bias[b] + 63;
    float sc[KT / 8][4];
#pragma unroll
    for (int nt = 0; nt < KT / 8; ++nt) sc[nt][0] = sc[nt][1] = sc[nt][2] = sc[nt][3] = 0.f;
#pragma unroll
    for (int kk = 0; kk < D / 16; ++kk) {
      const uint32_t a0 = *reinterpret_cast<const uint32_t *>(qw + kk * 16), a1 = *reinterpret_cast<const uint32_t *>(qw + 8 * LD + kk * 16);
      const uint32_t a2 = *reinterpret_cast<const uint32_t *>(qw + kk * 16 + 8), a3 = *reinterpret_cast<const uint32_t *>(qw + 8 * LD + kk * 16 + 8);
#pragma unroll
      for (int nt = 0; nt < KT / 8; ++nt) {
        const bf16 *kr = ks + (nt * 8 + gq) * LD + kk * 16 + 2 * t;
        mma_bf16(sc[nt], a0, a1, a2, a3, *reinterpret_cast<const uint32_t *>(kr), *reinterpret_cast<const uint32_t *>(kr + 8));
      }
    }
    float tm_lo = -INFINITY, tm_hi = -INFINITY;
#pragma unroll
    for (int nt = 0; nt < KT / 8; ++nt) {
      const int c = nt * 8 + 2 * t;
      const uint32_t j = j0 + c;
      sc[nt][0] = j < vis_lo && j >= see_lo ? fmaf(sc[nt][0], qs_lo, bs[(int)rl - c]) : -INFINITY;
      sc[nt][1] = j + 1 < vis_lo && j + 1 >= see_lo ? fmaf(sc[nt][1], qs_lo, bs[(int)rl - c - 1]) : -INFINITY;
      sc[nt][2] = j < vis_hi && j >= see_hi ? fmaf(sc[nt][2], qs_hi, bs[(int)rh - c]) : -INFINITY;
      sc[nt][3] = j + 1 < vis_hi && j + 1 >= see_hi ? fmaf(sc[nt][3], qs_hi, bs[(int)rh - c - 1]) : -INFINITY;
      tm_lo = fmaxf(tm_lo, fmaxf(sc[nt][0], sc[nt][1]));
      tm_hi = fmaxf(tm_hi, fmaxf(sc[nt][2], sc[nt][3]));
    }
#pragma unroll
    for (int w = 1; w < 4; w <<= 1) {
      tm_lo = fmaxf(tm_lo, __shfl_xor_sync(0xffffffffu, tm_lo, w));
      tm_hi = fmaxf(tm_hi, __shfl_xor_sync(0xffffffffu, tm_hi, w));
    }
    const float mn_lo = fmaxf(mx_lo, tm_lo), mn_hi = fmaxf(mx_hi, tm_hi);
    const float ref_lo = mn_lo == -INFINITY ? 0.f : mn_lo, ref_hi = mn_hi == -INFINITY ? 0.f : mn_hi;
    const float corr_lo = exp2f(mx_lo - ref_lo), corr_hi = exp2f(mx_hi - ref_hi);
    mx_lo = mn_lo;
    mx_hi = mn_hi;
    float rs_lo = 0.f, rs_hi = 0.f;
#pragma unroll
    for (int nt = 0; nt < KT / 8; ++nt) {
      sc[nt][0] = exp2f(sc[nt][0] - ref_lo);
      sc[nt][1] = exp2f(sc[nt][1] - ref_lo);
      sc[nt][2] = exp2f(sc[nt][2] - ref_hi);
      sc[nt][3] = exp2f(sc[nt][3] - ref_hi);
      rs_lo += sc[nt][0] + sc[nt][1];
      rs_hi += sc[nt][2] + sc[nt][3];
    }
    l_lo = l_lo * corr_lo + rs_lo;  // this thread's columns; summed over the four threads of a row at the end
    l_hi = l_hi * corr_hi + rs_hi;
#pragma unroll
    for (int i = 0; i < D / 8; ++i) {
      o[i][0] *= corr_lo;
      o[i][1] *= corr_lo;
      o[i][2] *= corr_hi;
      o[i][3] *= corr_hi;
    }
#pragma unroll
    for (int j16 = 0; j16 < KT / 16; ++j16) {
      const uint32_t a0 = pack_bf2(sc[2 * j16][0], sc[2 * j16][1]), a1 = pack_bf2(sc[2 * j16][2], sc[2 * j16][3]);
      const uint32_t a2 = pack_bf2(sc[2 * j16 + 1][0], sc[2 * j16 + 1][1]), a3 = pack_bf2(sc[2 * j16 + 1][2], sc[2 * j16 + 1][3]);
      const bf16 *vrow = (SEP ? sm.v[b] : ks) + (j16 * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * LD + ((lane >> 4) & 1) * 8;
#pragma unroll
      for (int dt = 0; dt < D / 16; ++dt) {
        uint32_t b0, b1, b2, b3;
        const uint32_t addr = (uint32_t)__cvta_generic_to_shared(vrow + dt * 16);
        asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(b0), "=r"(b1), "=r"(b2), "=r"(b3) : "r"(addr));
        mma_bf16(o[2 * dt], a0, a1, a2, a3, b0, b1);
        mma_bf16(o[2 * dt + 1], a0, a1, a2, a3, b2, b3);
      }
    }
  }
#pragma unroll
  for (int w = 1; w < 4; w <<= 1) {
    l_lo += __shfl_xor_sync(0xffffffffu, l_lo, w);
    l_hi += __shfl_xor_sync(0xffffffffu, l_hi, w);
  }
  const uint32_t ml = m0 + rl, mh = m0 + rh;
  float k_lo = 1.f, k_hi = 1.f;  // the sink may be the largest term: the outputs are rescaled to it
  if (p.sink) {
    const float sink = sink_log2(p, h), M_lo = fmaxf(mx_lo, sink), M_hi = fmaxf(mx_hi, sink);
    k_lo = exp2f(mx_lo - M_lo);
    k_hi = exp2f(mx_hi - M_hi);
    l_lo = l_lo * k_lo + exp2f(sink - M_lo);
    l_hi = l_hi * k_hi + exp2f(sink - M_hi);
  }
  const float f_lo = ml < T ? (p.gate ? p.gate[(size_t)ml * p.gate_ld + h] : 1.f) * k_lo / l_lo : 0.f;
  const float f_hi = mh < T ? (p.gate ? p.gate[(size_t)mh * p.gate_ld + h] : 1.f) * k_hi / l_hi : 0.f;
  bf16 *out = static_cast<bf16 *>(p.out) + (size_t)h * p.vp;
#pragma unroll
  for (int nt = 0; nt < D / 8; ++nt) {
    const uint32_t d = nt * 8 + 2 * t;
    if (d >= p.vp) continue;
    if (ml < T) *reinterpret_cast<uint32_t *>(out + (size_t)ml * p.out_ld + d) = pack_bf2(o[nt][0] * f_lo, o[nt][1] * f_lo);
    if (mh < T) *reinterpret_cast<uint32_t *>(out + (size_t)mh * p.out_ld + d) = pack_bf2(o[nt][2] * f_hi, o[nt][3] * f_hi);
  }
}

template <int D, bool SEP> cudaError_t launch_tile(const KvAttn &p, cudaStream_t s) {
  cudaError_t e = cudaFuncSetAttribute(kv_tile_kernel<D, SEP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sizeof(TileSmem<D, SEP>));
  if (e != cudaSuccess) return e;
  kv_tile_kernel<D, SEP><<<dim3(p.heads, (p.T + QT - 1) / QT), 128, sizeof(TileSmem<D, SEP>), s>>>(p);
  return cudaGetLastError();
}
template <bool SEP> cudaError_t launch_tile_d(const KvAttn &p, cudaStream_t s) {
  const uint32_t d = std::max(p.dp, p.vp);
  if (d <= 32) return launch_tile<32, SEP>(p, s);
  if (d <= 48) return launch_tile<48, SEP>(p, s);
  if (d <= 64) return launch_tile<64, SEP>(p, s);
  if (d <= 96) return launch_tile<96, SEP>(p, s);
  if (d <= 128) return launch_tile<128, SEP>(p, s);
  if (d <= 192) return launch_tile<192, SEP>(p, s);
  return launch_tile<256, SEP>(p, s);
}

constexpr uint32_t kTileRows = 16;  // from this many query rows the tile kernel is used

}  // namespace

size_t kv_attn_scratch_bytes(uint32_t T, uint32_t heads, uint32_t vp, uint32_t splits) {
  return splits < 2 ? 0 : (size_t)T * heads * 4 * splits * (vp + 4) * sizeof(float);  // at most heads (group) units of four records
}
uint32_t kv_attn_counters(uint32_t T, uint32_t heads) { return T * heads; }

cudaError_t launch_kv_attention(const KvAttn &p, bool f32, cudaStream_t s) {
  if (!p.T || !p.kv_heads || p.heads % p.kv_heads || p.dp % 16 || p.dp > 256 || p.vp % 16 || p.vp > 256 || (!p.vcache && p.vp != p.dp) || !p.splits || p.splits > kMaxSplits)
    return cudaErrorInvalidValue;
  if (!f32 && p.T >= kTileRows && !p.qk.q) return p.vcache ? launch_tile_d<true>(p, s) : launch_tile_d<false>(p, s);
  if (p.T > 65535 || (p.qk.q && (p.T != 1 || p.qk.pairs > kMaxPairs || p.qk.k_col % 8))) return cudaErrorInvalidValue;
  if (p.vcache) return f32 ? launch_row_d<float, true>(p, s) : launch_row_d<bf16, true>(p, s);
  return f32 ? launch_row_d<float, false>(p, s) : launch_row_d<bf16, false>(p, s);
}

}  // namespace vkl
