// Device side of rows.h: compute-type access and the epilogues every decoder kernel shares.
#pragma once
#include "common.cuh"
#include "rows.h"

namespace vkl {

__device__ __forceinline__ float bf_lo(uint32_t u) { return __uint_as_float(u << 16); }
__device__ __forceinline__ float bf_hi(uint32_t u) { return __uint_as_float(u & 0xffff0000u); }
__device__ __forceinline__ void unpack8(const uint4 &u, float (&v)[8]) {
  v[0] = bf_lo(u.x); v[1] = bf_hi(u.x); v[2] = bf_lo(u.y); v[3] = bf_hi(u.y);
  v[4] = bf_lo(u.z); v[5] = bf_hi(u.z); v[6] = bf_lo(u.w); v[7] = bf_hi(u.w);
}
__device__ __forceinline__ uint32_t pack_bf2(float lo, float hi) {
  const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<const uint32_t *>(&v);
}
// Eight consecutive values, 16-byte (bf16) or 32-byte (float) aligned.
__device__ __forceinline__ void load8(const bf16 *p, float (&v)[8]) { unpack8(*reinterpret_cast<const uint4 *>(p), v); }
__device__ __forceinline__ void load8(const float *p, float (&v)[8]) {
  const float4 a = *reinterpret_cast<const float4 *>(p), b = *reinterpret_cast<const float4 *>(p + 4);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ void store8(bf16 *p, const float *v) {
  *reinterpret_cast<uint4 *>(p) = make_uint4(pack_bf2(v[0], v[1]), pack_bf2(v[2], v[3]), pack_bf2(v[4], v[5]), pack_bf2(v[6], v[7]));
}
__device__ __forceinline__ void store8(float *p, const float *v) {
  *reinterpret_cast<float4 *>(p) = make_float4(v[0], v[1], v[2], v[3]);
  *reinterpret_cast<float4 *>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
}
__device__ __forceinline__ void store1(bf16 *p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ void store1(float *p, float v) { *p = v; }

__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float glu_act(uint32_t act, float limit, float g, float u) {
  if (act == GLU_CLAMPED) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g * sigmoid_f(1.702f * g) * (u + 1.0f);
  }
  return g * sigmoid_f(g) * u;
}
__device__ __forceinline__ float tanh_norm(float x, float alpha, float w, float b) { return tanhf(alpha * x) * w + b; }

// Sums of two numbers over a CTA of WARPS warps, the same order every time.
template <int WARPS> __device__ __forceinline__ float2 block_sum2(float a, float b) {
  __shared__ float2 part[WARPS];
  a = warp_sum(a);
  b = warp_sum(b);
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = make_float2(a, b);
  __syncthreads();
  float2 r = part[0];
#pragma unroll
  for (int w = 1; w < WARPS; ++w) {
    r.x += part[w].x;
    r.y += part[w].y;
  }
  return r;
}
__device__ __forceinline__ float square_sum8(const float (&v)[8], float s) {
#pragma unroll
  for (int i = 0; i < 8; ++i) s = fmaf(v[i], v[i], s);
  return s;
}
// RMS norm of one row, for one or two weights (RmsRows), by a CTA of WARPS warps.
template <class T, int WARPS> __device__ __forceinline__ void rms_row(const RmsRows &p, const float *x, T *h, T *h2) {
  float ss = 0.f;
  for (uint32_t n = threadIdx.x * 8; n < p.ldw; n += WARPS * 256) {
    float v[8];
    load8(x + n, v);
    ss = square_sum8(v, ss);
  }
  const float r = 1.0f / sqrtf(block_sum2<WARPS>(ss, 0.f).x / (float)p.width + p.eps);
  for (uint32_t n = threadIdx.x * 8; n < p.ldw; n += WARPS * 256) {
    float v[8], w[8], y[8];
    load8(x + n, v);
    load8(p.w + n, w);
#pragma unroll
    for (int i = 0; i < 8; ++i) y[i] = v[i] * r * w[i];
    store8(h + n, y);
    if (p.w2) {
      load8(p.w2 + n, w);
#pragma unroll
      for (int i = 0; i < 8; ++i) y[i] = v[i] * r * w[i];
      store8(h2 + n, y);
    }
  }
}
// Eight consecutive dimensions of a head, from dimension d on: norm (r times the weights, if any) and rotation; turn:
// cosine and sine per pair.
__device__ __forceinline__ void norm_and_turn(float (&v)[8], const float *w, float r, uint32_t d, const float2 *turn, uint32_t pairs) {
  if (w) {
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] *= r * w[i];
  }
#pragma unroll
  for (int i = 0; i < 8; i += 2) {
    if ((d + i) / 2 < pairs) {
      const float2 t = turn[(d + i) / 2];
      const float a = v[i], b = v[i + 1];
      v[i] = a * t.x - b * t.y;
      v[i + 1] = b * t.x + a * t.y;
    }
  }
}
constexpr uint32_t kMaxPairs = 128;  // head width at most 256
__device__ __forceinline__ float2 turn_of(uint32_t pos, float freq) {
  float s, c;
  sincosf((float)pos * freq, &s, &c);
  return make_float2(c, s);
}

__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float soft_cap(float v, float cap) { return cap > 0.f ? cap * tanhf(v / cap) : v; }

// x (already summed) of token m, column n: what follows a layer run (struct Residual).
template <class T> __device__ __forceinline__ void finish_residual(const Residual &r, uint32_t m, uint32_t n, float x) {
  const size_t o = (size_t)m * r.ldw + n;
  if (r.trace) r.trace[o] = x;
  if (r.emb) x += __bfloat162float(r.emb[(size_t)r.toks[m] * r.ldw + n]);
  if (r.step) x += r.step[n];
  r.x[o] = x;
  if (r.h) store1(static_cast<T *>(r.h) + o, tanh_norm(x, r.alpha, r.nw[n], r.nb[n]));
}

__device__ __forceinline__ const RowSeg &find_seg(const RowsOut &o, uint32_t n) {
  uint32_t i = 0;
  while (i + 1 < o.nseg && n >= o.seg[i].n1) ++i;
  return o.seg[i];
}
// c: padded column of a key or value row of width d
template <class T> __device__ __forceinline__ T *cache_slot(void *cache, uint32_t d, uint32_t maxlen, uint32_t pos, uint32_t c) {
  return static_cast<T *>(cache) + ((size_t)(c / d) * maxlen + pos) * d + c % d;
}
template <class T> __device__ __forceinline__ T *low_slot(const RowsOut &o, uint32_t m, uint32_t c) {
  return static_cast<T *>(o.low) + (c / o.low_ld) * o.low_stride + (size_t)m * o.low_ld + c % o.low_ld;
}

// 32 consecutive results (rows n0 .. n0 + 31 of the weights, one segment) of token m.
template <class T> __device__ __forceinline__ void rows_chunk(const RowsOut &o, uint32_t m, uint32_t n0, float (&v)[32]) {
  const RowSeg sg = find_seg(o, n0);
  if (o.bias) {
#pragma unroll
    for (int j = 0; j < 32; j += 4) {
      const float4 b = __ldg(reinterpret_cast<const float4 *>(o.bias + n0 + j));
      v[j] += b.x; v[j + 1] += b.y; v[j + 2] += b.z; v[j + 3] += b.w;
    }
  }
  const uint32_t c0 = n0 - sg.n0;
  switch (sg.kind) {
    case ROW_QUERY: {
      T *p = static_cast<T *>(o.q) + (size_t)m * o.q_ld + c0;
#pragma unroll
      for (int j = 0; j < 32; j += 8) store8(p + j, v + j);
      break;
    }
    case ROW_KEY: {
      const uint32_t pos = *o.pos + m;
#pragma unroll
      for (int j = 0; j < 32; j += 8)
        if (c0 + j < o.kv_heads * o.dp) store8(cache_slot<T>(o.kcache, o.dp, o.maxlen, pos, c0 + j), v + j);
      break;
    }
    case ROW_VALUE: {
      const uint32_t pos = *o.pos + m;
#pragma unroll
      for (int j = 0; j < 32; j += 8)
        if (c0 + j < o.kv_heads * o.vp) store8(cache_slot<T>(o.vcache, o.vp, o.maxlen, pos, c0 + j), v + j);
      break;
    }
    case ROW_LOW: {
      T *p = low_slot<T>(o, m, c0);  // low_ld is a multiple of 32
#pragma unroll
      for (int j = 0; j < 32; j += 8) store8(p + j, v + j);
      break;
    }
    case ROW_NONE: break;
    case ROW_HEAD_GATE: {
      float *p = o.gate + (size_t)m * o.gate_ld + c0;
#pragma unroll
      for (int j = 0; j < 32; j += 4)
        *reinterpret_cast<float4 *>(p + j) = make_float4(sigmoid_f(v[j]), sigmoid_f(v[j + 1]), sigmoid_f(v[j + 2]), sigmoid_f(v[j + 3]));
      break;
    }
    case ROW_GLU: {
      float y[16];
#pragma unroll
      for (int j = 0; j < 16; ++j) y[j] = glu_act(o.act, o.limit, v[j], v[16 + j]);
      T *p = static_cast<T *>(o.glu) + (size_t)m * o.glu_ld + c0 / 2;
      store8(p, y);
      store8(p + 8, y + 8);
      break;
    }
    case ROW_RESIDUAL: {
      const Residual &r = o.res;
      const size_t at = (size_t)m * r.ldw + n0;
      const uint32_t tok = r.emb ? r.toks[m] : 0u;
#pragma unroll
      for (int j = 0; j < 32; j += 8) {
        float x[8];
        load8(r.x + at + j, x);
#pragma unroll
        for (int i = 0; i < 8; ++i) x[i] += r.mult * (v[j + i] + (r.bias ? __ldg(r.bias + n0 + j + i) : 0.f));
        if (r.trace) store8(r.trace + at + j, x);
        if (r.emb) {
          float e[8];
          load8(r.emb + (size_t)tok * r.ldw + n0 + j, e);
#pragma unroll
          for (int i = 0; i < 8; ++i) x[i] += e[i];
        }
        if (r.step) {
#pragma unroll
          for (int i = 0; i < 8; ++i) x[i] += __ldg(r.step + n0 + j + i);
        }
        store8(r.x + at + j, x);
        if (r.h) {
#pragma unroll
          for (int i = 0; i < 8; ++i) x[i] = tanh_norm(x[i], r.alpha, __ldg(r.nw + n0 + j + i), __ldg(r.nb + n0 + j + i));
          store8(static_cast<T *>(r.h) + at + j, x);
        }
      }
      break;
    }
    default: {
      float *p = o.f32 + (size_t)m * o.f32_ld + c0;
#pragma unroll
      for (int j = 0; j < 32; j += 4)
        *reinterpret_cast<float4 *>(p + j) =
            make_float4(soft_cap(v[j] * o.scale, o.cap), soft_cap(v[j + 1] * o.scale, o.cap), soft_cap(v[j + 2] * o.scale, o.cap), soft_cap(v[j + 3] * o.scale, o.cap));
    }
  }
}

// One result of token 0 (row n of the weights; GLU rows go through rows_one_glu).
template <class T> __device__ __forceinline__ void rows_one(const RowsOut &o, const RowSeg &sg, uint32_t n, float v) {
  if (o.bias) v += o.bias[n];
  const uint32_t c = n - sg.n0;
  switch (sg.kind) {
    case ROW_QUERY: store1(static_cast<T *>(o.q) + c, v); break;
    case ROW_KEY:
      if (c < o.kv_heads * o.dp) store1(cache_slot<T>(o.kcache, o.dp, o.maxlen, *o.pos, c), v);
      break;
    case ROW_VALUE:
      if (c < o.kv_heads * o.vp) store1(cache_slot<T>(o.vcache, o.vp, o.maxlen, *o.pos, c), v);
      break;
    case ROW_LOW: store1(low_slot<T>(o, 0, c), v); break;
    case ROW_NONE: break;
    case ROW_HEAD_GATE: o.gate[c] = sigmoid_f(v); break;
    case ROW_RESIDUAL: finish_residual<T>(o.res, 0, n, o.res.x[n] + o.res.mult * (v + (o.res.bias ? o.res.bias[n] : 0.f))); break;
    default: o.f32[c] = soft_cap(v * o.scale, o.cap);
  }
}

}  // namespace vkl
