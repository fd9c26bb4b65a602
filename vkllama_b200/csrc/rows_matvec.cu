// One token through the rows of up to two weight matrices: the decode step's projections of the layer-list
// decoder designs, HBM-bound (every weight byte is read once).
//
// A unit is four rows. KS warps of a CTA share a unit, each taking every KS-th 256-column step of K, and a
// warp's lanes hold 8 columns each: four coalesced 128-bit weight loads per step and lane, eight inputs, 32
// fp32 FMAs. What becomes of a row is in its segment (rows.h), so one launch runs everything that reads the
// same input: keys, queries, head gates and the feed-forward's gate/up rows of a parallel block, and the
// gate/up rows of the experts that the token's id names. Rows may be split between two inputs (two norms of one
// stream), and a norm with statistics that leads to them is computed by every CTA for itself. The out-projection form sums, per output row, the
// attention's columns, the dense feed-forward's columns (one matrix, side by side) or the chosen experts'
// rows, and leaves the residual stream and the next norm's output behind.
#include <algorithm>

#include "rows.cuh"

namespace vkl {
namespace {

constexpr int kThreads = 256, kWarps = kThreads / 32;

template <class T> struct XVec;
template <> struct XVec<bf16> {
  uint4 u;
  __device__ void load(const bf16 *p) { u = *reinterpret_cast<const uint4 *>(p); }
  __device__ void get(float (&v)[8]) const { unpack8(u, v); }
};
template <> struct XVec<float> {
  float4 a, b;
  __device__ void load(const float *p) {
    a = *reinterpret_cast<const float4 *>(p);
    b = *reinterpret_cast<const float4 *>(p + 4);
  }
  __device__ void get(float (&v)[8]) const {
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
  }
};

// acc[i] += scale * <w[i], x> over this lane's columns k0, k0 + step, ...
template <class T> __device__ __forceinline__ void dot4(float (&acc)[4], const bf16 *w0, const bf16 *w1, const bf16 *w2, const bf16 *w3, const T *x, uint32_t k0,
                                                        uint32_t step, uint32_t K, float scale) {
#pragma unroll 2
  for (uint32_t k = k0; k < K; k += step) {
    const uint4 a = ldg_stream(w0 + k), b = ldg_stream(w1 + k), c = ldg_stream(w2 + k), d = ldg_stream(w3 + k);
    XVec<T> xv;
    xv.load(x + k);
    float f[8], w[8];
    xv.get(f);
#pragma unroll
    for (int i = 0; i < 8; ++i) f[i] *= scale;
    unpack8(a, w);
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[0] = fmaf(w[i], f[i], acc[0]);
    unpack8(b, w);
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[1] = fmaf(w[i], f[i], acc[1]);
    unpack8(c, w);
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[2] = fmaf(w[i], f[i], acc[2]);
    unpack8(d, w);
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[3] = fmaf(w[i], f[i], acc[3]);
  }
}

__device__ __forceinline__ void prefetch_l2(const void *p) { asm volatile("prefetch.global.L2 [%0];" ::"l"(p)); }

// NORM: the input is p.norm's output, computed here.
template <class T, int KS, bool OUT, bool NORM> __global__ void __launch_bounds__(kThreads) rows_matvec_kernel(const MvRows p) {
  constexpr uint32_t UPC = kWarps / KS;  // units a CTA works on at a time
  __shared__ float red[2][kWarps][4];
  const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, wg = warp / KS, ws = warp % KS;
  const uint32_t k0 = (ws * 32 + lane) * 8, step = KS * 256;
  const uint32_t gap = p.n2 - p.gap0;  // rows without a result
  const uint32_t u_main = (p.N - gap) / 4, u_exp = p.ne / 4, units = u_main + (OUT ? 0u : p.top * u_exp);
  auto first_row = [&](uint32_t u) { return u * 4 + (u * 4 >= p.gap0 ? gap : 0u); };
  const uint32_t rounds = (units + gridDim.x * UPC - 1) / (gridDim.x * UPC);
  // rows of unit u of a segment: four in a row, or two gate rows and the up rows of the same two outputs
  auto glu_row = [](uint32_t u) { return (u / 8) * 32 + (u % 8) * 2; };
  if (p.use_pdl) {
    // the weights do not depend on the kernel before: ask for the first unit's rows, then wait for it
    const uint32_t u = blockIdx.x * UPC + wg;
    if (u < u_main) {
      const bf16 *w = p.w + (size_t)first_row(u) * p.K;
      for (uint32_t k = k0, i = 0; k < p.K && i < 2; k += step, ++i)
        for (int r = 0; r < 4; ++r) prefetch_l2(w + (size_t)r * p.K + k);
    }
    asm volatile("griddepcontrol.wait;" ::: "memory");
    asm volatile("griddepcontrol.launch_dependents;");  // the next kernel asks for its weights as this one's CTAs make room
  }
  const T *x1 = static_cast<const T *>(p.x), *x2 = static_cast<const T *>(p.x2);
  if constexpr (NORM) {  // every CTA for itself
    extern __shared__ __align__(16) unsigned char xs_raw[];
    T *xs = reinterpret_cast<T *>(xs_raw);
    rms_row<T, kWarps>(p.norm, p.norm.x, xs, xs + p.K);
    __syncthreads();
    x1 = xs;
    x2 = xs + p.K;
  }
  const uint32_t tok = p.top ? *p.tok : 0u;
  for (uint32_t it = 0; it < rounds; ++it) {
    const uint32_t u = (it * gridDim.x + blockIdx.x) * UPC + wg;
    const bool active = u < units;
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    uint32_t n = 0, choice = 0;
    bool main_rows = true, glu = false;
    RowSeg sg = p.out.seg[0];
    if (active) {
      const T *x = x1;
      if (u < u_main) {
        n = first_row(u);
        if (p.n2 && n >= p.n2) x = x2;
        sg = find_seg(p.out, n);
        glu = !OUT && sg.kind == ROW_GLU;
        if (glu) n = sg.n0 + glu_row((n - sg.n0) / 4);
        const bf16 *w = p.w + (size_t)n * p.K, *w2 = w + (size_t)(glu ? 16 : 2) * p.K;
        dot4<T>(acc, w, w + p.K, w2, w2 + p.K, x, k0, step, p.K, 1.f);
        if (OUT) {
          for (uint32_t j = 0; j < p.top; ++j) {
            const int32_t e = p.table[(size_t)tok * p.top + j];
            const bf16 *v = p.we + ((size_t)e * p.N + n) * p.ke;
            dot4<T>(acc, v, v + p.ke, v + 2 * (size_t)p.ke, v + 3 * (size_t)p.ke, static_cast<const T *>(p.xe) + (size_t)j * p.xe_ld, k0, step, p.ke, p.xe_scale);
          }
        }
      } else if constexpr (!OUT) {
        main_rows = false;
        glu = true;
        choice = (u - u_main) / u_exp;
        n = glu_row((u - u_main) % u_exp);
        const int32_t e = p.table[(size_t)tok * p.top + choice];
        const bf16 *w = p.we + ((size_t)e * p.ne + n) * p.K, *w2 = w + (size_t)16 * p.K;
        dot4<T>(acc, w, w + p.K, w2, w2 + p.K, x, k0, step, p.K, 1.f);
      }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) acc[i] = warp_sum(acc[i]);
    if (KS > 1) {
      if (lane == 0) {
#pragma unroll
        for (int i = 0; i < 4; ++i) red[it & 1][warp][i] = acc[i];
      }
      __syncthreads();
      if (ws != 0) continue;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        acc[i] = red[it & 1][wg * KS][i];
#pragma unroll
        for (int w = 1; w < KS; ++w) acc[i] += red[it & 1][wg * KS + w][i];
      }
    }
    if (!active || lane >= (glu ? 2u : 4u)) continue;
    if (glu) {
      const float g = lane ? acc[1] : acc[0], up = lane ? acc[3] : acc[2];
      if (main_rows) {
        const uint32_t c = n - sg.n0;
        store1(static_cast<T *>(p.out.glu) + (c / 32) * 16 + c % 32 + lane, glu_act(p.out.act, p.out.limit, g, up));
      } else {
        store1(static_cast<T *>(p.xe) + (size_t)choice * p.xe_ld + (n / 32) * 16 + n % 32 + lane, glu_act(p.xe_act, p.out.limit, g, up));
      }
    } else {
      rows_one<T>(p.out, sg, n + lane, lane == 0 ? acc[0] : lane == 1 ? acc[1] : lane == 2 ? acc[2] : acc[3]);
    }
  }
}

template <class T, int KS, bool OUT, bool NORM> cudaError_t launch_t(const MvRows &p, uint32_t units, int sms, cudaStream_t s) {
  auto kern = rows_matvec_kernel<T, KS, OUT, NORM>;
  const size_t smem = NORM ? (p.norm.w2 ? 2 : 1) * (size_t)p.K * sizeof(T) : 0;
  auto resident = [](size_t bytes) {
    int n = 0;
    return cudaOccupancyMaxActiveBlocksPerMultiprocessor(&n, rows_matvec_kernel<T, KS, OUT, NORM>, kThreads, bytes) == cudaSuccess && n > 0 ? n : 1;
  };
  static const int without_norm = resident(0);
  const int per_sm = smem ? resident(smem) : without_norm;
  // one wave, every CTA with the same number of rounds (or one less)
  const uint32_t ctas = (units + kWarps / KS - 1) / (kWarps / KS), slots = (uint32_t)(sms * per_sm);
  const uint32_t rounds = (ctas + slots - 1) / slots;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3((ctas + rounds - 1) / rounds);
  cfg.blockDim = dim3(kThreads);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = s;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = p.use_pdl ? 1 : 0;
  return cudaLaunchKernelEx(&cfg, kern, p);
}

template <class T, bool OUT, bool NORM> cudaError_t launch_ks(const MvRows &p, int sms, cudaStream_t s) {
  const uint32_t units = (p.N - (p.n2 - p.gap0)) / 4 + (OUT ? 0u : p.top * (p.ne / 4));
  // enough warps to keep the memory system busy, as long as each has a step of K of its own
  uint32_t ks = 1;
  while (ks < 8 && units * ks < (uint32_t)sms * 24 && p.K >= 512 * ks) ks *= 2;
  switch (ks) {
    case 1: return launch_t<T, 1, OUT, NORM>(p, units, sms, s);
    case 2: return launch_t<T, 2, OUT, NORM>(p, units, sms, s);
    case 4: return launch_t<T, 4, OUT, NORM>(p, units, sms, s);
    default: return launch_t<T, 8, OUT, NORM>(p, units, sms, s);
  }
}

}  // namespace

bool rows_matvec_takes_norm(uint32_t K, bool two, bool f32) { return (two ? 2 : 1) * (size_t)K * (f32 ? 4 : 2) <= 46 * 1024; }

cudaError_t launch_rows_matvec(const MvRows &p, bool f32, int sms, cudaStream_t s) {
  if (p.norm.x && (p.norm.ldw != p.K || (p.n2 && !p.norm.w2) || !rows_matvec_takes_norm(p.K, p.norm.w2, f32))) return cudaErrorInvalidValue;
  if (!p.N || p.N % 32 || p.K % 64 || p.gap0 % 32 || p.n2 % 32 || p.gap0 > p.n2 || p.n2 > p.N || (p.top && (p.ke % 64 || p.ne % 32))) return cudaErrorInvalidValue;
  if (p.norm.x) return p.out_proj ? cudaErrorInvalidValue : f32 ? launch_ks<float, false, true>(p, sms, s) : launch_ks<bf16, false, true>(p, sms, s);
  if (f32) return p.out_proj ? launch_ks<float, true, false>(p, sms, s) : launch_ks<float, false, false>(p, sms, s);
  return p.out_proj ? launch_ks<bf16, true, false>(p, sms, s) : launch_ks<bf16, false, false>(p, sms, s);
}

}  // namespace vkl
