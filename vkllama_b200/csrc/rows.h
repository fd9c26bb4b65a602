// Parameters of the layer-list decoder kernels: "rows" of a weight matrix multiplied with one token
// (rows_matvec.cu) or many (gemm_tcgen05.cu in bfloat16, gemm_f32.cu in 32-bit), and what becomes of the
// results. All pointers are device pointers.
//
// Padding: every width is a multiple of 64 in memory (ldw), a head's a multiple of 16 (dp), and what a matrix
// does with its rows changes on 32-row boundaries only; the weights' padding is zero, so the kernels have no
// ragged edge and the padding of every activation stays zero.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

namespace vkl {

using bf16 = __nv_bfloat16;

// What the rows of a segment are.
enum RowKind : uint32_t {
  ROW_QUERY,      // + bias -> q [tokens, q_ld]
  ROW_KEY,        // + bias -> this token's row of the key cache [kv head][position][dp]
  ROW_HEAD_GATE,  // sigmoid -> gate [tokens, gate_ld] (fp32), one number per head
  ROW_GLU,        // 32 rows = 16 gate rows, then the 16 up rows of the same outputs -> glu [tokens, glu_ld]
  ROW_RESIDUAL,   // added to the residual stream, see Residual
  ROW_STORE,      // * scale, then the soft cap if there is one -> f32 [tokens, f32_ld]
  ROW_VALUE,      // this token's row of the value cache [kv head][position][vp]
  ROW_LOW,        // low_ld rows each of two low-rank inner vectors -> low [2][tokens, low_ld]
  ROW_NONE        // padding between two segments: no result
};
enum GluAct : uint32_t {
  GLU_SILU,     // the gate's SiLU times up
  GLU_CLAMPED   // gate cut off above the limit, up at both ends; quick-GELU of the gate times (1 + up)
};
struct RowSeg {
  uint32_t n0, n1;  // rows [n0, n1), multiples of 32
  uint32_t kind;
};

// The residual stream's step: x += mult * acc, then what comes between two layer runs (a loop's pass adds the token's
// embedding and the pass's vector), then the next norm if it is Dynamic Tanh, which needs no other element of the
// row and so runs in the epilogue of whatever wrote x.
struct Residual {
  float *x;             // [tokens, ldw]
  uint32_t ldw;
  float mult;
  const float *bias;    // [ldw] or null
  float *trace;         // optional [tokens, ldw]: x right after the layer run
  const bf16 *emb;      // next run's pass adds embed[token], or null
  const uint32_t *toks;
  const float *step;    // next run's pass adds this vector [ldw], or null
  void *h;              // next norm's output [tokens, ldw] in the compute type, or null: no norm here
  const float *nw, *nb; // Dynamic Tanh: h = tanh(alpha x) * nw + nb
  float alpha;
};

struct RowsOut {
  RowSeg seg[6];
  uint32_t nseg;
  const float *bias;    // per row, or null
  void *q;
  uint32_t q_ld;
  void *kcache;
  void *vcache;
  uint32_t kv_heads, dp, vp, maxlen;
  const uint32_t *pos;  // position of token 0
  void *low;
  uint32_t low_ld;
  size_t low_stride;    // elements between the two inner vectors of token 0
  float *gate;
  uint32_t gate_ld;
  void *glu;
  uint32_t glu_ld, act;
  float limit;
  float *f32;
  uint32_t f32_ld;
  float scale, cap;     // cap 0: none, else cap * tanh(. / cap)
  Residual res;
};

// ---- norms with statistics, rotation (norm_rows.cu) ----
// RMS norm of the residual stream with up to two weights (they share the statistic): h = x / rms(x) * w, the same
// for h2 and w2. The weights are what multiplies (a weight stored around zero has its 1 added when it is loaded).
struct RmsRows {
  const float *x;           // [T, ldw]
  uint32_t T, ldw, width;
  const float *w, *w2;      // w2 may be null
  void *h, *h2;             // [T, ldw] compute type
  float eps;
  int use_pdl;
};
cudaError_t launch_rms_rows(const RmsRows &p, bool f32, cudaStream_t s);

// RMS norm over all of a token's query rows and over all of its key rows, rotation of the first 2 * pairs dimensions
// of each head (neighbours 2i, 2i + 1 turn by position * freq[i]); queries stay where they are, keys go to the cache.
struct QkRows {
  void *q;                  // [T, q_ld] compute type: queries from column 0, raw keys from column k_col
  uint32_t q_ld, k_col;
  const float *qw, *kw;     // norm weights, padded like the rows; null: no norm
  float eps;
  const float *freq;
  uint32_t pairs;
  void *kcache;             // null: the layer has no keys of its own
  uint32_t T, heads, kv_heads, dim, dp, maxlen;
  const uint32_t *pos;
  int use_pdl;
};
cudaError_t launch_qk_rows(const QkRows &p, bool f32, cudaStream_t s);

// ---- one token: y = W x, weights bf16 [N, K], x in the compute type, fp32 accumulation (rows_matvec.cu) ----
struct MvRows {
  const bf16 *w;
  uint32_t N, K;
  const void *x;            // [K]
  const void *x2;           // rows from n2 on read this vector instead; null: none
  uint32_t n2, gap0;        // rows [gap0, n2) are padding and not computed (gap0 = n2: none)
  RmsRows norm;             // norm.x set: x (and x2, if norm.w2) are this norm's outputs, computed in the kernel
  // Routed experts. In-projection form: the chosen experts' gate/up rows (ne each, GLU order) read x too and
  // write xe [top, ke]. Out-projection form: N rows per expert over ke columns of xe, summed and weighted.
  const bf16 *we;
  uint32_t ne, ke, top;
  const int32_t *table;     // [vocab, top]: a token id's experts
  const uint32_t *tok;
  void *xe;
  uint32_t xe_ld, xe_act;
  float xe_scale;
  bool out_proj;
  int use_pdl;
  RowsOut out;
};
bool rows_matvec_takes_norm(uint32_t K, bool two, bool f32);  // whether the norm's outputs fit in a CTA
cudaError_t launch_rows_matvec(const MvRows &p, bool f32, int sms, cudaStream_t s);

// ---- many tokens: Y[M,N] = A[M,K] . W[N,K]^T ----
struct GemmRows {
  const void *a;            // [M, K] compute type
  const bf16 *w;            // [N, K]; grouped: [experts * N, K]
  uint32_t M, N, K;
  uint32_t n2;              // rows of w from n2 on (a multiple of kInputAlign) read A's rows M .. 2M - 1: a second input; 0: none
  const int32_t *tile_expert;  // grouped: expert of every 128-row tile of A (-1: no tokens), or null
  uint32_t w_rows;             // grouped: experts * N
  uint32_t *error;
  RowsOut out;
};
constexpr uint32_t kInputAlign = 256;  // no tile of the GEMMs crosses a multiple of this many weight rows
cudaError_t launch_gemm_rows_bf16(const GemmRows &p, cudaStream_t s);  // tcgen05
cudaError_t launch_gemm_rows_f32(const GemmRows &p, cudaStream_t s);   // true 32-bit

// ---- attention over a cache of keys and values, or of rows that are both (kv_attention.cu) ----
struct KvAttn {
  const void *q;            // [T, q_ld]
  uint32_t q_ld;
  const void *cache;        // [kv_heads][maxlen][dp]
  const void *vcache;       // [kv_heads][maxlen][vp], or null: the keys are the values (vp = dp)
  void *out;                // [T, out_ld], head h at column h * vp
  uint32_t out_ld;
  const float *gate;        // [T, gate_ld] or null
  uint32_t gate_ld;
  const float *bias;        // [heads][bias_n]: log2(e) * bias at distance n (the last entry from bias_n - 1 on), or null
  uint32_t bias_n;
  const uint32_t *pos;      // position of row 0
  uint32_t window;          // a query sees itself and the window - 1 positions before it; 0: all
  const float *sink;        // [heads] or null: one more term of a head's denominator, not scaled, without a value
  float scale;
  float temp_coef, temp_every;  // query temperature at p: 1 + temp_coef log(1 + k), k = whole temp_every-s in p + 1; temp_coef 0: none
  uint32_t T, heads, kv_heads, dp, vp, maxlen, splits;
  float *scratch;           // kv_attn_scratch_bytes
  uint32_t *counters;       // one per (row, head group), zero before and after
  QkRows qk;                // one token: qk.q set: q is raw, norm, rotation and the key's row of the cache are done here
  int use_pdl;
};
size_t kv_attn_scratch_bytes(uint32_t T, uint32_t heads, uint32_t vp, uint32_t splits);
uint32_t kv_attn_counters(uint32_t T, uint32_t heads);
cudaError_t launch_kv_attention(const KvAttn &p, bool f32, cudaStream_t s);

// ---- routing by a token-id table, and rows (experts.cu) ----
struct RouteTable {         // one routed layer
  const int32_t *table;     // [vocab, top]
  uint32_t top, experts;
  int32_t *slot;            // [T * top]: row of the grouped buffers that holds (token, choice)
  int32_t *token;           // [rows_pad]: token of a grouped row, -1: none
  int32_t *tile_expert;     // [rows_pad / 128]
};
// Rows of the grouped buffers for T tokens: every expert's tokens padded to whole 128-row tiles.
inline uint32_t route_rows(uint32_t T, uint32_t top, uint32_t experts) {
  const uint32_t n = T * top, used = n < experts ? n : experts;
  return (n / 128 + used) * 128;
}
cudaError_t launch_route(const RouteTable *layers, uint32_t n, uint32_t max_experts, const uint32_t *toks, uint32_t T, cudaStream_t s);
cudaError_t launch_gather_rows(const void *src, const int32_t *rows, uint32_t n, uint32_t row_bytes, void *dst, cudaStream_t s);
// x += sum over the token's choices of y[slot], then the residual step.
cudaError_t launch_combine(const float *y, uint32_t y_ld, const int32_t *slot, uint32_t top, uint32_t T, const Residual &r, bool f32, cudaStream_t s);
// x = scale * embed[token], then the residual step without its acc.
cudaError_t launch_embed_rows(const bf16 *emb, const uint32_t *toks, uint32_t T, float scale, const Residual &r, bool f32, cudaStream_t s);

// ---- gated delta rule with a decay per key channel (delta_rule.cu) ----
// Per head a state S [dim, vdim]: S <- g S, u = beta (v - S^T k), S <- S + k u^T, o = S^T q, then the RMS norm of o and
// a gate. Query, key and value are projections after a short causal convolution over time and SiLU, query and key unit
// vectors; decay and gate come from two-step projections, g = exp(-rate softplus(z + bias)), gate = sigmoid(z).
struct DeltaRows {
  const void *raw;          // [T, raw_ld] compute type: the projections, query | key | value columns
  uint32_t raw_ld, k_col, v_col;
  const float *taps;        // [raw_ld][ntaps], the last one is the current token's
  uint32_t ntaps;
  void *ring;               // [ntaps][raw_ld] compute type: the projections at position p in slot p % ntaps
  const uint32_t *pos;      // position of row 0; a sequence that starts at 0 finds state and ring empty
  uint32_t T, heads, kv_heads, dim, vdim, dp, vp;  // dp, vp: widths in memory, multiples of 32 and 16
  const float *bias, *rate; // [heads * dp]
  const float *beta;        // [T, beta_ld]
  uint32_t beta_ld;
  float *state;             // [heads][vp][dp]
  const float *norm;        // [vp]: weight of the output's RMS norm per head
  float eps;
  void *out;                // [T, out_ld] compute type, head h at column h * vp
  uint32_t out_ld;
  int use_pdl;
  // many tokens
  const float *z;           // [T, z_ld]: second steps of the projections, decays from column 0, gates from column z_gate
  uint32_t z_ld, z_gate;
  float *v;                 // [T][heads * vp]: values, which the recurrence replaces by its outputs
  float *blocks;            // delta_block_floats(...): what the recurrence needs of the keys, block by block
  uint32_t *error;          // set when a wait of the kernels runs out
  int sms;
  // one token
  const bf16 *wl;           // second steps' weights [., low_ld]: decay rows from 0, gate rows from z_gate
  const void *low;          // [2][low_ld] compute type: the first steps' results
  uint32_t low_ld;
};
constexpr uint32_t kDeltaSlice = 1024;  // tokens whose blocks are held at a time
size_t delta_block_floats(uint32_t T, uint32_t heads, uint32_t dp);
cudaError_t launch_delta_rows(const DeltaRows &p, bool f32, cudaStream_t s);  // T > 1; launches: delta_launches(T)
inline uint32_t delta_launches(uint32_t T) { return 2 * ((T + kDeltaSlice - 1) / kDeltaSlice) + 1; }
cudaError_t launch_delta_step(const DeltaRows &p, bool f32, cudaStream_t s);  // T = 1

// Places a bf16 tensor [rows, cols] into a padded matrix: row r -> (r / ra) * rb + r % ra + r0, columns alike.
struct PackMap {
  uint32_t ra, rb, r0, ca, cb, c0;
};
cudaError_t launch_pack_rows(const bf16 *src, uint32_t rows, uint32_t cols, bf16 *dst, uint32_t ld, const PackMap &m, cudaStream_t s);
cudaError_t launch_synth_bf16(bf16 *dst, uint64_t seed, uint64_t tensor, uint64_t n, float mean, float stdv, cudaStream_t s);

}  // namespace vkl
