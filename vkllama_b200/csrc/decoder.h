// Layer-list decoder designs: a model whose configuration lists its layers, each with a mixer and a
// feed-forward of its own sizes, read from a folder (config.json, model.safetensors). The mechanisms are
// parameters of the spec; a design is the function that fills the spec from its config (checkpoint.cu).
#pragma once
#include <map>
#include <set>
#include <string>
#include <vector>

#include "rows.h"
#include "runtime.h"

namespace vkl {
struct Marker;

// Rotary positions: pairs of neighbouring dimensions, optionally with the wavelengths beyond `original / high`
// stretched (fully, by `factor`, from `original / low` on).
struct RotSpec {
  uint32_t dims = 0;          // rotated dimensions of a head, 0: no rotation
  double base = 1.0;
  bool scaled = false;
  double factor = 1.0, low = 1.0, high = 1.0, original = 1.0;
};
// Grouped-query attention and what a design puts into it.
struct AttnSpec {
  uint32_t heads = 0, kv_heads = 0, dim = 0;
  uint32_t vdim = 0;          // 0: the keys are the values
  float scale = 1.f;
  bool proj_bias = false, head_gate = false, qk_norm = false, sink = false;
  float temp_coef = 0.f;      // query temperature, see KvAttn
  uint32_t temp_every = 1;
  uint32_t bias_max = 0;      // distance at which the bucketed bias saturates, 0: no bias; the buckets' number is the table's
  uint32_t window = 0;        // 0: every position before the query
  RotSpec rot;
  int kv_from = -1;           // layer whose keys and values are used instead of own ones
};
// Gated delta rule with a decay per key channel (rows.h: DeltaRows). The ranks are those of the decay's and the output
// gate's two-step projections.
struct DeltaSpec {
  uint32_t heads = 0, kv_heads = 0, dim = 0, vdim = 0, taps = 0, decay_rank = 0, gate_rank = 0;
};
enum MixerKind : uint32_t { MIX_ATTENTION, MIX_DELTA };
enum NormKind : uint32_t {
  NORM_TANH,         // Dynamic Tanh
  NORM_RMS_CENTRED   // RMS norm, the weight stored around zero
};
enum FfnKind : uint32_t { FFN_NONE, FFN_DENSE, FFN_TABLE_MOE };
struct FfnSpec {
  FfnKind kind = FFN_NONE;
  uint32_t act = GLU_SILU;    // of a dense layer or of an expert
  uint32_t ff = 0;            // width of a dense layer or of an expert
  float limit = 0.f;
  uint32_t experts = 0, top = 0;
};
struct LayerSpec {
  MixerKind mixer = MIX_ATTENTION;
  AttnSpec attn;
  DeltaSpec delta;
  FfnSpec ffn;
};
struct DecoderSpec {
  uint32_t vocab = 0, width = 0;
  std::vector<LayerSpec> layers;
  uint32_t loop_start = 0, loop_stop = 0, loop_times = 0;  // times 0: no loop
  float logit_scale = 1.f;
  NormKind norm = NORM_TANH;
  float norm_eps = 0.f;
  bool two_norms = false;     // the feed-forward reads a norm of its own
  float embed_scale = 1.f, residual_mult = 1.f, logit_cap = 0.f;  // cap 0: none
};

// Angle per position of rotated pair i.
double rotation_frequency(const RotSpec &r, uint32_t i);
// Bucket of a distance: the first half of the rows one by one, the rest logarithmic up to `far`.
uint32_t distance_bucket(uint32_t n, uint32_t rows, uint32_t far);

struct NormVec {  // Dynamic Tanh: w, b, alpha; RMS: w
  vkl_tensor *w = nullptr, *b = nullptr;
  float alpha = 0.f;
};
struct DecLayer {
  uint32_t dp = 0, vp = 0;       // key and value width of a head in memory
  uint32_t hd = 0;               // all heads' value columns rounded up to 64
  uint32_t qcols = 0, k_col = 0, v_col = 0;  // of a row of query projections (ROW_QUERY); what follows the queries in it
  uint32_t ffp = 0;              // feed-forward width in memory
  uint32_t n1 = 0, k2 = 0;       // rows of the in-projection, columns of the out-projection
  RowSeg seg[6];
  uint32_t nseg = 0, glu_row0 = 0, q_row0 = 0, k_row0 = 0, v_row0 = 0, g_row0 = 0, low_row0 = 0;
  uint32_t gap0 = 0, n2 = 0;     // padding rows before, and first row of, what reads the second norm (0, 0: one norm)
  NormVec norm, norm2;
  vkl_tensor *w1 = nullptr, *bias1 = nullptr;  // [keys | queries | head gates | gate/up], one matrix: they read the same input
  vkl_tensor *w2 = nullptr, *bias_o = nullptr; // [attention | feed-forward] columns side by side: they add into the same rows
  vkl_tensor *rel = nullptr;                   // [heads][rel_n]: log2(e) * bias at every distance
  uint32_t rel_n = 0;
  vkl_tensor *qw = nullptr, *kw = nullptr, *freq = nullptr, *sink = nullptr;  // query and key norm, angles, sinks
  // delta rule: convolution taps, second steps of decay and gate (one matrix, two inputs), its bias, the decays' rates, norm
  vkl_tensor *taps = nullptr, *wl = nullptr, *biasl = nullptr, *rate = nullptr, *onorm = nullptr;
  uint32_t lowp = 0, nl = 0, ln2 = 0;
  vkl_tensor *we1 = nullptr, *we2 = nullptr, *table = nullptr;  // experts: gate/up rows, down rows, token table
  vkl_tensor *slot = nullptr, *token = nullptr, *tile_expert = nullptr;  // routing of the current pass's tokens
};
struct LayerRun {
  uint32_t layer;
  bool add_embedding = false;  // before the run: x += embed[token]
  int step = -1;               // before the run: x += loop.step[step]
};

struct Decoder {
  DecoderSpec spec;
  bool f32 = false;            // everything in 32-bit
  bool recurrent = false;      // some layer has a state: a sequence continues where the last pass ended, or starts at 0
  static constexpr size_t kNowhere = ~(size_t)0;
  size_t filled = kNowhere;    // tokens in the states; kNowhere: unknown, only position 0 can follow
  uint32_t ldw = 0, vocab_p = 0;
  std::vector<DecLayer> L;
  std::vector<LayerRun> runs;  // layer runs in order; run i's caches and states are in vkl_model::L[i]
  vkl_tensor *emb = nullptr, *head = nullptr, *step = nullptr;
  NormVec final_norm;
  std::vector<std::string> names;  // every tensor of the checkpoint
  std::set<std::string> loaded;
  // activations for vkl_model::cap_T rows
  vkl_tensor *x = nullptr, *h = nullptr, *q = nullptr, *gate = nullptr, *a2 = nullptr;
  vkl_tensor *low = nullptr, *dv = nullptr, *dz = nullptr, *dblocks = nullptr;  // delta rule
  vkl_tensor *xe = nullptr, *hp = nullptr, *tp = nullptr, *y = nullptr;  // experts: one token; grouped rows
  vkl_tensor *want = nullptr, *hw = nullptr, *logits_rows = nullptr, *trace = nullptr;
  uint32_t low_max = 0, dv_max = 0, dz_max = 0;
  uint32_t qld_max = 0, gld_max = 0, k2_max = 0, top_max = 0, ffe_max = 0, experts_max = 0, heads_max = 0;
  vkl_tensor *attn_scratch = nullptr, *attn_counters = nullptr;
  uint32_t counters_n = 0;
  uint32_t launches_per_token = 0;
  // what the next pass leaves besides the last row's logits (host side, set before decoder_run)
  std::vector<int32_t> want_rows;  // rows whose logits go to logits_rows
  bool tracing = false;            // residual stream after every layer run -> trace [runs][T][ldw]
  ~Decoder();
};

// Creates a model for the spec; maxlen positions per sequence, compute in 32-bit or bfloat16.
int decoder_create(vkl_device *dev, const DecoderSpec &spec, uint32_t maxlen, bool f32, vkl_model **out);
int decoder_set_weight(vkl_model *m, const char *name, int dtype, const void *data, size_t bytes);
// The shape a checkpoint gives for a tensor against the spec's.
int decoder_check_shape(vkl_model *m, const char *name, const std::vector<uint32_t> &dims);
int decoder_synth(vkl_model *m, uint64_t seed, float wstd, float nstd);
int decoder_ready(const vkl_model *m);
int decoder_ensure_rows(vkl_model *m, uint32_t T);
// Before and after passes that take a sequence from position `offset` to `end`: refuses a position that the recurrent
// states are not at. In between (and if something fails) the states count as unknown.
int decoder_begin(vkl_model *m, size_t offset);
void decoder_end(vkl_model *m, size_t end);
// One pass over T tokens in vkl_model::toks from the position in vkl_model::state: appends to the caches, leaves
// the last row's fp32 logits in logits32 and its arg-max in state[2].
int decoder_run(vkl_model *m, uint32_t T, bool pdl, Marker *mk);

}  // namespace vkl
