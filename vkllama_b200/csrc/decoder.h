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

// Attention whose keys are its values: grouped heads, biases on the projections, no rotation.
struct AttnSpec {
  uint32_t heads = 0, kv_heads = 0, dim = 0;
  float scale = 1.f;
  float temp_coef = 0.f;      // query temperature, see KvAttn
  uint32_t temp_every = 1;
  uint32_t bias_max = 0;      // distance at which the bucketed bias saturates; the buckets' number is the table's
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
  AttnSpec attn;
  FfnSpec ffn;
};
struct DecoderSpec {
  uint32_t vocab = 0, width = 0;
  std::vector<LayerSpec> layers;
  uint32_t loop_start = 0, loop_stop = 0, loop_times = 0;  // times 0: no loop
  float logit_scale = 1.f;
};

// Bucket of a distance: the first half of the rows one by one, the rest logarithmic up to `far`.
uint32_t distance_bucket(uint32_t n, uint32_t rows, uint32_t far);

struct NormVec {  // Dynamic Tanh
  vkl_tensor *w = nullptr, *b = nullptr;
  float alpha = 0.f;
};
struct DecLayer {
  uint32_t dp = 0, hd = 0;       // head width in memory, all heads' columns rounded up to 64
  uint32_t ffp = 0;              // feed-forward width in memory
  uint32_t n1 = 0, k2 = 0;       // rows of the in-projection, columns of the out-projection
  RowSeg seg[4];
  uint32_t nseg = 0, glu_row0 = 0, q_row0 = 0, g_row0 = 0;
  NormVec norm;
  vkl_tensor *w1 = nullptr, *bias1 = nullptr;  // [keys | queries | head gates | gate/up], one matrix: they read the same input
  vkl_tensor *w2 = nullptr, *bias_o = nullptr; // [attention | feed-forward] columns side by side: they add into the same rows
  vkl_tensor *rel = nullptr;                   // [heads][rel_n]: log2(e) * bias at every distance
  uint32_t rel_n = 0;
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
  uint32_t ldw = 0, vocab_p = 0;
  std::vector<DecLayer> L;
  std::vector<LayerRun> runs;  // layer runs in order; run i's key cache is vkl_model::L[i].kcache
  vkl_tensor *emb = nullptr, *head = nullptr, *step = nullptr;
  NormVec final_norm;
  std::vector<std::string> names;  // every tensor of the checkpoint
  std::set<std::string> loaded;
  // activations for vkl_model::cap_T rows
  vkl_tensor *x = nullptr, *h = nullptr, *q = nullptr, *gate = nullptr, *a2 = nullptr;
  vkl_tensor *xe = nullptr, *hp = nullptr, *tp = nullptr, *y = nullptr;  // experts: one token; grouped rows
  vkl_tensor *want = nullptr, *hw = nullptr, *logits_rows = nullptr, *trace = nullptr;
  uint32_t hd_max = 0, qld_max = 0, gld_max = 0, k2_max = 0, top_max = 0, ffe_max = 0, experts_max = 0, heads_max = 0;
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
// One pass over T tokens in vkl_model::toks from the position in vkl_model::state: appends to the caches, leaves
// the last row's fp32 logits in logits32 and its arg-max in state[2].
int decoder_run(vkl_model *m, uint32_t T, bool pdl, Marker *mk);

}  // namespace vkl
