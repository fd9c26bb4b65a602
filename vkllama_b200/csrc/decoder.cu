// The layer-list decoder designs on this library's model driver: weight placement, buffers and the pass over
// T tokens that vkl_model_forward and vkl_model_generate run (model.cu owns caches, token loop, decode graph,
// arg-max and sampling input).
//
// A layer is a parallel block: both sublayers read the same residual stream, through one norm or through one each,
// and add to it together, so
//   * everything that reads the stream's norms is ONE matrix (keys, queries, values, head gates, gate/up); with two
//     norms its last rows take the second one as their input,
//   * everything that adds to the stream is ONE matrix over the concatenated inputs,
//   * a norm without statistics (Dynamic Tanh) is computed by the epilogue that completes the stream.
// A design with Dynamic Tanh takes three kernels per layer and token (in-projection, attention, out-projection) for
// decode and for prompts alike; norms with statistics, rotation and the delta rule's steps come between. Layers with routed experts: in decode the experts' rows are extra units of the same two
// launches; prompts group the tokens by expert and run two grouped GEMMs and a combine step.
#include <math.h>
#include <stdlib.h>
#include <string.h>

#include <algorithm>

#include "decoder.h"
#include "model.h"

namespace vkl {

uint32_t distance_bucket(uint32_t n, uint32_t rows, uint32_t far) {
  const uint32_t half = rows / 2;
  if (n < half) return n;
  const double v = log((double)n / half) / log((double)far / half) * (rows - half), near = rint(v);
  // a distance that is exactly a bucket's first one must not fall below it by a rounding
  const double k = fabs(v - near) < 1e-9 * std::max(1.0, fabs(near)) ? near : floor(v);
  return std::min(rows - 1, half + (uint32_t)k);
}

double rotation_frequency(const RotSpec &r, uint32_t i) {
  const double f = pow(r.base, -2.0 * i / r.dims), len = 2.0 * M_PI / f;
  if (!r.scaled || len < r.original / r.high) return f;
  if (len > r.original / r.low) return f / r.factor;
  const double s = (r.original / len - r.low) / (r.high - r.low);
  return (1.0 - s) * f / r.factor + s * f;
}

Decoder::~Decoder() {
  for (DecLayer &l : L)
    for (vkl_tensor *t : {l.norm.w, l.norm.b, l.norm2.w, l.norm2.b, l.qw, l.kw, l.freq, l.sink, l.taps, l.wl, l.biasl, l.rate, l.onorm, l.w1, l.bias1, l.w2, l.bias_o, l.rel, l.we1, l.we2, l.table, l.slot, l.token, l.tile_expert}) vkl_tensor_release(t);
  for (vkl_tensor *t : {emb, head, step, final_norm.w, final_norm.b, x, h, q, gate, a2, low, dv, dz, dblocks, xe, hp, tp, y, want, hw, logits_rows, trace, attn_scratch, attn_counters}) vkl_tensor_release(t);
}

namespace {

uint32_t up_to(uint32_t n, uint32_t k) { return (n + k - 1) / k * k; }
int compute_dtype(const Decoder *d) { return d->f32 ? VKL_FP32 : VKL_BF16; }
size_t elem(const Decoder *d) { return d->f32 ? 4 : 2; }

int zeros(vkl_model *m, vkl_tensor **t, size_t c, size_t h, size_t w, int dtype) {
  VKL_OKAY(ensure_tensor(m->dev, t, c, h, w, dtype));
  VKL_CUDA(cudaMemsetAsync((*t)->data(), 0, (*t)->device_bytes(), m->stream));
  return VKL_OK;
}

// Where a checkpoint tensor goes.
struct Target {
  enum Kind { MATRIX, VECTOR, SCALAR, DISTANCE, TABLE, RATE } kind = MATRIX;  // RATE: exp of one number per head, for every row of it
  vkl_tensor *dst = nullptr;
  uint32_t rows = 0, cols = 0, ld = 0;
  size_t row_base = 0;       // first row of dst (one of several matrices in it)
  PackMap map = {1u << 30, 0, 0, 1u << 30, 0, 0};
  float *scalar = nullptr;
  float add = 0.f;           // VECTOR: added to every element
  bool optional = false;     // a checkpoint may have it, nothing reads it
  DecLayer *layer = nullptr;
  const LayerSpec *spec = nullptr;
  float synth_mean = 0.f, synth_std = -1.f;  // std < 0: the weight matrices'
};

bool norm_target(Decoder *d, NormVec &n, const std::string &rest, Target *t) {
  t->kind = Target::VECTOR;
  t->rows = d->spec.width;
  t->cols = 1;
  if (d->spec.norm == NORM_RMS_CENTRED) {
    if (!rest.empty()) return false;
    t->dst = n.w;
    t->add = 1.f;
    t->synth_std = -2.f;
    return true;
  }
  if (rest.empty()) {
    t->dst = n.w;
    t->synth_mean = 1.f;
    t->synth_std = -2.f;  // the norms'
  } else if (rest == ".b") {
    t->dst = n.b;
    t->synth_std = -2.f;
  } else if (rest == ".alpha") {
    t->kind = Target::SCALAR;
    t->rows = 1;
    t->scalar = &n.alpha;
    t->synth_mean = 0.5f;
    t->synth_std = 0.f;
  } else {
    return false;
  }
  return true;
}

// The tensors of a delta-rule mixer; what is left of their names after "mix.".
bool delta_target(Decoder *d, DecLayer &l, const DeltaSpec &p, const std::string &s, Target *t) {
  const uint32_t W = d->spec.width;
  auto matrix = [&](vkl_tensor *dst, uint32_t rows, uint32_t cols, uint32_t ld, uint32_t row0) {
    t->kind = Target::MATRIX;
    t->dst = dst;
    t->rows = rows;
    t->cols = cols;
    t->ld = ld;
    t->map.r0 = row0;
  };
  auto heads_rows = [&](uint32_t from, uint32_t to) { t->map.ra = from; t->map.rb = to; };
  auto vector = [&](vkl_tensor *dst, uint32_t n) { t->kind = Target::VECTOR; t->dst = dst; t->rows = n; t->cols = 1; };
  const std::string side = s.substr(0, 1);
  if (side == "q" || side == "k" || side == "v") {
    const bool v = side == "v";
    const uint32_t n = v ? p.heads : p.kv_heads, w = v ? p.vdim : p.dim, wp = v ? l.vp : l.dp, col = v ? l.v_col : side == "k" ? l.k_col : 0;
    if (s.size() == 1) {
      matrix(l.w1, n * w, W, d->ldw, l.q_row0 + col);
      heads_rows(w, wp);
      return true;
    }
    if (s.substr(1) == ".conv") {  // [channels, taps], channels placed like the rows of the projection
      vector(l.taps, n * w);
      t->cols = p.taps;
      t->map.ra = w * p.taps;
      t->map.rb = wp * p.taps;
      t->map.r0 = col * p.taps;
      t->synth_std = 0.5f;
      return true;
    }
    return false;
  }
  if (s == "b") { matrix(l.w1, p.heads, W, d->ldw, l.g_row0); return true; }
  if (s == "a1") { matrix(l.w1, p.decay_rank, W, d->ldw, l.low_row0); return true; }
  if (s == "g1") { matrix(l.w1, p.gate_rank, W, d->ldw, l.low_row0 + l.lowp); return true; }
  if (s == "a2") { matrix(l.wl, p.heads * p.dim, p.decay_rank, l.lowp, 0); heads_rows(p.dim, l.dp); return true; }
  if (s == "g2") { matrix(l.wl, p.heads * p.vdim, p.gate_rank, l.lowp, l.ln2); heads_rows(p.vdim, l.vp); return true; }
  if (s == "dt_bias") { vector(l.biasl, p.heads * p.dim); heads_rows(p.dim, l.dp); t->synth_std = 1.f; return true; }
  if (s == "norm") { vector(l.onorm, p.vdim); t->synth_mean = 1.f; t->synth_std = -2.f; return true; }
  if (s == "A_log") {
    vector(l.rate, p.heads);
    t->kind = Target::RATE;
    heads_rows(p.dim, l.dp);
    t->synth_std = 0.5f;
    return true;
  }
  if (s == "o") {
    matrix(l.w2, W, p.heads * p.vdim, l.k2, 0);
    t->map.ca = p.vdim;
    t->map.cb = l.vp;
    return true;
  }
  return false;
}

bool layer_target(Decoder *d, uint32_t i, const std::string &s, Target *t) {
  DecLayer &l = d->L[i];
  const LayerSpec &p = d->spec.layers[i];
  const AttnSpec &a = p.attn;
  const FfnSpec &f = p.ffn;
  const uint32_t W = d->spec.width, vdim = a.vdim ? a.vdim : a.dim;
  t->layer = &l;
  t->spec = &p;
  auto matrix = [&](vkl_tensor *dst, uint32_t rows, uint32_t cols, uint32_t ld) {
    t->kind = Target::MATRIX;
    t->dst = dst;
    t->rows = rows;
    t->cols = cols;
    t->ld = ld;
  };
  auto heads_rows = [&](uint32_t row0) { t->map.ra = a.dim; t->map.rb = l.dp; t->map.r0 = row0; };
  auto glu_rows = [&](uint32_t row0, bool up) { t->map.ra = 16; t->map.rb = 32; t->map.r0 = row0 + (up ? 16 : 0); };
  auto as_vector = [&](vkl_tensor *dst) { t->kind = Target::VECTOR; t->dst = dst; t->cols = 1; };
  if (s.rfind("norm1", 0) == 0) return norm_target(d, l.norm, s.substr(5), t);
  if (d->spec.two_norms && s.rfind("norm2", 0) == 0) {
    t->optional = f.kind == FFN_NONE;
    return norm_target(d, l.norm2, s.substr(5), t);
  }
  if (p.mixer == MIX_DELTA && s.rfind("mix.", 0) == 0) return delta_target(d, l, p.delta, s.substr(4), t);
  const bool own_kv = a.kv_from < 0;
  if (s == "mix.q" || (a.proj_bias && s == "mix.q.b")) {
    matrix(l.w1, a.heads * a.dim, W, d->ldw);
    heads_rows(l.q_row0);
    if (s == "mix.q.b") as_vector(l.bias1);
    return true;
  }
  if (own_kv && (s == "mix.k" || (a.proj_bias && s == "mix.k.b"))) {
    matrix(l.w1, a.kv_heads * a.dim, W, d->ldw);
    heads_rows(l.k_row0);
    if (s == "mix.k.b") as_vector(l.bias1);
    return true;
  }
  if (own_kv && a.vdim && s == "mix.v") {
    matrix(l.w1, a.kv_heads * a.vdim, W, d->ldw);
    t->map.ra = a.vdim;
    t->map.rb = l.vp;
    t->map.r0 = l.v_row0;
    return true;
  }
  if (a.qk_norm && (s == "mix.q.norm" || (own_kv && s == "mix.k.norm"))) {
    const bool q = s == "mix.q.norm";
    t->rows = (q ? a.heads : a.kv_heads) * a.dim;
    as_vector(q ? l.qw : l.kw);
    heads_rows(0);
    t->synth_mean = 1.f;
    t->synth_std = -2.f;
    return true;
  }
  if (a.sink && s == "mix.sink") {
    t->rows = a.heads;
    as_vector(l.sink);
    t->synth_std = 1.f;
    return true;
  }
  if (a.head_gate && s == "mix.g") {
    matrix(l.w1, a.heads, W, d->ldw);
    t->map.r0 = l.g_row0;
    return true;
  }
  if (s == "mix.o") {
    matrix(l.w2, W, a.heads * vdim, l.k2);
    t->map.ca = vdim;
    t->map.cb = l.vp;
    return true;
  }
  if (a.proj_bias && s == "mix.o.b") {
    t->rows = W;
    as_vector(l.bias_o);
    return true;
  }
  if (a.bias_max && s == "mix.rel") {
    t->kind = Target::DISTANCE;
    t->dst = l.rel;
    return true;
  }
  if (f.kind == FFN_DENSE) {
    if (s == "mlp.gate" || s == "mlp.up") {
      matrix(l.w1, f.ff, W, d->ldw);
      glu_rows(l.glu_row0, s == "mlp.up");
      return true;
    }
    if (s == "mlp.down") {
      matrix(l.w2, W, f.ff, l.k2);
      t->map.c0 = l.hd;
      return true;
    }
  }
  if (f.kind == FFN_TABLE_MOE) {
    if (s == "mlp.table") {
      t->kind = Target::TABLE;
      t->dst = l.table;
      t->rows = d->spec.vocab;
      t->cols = f.top;
      return true;
    }
    unsigned e = 0;
    int at = 0;
    if (sscanf(s.c_str(), "mlp.e%u.%n", &e, &at) == 1 && at && e < f.experts) {
      const std::string w = s.substr(at);
      if (w == "gate" || w == "up") {
        matrix(l.we1, f.ff, W, d->ldw);
        t->row_base = (size_t)e * 2 * l.ffp;
        glu_rows(0, w == "up");
        return true;
      }
      if (w == "down") {
        matrix(l.we2, W, f.ff, l.ffp);
        t->row_base = (size_t)e * d->ldw;
        return true;
      }
    }
  }
  return false;
}

bool find_target(Decoder *d, const std::string &name, Target *t) {
  *t = Target();
  if (name == "embed" || name == "head") {
    t->dst = name == "embed" ? d->emb : d->head;
    t->rows = d->spec.vocab;
    t->cols = d->spec.width;
    t->ld = d->ldw;
    if (name == "embed") t->synth_std = 1.f;
    return true;
  }
  if (name == "loop.step" && d->spec.loop_times) {  // [times, width] -> fp32 rows of ldw
    t->kind = Target::VECTOR;
    t->dst = d->step;
    t->rows = d->spec.loop_times * d->spec.width;
    t->cols = 1;
    t->map.ra = d->spec.width;
    t->map.rb = d->ldw;
    t->synth_std = -2.f;
    return true;
  }
  if (name.rfind("final.norm", 0) == 0) return norm_target(d, d->final_norm, name.substr(10), t);
  unsigned i = 0;
  int at = 0;
  if (sscanf(name.c_str(), "l%u.%n", &i, &at) == 1 && at && i < d->L.size()) return layer_target(d, i, name.substr(at), t);
  return false;
}

float bf16_value(const uint8_t *p) {
  uint16_t u;
  memcpy(&u, p, 2);
  const uint32_t w = (uint32_t)u << 16;
  float v;
  memcpy(&v, &w, 4);
  return v;
}

// The distance table as one number per distance, in units of log2 (the attention's exponentials are base 2).
int set_distance(vkl_model *m, DecLayer *l, const LayerSpec *p, const std::vector<float> &rel) {
  const uint32_t H = p->attn.heads, B = (uint32_t)(rel.size() / H), n = l->rel_n;
  if (B < 2 || B * H != rel.size()) return fail(VKL_INVALID_ARGUMENT, "model_set_weight: a distance table of %zu numbers for %u heads", rel.size(), H);
  if (p->attn.bias_max <= B / 2) return fail(VKL_INVALID_ARGUMENT, "model_set_weight: bias_max %u does not exceed half of the table's %u rows", p->attn.bias_max, B);
  std::vector<float> out((size_t)H * n);
  for (uint32_t j = 0; j < n; ++j) {
    const uint32_t b = distance_bucket(j, B, p->attn.bias_max);
    for (uint32_t h = 0; h < H; ++h) out[(size_t)h * n + j] = (float)(rel[(size_t)b * H + h] * 1.4426950408889634);
  }
  VKL_CUDA(cudaMemcpyAsync(l->rel->data(), out.data(), out.size() * 4, cudaMemcpyHostToDevice, m->stream));
  VKL_CUDA(cudaStreamSynchronize(m->stream));
  return VKL_OK;
}

// All tensor names of the spec, the order of the synthetic weights' ids.
std::vector<std::string> tensor_names(const DecoderSpec &s) {
  std::vector<std::string> n = {"embed", "head"};
  if (s.loop_times) n.push_back("loop.step");
  auto norm = [&](const std::string &p) {
    n.push_back(p);
    if (s.norm == NORM_TANH)
      for (const char *e : {".b", ".alpha"}) n.push_back(p + e);
  };
  norm("final.norm");
  for (size_t i = 0; i < s.layers.size(); ++i) {
    const std::string l = "l" + std::to_string(i) + ".";
    const FfnSpec &f = s.layers[i].ffn;
    norm(l + "norm1");
    if (s.two_norms && f.kind != FFN_NONE) norm(l + "norm2");
    auto mix = [&](bool have, const char *k) {
      if (have) n.push_back(l + "mix." + k);
    };
    if (s.layers[i].mixer == MIX_DELTA) {
      for (const char *k : {"q", "q.conv", "k", "k.conv", "v", "v.conv", "b", "A_log", "norm", "a1", "a2", "dt_bias", "g1", "g2", "o"}) mix(true, k);
    } else {
      const AttnSpec &a = s.layers[i].attn;
      const bool own = a.kv_from < 0;
      mix(true, "q");
      mix(a.proj_bias, "q.b");
      mix(own, "k");
      mix(own && a.proj_bias, "k.b");
      mix(own && a.vdim, "v");
      mix(a.qk_norm, "q.norm");
      mix(own && a.qk_norm, "k.norm");
      mix(a.sink, "sink");
      mix(a.bias_max, "rel");
      mix(a.head_gate, "g");
      mix(true, "o");
      mix(a.proj_bias, "o.b");
    }
    if (f.kind == FFN_DENSE)
      for (const char *k : {"gate", "up", "down"}) n.push_back(l + "mlp." + k);
    if (f.kind == FFN_TABLE_MOE) {
      for (uint32_t e = 0; e < f.experts; ++e)
        for (const char *k : {"gate", "up", "down"}) n.push_back(l + "mlp.e" + std::to_string(e) + "." + k);
      n.push_back(l + "mlp.table");
    }
  }
  return n;
}

int check_spec(const DecoderSpec &s, uint32_t maxlen) {
  if (!s.vocab || !s.width || !maxlen || s.layers.empty()) return fail(VKL_INVALID_ARGUMENT, "model: empty vocabulary, width, context or layer list");
  if (s.loop_times && (s.loop_start >= s.loop_stop || s.loop_stop > s.layers.size()))
    return fail(VKL_INVALID_ARGUMENT, "model: the loop runs layers %u .. %u of %zu", s.loop_start, s.loop_stop, s.layers.size());
  for (size_t i = 0; i < s.layers.size(); ++i) {
    const LayerSpec &l = s.layers[i];
    if (l.mixer == MIX_DELTA) {
      const DeltaSpec &p = l.delta;
      if (!p.heads || !p.kv_heads || p.heads % p.kv_heads || !p.dim || !p.vdim || !p.taps || !p.decay_rank || !p.gate_rank)
        return fail(VKL_INVALID_ARGUMENT, "model: a delta rule of %u heads over %u key heads, widths %u and %u, %u taps, ranks %u and %u", p.heads, p.kv_heads, p.dim, p.vdim, p.taps,
                    p.decay_rank, p.gate_rank);
      if (p.dim > 256 || p.vdim > 256) return fail(VKL_UNIMPLEMENTED, "model: a delta rule of widths %u and %u (at most 256)", p.dim, p.vdim);
      if (s.loop_times) return fail(VKL_UNIMPLEMENTED, "model: recurrent layers and a loop over layers");
    }
    const FfnSpec &f = l.ffn;
    if (f.kind != FFN_NONE && !f.ff) return fail(VKL_INVALID_ARGUMENT, "model: a feed-forward of width 0");
    if (f.kind == FFN_TABLE_MOE && (!f.experts || !f.top || f.top > f.experts || f.experts > 4096))
      return fail(VKL_INVALID_ARGUMENT, "model: %u of %u experts", f.top, f.experts);
    if (f.kind == FFN_TABLE_MOE && s.two_norms) return fail(VKL_UNIMPLEMENTED, "model: routed experts with a norm of their own");
    if (l.mixer == MIX_DELTA) continue;
    const AttnSpec &a = l.attn;
    if (!a.heads || !a.kv_heads || a.heads % a.kv_heads || !a.dim) return fail(VKL_INVALID_ARGUMENT, "model: %u heads over %u key heads of width %u", a.heads, a.kv_heads, a.dim);
    if (a.dim > 256 || a.vdim > 256) return fail(VKL_UNIMPLEMENTED, "model: head width %u, %u (at most 256)", a.dim, a.vdim);
    if (a.rot.dims % 2 || a.rot.dims > a.dim) return fail(VKL_INVALID_ARGUMENT, "model: a rotation of %u of %u dimensions", a.rot.dims, a.dim);
    if ((a.qk_norm || a.rot.dims) && (a.proj_bias || !a.vdim)) return fail(VKL_UNIMPLEMENTED, "model: normed or rotated keys that are values or have a bias");
    if (a.kv_from >= 0) {
      const LayerSpec *o = (size_t)a.kv_from < i ? &s.layers[a.kv_from] : nullptr;
      if (s.loop_times) return fail(VKL_UNIMPLEMENTED, "model: shared caches and a loop over layers");
      if (!o || o->mixer != MIX_ATTENTION || o->attn.kv_from >= 0) return fail(VKL_INVALID_ARGUMENT, "model: layer %zu uses the cache of layer %d", i, a.kv_from);
      if (o->attn.kv_heads != a.kv_heads || o->attn.dim != a.dim || o->attn.vdim != a.vdim)
        return fail(VKL_INVALID_ARGUMENT, "model: layer %zu uses the cache of layer %d, which has other sizes", i, a.kv_from);
    }
    if (!a.temp_every) return fail(VKL_INVALID_ARGUMENT, "model: the query temperature's period is 0");
  }
  return VKL_OK;
}

int new_norm(vkl_model *m, NormVec *n, uint32_t ldw) {
  VKL_OKAY(zeros(m, &n->w, 1, 1, ldw, VKL_FP32));
  if (m->dec->spec.norm != NORM_TANH) return VKL_OK;
  return zeros(m, &n->b, 1, 1, ldw, VKL_FP32);
}

// Buffers of one token that the layer needs, and its mixer's own vectors and matrices.
int build_attention(vkl_model *m, DecLayer &l, const AttnSpec &a) {
  Decoder *d = m->dec.get();
  l.rel_n = a.bias_max ? std::min(a.bias_max, m->cfg.maxlen) + 1 : 0;
  if (a.bias_max) VKL_OKAY(zeros(m, &l.rel, 1, a.heads, l.rel_n, VKL_FP32));
  if (a.sink) VKL_OKAY(zeros(m, &l.sink, 1, 1, a.heads, VKL_FP32));
  if (a.qk_norm) VKL_OKAY(zeros(m, &l.qw, 1, 1, a.heads * l.dp, VKL_FP32));
  if (a.qk_norm && a.kv_from < 0) VKL_OKAY(zeros(m, &l.kw, 1, 1, a.kv_heads * l.dp, VKL_FP32));
  if (a.rot.dims) {
    std::vector<float> f(a.rot.dims / 2);
    for (uint32_t i = 0; i < f.size(); ++i) f[i] = (float)rotation_frequency(a.rot, i);
    VKL_OKAY(zeros(m, &l.freq, 1, 1, f.size(), VKL_FP32));
    VKL_CUDA(cudaMemcpyAsync(l.freq->data(), f.data(), f.size() * 4, cudaMemcpyHostToDevice, m->stream));
    VKL_CUDA(cudaStreamSynchronize(m->stream));
  }
  d->gld_max = std::max(d->gld_max, up_to(a.heads, 32));
  d->heads_max = std::max(d->heads_max, a.heads);
  return VKL_OK;
}

int build_delta(vkl_model *m, DecLayer &l, const DeltaSpec &p) {
  Decoder *d = m->dec.get();
  d->recurrent = true;
  l.ln2 = up_to(p.heads * l.dp, kInputAlign);
  l.nl = l.ln2 + up_to(p.heads * l.vp, 32);
  VKL_OKAY(zeros(m, &l.taps, 1, l.qcols, p.taps, VKL_FP32));
  VKL_OKAY(zeros(m, &l.wl, 1, l.nl, l.lowp, VKL_BF16));
  VKL_OKAY(zeros(m, &l.biasl, 1, 1, l.nl, VKL_FP32));
  VKL_OKAY(zeros(m, &l.rate, 1, 1, l.ln2, VKL_FP32));
  VKL_OKAY(zeros(m, &l.onorm, 1, 1, l.vp, VKL_FP32));
  d->low_max = std::max(d->low_max, l.lowp);
  d->dv_max = std::max(d->dv_max, p.heads * l.vp);
  d->dz_max = std::max(d->dz_max, l.nl);
  d->gld_max = std::max(d->gld_max, up_to(p.heads, 32));
  return VKL_OK;
}

int build(vkl_model *m) {
  Decoder *d = m->dec.get();
  const DecoderSpec &s = d->spec;
  d->ldw = up_to(s.width, 64);
  d->vocab_p = up_to(s.vocab, 32);
  VKL_OKAY(zeros(m, &d->emb, 1, s.vocab, d->ldw, VKL_BF16));
  VKL_OKAY(zeros(m, &d->head, 1, d->vocab_p, d->ldw, VKL_BF16));
  if (s.loop_times) VKL_OKAY(zeros(m, &d->step, 1, s.loop_times, d->ldw, VKL_FP32));
  VKL_OKAY(new_norm(m, &d->final_norm, d->ldw));
  d->L.resize(s.layers.size());
  for (size_t i = 0; i < s.layers.size(); ++i) {
    DecLayer &l = d->L[i];
    const LayerSpec &p = s.layers[i];
    const AttnSpec &a = p.attn;
    const FfnSpec &f = p.ffn;
    const bool delta = p.mixer == MIX_DELTA;
    l.ffp = f.kind == FFN_NONE ? 0 : up_to(f.ff, 64);
    uint32_t n = 0;
    auto seg = [&](uint32_t rows, uint32_t kind) {
      const uint32_t at = n;
      n += up_to(rows, 32);
      l.seg[l.nseg++] = RowSeg{at, n, kind};
      return at;
    };
    if (delta) {
      const DeltaSpec &r = p.delta;
      l.dp = up_to(r.dim, 32);
      l.vp = up_to(r.vdim, 16);
      l.lowp = up_to(std::max(r.decay_rank, r.gate_rank), 64);
      l.k_col = r.kv_heads * l.dp;
      l.v_col = 2 * l.k_col;
      l.qcols = up_to(l.v_col + r.heads * l.vp, 32);
      l.q_row0 = seg(l.qcols, ROW_QUERY);
      l.low_row0 = seg(2 * l.lowp, ROW_LOW);
      l.g_row0 = seg(r.heads, ROW_HEAD_GATE);
      l.hd = up_to(r.heads * l.vp, 64);
      VKL_OKAY(build_delta(m, l, r));
    } else {
      l.dp = up_to(a.dim, 16);
      l.vp = a.vdim ? up_to(a.vdim, 16) : l.dp;
      l.hd = up_to(a.heads * l.vp, 64);
      const uint32_t qn = up_to(a.heads * l.dp, 32), kn = up_to(a.kv_heads * l.dp, 32);
      const bool own = a.kv_from < 0, prep = a.qk_norm || a.rot.dims;  // prep: the keys are not yet what the cache holds
      l.qcols = qn;
      if (prep && own) {
        l.k_col = qn;
        l.qcols += kn;
        l.q_row0 = seg(l.qcols, ROW_QUERY);
        l.k_row0 = l.q_row0 + l.k_col;
      } else {
        if (own) l.k_row0 = seg(kn, ROW_KEY);
        l.q_row0 = seg(qn, ROW_QUERY);
      }
      if (own && a.vdim) l.v_row0 = seg(a.kv_heads * l.vp, ROW_VALUE);
      if (a.head_gate) l.g_row0 = seg(a.heads, ROW_HEAD_GATE);
      VKL_OKAY(build_attention(m, l, a));
    }
    if (f.kind == FFN_DENSE) {
      if (s.two_norms) {
        l.gap0 = n;
        l.n2 = up_to(n, kInputAlign);
        if (l.n2 > n) seg(l.n2 - n, ROW_NONE);
      }
      l.glu_row0 = seg(2 * l.ffp, ROW_GLU);
    }
    l.n1 = n;
    l.k2 = l.hd + (f.kind == FFN_DENSE ? l.ffp : 0);
    VKL_OKAY(new_norm(m, &l.norm, d->ldw));
    if (s.two_norms) VKL_OKAY(new_norm(m, &l.norm2, d->ldw));
    VKL_OKAY(zeros(m, &l.w1, 1, l.n1, d->ldw, VKL_BF16));
    VKL_OKAY(zeros(m, &l.w2, 1, d->ldw, l.k2, VKL_BF16));
    if (!delta && a.proj_bias) {
      VKL_OKAY(zeros(m, &l.bias1, 1, 1, l.n1, VKL_FP32));
      VKL_OKAY(zeros(m, &l.bias_o, 1, 1, d->ldw, VKL_FP32));
    }
    if (f.kind == FFN_TABLE_MOE) {
      VKL_OKAY(zeros(m, &l.we1, f.experts, 2 * l.ffp, d->ldw, VKL_BF16));
      VKL_OKAY(zeros(m, &l.we2, f.experts, d->ldw, l.ffp, VKL_BF16));
      VKL_OKAY(zeros(m, &l.table, 1, s.vocab, f.top, VKL_UINT32));
      d->top_max = std::max(d->top_max, f.top);
      d->ffe_max = std::max(d->ffe_max, l.ffp);
      d->experts_max = std::max(d->experts_max, f.experts);
    }
    d->qld_max = std::max(d->qld_max, l.qcols);
    d->k2_max = std::max(d->k2_max, l.k2);
  }
  const uint32_t nl = (uint32_t)s.layers.size(), lo = s.loop_times ? s.loop_start : nl, hi = s.loop_times ? s.loop_stop : nl;
  for (uint32_t i = 0; i < lo; ++i) d->runs.push_back(LayerRun{i});
  for (uint32_t t = 0; t < s.loop_times; ++t)
    for (uint32_t i = lo; i < hi; ++i) {
      LayerRun r{i};
      if (i == lo) {
        r.add_embedding = t > 0;
        r.step = (int)t;
      }
      d->runs.push_back(r);
    }
  for (uint32_t i = hi; i < nl; ++i) d->runs.push_back(LayerRun{i});
  m->cfg.layers = (uint32_t)d->runs.size();
  m->L.resize(d->runs.size());
  for (size_t r = 0; r < d->runs.size(); ++r) {
    const uint32_t i = d->runs[r].layer;
    const LayerSpec &p = s.layers[i];
    const DecLayer &l = d->L[i];
    if (p.mixer == MIX_DELTA) {
      VKL_OKAY(zeros(m, &m->L[r].state, p.delta.heads, l.vp, l.dp, VKL_FP32));
      VKL_OKAY(zeros(m, &m->L[r].ring, 1, p.delta.taps, l.qcols, compute_dtype(d)));
    } else if (p.attn.kv_from < 0) {
      VKL_OKAY(zeros(m, &m->L[r].kcache, p.attn.kv_heads, m->cfg.maxlen, l.dp, compute_dtype(d)));
      if (p.attn.vdim) VKL_OKAY(zeros(m, &m->L[r].vcache, p.attn.kv_heads, m->cfg.maxlen, l.vp, compute_dtype(d)));
    }
  }
  d->names = tensor_names(s);
  return VKL_OK;
}

// The residual step that follows layer run `r` (-1: the embedding): what the next run adds first, and its norm.
Residual residual_after(vkl_model *m, int r) {
  Decoder *d = m->dec.get();
  Residual o = {};
  o.x = (float *)d->x->data();
  o.ldw = d->ldw;
  o.mult = d->spec.residual_mult;
  const NormVec *n = &d->final_norm;
  if ((size_t)(r + 1) < d->runs.size()) {
    const LayerRun &next = d->runs[r + 1];
    n = &d->L[next.layer].norm;
    if (next.add_embedding) {
      o.emb = (const bf16 *)d->emb->data();
      o.toks = (const uint32_t *)m->toks->data();
    }
    if (next.step >= 0) o.step = (const float *)d->step->data() + (size_t)next.step * d->ldw;
  }
  if (d->spec.norm != NORM_TANH) return o;  // a kernel of its own: norm_after
  o.h = d->h->data();
  o.nw = (const float *)n->w->data();
  o.nb = (const float *)n->b->data();
  o.alpha = n->alpha;
  return o;
}

// The norm with statistics that follows layer run `r` (-1: the embedding), of both sublayers' inputs or the final one:
// a kernel of its own for several tokens, for one part of the matrix product that reads it.
RmsRows norm_of(vkl_model *m, int r, uint32_t T) {
  Decoder *d = m->dec.get();
  RmsRows p = {};
  if (d->spec.norm == NORM_TANH) return p;
  p.x = (const float *)d->x->data();
  p.T = T;
  p.ldw = d->ldw;
  p.width = d->spec.width;
  p.eps = d->spec.norm_eps;
  p.h = d->h->data();
  p.w = (const float *)d->final_norm.w->data();
  if ((size_t)(r + 1) < d->runs.size()) {
    const DecLayer &l = d->L[d->runs[r + 1].layer];
    p.w = (const float *)l.norm.w->data();
    if (l.n2) {
      p.w2 = (const float *)l.norm2.w->data();
      p.h2 = d->h->data() + (size_t)T * d->ldw * elem(d);  // the second input of the in-projection follows the first
    }
  }
  return p;
}
bool norm_in_matvec(const Decoder *d, uint32_t T) { return T == 1 && rows_matvec_takes_norm(d->ldw, d->spec.two_norms, d->f32); }
int norm_after(vkl_model *m, int r, uint32_t T, bool pdl) {
  Decoder *d = m->dec.get();
  RmsRows p = norm_of(m, r, T);
  if (!p.x || norm_in_matvec(d, T)) return VKL_OK;
  p.use_pdl = pdl;
  VKL_LAUNCH(1, launch_rms_rows(p, d->f32, m->stream));
  return VKL_OK;
}
}  // namespace

int decoder_create(vkl_device *dev, const DecoderSpec &spec, uint32_t maxlen, bool f32, vkl_model **out) {
  VKL_OKAY(check_spec(spec, maxlen));
  VKL_CUDA(cudaSetDevice(dev->ordinal));
  vkl_model *m = new vkl_model();
  m->dev = dev;
  m->cfg = vkl_model_config{};
  m->cfg.dim = spec.width;
  for (const LayerSpec &l : spec.layers) m->cfg.heads = std::max(m->cfg.heads, l.mixer == MIX_DELTA ? l.delta.heads : l.attn.heads);
  m->cfg.vocab = spec.vocab;
  m->cfg.maxlen = maxlen;
  m->cfg.weight_dtype = VKL_BF16;
  m->cfg.tp_size = 1;
  m->vocab_l = spec.vocab;
  m->dec.reset(new Decoder());
  m->dec->spec = spec;
  m->dec->f32 = f32;
  int st = model_init_common(m);
  if (st == VKL_OK) st = build(m);
  if (st == VKL_OK) st = decoder_ensure_rows(m, 1);
  if (st == VKL_OK && cudaStreamSynchronize(m->stream) != cudaSuccess) st = fail(VKL_INTERNAL, "model: %s", cudaGetErrorString(cudaGetLastError()));
  if (st != VKL_OK) {
    vkl_model_destroy(m);
    return st;
  }
  *out = m;
  return VKL_OK;
}

int decoder_ensure_rows(vkl_model *m, uint32_t T) {
  if (T <= m->cap_T) return VKL_OK;
  Decoder *d = m->dec.get();
  model_drop_graph(m);
  VKL_CUDA(cudaStreamSynchronize(m->stream));
  const int ct = compute_dtype(d);
  VKL_OKAY(zeros(m, &d->x, 1, T, d->ldw, VKL_FP32));
  VKL_OKAY(zeros(m, &d->h, d->spec.two_norms ? 2 : 1, T, d->ldw, ct));
  VKL_OKAY(zeros(m, &d->q, 1, T, d->qld_max, ct));
  VKL_OKAY(zeros(m, &d->gate, 1, T, d->gld_max, VKL_FP32));
  if (d->recurrent) {
    VKL_OKAY(zeros(m, &d->low, 2, T, d->low_max, ct));
    if (T > 1) {
      VKL_OKAY(zeros(m, &d->dv, 1, T, d->dv_max, VKL_FP32));
      VKL_OKAY(zeros(m, &d->dz, 1, T, d->dz_max, VKL_FP32));
      size_t most = 0;
      for (size_t i = 0; i < d->L.size(); ++i)
        if (d->spec.layers[i].mixer == MIX_DELTA) most = std::max(most, delta_block_floats(T, d->spec.layers[i].delta.heads, d->L[i].dp));
      VKL_OKAY(zeros(m, &d->dblocks, 1, 1, most, VKL_FP32));
    }
  }
  VKL_OKAY(zeros(m, &d->a2, 1, T, d->k2_max, ct));
  VKL_OKAY(zeros(m, &m->toks, 1, 1, T, VKL_UINT32));
  if (d->top_max) {
    VKL_OKAY(zeros(m, &d->xe, 1, d->top_max, d->ffe_max, ct));
    uint32_t rows = 0;
    for (size_t i = 0; i < d->L.size(); ++i) {
      const FfnSpec &f = d->spec.layers[i].ffn;
      if (f.kind != FFN_TABLE_MOE) continue;
      const uint32_t n = route_rows(T, f.top, f.experts);
      rows = std::max(rows, n);
      VKL_OKAY(zeros(m, &d->L[i].slot, 1, 1, (size_t)T * f.top, VKL_UINT32));
      VKL_OKAY(zeros(m, &d->L[i].token, 1, 1, n, VKL_UINT32));
      VKL_OKAY(zeros(m, &d->L[i].tile_expert, 1, 1, n / 128, VKL_UINT32));
    }
    if (T > 1) {
      VKL_OKAY(zeros(m, &d->hp, 1, rows, d->ldw, ct));
      VKL_OKAY(zeros(m, &d->tp, 1, rows, d->ffe_max, ct));
      VKL_OKAY(zeros(m, &d->y, 1, rows, d->ldw, VKL_FP32));
    }
  }
  // decode: enough cache ranges to spread a few key heads over the SMs; longer calls have rows enough
  m->splits = 1;
  for (size_t i = 0; i < d->L.size(); ++i) {
    if (d->spec.layers[i].mixer != MIX_ATTENTION) continue;
    const AttnSpec &a = d->spec.layers[i].attn;
    const uint32_t per = a.heads / a.kv_heads, units = a.kv_heads * ((per + 3) / 4);
    m->splits = std::max(m->splits, std::min(32u, (uint32_t)(6 * m->dev->prop.multiProcessorCount) / units));
  }
  size_t sc = 0;
  for (size_t i = 0; i < d->L.size(); ++i) sc = std::max(sc, kv_attn_scratch_bytes(1, d->spec.layers[i].attn.heads, d->L[i].vp, m->splits));
  VKL_OKAY(zeros(m, &d->attn_scratch, 1, 1, sc / 4 + 4, VKL_FP32));
  VKL_OKAY(zeros(m, &d->attn_counters, 1, 1, kv_attn_counters(1, d->heads_max) + 1, VKL_UINT32));
  m->cap_T = T;
  return VKL_OK;
}

int decoder_ready(const vkl_model *m) {
  const Decoder *d = m->dec.get();
  for (const std::string &n : d->names)
    if (!d->loaded.count(n)) return fail(VKL_FAILED_PRECONDITION, "model: tensor %s is not set", n.c_str());
  return VKL_OK;
}

int decoder_check_shape(vkl_model *m, const char *name, const std::vector<uint32_t> &dims) {
  Decoder *d = m->dec.get();
  Target t;
  if (!find_target(d, name, &t)) return fail(VKL_INVALID_ARGUMENT, "model: tensor name '%s' is not part of this model", name);
  size_t n = 1;
  for (uint32_t k : dims) n *= k;
  bool ok = n == (size_t)t.rows * t.cols;
  if (t.kind == Target::MATRIX || t.kind == Target::TABLE || t.cols > 1) ok = dims.size() == 2 && dims[0] == t.rows && dims[1] == t.cols;
  if (t.kind == Target::DISTANCE) ok = dims.size() == 2 && dims[1] == t.spec->attn.heads;
  if (!ok) return fail(VKL_INVALID_ARGUMENT, "model: tensor %s does not have the configuration's shape [%u, %u]", name, t.rows, t.cols);
  return VKL_OK;
}

int decoder_set_weight(vkl_model *m, const char *name, int dtype, const void *data, size_t bytes) {
  Decoder *d = m->dec.get();
  Target t;
  if (!find_target(d, name, &t)) return fail(VKL_INVALID_ARGUMENT, "model_set_weight: tensor name '%s' is not part of this model", name);
  if (dtype != (t.kind == Target::TABLE ? VKL_UINT32 : VKL_BF16)) return fail(VKL_INVALID_ARGUMENT, "model_set_weight: %s has dtype %d", name, dtype);
  const size_t n = t.kind == Target::DISTANCE ? bytes / 2 : (size_t)t.rows * t.cols;
  if (bytes != n * (t.kind == Target::TABLE ? 4 : 2)) return fail(VKL_INVALID_ARGUMENT, "model_set_weight: %s is [%u, %u], got %zu bytes", name, t.rows, t.cols, bytes);
  model_drop_graph(m);  // it holds scalars by value
  const uint8_t *src = (const uint8_t *)data;
  switch (t.kind) {
    case Target::SCALAR: *t.scalar = bf16_value(src); break;
    case Target::RATE: {
      std::vector<float> v(t.dst->size());
      for (uint32_t h = 0; h < t.rows; ++h)
        for (uint32_t i = 0; i < t.map.ra; ++i) v[(size_t)h * t.map.rb + i] = (float)exp((double)bf16_value(src + 2 * h));
      VKL_CUDA(cudaMemcpyAsync(t.dst->data(), v.data(), v.size() * 4, cudaMemcpyHostToDevice, m->stream));
      VKL_CUDA(cudaStreamSynchronize(m->stream));
      break;
    }
    case Target::DISTANCE: {
      std::vector<float> v(n);
      for (size_t i = 0; i < n; ++i) v[i] = bf16_value(src + 2 * i);
      VKL_OKAY(set_distance(m, t.layer, t.spec, v));
      break;
    }
    case Target::TABLE: {
      const uint32_t E = t.spec->ffn.experts;
      for (size_t i = 0; i < n; ++i) {
        uint32_t e;
        memcpy(&e, src + 4 * i, 4);
        if (e >= E) return fail(VKL_OUT_OF_RANGE, "model_set_weight: %s names expert %d of %u", name, (int)e, E);
      }
      VKL_CUDA(cudaMemcpyAsync(t.dst->data(), data, bytes, cudaMemcpyHostToDevice, m->stream));
      VKL_CUDA(cudaStreamSynchronize(m->stream));
      break;
    }
    case Target::VECTOR: {
      std::vector<float> v(t.dst->size());
      VKL_CUDA(cudaMemcpyAsync(v.data(), t.dst->data(), v.size() * 4, cudaMemcpyDeviceToHost, m->stream));  // other tensors' parts stay
      VKL_CUDA(cudaStreamSynchronize(m->stream));
      for (uint32_t i = 0; i < t.rows * t.cols; ++i) v[(size_t)(i / t.map.ra) * t.map.rb + i % t.map.ra + t.map.r0] = bf16_value(src + 2 * (size_t)i) + t.add;
      VKL_CUDA(cudaMemcpyAsync(t.dst->data(), v.data(), v.size() * 4, cudaMemcpyHostToDevice, m->stream));
      VKL_CUDA(cudaStreamSynchronize(m->stream));
      break;
    }
    case Target::MATRIX: {
      void *tmp = nullptr;
      VKL_OKAY(m->dev->alloc(bytes, &tmp));
      cudaError_t e = cudaMemcpyAsync(tmp, data, bytes, cudaMemcpyHostToDevice, m->stream);
      if (e == cudaSuccess) e = launch_pack_rows((const bf16 *)tmp, t.rows, t.cols, (bf16 *)t.dst->data() + t.row_base * t.ld, t.ld, t.map, m->stream);
      if (e == cudaSuccess) e = cudaStreamSynchronize(m->stream);
      m->dev->release(tmp, bytes);
      count_launches(1);
      if (e != cudaSuccess) return fail(VKL_INTERNAL, "model_set_weight: %s: %s", name, cudaGetErrorString(e));
    }
  }
  d->loaded.insert(name);
  return VKL_OK;
}

int decoder_synth(vkl_model *m, uint64_t seed, float wstd, float nstd) {
  Decoder *d = m->dec.get();
  size_t most = 0;
  for (const std::string &n : d->names) {
    Target t;
    if (find_target(d, n, &t)) most = std::max(most, (size_t)t.rows * t.cols * 2);
  }
  const uint32_t rel_rows = 32;
  for (const LayerSpec &l : d->spec.layers)
    if (l.mixer == MIX_ATTENTION) most = std::max(most, (size_t)rel_rows * l.attn.heads * 2);
  void *tmp = nullptr;
  VKL_OKAY(m->dev->alloc(most, &tmp));
  int st = VKL_OK;
  for (size_t i = 0; i < d->names.size() && st == VKL_OK; ++i) {
    const std::string &name = d->names[i];
    Target t;
    if (!find_target(d, name, &t)) continue;
    if (t.kind == Target::TABLE) {  // distinct experts per token: consecutive ones from a mixed start
      std::vector<uint32_t> v((size_t)t.rows * t.cols);
      for (uint32_t r = 0; r < t.rows; ++r)
        for (uint32_t c = 0; c < t.cols; ++c) v[(size_t)r * t.cols + c] = (uint32_t)(((r + seed + i) * 2654435761ull >> 7) + c) % t.spec->ffn.experts;
      st = decoder_set_weight(m, name.c_str(), VKL_UINT32, v.data(), v.size() * 4);
      continue;
    }
    const uint32_t rows = t.kind == Target::DISTANCE ? rel_rows * t.spec->attn.heads : t.rows, cols = t.kind == Target::DISTANCE ? 1 : t.cols;
    const size_t n = (size_t)rows * cols;
    const float sd = t.synth_std == -1.f ? wstd : t.synth_std == -2.f ? nstd : t.synth_std;
    cudaError_t e = launch_synth_bf16((bf16 *)tmp, seed, i, n, t.synth_mean, sd, m->stream);
    if (t.kind == Target::MATRIX) {
      if (e == cudaSuccess) e = launch_pack_rows((const bf16 *)tmp, rows, cols, (bf16 *)t.dst->data() + t.row_base * t.ld, t.ld, t.map, m->stream);
      d->loaded.insert(name);
      count_launches(2);
    } else {
      std::vector<uint8_t> host(n * 2);
      if (e == cudaSuccess) e = cudaMemcpyAsync(host.data(), tmp, n * 2, cudaMemcpyDeviceToHost, m->stream);
      if (e == cudaSuccess) e = cudaStreamSynchronize(m->stream);
      if (e == cudaSuccess) st = decoder_set_weight(m, name.c_str(), VKL_BF16, host.data(), host.size());
    }
    if (e != cudaSuccess) st = fail(VKL_INTERNAL, "model_synth_weights: %s", cudaGetErrorString(e));
  }
  model_drop_graph(m);
  cudaStreamSynchronize(m->stream);
  m->dev->release(tmp, most);
  return st;
}

int decoder_begin(vkl_model *m, size_t offset) {
  Decoder *d = m->dec.get();
  if (d->recurrent && offset && offset != d->filled) {
    if (d->filled == Decoder::kNowhere) return fail(VKL_FAILED_PRECONDITION, "model: position %zu cannot follow, the recurrent states are not those of a sequence (start at 0)", offset);
    return fail(VKL_FAILED_PRECONDITION, "model: position %zu cannot follow, the recurrent states have taken %zu tokens (continue there or start at 0)", offset, d->filled);
  }
  d->filled = Decoder::kNowhere;
  return VKL_OK;
}
void decoder_end(vkl_model *m, size_t end) { m->dec->filled = end; }

#define MARK(c) do { if (mk) mk->mark(c); } while (0)
#define MARK_NORM() do { if (d->spec.norm != NORM_TANH && !norm_in_matvec(d, T)) MARK(9); } while (0)

namespace {
// The delta rule's steps between the projections of layer run r.
int run_delta(vkl_model *m, size_t r, uint32_t T, bool pdl) {
  Decoder *d = m->dec.get();
  DecLayer &l = d->L[d->runs[r].layer];
  const DeltaSpec &a = d->spec.layers[d->runs[r].layer].delta;
  const bool f32 = d->f32;
  cudaStream_t s = m->stream;
  DeltaRows p = {};
  p.raw = d->q->data();
  p.raw_ld = l.qcols;
  p.k_col = l.k_col;
  p.v_col = l.v_col;
  p.taps = (const float *)l.taps->data();
  p.ntaps = a.taps;
  p.ring = m->L[r].ring->data();
  p.pos = m->pos_dev();
  p.T = T;
  p.heads = a.heads;
  p.kv_heads = a.kv_heads;
  p.dim = a.dim;
  p.vdim = a.vdim;
  p.dp = l.dp;
  p.vp = l.vp;
  p.bias = (const float *)l.biasl->data();
  p.rate = (const float *)l.rate->data();
  p.beta = (const float *)d->gate->data();
  p.beta_ld = d->gld_max;
  p.state = (float *)m->L[r].state->data();
  p.norm = (const float *)l.onorm->data();
  p.eps = d->spec.norm_eps;
  p.out = d->a2->data();
  p.out_ld = l.k2;
  p.use_pdl = pdl;
  p.z_gate = l.ln2;
  if (T == 1) {
    p.wl = (const bf16 *)l.wl->data();
    p.low = d->low->data();
    p.low_ld = l.lowp;
    VKL_LAUNCH(1, launch_delta_step(p, f32, s));
    return VKL_OK;
  }
  // the second steps of the decays' and the gates' projections: one matrix over two inputs
  GemmRows g = {};
  g.a = d->low->data();
  g.w = (const bf16 *)l.wl->data();
  g.M = T;
  g.N = l.nl;
  g.K = l.lowp;
  g.n2 = l.ln2;
  g.out.seg[0] = RowSeg{0, l.nl, ROW_STORE};
  g.out.nseg = 1;
  g.out.f32 = (float *)d->dz->data();
  g.out.f32_ld = l.nl;
  g.out.scale = 1.f;
  g.error = (uint32_t *)m->state->data() + 6;
  m->gemm_used = true;
  VKL_LAUNCH(1, f32 ? launch_gemm_rows_f32(g, s) : launch_gemm_rows_bf16(g, s));
  p.z = g.out.f32;
  p.z_ld = l.nl;
  p.v = (float *)d->dv->data();
  p.blocks = (float *)d->dblocks->data();
  p.error = g.error;
  p.sms = m->dev->prop.multiProcessorCount;
  VKL_LAUNCH(delta_launches(T), launch_delta_rows(p, f32, s));
  return VKL_OK;
}
}  // namespace

int decoder_run(vkl_model *m, uint32_t T, bool pdl, Marker *mk) {
  Decoder *d = m->dec.get();
  cudaStream_t s = m->stream;
  const int sms = m->dev->prop.multiProcessorCount;
  const bool one = T == 1, f32 = d->f32;
  const uint32_t *toks = (const uint32_t *)m->toks->data();
  const size_t es = elem(d);
  const uint64_t launches0 = vkl_kernel_launches();
  auto gemm = [&](GemmRows &g) -> int {
    g.error = (uint32_t *)m->state->data() + 6;
    m->gemm_used = true;
    VKL_LAUNCH(1, f32 ? launch_gemm_rows_f32(g, s) : launch_gemm_rows_bf16(g, s));
    return VKL_OK;
  };
  MARK(-1);
  if (!one && d->top_max) {
    std::vector<RouteTable> rt;
    for (size_t i = 0; i < d->L.size(); ++i) {
      const FfnSpec &f = d->spec.layers[i].ffn;
      DecLayer &l = d->L[i];
      if (f.kind == FFN_TABLE_MOE)
        rt.push_back(RouteTable{(const int32_t *)l.table->data(), f.top, f.experts, (int32_t *)l.slot->data(), (int32_t *)l.token->data(), (int32_t *)l.tile_expert->data()});
    }
    VKL_LAUNCH((rt.size() + 31) / 32, launch_route(rt.data(), (uint32_t)rt.size(), d->experts_max, toks, T, s));
  }
  VKL_LAUNCH(1, launch_embed_rows((const bf16 *)d->emb->data(), toks, T, d->spec.embed_scale, residual_after(m, -1), f32, s));
  MARK(0);
  VKL_OKAY(norm_after(m, -1, T, false));
  MARK_NORM();
  for (size_t r = 0; r < d->runs.size(); ++r) {
    const uint32_t i = d->runs[r].layer;
    DecLayer &l = d->L[i];
    const AttnSpec &a = d->spec.layers[i].attn;
    const FfnSpec &f = d->spec.layers[i].ffn;
    const bool moe = f.kind == FFN_TABLE_MOE, delta = d->spec.layers[i].mixer == MIX_DELTA;
    const Layer &own = m->L[r], &kv = m->L[delta || a.kv_from < 0 ? r : (size_t)a.kv_from];  // no loop where a layer uses another's cache
    // --- everything that reads the stream's norms
    RowsOut in = {};
    std::copy(l.seg, l.seg + l.nseg, in.seg);
    in.nseg = l.nseg;
    in.bias = l.bias1 ? (const float *)l.bias1->data() : nullptr;
    in.q = d->q->data();
    in.q_ld = l.qcols;
    in.kcache = own.kcache ? own.kcache->data() : nullptr;
    in.vcache = own.vcache ? own.vcache->data() : nullptr;
    in.kv_heads = a.kv_heads;
    in.dp = l.dp;
    in.vp = l.vp;
    if (delta) {
      in.low = d->low->data();
      in.low_ld = l.lowp;
      in.low_stride = (size_t)T * l.lowp;
    }
    in.maxlen = m->cfg.maxlen;
    in.pos = m->pos_dev();
    in.gate = (float *)d->gate->data();
    in.gate_ld = d->gld_max;
    in.glu = d->a2->data() + (size_t)l.hd * es;
    in.glu_ld = l.k2;
    in.act = f.act;
    in.limit = f.limit;
    if (one) {
      MvRows p = {};
      p.w = (const bf16 *)l.w1->data();
      p.N = l.n1;
      p.K = d->ldw;
      p.x = d->h->data();
      if (l.n2) p.x2 = d->h->data() + (size_t)d->ldw * es;
      if (norm_in_matvec(d, T)) p.norm = norm_of(m, (int)r - 1, T);
      p.n2 = l.n2;
      p.gap0 = l.gap0;
      p.out = in;
      if (moe) {
        p.we = (const bf16 *)l.we1->data();
        p.ne = 2 * l.ffp;
        p.ke = l.ffp;
        p.top = f.top;
        p.table = (const int32_t *)l.table->data();
        p.tok = toks;
        p.xe = d->xe->data();
        p.xe_ld = d->ffe_max;
        p.xe_act = f.act;
      }
      p.use_pdl = pdl;
      VKL_LAUNCH(1, launch_rows_matvec(p, f32, sms, s));
    } else {
      GemmRows g = {};
      g.a = d->h->data();
      g.w = (const bf16 *)l.w1->data();
      g.M = T;
      g.N = l.n1;
      g.K = d->ldw;
      g.n2 = l.n2;
      g.out = in;
      VKL_OKAY(gemm(g));
    }
    MARK(1);
    if (delta) {
      VKL_OKAY(run_delta(m, r, T, one && pdl));
      MARK(8);
    } else {
      KvAttn at = {};
      if (a.qk_norm || a.rot.dims) {
        QkRows p = {};
        p.q = d->q->data();
        p.q_ld = l.qcols;
        p.k_col = l.k_col;
        if (l.qw) p.qw = (const float *)l.qw->data();
        if (l.kw) p.kw = (const float *)l.kw->data();
        p.eps = d->spec.norm_eps;
        if (l.freq) p.freq = (const float *)l.freq->data();
        p.pairs = a.rot.dims / 2;
        if (own.kcache) p.kcache = own.kcache->data();
        p.T = T;
        p.heads = a.heads;
        p.kv_heads = a.kv_heads;
        p.dim = a.dim;
        p.dp = l.dp;
        p.maxlen = m->cfg.maxlen;
        p.pos = m->pos_dev();
        if (one) at.qk = p;  // part of the attention kernel
        else VKL_LAUNCH(1, launch_qk_rows(p, f32, s));
      }
      at.q = d->q->data();
      at.q_ld = l.qcols;
      at.cache = kv.kcache->data();
      if (kv.vcache) at.vcache = kv.vcache->data();
      at.vp = l.vp;
      at.window = a.window;
      if (l.sink) at.sink = (const float *)l.sink->data();
      at.out = d->a2->data();
      at.out_ld = l.k2;
      if (a.head_gate) at.gate = (const float *)d->gate->data();
      at.gate_ld = d->gld_max;
      if (l.rel) at.bias = (const float *)l.rel->data();
      at.bias_n = l.rel_n;
      at.pos = m->pos_dev();
      at.scale = a.scale;
      at.temp_coef = a.temp_coef;
      at.temp_every = (float)a.temp_every;
      at.T = T;
      at.heads = a.heads;
      at.kv_heads = a.kv_heads;
      at.dp = l.dp;
      at.maxlen = m->cfg.maxlen;
      at.splits = one ? m->splits : 1;
      at.scratch = (float *)d->attn_scratch->data();
      at.counters = (uint32_t *)d->attn_counters->data();
      at.use_pdl = one && pdl;
      VKL_LAUNCH(1, launch_kv_attention(at, f32, s));
      MARK(2);
    }
    // --- everything that adds to the stream, and the next run's norm
    RowsOut out = {};
    out.seg[0] = RowSeg{0, d->ldw, ROW_RESIDUAL};
    out.nseg = 1;
    Residual res = residual_after(m, (int)r);
    if (d->tracing) res.trace = (float *)d->trace->data() + r * (size_t)T * d->ldw;
    if (l.bias_o) res.bias = (const float *)l.bias_o->data();
    if (one) {
      MvRows p = {};
      p.w = (const bf16 *)l.w2->data();
      p.N = d->ldw;
      p.K = l.k2;
      p.x = d->a2->data();
      p.out = out;
      p.out.res = res;
      p.out_proj = true;
      if (moe) {
        p.we = (const bf16 *)l.we2->data();
        p.ke = l.ffp;
        p.top = f.top;
        p.table = (const int32_t *)l.table->data();
        p.tok = toks;
        p.xe = d->xe->data();
        p.xe_ld = d->ffe_max;
        p.xe_scale = 1.0f / (float)f.top;
      }
      p.use_pdl = pdl;
      VKL_LAUNCH(1, launch_rows_matvec(p, f32, sms, s));
      MARK(5);
      VKL_OKAY(norm_after(m, (int)r, T, pdl));
      MARK_NORM();
      continue;
    }
    if (moe) {
      const uint32_t rows = route_rows(T, f.top, f.experts);
      VKL_LAUNCH(1, launch_gather_rows(d->h->data(), (const int32_t *)l.token->data(), rows, (uint32_t)(d->ldw * es), d->hp->data(), s));
      GemmRows g = {};
      g.a = d->hp->data();
      g.w = (const bf16 *)l.we1->data();
      g.M = rows;
      g.N = 2 * l.ffp;
      g.K = d->ldw;
      g.tile_expert = (const int32_t *)l.tile_expert->data();
      g.w_rows = f.experts * g.N;
      g.out.seg[0] = RowSeg{0, g.N, ROW_GLU};
      g.out.nseg = 1;
      g.out.glu = d->tp->data();
      g.out.glu_ld = l.ffp;
      g.out.act = f.act;
      g.out.limit = f.limit;
      VKL_OKAY(gemm(g));
      MARK(4);
      g.a = d->tp->data();
      g.w = (const bf16 *)l.we2->data();
      g.N = d->ldw;
      g.K = l.ffp;
      g.w_rows = f.experts * g.N;
      g.out = RowsOut{};
      g.out.seg[0] = RowSeg{0, g.N, ROW_STORE};
      g.out.nseg = 1;
      g.out.f32 = (float *)d->y->data();
      g.out.f32_ld = d->ldw;
      g.out.scale = 1.0f / (float)f.top;
      VKL_OKAY(gemm(g));
      MARK(5);
    }
    GemmRows g = {};
    g.a = d->a2->data();
    g.w = (const bf16 *)l.w2->data();
    g.M = T;
    g.N = d->ldw;
    g.K = l.k2;
    g.out = out;
    if (moe) {  // the stream is complete only after the combine step: no norm yet
      g.out.res.x = res.x;
      g.out.res.ldw = res.ldw;
      g.out.res.mult = res.mult;
      g.out.res.bias = res.bias;
    } else {
      g.out.res = res;
    }
    VKL_OKAY(gemm(g));
    MARK(3);
    if (moe) {
      VKL_LAUNCH(1, launch_combine((const float *)d->y->data(), d->ldw, (const int32_t *)l.slot->data(), f.top, T, res, f32, s));
      MARK(5);
    }
    VKL_OKAY(norm_after(m, (int)r, T, false));
    MARK_NORM();
  }
  // --- output layer: the last row for the token loop, and the rows a caller asked for
  MvRows p = {};
  p.w = (const bf16 *)d->head->data();
  p.N = d->vocab_p;
  p.K = d->ldw;
  p.x = d->h->data() + (size_t)(T - 1) * d->ldw * es;
  if (norm_in_matvec(d, T)) p.norm = norm_of(m, (int)d->runs.size() - 1, T);
  p.out.seg[0] = RowSeg{0, d->vocab_p, ROW_STORE};
  p.out.nseg = 1;
  p.out.f32 = (float *)m->logits32->data();
  p.out.f32_ld = d->vocab_p;
  p.out.scale = d->spec.logit_scale;
  p.out.cap = d->spec.logit_cap;
  p.use_pdl = one && pdl;
  VKL_LAUNCH(1, launch_rows_matvec(p, f32, sms, s));
  MARK(6);
  if (!d->want_rows.empty()) {
    const uint32_t n = (uint32_t)d->want_rows.size();
    VKL_OKAY(ensure_tensor(m->dev, &d->want, 1, 1, n, VKL_UINT32));
    VKL_OKAY(ensure_tensor(m->dev, &d->hw, 1, n, d->ldw, compute_dtype(d)));
    VKL_OKAY(ensure_tensor(m->dev, &d->logits_rows, 1, n, d->vocab_p, VKL_FP32));
    VKL_CUDA(cudaMemcpyAsync(d->want->data(), d->want_rows.data(), (size_t)n * 4, cudaMemcpyHostToDevice, s));
    VKL_LAUNCH(1, launch_gather_rows(d->h->data(), (const int32_t *)d->want->data(), n, (uint32_t)(d->ldw * es), d->hw->data(), s));
    GemmRows g = {};
    g.a = d->hw->data();
    g.w = p.w;
    g.M = n;
    g.N = d->vocab_p;
    g.K = d->ldw;
    g.out = p.out;
    g.out.f32 = (float *)d->logits_rows->data();
    VKL_OKAY(gemm(g));
  }
  VKL_LAUNCH(2, launch_argmax_f32((const float *)m->logits32->data(), m->next_dev(), m->argpart->data(), 1, m->vocab_l, s));
  MARK(7);
  if (one) d->launches_per_token = (uint32_t)(vkl_kernel_launches() - launches0);
  return VKL_OK;
}

}  // namespace vkl
