// Checkpoint folders (config.json, model.safetensors) and the registry of decoder architectures.
//
// The JSON reader takes the whole grammar that config files use; the safetensors reader maps the file and hands
// every tensor to vkl_model_set_weight by name. An architecture is one entry of kArchitectures: its name as
// config.json gives it and the function that turns the config (and, where the config leaves a size to a tensor, the
// tensors' shapes) into a DecoderSpec.
#include <ctype.h>
#include <errno.h>
#include <fcntl.h>
#include <math.h>
#include <stdlib.h>
#include <string.h>
#include <sys/mman.h>
#include <sys/stat.h>
#include <unistd.h>

#include <map>
#include <memory>
#include <utility>

#include "decoder.h"
#include "runtime.h"

using namespace vkl;

namespace {

// ------------------------------------------------------------------------------------------ JSON
struct Json {
  enum Kind { NUL, BOOL, NUMBER, STRING, ARRAY, OBJECT } kind = NUL;
  double num = 0;
  bool boolean = false;
  std::string str;
  std::vector<Json> items;
  std::vector<std::pair<std::string, Json>> fields;
  const Json *get(const char *key) const {
    for (const auto &f : fields)
      if (f.first == key) return &f.second;
    return nullptr;
  }
};

struct JsonReader {
  const char *p, *end;
  bool ok = true;
  int depth = 0;
  void ws() {
    while (p < end && (*p == ' ' || *p == '\n' || *p == '\t' || *p == '\r')) ++p;
  }
  bool fail_() { return ok = false; }
  bool lit(const char *s) {
    const size_t n = strlen(s);
    if ((size_t)(end - p) < n || memcmp(p, s, n)) return fail_();
    p += n;
    return true;
  }
  static void utf8(std::string *o, unsigned c) {
    if (c < 0x80) {
      o->push_back((char)c);
    } else if (c < 0x800) {
      o->push_back((char)(0xc0 | (c >> 6)));
      o->push_back((char)(0x80 | (c & 63)));
    } else {
      o->push_back((char)(0xe0 | (c >> 12)));
      o->push_back((char)(0x80 | ((c >> 6) & 63)));
      o->push_back((char)(0x80 | (c & 63)));
    }
  }
  bool string(std::string *o) {
    if (p >= end || *p != '"') return fail_();
    for (++p; p < end && *p != '"'; ++p) {
      if (*p != '\\') {
        o->push_back(*p);
        continue;
      }
      if (++p >= end) return fail_();
      switch (*p) {
        case 'n': o->push_back('\n'); break;
        case 't': o->push_back('\t'); break;
        case 'r': o->push_back('\r'); break;
        case 'b': o->push_back('\b'); break;
        case 'f': o->push_back('\f'); break;
        case 'u': {
          if (end - p < 5) return fail_();
          unsigned c = 0;
          for (int i = 1; i <= 4; ++i) {
            if (!isxdigit((unsigned char)p[i])) return fail_();
            c = c * 16 + (unsigned)(isdigit((unsigned char)p[i]) ? p[i] - '0' : tolower(p[i]) - 'a' + 10);
          }
          utf8(o, c);
          p += 4;
          break;
        }
        default: o->push_back(*p);
      }
    }
    if (p >= end) return fail_();
    ++p;
    return true;
  }
  bool value(Json *j) {
    ws();
    if (!ok || p >= end || ++depth > 64) return fail_();
    switch (*p) {
      case '{':
        j->kind = Json::OBJECT;
        for (++p, ws(); p < end && *p != '}'; ws()) {
          if (!j->fields.empty()) {
            if (*p != ',') return fail_();
            ++p;
            ws();
          }
          j->fields.emplace_back();
          if (!string(&j->fields.back().first)) return false;
          ws();
          if (p >= end || *p != ':') return fail_();
          ++p;
          if (!value(&j->fields.back().second)) return false;
        }
        if (p >= end) return fail_();
        ++p;
        break;
      case '[':
        j->kind = Json::ARRAY;
        for (++p, ws(); p < end && *p != ']'; ws()) {
          if (!j->items.empty()) {
            if (*p != ',') return fail_();
            ++p;
          }
          j->items.emplace_back();
          if (!value(&j->items.back())) return false;
        }
        if (p >= end) return fail_();
        ++p;
        break;
      case '"':
        j->kind = Json::STRING;
        if (!string(&j->str)) return false;
        break;
      case 't': j->kind = Json::BOOL; j->boolean = true; if (!lit("true")) return false; break;
      case 'f': j->kind = Json::BOOL; if (!lit("false")) return false; break;
      case 'n': if (!lit("null")) return false; break;
      default: {
        std::string t;
        while (p < end && (isalnum((unsigned char)*p) || *p == '-' || *p == '+' || *p == '.')) t.push_back(*p++);
        char *e = nullptr;
        j->kind = Json::NUMBER;
        j->num = strtod(t.c_str(), &e);
        if (t.empty() || !e || *e) return fail_();
      }
    }
    --depth;
    return true;
  }
};

int parse_json(const char *text, size_t n, const char *what, Json *out) {
  JsonReader r{text, text + n};
  const bool got = r.value(out);
  r.ws();
  if (!got || r.p != r.end) return fail(VKL_INVALID_ARGUMENT, "%s: malformed JSON at byte %zu", what, (size_t)(r.p - text));
  return VKL_OK;
}

// Field access that names what is missing.
int get_number(const Json &o, const char *key, double *out) {
  const Json *j = o.get(key);
  if (!j || j->kind != Json::NUMBER) return fail(VKL_INVALID_ARGUMENT, "config: number '%s' is missing", key);
  *out = j->num;
  return VKL_OK;
}
int get_u32(const Json &o, const char *key, uint32_t *out) {
  double v = 0;
  VKL_OKAY(get_number(o, key, &v));
  if (v < 0 || v > 4294967295.0 || v != floor(v)) return fail(VKL_INVALID_ARGUMENT, "config: '%s' is not a whole number", key);
  *out = (uint32_t)v;
  return VKL_OK;
}
int get_f32(const Json &o, const char *key, float *out) {
  double v = 0;
  VKL_OKAY(get_number(o, key, &v));
  *out = (float)v;
  return VKL_OK;
}
int get_object(const Json &o, const char *key, const Json **out) {
  *out = o.get(key);
  if (!*out || (*out)->kind != Json::OBJECT) return fail(VKL_INVALID_ARGUMENT, "config: object '%s' is missing", key);
  return VKL_OK;
}
bool absent(const Json *j) { return !j || j->kind == Json::NUL; }

// Shapes of a checkpoint's tensors, for the sizes that a config leaves to them.
using Shapes = std::map<std::string, std::vector<uint32_t>>;
int read_shapes(const Json &header, Shapes *out) {
  for (const auto &t : header.fields) {
    if (t.first == "__metadata__") continue;
    const Json *shape = t.second.get("shape");
    if (!shape || shape->kind != Json::ARRAY) return fail(VKL_INVALID_ARGUMENT, "model: tensor %s has no shape", t.first.c_str());
    std::vector<uint32_t> &d = (*out)[t.first];
    for (const Json &k : shape->items) {
      if (k.kind != Json::NUMBER || k.num < 0 || k.num > 4294967295.0) return fail(VKL_INVALID_ARGUMENT, "model: tensor %s has a malformed shape", t.first.c_str());
      d.push_back((uint32_t)k.num);
    }
  }
  return VKL_OK;
}
int get_rows(const Shapes &shapes, const std::string &name, uint32_t *out) {
  const auto it = shapes.find(name);
  if (it == shapes.end() || it->second.size() != 2) return fail(VKL_INVALID_ARGUMENT, "model: the shape of tensor %s is needed", name.c_str());
  *out = it->second[0];
  return VKL_OK;
}

// -------------------------------------------------------------------------------------- Rumalorn
// Parallel blocks under Dynamic Tanh norms; attention whose keys are its values, with a bucketed distance bias,
// a query temperature and head gates; dense clamped or table-routed SiLU feed-forwards; a loop over some layers.
int rumalorn_spec(const Json &c, const Shapes &, DecoderSpec *s) {
  VKL_OKAY(get_u32(c, "vocab", &s->vocab));
  VKL_OKAY(get_u32(c, "width", &s->width));
  VKL_OKAY(get_f32(c, "logit_scale", &s->logit_scale));
  const Json *loop = c.get("loop");
  if (!absent(loop)) {
    VKL_OKAY(get_u32(*loop, "start", &s->loop_start));
    VKL_OKAY(get_u32(*loop, "stop", &s->loop_stop));
    VKL_OKAY(get_u32(*loop, "times", &s->loop_times));
    if (!s->loop_times) return fail(VKL_INVALID_ARGUMENT, "config: a loop of 0 times");
  }
  const Json *layers = c.get("layers");
  if (absent(layers) || layers->kind != Json::ARRAY) return fail(VKL_INVALID_ARGUMENT, "config: 'layers' is missing");
  for (const Json &j : layers->items) {
    LayerSpec l;
    const Json *type = j.get("type"), *mix = nullptr;
    if (!type || type->str != "attention") return fail(VKL_UNIMPLEMENTED, "config: layer type '%s'", type ? type->str.c_str() : "");
    VKL_OKAY(get_object(j, "mixer", &mix));
    AttnSpec &a = l.attn;
    uint32_t vdim = 0;
    a.proj_bias = a.head_gate = true;
    VKL_OKAY(get_u32(*mix, "heads", &a.heads));
    VKL_OKAY(get_u32(*mix, "kv_heads", &a.kv_heads));
    VKL_OKAY(get_u32(*mix, "dim", &a.dim));
    VKL_OKAY(get_f32(*mix, "scale", &a.scale));
    VKL_OKAY(get_u32(*mix, "bias_max", &a.bias_max));
    if (!absent(mix->get("vdim"))) {
      VKL_OKAY(get_u32(*mix, "vdim", &vdim));
      if (vdim != a.dim) return fail(VKL_INVALID_ARGUMENT, "config: keys of width %u cannot be values of width %u", a.dim, vdim);
    }
    const Json *qt = mix->get("q_temp");
    if (!absent(qt)) {
      VKL_OKAY(get_f32(*qt, "coef", &a.temp_coef));
      VKL_OKAY(get_u32(*qt, "every", &a.temp_every));
    }
    const Json *mlp = j.get("mlp");
    if (!absent(mlp)) {
      FfnSpec &f = l.ffn;
      const Json *kind = mlp->get("kind");
      if (kind && kind->str == "dense") {
        f.kind = FFN_DENSE;
        f.act = GLU_CLAMPED;
        VKL_OKAY(get_u32(*mlp, "ff", &f.ff));
        VKL_OKAY(get_f32(*mlp, "limit", &f.limit));
      } else if (kind && kind->str == "moe") {
        const Json *ex = nullptr, *ro = nullptr;
        f.kind = FFN_TABLE_MOE;
        f.act = GLU_SILU;
        VKL_OKAY(get_object(*mlp, "expert", &ex));
        VKL_OKAY(get_object(*mlp, "router", &ro));
        VKL_OKAY(get_u32(*ex, "ff", &f.ff));
        VKL_OKAY(get_u32(*ro, "experts", &f.experts));
        VKL_OKAY(get_u32(*ro, "top", &f.top));
      } else {
        return fail(VKL_UNIMPLEMENTED, "config: feed-forward kind '%s'", kind ? kind->str.c_str() : "");
      }
    }
    s->layers.push_back(l);
  }
  return VKL_OK;
}

// --------------------------------------------------------------------------------------- Kupuzen
// Parallel sublayers under centred RMS norms of their own; windowed attention with sinks, normed and rotated queries
// and keys and caches that later layers may share; a gated delta rule with a decay per key channel; dense SiLU
// feed-forwards; scaled embedding and residual, soft-capped logits.
int kupuzen_attention(const Json &mix, AttnSpec *a) {
  VKL_OKAY(get_u32(mix, "heads", &a->heads));
  VKL_OKAY(get_u32(mix, "kv_heads", &a->kv_heads));
  VKL_OKAY(get_u32(mix, "dim", &a->dim));
  VKL_OKAY(get_u32(mix, "vdim", &a->vdim));
  VKL_OKAY(get_f32(mix, "scale", &a->scale));
  if (!a->vdim) return fail(VKL_INVALID_ARGUMENT, "config: values of width 0");
  a->qk_norm = a->sink = true;
  const Json *mask = mix.get("mask"), *rot = mix.get("rot");
  if (!absent(mask)) {
    VKL_OKAY(get_u32(*mask, "size", &a->window));
    if (!a->window) return fail(VKL_INVALID_ARGUMENT, "config: a window of 0 positions");
  }
  if (!absent(rot)) {
    VKL_OKAY(get_u32(*rot, "dims", &a->rot.dims));
    VKL_OKAY(get_number(*rot, "base", &a->rot.base));
    const Json *sc = rot->get("scaling");
    if (!absent(sc)) {
      a->rot.scaled = true;
      VKL_OKAY(get_number(*sc, "factor", &a->rot.factor));
      VKL_OKAY(get_number(*sc, "low", &a->rot.low));
      VKL_OKAY(get_number(*sc, "high", &a->rot.high));
      VKL_OKAY(get_number(*sc, "original", &a->rot.original));
    }
  }
  if (!absent(mix.get("kv_from"))) {
    uint32_t j = 0;
    VKL_OKAY(get_u32(mix, "kv_from", &j));
    a->kv_from = (int)j;
  }
  return VKL_OK;
}
int kupuzen_spec(const Json &c, const Shapes &shapes, DecoderSpec *s) {
  const Json *norm = nullptr, *emb = c.get("embedding"), *layers = c.get("layers");
  VKL_OKAY(get_u32(c, "vocab", &s->vocab));
  VKL_OKAY(get_u32(c, "width", &s->width));
  VKL_OKAY(get_object(c, "norm", &norm));
  VKL_OKAY(get_f32(*norm, "eps", &s->norm_eps));
  VKL_OKAY(get_f32(c, "residual_mult", &s->residual_mult));
  if (!absent(emb)) VKL_OKAY(get_f32(*emb, "scale", &s->embed_scale));
  if (!absent(c.get("logit_softcap"))) VKL_OKAY(get_f32(c, "logit_softcap", &s->logit_cap));
  s->norm = NORM_RMS_CENTRED;
  s->two_norms = true;
  if (absent(layers) || layers->kind != Json::ARRAY) return fail(VKL_INVALID_ARGUMENT, "config: 'layers' is missing");
  for (const Json &j : layers->items) {
    LayerSpec l;
    const Json *type = j.get("type"), *mix = nullptr;
    VKL_OKAY(get_object(j, "mixer", &mix));
    if (type && type->str == "attention") {
      VKL_OKAY(kupuzen_attention(*mix, &l.attn));
    } else if (type && type->str == "channel_delta") {
      const std::string p = "l" + std::to_string(s->layers.size()) + ".mix.";
      l.mixer = MIX_DELTA;
      VKL_OKAY(get_u32(*mix, "heads", &l.delta.heads));
      VKL_OKAY(get_u32(*mix, "kv_heads", &l.delta.kv_heads));
      VKL_OKAY(get_u32(*mix, "dim", &l.delta.dim));
      VKL_OKAY(get_u32(*mix, "vdim", &l.delta.vdim));
      VKL_OKAY(get_u32(*mix, "conv", &l.delta.taps));
      VKL_OKAY(get_rows(shapes, p + "a1", &l.delta.decay_rank));
      VKL_OKAY(get_rows(shapes, p + "g1", &l.delta.gate_rank));
    } else {
      return fail(VKL_UNIMPLEMENTED, "config: layer type '%s'", type ? type->str.c_str() : "");
    }
    const Json *mlp = j.get("mlp");
    if (!absent(mlp)) {
      const Json *kind = mlp->get("kind");
      if (!kind || kind->str != "dense") return fail(VKL_UNIMPLEMENTED, "config: feed-forward kind '%s'", kind ? kind->str.c_str() : "");
      l.ffn.kind = FFN_DENSE;
      l.ffn.act = GLU_SILU;
      VKL_OKAY(get_u32(*mlp, "ff", &l.ffn.ff));
    }
    s->layers.push_back(l);
  }
  return VKL_OK;
}

struct Architecture {
  const char *name;
  int (*spec)(const Json &config, const Shapes &shapes, DecoderSpec *out);
};
const Architecture kArchitectures[] = {
    {"Rumalorn", rumalorn_spec},
    {"Kupuzen", kupuzen_spec},
};

int spec_of(const char *text, size_t n, const Shapes &shapes, DecoderSpec *out) {
  Json c;
  VKL_OKAY(parse_json(text, n, "config", &c));
  const Json *name = c.get("architecture");
  if (!name || name->kind != Json::STRING) return fail(VKL_INVALID_ARGUMENT, "config: 'architecture' is missing");
  for (const Architecture &a : kArchitectures)
    if (name->str == a.name) return a.spec(c, shapes, out);
  return fail(VKL_UNIMPLEMENTED, "config: architecture '%s' is not registered (%s)", name->str.c_str(), vkl_model_architectures());
}

struct Mapping {
  const uint8_t *p = nullptr;
  size_t n = 0;
  ~Mapping() {
    if (p) munmap((void *)p, n);
  }
  int open_file(const std::string &path) {
    const int fd = open(path.c_str(), O_RDONLY);
    if (fd < 0) return fail(VKL_NOT_FOUND, "model_load: %s: %s", path.c_str(), strerror(errno));
    struct stat st;
    void *v = MAP_FAILED;
    if (fstat(fd, &st) == 0 && st.st_size > 0) v = mmap(nullptr, (size_t)st.st_size, PROT_READ, MAP_PRIVATE, fd, 0);
    close(fd);
    if (v == MAP_FAILED) return fail(VKL_INVALID_ARGUMENT, "model_load: %s cannot be mapped", path.c_str());
    p = (const uint8_t *)v;
    n = (size_t)st.st_size;
    return VKL_OK;
  }
};

// A safetensors file: its header, and every tensor by name.
struct Safetensors {
  std::string path;
  Mapping f;
  Json head;
  size_t data = 0;
  int open_file(const std::string &p) {
    path = p;
    VKL_OKAY(f.open_file(path));
    uint64_t hn = 0;
    if (f.n < 8) return fail(VKL_INVALID_ARGUMENT, "model_load: %s is too short", path.c_str());
    memcpy(&hn, f.p, 8);
    if (hn > f.n - 8) return fail(VKL_INVALID_ARGUMENT, "model_load: %s: the header runs past the end", path.c_str());
    data = 8 + (size_t)hn;
    return parse_json((const char *)f.p + 8, (size_t)hn, path.c_str(), &head);
  }
  int load(vkl_model *m) const {
    Shapes shapes;
    VKL_OKAY(read_shapes(head, &shapes));
    for (const auto &t : head.fields) {
      if (t.first == "__metadata__") continue;
      const Json *dt = t.second.get("dtype"), *off = t.second.get("data_offsets");
      if (!dt || !off || off->items.size() != 2) return fail(VKL_INVALID_ARGUMENT, "model_load: %s: entry %s is malformed", path.c_str(), t.first.c_str());
      const double a = off->items[0].num, b = off->items[1].num;
      if (!(a >= 0 && a <= b && b <= (double)(f.n - data))) return fail(VKL_OUT_OF_RANGE, "model_load: tensor %s runs past the end of %s", t.first.c_str(), path.c_str());
      const int dtype = dt->str == "BF16" ? VKL_BF16 : dt->str == "I32" ? VKL_UINT32 : -1;
      if (dtype < 0) return fail(VKL_UNIMPLEMENTED, "model_load: tensor %s has dtype %s (BF16 or I32)", t.first.c_str(), dt->str.c_str());
      VKL_OKAY(decoder_check_shape(m, t.first.c_str(), shapes[t.first]));
      VKL_OKAY(vkl_model_set_weight(m, t.first.c_str(), dtype, f.p + data + (size_t)a, (size_t)(b - a)));
    }
    return VKL_OK;
  }
};

int create(vkl_device *dev, const char *config_json, const Shapes &shapes, uint32_t maxlen, int compute_dtype, vkl_model **out) {
  if (compute_dtype != VKL_BF16 && compute_dtype != VKL_FP32) return fail(VKL_INVALID_ARGUMENT, "model_create_config: compute dtype %d (BF16 or FP32)", compute_dtype);
  DecoderSpec s;
  VKL_OKAY(spec_of(config_json, strlen(config_json), shapes, &s));
  if (!dev) return fail(VKL_INVALID_ARGUMENT, "model_create_config: null device");
  return decoder_create(dev, s, maxlen, compute_dtype == VKL_FP32, out);
}

}  // namespace

extern "C" {

const char *vkl_model_architectures(void) {
  static const std::string names = [] {
    std::string s;
    for (const Architecture &a : kArchitectures) s += (s.empty() ? "" : ",") + std::string(a.name);
    return s;
  }();
  return names.c_str();
}

int vkl_model_create_config(vkl_device *dev, const char *config_json, uint32_t maxlen, int compute_dtype, vkl_model **out) {
  return vkl_model_create_config_shapes(dev, config_json, nullptr, maxlen, compute_dtype, out);
}

int vkl_model_create_config_shapes(vkl_device *dev, const char *config_json, const char *shapes_json, uint32_t maxlen, int compute_dtype, vkl_model **out) {
  if (!config_json || !out) return fail(VKL_INVALID_ARGUMENT, "model_create_config: null argument");
  Shapes shapes;
  if (shapes_json) {
    Json j;
    VKL_OKAY(parse_json(shapes_json, strlen(shapes_json), "shapes", &j));
    VKL_OKAY(read_shapes(j, &shapes));
  }
  return create(dev, config_json, shapes, maxlen, compute_dtype, out);
}

int vkl_model_load_folder(vkl_device *dev, const char *path, uint32_t maxlen, int compute_dtype, vkl_model **out) {
  if (!path || !out) return fail(VKL_INVALID_ARGUMENT, "model_load_folder: null argument");
  const std::string dir(path);
  std::string text;
  {
    Mapping f;
    VKL_OKAY(f.open_file(dir + "/config.json"));
    text.assign((const char *)f.p, f.n);
  }
  Safetensors f;
  VKL_OKAY(f.open_file(dir + "/model.safetensors"));
  Shapes shapes;
  VKL_OKAY(read_shapes(f.head, &shapes));
  vkl_model *m = nullptr;
  VKL_OKAY(create(dev, text.c_str(), shapes, maxlen, compute_dtype, &m));
  int st = f.load(m);
  if (st == VKL_OK) st = decoder_ready(m);
  if (st != VKL_OK) {
    vkl_model_destroy(m);
    return st;
  }
  *out = m;
  return VKL_OK;
}

int vkl_distance_bucket(uint32_t n, uint32_t rows, uint32_t far) { return rows < 2 || far <= rows / 2 ? -1 : (int)distance_bucket(n, rows, far); }

}  // extern "C"
