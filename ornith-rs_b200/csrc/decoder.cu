// Decoders around a float32 residual stream whose sublayers read the stream itself: y = mixer(x) or ff(x).
//
// Peratar: latent attention, dense xIELU feed-forwards
//   x <- x + norm(y * sigmoid(W x + b))   a result is gated from the same input, then normed
//   X_(i+1) = the stream after layer i;  what goes on is sum_j a_ij X_j over all of them so far
//   logits = cap * tanh(head(norm(x)) / cap)
// Dokulorn: a decayed state (retention), or grouped attention and a decayed state side by side (parallel);
// dense gated feed-forwards
//   x <- norm(alpha x + y), y of a parallel mixer = (norm_l(y_l) + norm_r(y_r)) / 2
//   logits = embed(norm(x)), the embedding table itself
//
// Three routes through the same layers, equal to rounding:
//   * windows of 1..4 rows (decoding): three to seven kernels a layer (dense.cu and the mixers), programmatic
//     dependents, capturable into CUDA graphs: every position-dependent size is read on the device;
//   * prompt chunks: tensor-core products with bias and activation in their epilogue, the mixers' chunk
//     forms, one row kernel per sublayer;
//   * the control route, one plain kernel per operation: models loaded in float32, and ORN_UNFUSED=1.
#include <algorithm>
#include <cmath>
#include <cstring>
#include <memory>
#include <string>
#include <vector>

#include "arch.h"
#include "decayed.h"
#include "dense.h"
#include "fused.h"
#include "grouped.h"
#include "heads.h"
#include "latent.h"
#include "model_types.h"

#define CK(call)                     \
  do {                               \
    int rc__ = (call);               \
    if (rc__ != ORN_OK) return rc__; \
  } while (0)

using namespace orna;

namespace {

// ------------------------------------------------------------------ configuration
enum MixKind { MIX_LATENT, MIX_DECAYED, MIX_PARALLEL };  // parallel: grouped attention beside a decayed state
struct LayerSpec {
  MixKind kind = MIX_LATENT;
  LatentDims mix;
  double rot_base = 1.0;
  int kv_from = -1;  // the layer whose cache this one reads, -1: its own
  GroupedDims att;
  double att_base = 1.0;
  DecayedDims lin;
  double lin_base = 1.0;
  std::vector<double> decay;      // per head of lin
  int lin_act = ACT_NONE;         // of its q, k and v
  int lin_gate = ACT_SIGMOID;     // of its output gate
  int lin_group = 1;              // entries of its result that are normed together
  int ff = 0;                     // 0: no feed-forward
  bool attends() const { return kind == MIX_PARALLEL; }
  bool decays() const { return kind != MIX_LATENT; }
};
enum ResidualForm { RES_GATED_AVERAGE, RES_POST_NORM };
struct Spec {
  ResidualForm form = RES_GATED_AVERAGE;
  int width = 0, vocab = 0;
  float eps = 0.f, softcap = 0.f;
  float embed_scale = 1.f, alpha = 1.f, w_add = 0.f;  // RES_POST_NORM: w_add + w is a norm's weight
  bool tied = false;                                  // the head is the embedding table
  std::vector<LayerSpec> layers;
};
struct LayerW {
  orn_linear *q = nullptr, *dkv = nullptr, *uk = nullptr, *uv = nullptr, *g = nullptr, *o = nullptr;
  orn_linear *rg1 = nullptr, *rg2 = nullptr, *up = nullptr, *down = nullptr;
  bf16_t *norm1 = nullptr, *norm2 = nullptr, *dkv_norm = nullptr, *rg1_b = nullptr, *rg2_b = nullptr;
  bf16_t *up_b = nullptr, *down_b = nullptr, *act = nullptr, *dwa = nullptr;
  orn_linear *k = nullptr, *v = nullptr, *lq = nullptr, *lk = nullptr, *lv = nullptr, *lg = nullptr, *lo = nullptr, *gate = nullptr;
  bf16_t *sink = nullptr, *lnorm = nullptr, *out_l = nullptr, *out_r = nullptr;
};
// activation scratch for `rows` rows
struct Scratch {
  int rows = 0;
  std::vector<void*> allocs;
  uint32_t* ids = nullptr;
  float *streams = nullptr, *x = nullptr, *xm = nullptr, *part = nullptr, *kv = nullptr, *g = nullptr, *rg = nullptr, *y = nullptr;
  float* rg_prev = nullptr;  // the gate logits a fused window kernel still reads while it writes the next ones
  float *partial = nullptr, *ml = nullptr;
  uint8_t *xa = nullptr, *q = nullptr, *qa = nullptr, *att = nullptr, *u = nullptr, *normed = nullptr;
  // grouped attention: keys, values, gate; decayed state: queries, keys, values, gate, result, gated result
  uint8_t *ak = nullptr, *av = nullptr, *ag = nullptr, *lq = nullptr, *lk = nullptr, *lv = nullptr, *lg = nullptr, *la = nullptr;
  float *lo = nullptr, *y2 = nullptr;
  uint8_t *ug = nullptr, *chunk = nullptr;  // activated gate of the feed-forward; the decayed state's chunk scratch
  size_t stream_stride = 0;
};
}  // namespace

struct orn_decoder {
  Spec spec;
  std::vector<LayerW> w;
  bf16_t* final_norm = nullptr;
  orn_linear* head = nullptr;
  std::vector<void*> tables;  // rotation frequencies, powers of decays
  uint8_t* window_scratch = nullptr;  // grouped attention's key ranges
  int ldak = 8, ldav = 8, ldag = 8, ldlq = 8, ldlv = 8;
  int ldD = 0, ldq = 0, ldkv = 0, ldg = 0, ldatt = 0, ldu = 0;
  Scratch win, wide;         // windows (its addresses are in captured graphs); prompt chunks
  bf16_t *kx = nullptr, *vx = nullptr;  // expanded keys and values of one layer
  int exp_rows = 0, ldkx = 0, ldvx = 0;
  float* logits = nullptr;   // [kMaxRows][vocab]
  bool f32 = false;
};

namespace {

struct FieldError {
  std::string what;
};
double need_num(const JVal* o, const char* k, const std::string& where) {
  const JVal* v = o ? o->get(k) : nullptr;
  if (!v || v->type != JVal::Num) throw FieldError{where + "." + k + " is missing or not a number"};
  return v->num;
}
int need_int(const JVal* o, const char* k, const std::string& where, int lo) {
  const double d = need_num(o, k, where);
  if (d != std::floor(d) || d < lo || d > 2e9) throw FieldError{where + "." + k + " is out of range"};
  return (int)d;
}
const JVal* need_obj(const JVal* o, const char* k, const std::string& where) {
  const JVal* v = o ? o->get(k) : nullptr;
  if (!v || v->type != JVal::Obj) throw FieldError{where + "." + k + " is missing or not an object"};
  return v;
}
bool is_null(const JVal* v) { return v == nullptr || v->type == JVal::Null; }

void parse_sizes(const JVal& c, Spec* s) {
  s->width = need_int(&c, "width", "config", 1);
  s->vocab = need_int(&c, "vocab", "config", 1);
  s->eps = (float)need_num(c.get("norm"), "eps", "norm");
}
const JVal* parse_layers(const JVal& c) {
  const JVal* ls = c.get("layers");
  if (!ls || ls->type != JVal::Arr || ls->arr.empty()) throw FieldError{"layers is missing or empty"};
  return ls;
}
int parse_ff(const JVal& l, const std::string& at) {
  const JVal* f = l.get("mlp");
  if (is_null(f)) return 0;
  const JVal* k = f->get("kind");
  if (!k || k->str != "dense") throw FieldError{at + ".mlp.kind is not a feed-forward of this architecture"};
  return need_int(f, "ff", at + ".mlp", 1);
}
// a rotation over `dim` entries: base and turned entries; without one nothing turns
void parse_rot(const JVal* m, const std::string& at, int dim, double* base, int* dims) {
  *dims = 0;
  const JVal* r = m->get("rot");
  if (is_null(r)) return;
  *base = need_num(r, "base", at + ".rot");
  *dims = need_int(r, "dims", at + ".rot", 0);
  if (*dims % 2 || *dims > dim || *base <= 0) throw FieldError{at + ".rot does not fit the head"};
}

// ---- Dokulorn
void parse_decayed(const JVal* m, const std::string& at, LayerSpec* L) {
  DecayedDims& D = L->lin;
  D.heads = need_int(m, "heads", at, 1);
  D.dim = need_int(m, "dim", at, 1);
  D.vdim = need_int(m, "vdim", at, 1);
  const JVal* d = m->get("decay");
  if (!d || d->type != JVal::Arr || d->arr.size() != (size_t)D.heads) throw FieldError{at + ".decay is not one number per head"};
  for (const JVal& g : d->arr) {
    if (g.type != JVal::Num || g.num < 0.0 || g.num > 1.0) throw FieldError{at + ".decay is not between 0 and 1"};
    L->decay.push_back(g.num);
  }
}
void parse_grouped(const JVal* m, const std::string& at, float eps, LayerSpec* L) {
  GroupedDims& D = L->att;
  D.heads = need_int(m, "heads", at, 1);
  D.kv_heads = need_int(m, "kv_heads", at, 1);
  if (D.heads % D.kv_heads) throw FieldError{at + ".kv_heads does not divide heads"};
  D.dim = need_int(m, "dim", at, 1);
  D.vdim = need_int(m, "vdim", at, 1);
  D.scale = (float)need_num(m, "scale", at);
  if (!is_null(m->get("softcap"))) {
    D.softcap = (float)need_num(m, "softcap", at);
    if (!(D.softcap > 0.f)) throw FieldError{at + ".softcap is not positive"};
  }
  D.eps = eps;
  parse_rot(m, at, D.dim, &L->att_base, &D.rot_dims);
}
Spec parse_dokulorn(const JVal& c) {
  Spec s;
  s.form = RES_POST_NORM;
  s.tied = true;
  s.w_add = 1.f;
  parse_sizes(c, &s);
  s.alpha = (float)need_num(&c, "postln_alpha", "config");
  s.embed_scale = (float)need_num(need_obj(&c, "embedding", "config"), "scale", "embedding");
  const JVal* ls = parse_layers(c);
  for (size_t i = 0; i < ls->arr.size(); ++i) {
    const JVal& l = ls->arr[i];
    const std::string at = "layers[" + std::to_string(i) + "]", am = at + ".mixer";
    const JVal* ty = l.get("type");
    const JVal* m = need_obj(&l, "mixer", at);
    LayerSpec L;
    if (ty && ty->str == "retention") {
      L.kind = MIX_DECAYED;
      parse_decayed(m, am, &L);
      parse_rot(m, am, L.lin.dim, &L.lin_base, &L.lin.rot_dims);
      L.lin.k_scale = (float)(1.0 / std::sqrt((double)L.lin.dim));
      L.lin_gate = ACT_SILU;
      L.lin_group = L.lin.vdim;
    } else if (ty && ty->str == "parallel") {
      L.kind = MIX_PARALLEL;
      parse_grouped(need_obj(m, "left", am), am + ".left", s.eps, &L);
      parse_decayed(need_obj(m, "right", am), am + ".right", &L);
      L.lin_act = ACT_SILU;
      L.lin_gate = ACT_SIGMOID;
      L.lin_group = L.lin.heads * L.lin.vdim;
    } else {
      throw FieldError{at + ".type is not a mixer of this architecture"};
    }
    L.ff = parse_ff(l, at);
    s.layers.push_back(L);
  }
  return s;
}

// ---- Peratar
Spec parse_peratar(const JVal& c) {
  Spec s;
  parse_sizes(c, &s);
  if (!is_null(c.get("logit_softcap"))) s.softcap = (float)need_num(&c, "logit_softcap", "config");
  const JVal* ls = parse_layers(c);
  for (size_t i = 0; i < ls->arr.size(); ++i) {
    const JVal& l = ls->arr[i];
    const std::string at = "layers[" + std::to_string(i) + "]";
    const JVal* ty = l.get("type");
    if (!ty || ty->str != "latent_attention") throw FieldError{at + ".type is not a mixer of this architecture"};
    const JVal* m = l.get("mixer");
    LayerSpec L;
    L.mix.heads = need_int(m, "heads", at + ".mixer", 1);
    L.mix.dim = need_int(m, "dim", at + ".mixer", 0);
    L.mix.rot_dim = need_int(m, "rot_dim", at + ".mixer", 0);
    L.mix.vdim = need_int(m, "vdim", at + ".mixer", 1);
    L.mix.kv_rank = need_int(m, "kv_rank", at + ".mixer", 1);
    L.mix.scale = (float)need_num(m, "scale", at + ".mixer");
    L.mix.eps = s.eps;
    if (L.mix.rot_dim > 0) {
      const JVal* r = m->get("rot");
      L.rot_base = need_num(r, "base", at + ".mixer.rot");
      L.mix.rot_dims = need_int(r, "dims", at + ".mixer.rot", 0);
      if (L.mix.rot_dims % 2 || L.mix.rot_dims > L.mix.rot_dim || L.rot_base <= 0)
        throw FieldError{at + ".mixer.rot does not fit rot_dim"};
    }
    if (L.mix.qk() < 1) throw FieldError{at + ".mixer has no query dimensions"};
    if (!is_null(m->get("kv_from"))) {
      L.kv_from = need_int(m, "kv_from", at + ".mixer", 0);
      if (L.kv_from >= (int)i) throw FieldError{at + ".mixer.kv_from is not an earlier layer"};
      const LayerSpec& o = s.layers[L.kv_from];
      if (o.kv_from >= 0 || o.mix.kv_rank != L.mix.kv_rank || o.mix.rot_dim != L.mix.rot_dim)
        throw FieldError{at + ".mixer.kv_from names a layer without a cache of these sizes"};
    }
    L.ff = parse_ff(l, at);
    s.layers.push_back(L);
  }
  return s;
}

// Every weight by name and shape; K == 0: a vector of O entries.
struct WeightDesc {
  std::string name;
  int O, K;
};
void decayed_weights(const Spec& s, const LayerSpec& L, const std::string& p, std::vector<WeightDesc>* t) {
  const DecayedDims& D = L.lin;
  t->push_back({p + "q", D.heads * D.dim, s.width});
  t->push_back({p + "k", D.heads * D.dim, s.width});
  t->push_back({p + "v", D.heads * D.vdim, s.width});
  t->push_back({p + "g", D.heads * D.vdim, s.width});
  t->push_back({p + "o", s.width, D.heads * D.vdim});
}
std::vector<WeightDesc> dokulorn_weights(const Spec& s) {
  std::vector<WeightDesc> t;
  t.push_back({"embed", s.vocab, s.width});
  for (size_t i = 0; i < s.layers.size(); ++i) {
    const LayerSpec& L = s.layers[i];
    const std::string p = "l" + std::to_string(i) + ".";
    t.push_back({p + "norm1", s.width, 0});
    if (L.kind == MIX_DECAYED) {
      decayed_weights(s, L, p + "mix.", &t);
    } else {
      const GroupedDims& a = L.att;
      t.push_back({p + "mix.left.q", a.heads * a.dim, s.width});
      t.push_back({p + "mix.left.k", a.kv_heads * a.dim, s.width});
      t.push_back({p + "mix.left.v", a.kv_heads * a.vdim, s.width});
      t.push_back({p + "mix.left.sink", a.heads, 0});
      t.push_back({p + "mix.left.g", a.heads * a.vdim, s.width});
      t.push_back({p + "mix.left.o", s.width, a.heads * a.vdim});
      t.push_back({p + "mix.left.out", s.width, 0});
      decayed_weights(s, L, p + "mix.right.", &t);
      t.push_back({p + "mix.right.norm", L.lin.heads * L.lin.vdim, 0});
      t.push_back({p + "mix.right.out", s.width, 0});
    }
    if (L.ff > 0) {
      t.push_back({p + "norm2", s.width, 0});
      t.push_back({p + "mlp.gate", L.ff, s.width});
      t.push_back({p + "mlp.up", L.ff, s.width});
      t.push_back({p + "mlp.down", s.width, L.ff});
    }
  }
  t.push_back({"final.norm", s.width, 0});
  return t;
}
std::vector<WeightDesc> weight_table(const Spec& s) {
  if (s.form == RES_POST_NORM) return dokulorn_weights(s);
  std::vector<WeightDesc> t;
  t.push_back({"embed", s.vocab, s.width});
  for (size_t i = 0; i < s.layers.size(); ++i) {
    const LayerSpec& L = s.layers[i];
    const LatentDims& m = L.mix;
    const std::string p = "l" + std::to_string(i) + ".";
    t.push_back({p + "norm1", s.width, 0});
    t.push_back({p + "mix.q", m.heads * m.qk(), s.width});
    if (L.kv_from < 0) {
      t.push_back({p + "mix.dkv", m.kv_rank + m.rot_dim, s.width});
      t.push_back({p + "mix.dkv.norm", m.kv_rank, 0});
    }
    if (m.dim > 0) t.push_back({p + "mix.uk", m.heads * m.dim, m.kv_rank});
    t.push_back({p + "mix.uv", m.heads * m.vdim, m.kv_rank});
    t.push_back({p + "mix.g", m.heads, s.width});
    t.push_back({p + "mix.o", s.width, m.heads * m.vdim});
    t.push_back({p + "rg1", s.width, s.width});
    t.push_back({p + "rg1.b", s.width, 0});
    if (L.ff > 0) {
      t.push_back({p + "norm2", s.width, 0});
      t.push_back({p + "mlp.up", L.ff, s.width});
      t.push_back({p + "mlp.up.b", L.ff, 0});
      t.push_back({p + "mlp.down", s.width, L.ff});
      t.push_back({p + "mlp.down.b", s.width, 0});
      t.push_back({p + "mlp.act", 2, 0});
      t.push_back({p + "rg2", s.width, s.width});
      t.push_back({p + "rg2.b", s.width, 0});
    }
    t.push_back({p + "dwa", (int)i + 2, 0});
  }
  t.push_back({"final.norm", s.width, 0});
  t.push_back({"head", s.vocab, s.width});
  return t;
}

// ------------------------------------------------------------------ create, load, finalize
int decoder_create(orn_ctx* ctx, const JVal& cfg, int max_ctx, int dtype, const orn_arch* arch, Spec (*parse)(const JVal&), orn_model** out) {
  if (dtype != ORN_DT_BF16 && dtype != ORN_DT_F32) ORN_FAIL(ctx, ORN_ERR_ARG, "model: unknown data type");
  if (max_ctx < 1) ORN_FAIL(ctx, ORN_ERR_ARG, "model: max_ctx must be positive");
  std::unique_ptr<orn_decoder> d(new orn_decoder());
  try {
    d->spec = parse(cfg);
  } catch (const FieldError& e) {
    ORN_FAIL(ctx, ORN_ERR_ARG, "config.json: " + e.what);
  }
  d->f32 = dtype == ORN_DT_F32;
  orn_model* m = new orn_model();
  m->ctx = ctx;
  m->arch = arch;
  m->cfg = orn_config{};
  m->cfg.hidden = d->spec.width;
  m->cfg.n_layers = (int)d->spec.layers.size();
  m->cfg.vocab = d->spec.vocab;
  m->cfg.rms_eps = d->spec.eps;
  m->cfg.max_ctx = max_ctx;
  m->dtype = dtype;
  m->row_ld = pad8(d->spec.width);
  m->dec = d.release();
  *out = m;
  return ORN_OK;
}

int peratar_create(orn_ctx* ctx, const JVal& cfg, int max_ctx, int dtype, orn_model** out) {
  return decoder_create(ctx, cfg, max_ctx, dtype, &kArchPeratar, parse_peratar, out);
}
int dokulorn_create(orn_ctx* ctx, const JVal& cfg, int max_ctx, int dtype, orn_model** out) {
  return decoder_create(ctx, cfg, max_ctx, dtype, &kArchDokulorn, parse_dokulorn, out);
}

// a matrix [O, K] with rows padded to a multiple of 8 by zeros
int add_matrix(orn_model* m, const std::string& name, int O, int K, const uint16_t* host) {
  const int Kp = pad8(K);
  std::vector<uint16_t> buf;
  if (Kp != K) {
    buf.assign((size_t)O * Kp, 0);
    for (int o = 0; o < O; ++o) memcpy(&buf[(size_t)o * Kp], host + (size_t)o * K, 2 * (size_t)K);
    host = buf.data();
  }
  orn_linear* L = nullptr;
  CK(orn_linear_create(m->ctx, ORN_BF16, 1, O, Kp, host, nullptr, nullptr, &L));
  return orn_model_set_linear(m, name.c_str(), L);
}

int decoder_load(orn_ctx* ctx, const std::string& dir, const JVal& cfg, int max_ctx, int dtype,
                 int (*create)(orn_ctx*, const JVal&, int, int, orn_model**), orn_model** out) {
  Store st;
  std::string err;
  if (!open_shards(dir, &st, &err)) ORN_FAIL(ctx, ORN_ERR_IO, err);
  orn_model* m = nullptr;
  CK(create(ctx, cfg, max_ctx, dtype, &m));
  auto fail = [&](int code, const std::string& msg) {
    orn_model_destroy(m);
    ctx->err = msg;
    return code;
  };
  for (const WeightDesc& w : weight_table(m->dec->spec)) {
    auto it = st.tensors.find(w.name);
    if (it == st.tensors.end()) return fail(ORN_ERR_IO, "missing tensor " + w.name);
    const TInfo& t = it->second;
    const bool shape_ok = w.K ? (t.shape.size() == 2 && t.shape[0] == w.O && t.shape[1] == w.K) : (t.shape.size() == 1 && t.shape[0] == w.O);
    if (t.dtype != "BF16" || !shape_ok || !bytes_match(t, 2)) return fail(ORN_ERR_ARG, "tensor is not bf16 of the configured shape: " + w.name);
    std::vector<uint16_t> host((size_t)numel(t));  // the file's bytes may be unaligned
    memcpy(host.data(), t.data, t.nbytes);
    const int rc = w.K ? add_matrix(m, w.name, w.O, w.K, host.data()) : orn_model_set_tensor(m, w.name.c_str(), host.data(), host.size());
    if (rc != ORN_OK) {
      const std::string msg = ctx->err;
      return fail(rc, msg);
    }
  }
  *out = m;
  return ORN_OK;
}

int peratar_load(orn_ctx* ctx, const std::string& dir, const JVal& cfg, int max_ctx, int dtype, orn_model** out) {
  return decoder_load(ctx, dir, cfg, max_ctx, dtype, peratar_create, out);
}
int dokulorn_load(orn_ctx* ctx, const std::string& dir, const JVal& cfg, int max_ctx, int dtype, orn_model** out) {
  return decoder_load(ctx, dir, cfg, max_ctx, dtype, dokulorn_create, out);
}

uint64_t mix64(uint64_t x) {
  x += 0x9e3779b97f4a7c15ull;
  x = (x ^ (x >> 30)) * 0xbf58476d1ce4e5b9ull;
  x = (x ^ (x >> 27)) * 0x94d049bb133111ebull;
  return x ^ (x >> 31);
}

// seeded synthetic weights: matrices ~ 1 / sqrt(K), norms' weights near 1, each average mostly its newest stream
int decoder_init_random(orn_model* m, uint64_t seed) {
  orn_ctx* ctx = m->ctx;
  uint64_t n = 0;
  const Spec& s = m->dec->spec;
  for (const WeightDesc& w : weight_table(s)) {
    const uint64_t sd = mix64(seed + (++n));
    if (w.K) {
      if (w.K % 8) ORN_FAIL(ctx, ORN_ERR_ARG, "init_random: row lengths must be multiples of 8");
      orn_linear* L = nullptr;
      const float std = w.name == "embed" && !s.tied ? 1.0f : 1.0f / std::sqrt((float)w.K);
      CK(orn_linear_create_random(ctx, ORN_BF16, 1, w.O, w.K, sd, std, &L));
      CK(orn_model_set_linear(m, w.name.c_str(), L));
    } else {
      const bool plain_norm = ends_with(w.name, "mix.right.norm") || ends_with(w.name, ".out");
      const bool norm = plain_norm || w.name.find("norm") != std::string::npos;
      const float mean = !norm ? 0.0f : plain_norm ? 1.0f : 1.0f - s.w_add;
      const bool dwa = ends_with(w.name, ".dwa");
      void* d = nullptr;
      CK(orn_alloc(ctx, (size_t)w.O * 2, &d));
      int rc = k_fill_bf16(ctx, ctx->stream, (bf16_t*)d, w.O, sd, mean, norm ? 0.05f : dwa ? 0.1f : 0.3f);
      if (rc != ORN_OK) { cudaFree(d); return rc; }
      if (dwa) {
        const uint16_t one = 0x3f80;
        rc = orn_upload(ctx, (bf16_t*)d + (w.O - 1), &one, 2);
        if (rc != ORN_OK) { cudaFree(d); return rc; }
      }
      auto it = m->tensors.find(w.name);
      if (it != m->tensors.end()) cudaFree(it->second.p);
      m->tensors[w.name] = Tensor{(bf16_t*)d, (size_t)w.O};
    }
  }
  return orn_sync(ctx);
}

size_t act_bytes(const orn_decoder* d) { return d->f32 ? 4 : 2; }

bool unfused_env() {
  static const bool v = [] { const char* e = getenv("ORN_UNFUSED"); return e && e[0] == '1'; }();
  return v;
}
bool plain_route(const orn_model* m) { return m->dec->f32 || unfused_env(); }

void release_scratch(Scratch& w) {
  for (void* p : w.allocs) cudaFree(p);
  w = Scratch();
}

constexpr int kAbsorbMaxRows = 32;  // chunks up to this many rows attend in absorbed form

bool expand_layer(const orn_model* m, int i, int T) {
  const orn_decoder* d = m->dec;
  return d->spec.layers[i].kind == MIX_LATENT && !plain_route(m) && T > kAbsorbMaxRows && latent_flash_ok(d->spec.layers[i].mix, d->ldq);
}
bool attn_plain(const orn_model* m, const LatentDims& D) { return plain_route(m) || !latent_attn_tensor_ok(D); }

int reserve(orn_model* m, Scratch& w, int rows) {
  if (w.rows >= rows) return ORN_OK;
  orn_ctx* ctx = m->ctx;
  ORN_CHECK_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
  release_scratch(w);
  orn_decoder* d = m->dec;
  const size_t R = rows, A = act_bytes(d), D = d->ldD;
  int rc = ORN_OK;
  auto take = [&](auto** p, size_t bytes) {
    if (rc != ORN_OK) return;
    void* v = nullptr;
    rc = orn_alloc(ctx, bytes ? bytes : 16, &v);
    if (rc != ORN_OK) return;
    w.allocs.push_back(v);
    rc = orn_memset(ctx, v, 0, bytes);  // row padding stays zero from here on
    *p = reinterpret_cast<std::remove_reference_t<decltype(**p)>*>(v);
  };
  const size_t L = d->spec.layers.size();
  take(&w.ids, R * 4);
  take(&w.x, R * D * 4); take(&w.xm, R * D * 4); take(&w.y, R * D * 4);
  if (d->spec.form == RES_GATED_AVERAGE) {
    w.stream_stride = R * D;
    take(&w.streams, (L + 1) * w.stream_stride * 4);
    take(&w.part, R * D * 4); take(&w.rg, R * D * 4); take(&w.rg_prev, R * D * 4);
  }
  bool attends = false, decays = false, glu = false;
  size_t chunk = 0;
  for (const LayerSpec& y : d->spec.layers) {
    attends = attends || y.attends();
    decays = decays || y.decays();
    glu = glu || (y.ff > 0 && d->spec.form == RES_POST_NORM);
    if (y.decays() && rows > kMaxRows) chunk = std::max(chunk, decayed_chunk_scratch(y.lin, rows));
  }
  if (attends) { take(&w.ak, R * d->ldak * A); take(&w.av, R * d->ldav * A); take(&w.ag, R * d->ldag * A); take(&w.y2, R * D * 4); }
  if (decays) {
    take(&w.lq, R * d->ldlq * A); take(&w.lk, R * d->ldlq * A); take(&w.lv, R * d->ldlv * A); take(&w.lg, R * d->ldlv * A);
    take(&w.la, R * d->ldlv * A); take(&w.lo, R * d->ldlv * 4);
    if (!plain_route(m) && chunk > 0) take(&w.chunk, chunk);
  }
  if (glu) take(&w.ug, R * d->ldu * A);
  take(&w.kv, R * d->ldkv * 4); take(&w.g, R * d->ldg * 4);
  take(&w.q, R * d->ldq * A); take(&w.att, R * d->ldatt * A); take(&w.u, R * d->ldu * A); take(&w.normed, R * D * A);
  if (d->f32) w.xa = reinterpret_cast<uint8_t*>(w.x);
  else take(&w.xa, R * D * A);
  // absorbed attention: queries, partial sums
  size_t qa = 0, part = 0, ml = 0;
  for (size_t i = 0; i < L; ++i) {
    if (d->spec.layers[i].kind != MIX_LATENT) continue;
    const LatentDims& M = d->spec.layers[i].mix;
    // the widest window that attends in absorbed form
    const int wide_rows = expand_layer(m, (int)i, rows) ? std::min(rows, kAbsorbMaxRows) : rows;
    const size_t rh = (size_t)wide_rows * M.heads;
    qa = std::max(qa, rh * M.row());
    size_t sp = 1;
    for (int t = 1; t <= wide_rows; ++t) {
      const size_t s = (size_t)latent_splits(ctx, M, t, attn_plain(m, M)) * t;
      sp = std::max(sp, s);
    }
    part = std::max(part, sp * M.heads * M.kv_rank);
    ml = std::max(ml, sp * M.heads * 2);
  }
  take(&w.qa, qa * A); take(&w.partial, part * 4); take(&w.ml, ml * 4);
  if (rc != ORN_OK) { release_scratch(w); return rc; }
  w.rows = rows;
  return ORN_OK;
}

// device tables of a rotation and of a head's powers
template <typename T>
int upload_table(orn_model* m, const std::vector<T>& v, const T** out) {
  void* p = nullptr;
  CK(orn_alloc(m->ctx, std::max<size_t>(1, v.size()) * sizeof(T), &p));
  m->dec->tables.push_back(p);
  *out = reinterpret_cast<const T*>(p);
  return v.empty() ? ORN_OK : orn_upload(m->ctx, p, v.data(), v.size() * sizeof(T));
}
std::vector<double> rotation_table(double base, int dims) {
  std::vector<double> f(dims / 2);
  for (int e = 0; e < dims / 2; ++e) f[e] = std::pow(base, -2.0 * e / dims);
  return f;
}

int decoder_finalize(orn_model* m) {
  if (m->finalized) return ORN_OK;
  orn_ctx* ctx = m->ctx;
  orn_decoder* d = m->dec;
  const Spec& s = d->spec;
  for (const WeightDesc& w : weight_table(s)) {
    if (w.K) {
      auto it = m->lins.find(w.name);
      if (it == m->lins.end()) ORN_FAIL(ctx, ORN_ERR_STATE, "model: missing weight " + w.name);
      if (it->second->kind != ORN_BF16 || it->second->E != 1 || it->second->O != w.O || it->second->K != pad8(w.K))
        ORN_FAIL(ctx, ORN_ERR_ARG, "model: wrong shape or format for " + w.name);
    } else {
      auto it = m->tensors.find(w.name);
      if (it == m->tensors.end()) ORN_FAIL(ctx, ORN_ERR_STATE, "model: missing tensor " + w.name);
      if (it->second.n != (size_t)w.O) ORN_FAIL(ctx, ORN_ERR_ARG, "model: wrong size for " + w.name);
    }
  }
  auto lin = [&](const std::string& n) { auto it = m->lins.find(n); return it == m->lins.end() ? nullptr : it->second; };
  auto ten = [&](const std::string& n) { auto it = m->tensors.find(n); return it == m->tensors.end() ? nullptr : it->second.p; };
  m->embed = lin("embed");
  m->lm_head = d->head = s.tied ? m->embed : lin("head");
  d->final_norm = ten("final.norm");
  d->w.assign(s.layers.size(), LayerW());
  for (void* p : d->tables) cudaFree(p);
  d->tables.clear();
  size_t window_bytes = 0;
  d->ldD = pad8(s.width);
  d->ldkv = d->ldg = d->ldq = d->ldatt = 8;
  d->ldu = d->ldkx = d->ldvx = 8;
  for (size_t i = 0; i < s.layers.size(); ++i) {
    const std::string p = "l" + std::to_string(i) + ".";
    LayerW& w = d->w[i];
    w.q = lin(p + "mix.q"); w.dkv = lin(p + "mix.dkv"); w.uk = lin(p + "mix.uk"); w.uv = lin(p + "mix.uv");
    w.g = lin(p + "mix.g"); w.o = lin(p + "mix.o"); w.rg1 = lin(p + "rg1"); w.rg2 = lin(p + "rg2");
    w.up = lin(p + "mlp.up"); w.down = lin(p + "mlp.down");
    w.norm1 = ten(p + "norm1"); w.norm2 = ten(p + "norm2"); w.dkv_norm = ten(p + "mix.dkv.norm");
    w.rg1_b = ten(p + "rg1.b"); w.rg2_b = ten(p + "rg2.b"); w.up_b = ten(p + "mlp.up.b"); w.down_b = ten(p + "mlp.down.b");
    w.act = ten(p + "mlp.act"); w.dwa = ten(p + "dwa");
    LayerSpec& L = d->spec.layers[i];
    d->ldu = std::max(d->ldu, pad8(L.ff));
    if (L.decays()) {
      const std::string pl = p + (L.attends() ? "mix.right." : "mix.");
      w.lq = lin(pl + "q"); w.lk = lin(pl + "k"); w.lv = lin(pl + "v"); w.lg = lin(pl + "g"); w.lo = lin(pl + "o");
      w.lnorm = ten(pl + "norm"); w.out_r = ten(pl + "out");
      w.gate = lin(p + "mlp.gate");
      DecayedDims& D = L.lin;
      d->ldlq = std::max(d->ldlq, pad8(D.heads * D.dim));
      d->ldlv = std::max(d->ldlv, pad8(D.heads * D.vdim));
      CK(upload_table(m, rotation_table(L.lin_base, D.rot_dims), &D.freq));
      std::vector<float> gp;
      for (double g : L.decay)
        for (int e = 0; e <= kDecayChunk; ++e) gp.push_back((float)std::pow(g, (double)e));
      CK(upload_table(m, gp, &D.gpow));
      if (L.attends()) {
        const std::string pa = p + "mix.left.";
        w.q = lin(pa + "q"); w.k = lin(pa + "k"); w.v = lin(pa + "v"); w.g = lin(pa + "g"); w.o = lin(pa + "o");
        w.sink = ten(pa + "sink"); w.out_l = ten(pa + "out");
        GroupedDims& G = L.att;
        G.sink = w.sink;
        d->ldq = std::max(d->ldq, pad8(G.heads * G.dim));
        d->ldak = std::max(d->ldak, pad8(G.kv_heads * G.dim));
        d->ldav = std::max(d->ldav, pad8(G.kv_heads * G.vdim));
        d->ldag = std::max(d->ldag, pad8(G.heads * G.vdim));
        d->ldatt = std::max(d->ldatt, pad8(G.heads * G.vdim));
        CK(upload_table(m, rotation_table(L.att_base, G.rot_dims), &G.freq));
        window_bytes = std::max(window_bytes, grouped_window_scratch(ctx, G));
      }
      continue;
    }
    LatentDims& M = L.mix;
    d->ldq = std::max(d->ldq, pad8(M.heads * M.qk()));
    d->ldkv = std::max(d->ldkv, pad8(M.kv_rank + M.rot_dim));
    d->ldg = std::max(d->ldg, pad8(M.heads));
    d->ldatt = std::max(d->ldatt, pad8(M.heads * M.vdim));
    d->ldkx = std::max(d->ldkx, pad8(M.heads * M.dim));
    d->ldvx = std::max(d->ldvx, pad8(M.heads * M.vdim));
    const std::vector<double> f = rotation_table(L.rot_base, M.rot_dims);
    CK(upload_table(m, std::vector<float>(f.begin(), f.end()), &M.freq));
  }
  Workspace& ws = m->ws;
  auto take = [&](auto** p, size_t bytes) -> int {
    void* v = nullptr;
    CK(orn_alloc(ctx, bytes, &v));
    m->ws_allocs.push_back(v);
    *p = reinterpret_cast<std::remove_reference_t<decltype(**p)>*>(v);
    return orn_memset(ctx, v, 0, bytes);
  };
  const size_t row = (size_t)d->ldD * act_bytes(d);
  CK(take(&ws.ids, 32)); CK(take(&ws.targets, 32)); CK(take(&ws.window, 32)); CK(take(&ws.local, 4)); CK(take(&ws.mailbox, 64));
  CK(take(&ws.vh, kMaxRows * row)); CK(take(&ws.hrow, row));
  CK(take(&ws.greedy_scratch, 4 * greedy_scratch_floats(kMaxRows, s.vocab)));
  CK(take(&d->logits, 4 * (size_t)kMaxRows * s.vocab));
  if (window_bytes > 0) CK(take(&d->window_scratch, window_bytes));
  CK(reserve(m, d->win, kMaxRows));
  for (int i = 0; i < 4; ++i) ORN_CHECK_CUDA(ctx, cudaEventCreate(&m->ev[i]));
  m->finalized = true;
  return ORN_OK;
}

void decoder_release(orn_model* m) {
  orn_decoder* d = m->dec;
  if (!d) return;
  release_scratch(d->win);
  release_scratch(d->wide);
  for (void* p : d->tables) cudaFree(p);
  cudaFree(d->kx);
  cudaFree(d->vx);
  delete d;
  m->dec = nullptr;
}

// ------------------------------------------------------------------ cache
// latent attention: one row per position and owning layer; grouped attention: a key and a value row per
// position; a decayed state: a ring of states, of which a window of rows fills one slot per row
int grouped_row_k(const LayerSpec& L) { return pad8(L.att.kv_heads * L.att.dim); }
int grouped_row_v(const LayerSpec& L) { return pad8(L.att.kv_heads * L.att.vdim); }

int decoder_cache_init(orn_cache* c) {
  orn_model* m = c->m;
  const Spec& s = m->dec->spec;
  const size_t n = s.layers.size(), A = act_bytes(m->dec), cap = m->cfg.max_ctx;
  c->latent.assign(n, nullptr);
  c->kc.assign(n, nullptr);
  c->vc.assign(n, nullptr);
  c->ring.assign(n, nullptr);
  auto zeroed = [&](void** p, size_t bytes) -> int {
    CK(orn_alloc(m->ctx, bytes, p));
    return orn_memset(m->ctx, *p, 0, bytes);
  };
  for (size_t i = 0; i < n; ++i) {
    const LayerSpec& L = s.layers[i];
    if (L.kind == MIX_LATENT && L.kv_from < 0) CK(zeroed(&c->latent[i], cap * L.mix.row() * A));
    if (L.attends()) {
      CK(zeroed((void**)&c->kc[i], cap * grouped_row_k(L) * A));
      CK(zeroed((void**)&c->vc[i], cap * grouped_row_v(L) * A));
    }
    if (L.decays()) CK(orn_alloc(m->ctx, kRing * L.lin.state() * sizeof(float), (void**)&c->ring[i]));
  }
  for (size_t i = 0; i < n; ++i)
    if (s.layers[i].kv_from >= 0) c->latent[i] = c->latent[s.layers[i].kv_from];
  return ORN_OK;
}
// rows beyond the position are never read; the states start at zero
int decoder_cache_reset(orn_cache* c) {
  const Spec& s = c->m->dec->spec;
  for (size_t i = 0; i < s.layers.size(); ++i)
    if (s.layers[i].decays()) CK(orn_memset(c->m->ctx, c->ring[i], 0, kRing * s.layers[i].lin.state() * sizeof(float)));
  return ORN_OK;
}
void decoder_cache_release(orn_cache* c) {  // keys, values and states go with the cache itself
  const Spec& s = c->m->dec->spec;
  for (size_t i = 0; i < c->latent.size(); ++i)
    if (s.layers[i].kv_from < 0) cudaFree(c->latent[i]);
  c->latent.clear();
}

// ------------------------------------------------------------------ products
constexpr int kInputJobs = 8;  // most matrices that read a layer's input

// y_j = act(x W_j^T + b) of up to kInputJobs matrices over the same rows
int products(orn_model* m, const void* x, int ldx, int T, const DenseJob* jobs, int n) {
  orn_ctx* ctx = m->ctx;
  if (plain_route(m)) {
    for (int j = 0; j < n; ++j) {
      DenseJob job = jobs[j];
      if (m->dec->f32) job.out_f32 = true;
      CK(k_linear_plain(ctx, ctx->stream, job.lin, x, m->dec->f32, ldx, T, job));
    }
    return ORN_OK;
  }
  for (int j0 = 0; j0 < n; j0 += 4) {  // four to a launch
    const orn_linear* Ls[4];
    void* ys[4];
    int ldys[4];
    QGemmEpi epi[4];
    const int k = std::min(4, n - j0);
    for (int j = 0; j < k; ++j) {
      const DenseJob& J = jobs[j0 + j];
      Ls[j] = J.lin; ys[j] = J.y; ldys[j] = J.ldy;
      epi[j].bias = J.bias; epi[j].act = J.act; epi[j].out_f32 = J.out_f32;
      epi[j].mul = reinterpret_cast<const bf16_t*>(J.mul);
    }
    CK(f_qgemm_multi(ctx, ctx->stream, Ls, ys, ldys, k, reinterpret_cast<const bf16_t*>(x), T, nullptr, nullptr, 0, 0, epi, ldx));
  }
  return ORN_OK;
}

// the products that read a layer's input, into the scratch; returns how many
int input_jobs(orn_model* m, Scratch& w, int i, DenseJob* j) {
  orn_decoder* d = m->dec;
  const LayerW& W = d->w[i];
  const LayerSpec& ly = d->spec.layers[i];
  int n = 0;
  if (ly.kind != MIX_LATENT) {
    auto add = [&](const orn_linear* lin, void* y, int ldy, int act) {
      j[n] = DenseJob(); j[n].lin = lin; j[n].y = y; j[n].ldy = ldy; j[n].out_f32 = d->f32; j[n].act.kind = act; ++n;
    };
    if (ly.attends()) {
      add(W.q, w.q, d->ldq, ACT_NONE); add(W.k, w.ak, d->ldak, ACT_NONE); add(W.v, w.av, d->ldav, ACT_NONE); add(W.g, w.ag, d->ldag, ACT_NONE);
    }
    add(W.lq, w.lq, d->ldlq, ly.lin_act); add(W.lk, w.lk, d->ldlq, ly.lin_act); add(W.lv, w.lv, d->ldlv, ly.lin_act);
    add(W.lg, w.lg, d->ldlv, ACT_NONE);
    return n;
  }
  j[n] = DenseJob(); j[n].lin = W.q; j[n].y = w.q; j[n].ldy = d->ldq; j[n].out_f32 = d->f32; ++n;
  if (d->spec.layers[i].kv_from < 0) { j[n] = DenseJob(); j[n].lin = W.dkv; j[n].y = w.kv; j[n].ldy = d->ldkv; ++n; }
  j[n] = DenseJob(); j[n].lin = W.g; j[n].y = w.g; j[n].ldy = d->ldg; ++n;
  j[n] = DenseJob(); j[n].lin = W.rg1; j[n].y = w.rg; j[n].ldy = d->ldD; ++n;
  return n;
}
int ff_jobs(orn_model* m, Scratch& w, int i, DenseJob* j) {
  orn_decoder* d = m->dec;
  const LayerW& W = d->w[i];
  j[0] = DenseJob(); j[0].lin = W.up; j[0].y = w.u; j[0].ldy = d->ldu; j[0].out_f32 = d->f32; j[0].bias = W.up_b;
  j[0].act.kind = ACT_XIELU; j[0].act.pq = W.act;
  j[1] = DenseJob(); j[1].lin = W.rg2; j[1].y = w.rg; j[1].ldy = d->ldD;
  return 2;
}
DenseJob down_job(orn_model* m, Scratch& w, int i) {
  DenseJob j;
  j.lin = m->dec->w[i].down; j.y = w.y; j.ldy = m->dec->ldD; j.bias = m->dec->w[i].down_b;
  return j;
}
DenseJob o_job(orn_model* m, Scratch& w, int i) {
  DenseJob j;
  j.lin = m->dec->w[i].o; j.y = w.y; j.ldy = m->dec->ldD;
  return j;
}
// the output products of a mixer: into w.y (a decayed state alone, or the attention) and w.y2
DenseJob lin_o_job(orn_model* m, Scratch& w, int i) {
  DenseJob j;
  j.lin = m->dec->w[i].lo; j.y = m->dec->spec.layers[i].attends() ? w.y2 : w.y; j.ldy = m->dec->ldD;
  return j;
}
DenseJob head_job(orn_model* m, float* logits) {
  DenseJob j;
  j.lin = m->dec->head; j.y = logits; j.ldy = m->dec->spec.vocab;
  if (m->dec->spec.softcap > 0.f) { j.act.kind = ACT_SOFTCAP; j.act.cap = m->dec->spec.softcap; }
  return j;
}
// the gate, norm and residual add after sublayer `sub` of layer i; with avg also the layer's depth average
ResidualStep residual(orn_model* m, Scratch& w, int i, int sub, bool avg) {
  orn_decoder* d = m->dec;
  const LayerW& W = d->w[i];
  ResidualStep r;
  r.y = w.y; r.gate = w.rg; r.gate_b = sub == 1 ? W.rg1_b : W.rg2_b; r.w = sub == 1 ? W.norm1 : W.norm2;
  r.width = d->spec.width; r.ld = d->ldD; r.eps = d->spec.eps;
  if (avg) { r.n_avg = i + 2; r.a = W.dwa; r.streams = w.streams; r.stream_stride = w.stream_stride; }
  return r;
}

// the residual after sublayer `sub` of layer i, normed after its sum
PostNormStep post_norm(orn_model* m, Scratch& w, int i, int sub) {
  orn_decoder* d = m->dec;
  const LayerW& W = d->w[i];
  const Spec& s = d->spec;
  PostNormStep r;
  r.y = w.y; r.w = sub == 1 ? W.norm1 : W.norm2; r.w_add = s.w_add; r.alpha = s.alpha; r.eps = s.eps; r.width = s.width; r.ld = d->ldD;
  if (sub == 1 && s.layers[i].attends()) { r.y2 = w.y2; r.wl = W.out_l; r.wr = W.out_r; }
  return r;
}
GroupGate lin_gate(orn_model* m, Scratch& w, int i) {
  orn_decoder* d = m->dec;
  const LayerSpec& ly = d->spec.layers[i];
  GroupGate g;
  g.o = w.lo; g.ldo = d->ldlv; g.gate = w.lg; g.ldg = d->ldlv; g.n = ly.lin.heads * ly.lin.vdim; g.group = ly.lin_group;
  g.w = d->w[i].lnorm; g.act = ly.lin_gate; g.eps = d->spec.eps;
  return g;
}
GroupedArgs grouped_args(orn_model* m, orn_cache* c, Scratch& w, int i, int T) {
  orn_decoder* d = m->dec;
  const LayerSpec& ly = d->spec.layers[i];
  GroupedArgs a;
  a.T = T; a.q = w.q; a.ldq = d->ldq; a.k = w.ak; a.ldk = d->ldak; a.v = w.av; a.ldv = d->ldav;
  a.kc = c->kc[i]; a.vc = c->vc[i]; a.ldkc = grouped_row_k(ly); a.ldvc = grouped_row_v(ly); a.cap = m->cfg.max_ctx; a.pos = c->pos;
  a.gate = w.ag; a.ldg = d->ldag; a.att = w.att; a.ldatt = d->ldatt;
  return a;
}
DecayedArgs decayed_args(orn_model* m, orn_cache* c, Scratch& w, int i, int T, bool keep_all) {
  orn_decoder* d = m->dec;
  DecayedArgs a;
  a.T = T; a.q = w.lq; a.ldq = d->ldlq; a.k = w.lk; a.ldk = d->ldlq; a.v = w.lv; a.ldv = d->ldlv;
  a.ring = c->ring[i]; a.nring = kRing; a.cur = c->cur; a.keep_all = keep_all; a.pos = c->pos; a.o = w.lo; a.ldo = d->ldlv;
  return a;
}

int copy_tap(orn_model* m, int i, const float* x, int T) {
  if (m->tap == nullptr) return ORN_OK;
  const int D = m->dec->spec.width;
  ORN_CHECK_CUDA(m->ctx, cudaMemcpy2DAsync(m->tap + ((size_t)i * m->tap_rows + m->tap_at) * D, (size_t)D * 4, x, (size_t)m->dec->ldD * 4,
                                           (size_t)D * 4, T, cudaMemcpyDeviceToDevice, m->ctx->stream));
  return ORN_OK;
}

// absorbed attention of T rows: queries, partial sums, output rows in w.att
int attend_absorbed(orn_model* m, orn_cache* c, Scratch& w, int i, int T, const StreamSum& sum) {
  orn_ctx* ctx = m->ctx;
  cudaStream_t s = ctx->stream;
  orn_decoder* d = m->dec;
  const LayerSpec& L = d->spec.layers[i];
  const LayerW& W = d->w[i];
  const bool plain = attn_plain(m, L.mix);
  const int cap = m->cfg.max_ctx, splits = latent_splits(ctx, L.mix, T, plain);
  orn_linear none;
  CK(k_latent_absorb(ctx, s, L.mix, T, w.q, d->ldq, W.uk ? W.uk : &none, L.kv_from < 0 ? w.kv : nullptr, d->ldkv, W.dkv_norm, c->latent[i], cap,
                     c->pos, w.qa, sum, d->f32));
  CK(k_latent_attn(ctx, s, L.mix, T, w.qa, c->latent[i], cap, c->pos, splits, w.partial, w.ml, plain, d->f32));
  return k_latent_out(ctx, s, L.mix, T, W.uv, w.partial, w.ml, splits, c->pos, w.g, d->ldg, w.att, d->ldatt, plain, d->f32);
}

int reserve_expanded(orn_model* m, int rows) {
  orn_decoder* d = m->dec;
  if (d->exp_rows >= rows) return ORN_OK;
  ORN_CHECK_CUDA(m->ctx, cudaStreamSynchronize(m->ctx->stream));
  cudaFree(d->kx); cudaFree(d->vx);
  d->kx = d->vx = nullptr;
  d->exp_rows = 0;
  const int n = std::min(m->cfg.max_ctx, std::max(rows, 2048));
  CK(orn_alloc(m->ctx, (size_t)n * d->ldkx * 2, (void**)&d->kx));
  CK(orn_alloc(m->ctx, (size_t)n * d->ldvx * 2, (void**)&d->vx));
  d->exp_rows = n;
  return ORN_OK;
}

int attend_expanded(orn_model* m, orn_cache* c, Scratch& w, int i, int T) {
  orn_ctx* ctx = m->ctx;
  cudaStream_t s = ctx->stream;
  orn_decoder* d = m->dec;
  const LayerSpec& L = d->spec.layers[i];
  const LayerW& W = d->w[i];
  const int n = c->h_pos + T;  // cached positions once this chunk's rows are in
  CK(k_latent_rows(ctx, s, L.mix, T, L.kv_from < 0 ? w.kv : nullptr, d->ldkv, W.dkv_norm, c->latent[i], m->cfg.max_ctx, c->pos, w.q, d->ldq, true, d->f32));
  const orn_linear* Ls[2] = {W.uv, W.uk};
  void* ys[2] = {d->vx, d->kx};
  const int ldys[2] = {d->ldvx, d->ldkx};
  CK(f_qgemm_multi(ctx, s, Ls, ys, ldys, W.uk ? 2 : 1, reinterpret_cast<const bf16_t*>(c->latent[i]), n, nullptr, nullptr, 0, 0, nullptr, L.mix.row()));
  return k_latent_flash(ctx, s, L.mix, T, (const bf16_t*)w.q, d->ldq, d->kx, d->ldkx, d->vx, d->ldvx, (const bf16_t*)c->latent[i], m->cfg.max_ctx, c->pos, w.g,
                        d->ldg, (bf16_t*)w.att, d->ldatt);
}

// grouped attention over rows: turn, norm and append, then attend; result in w.att
int attend_grouped(orn_model* m, orn_cache* c, Scratch& w, int i, int T) {
  orn_ctx* ctx = m->ctx;
  cudaStream_t s = ctx->stream;
  orn_decoder* d = m->dec;
  const GroupedDims& G = d->spec.layers[i].att;
  const GroupedArgs a = grouped_args(m, c, w, i, T);
  HeadRows h[3];
  h[0].src = w.q; h[0].ld_src = a.ldq; h[0].dst = w.q; h[0].ld_dst = a.ldq; h[0].heads = G.heads; h[0].dim = G.dim;
  h[1].src = w.ak; h[1].ld_src = a.ldk; h[1].dst = a.kc; h[1].ld_dst = a.ldkc; h[1].heads = G.kv_heads; h[1].dim = G.dim;
  for (int j = 0; j < 2; ++j) { h[j].rot_dims = G.rot_dims; h[j].freq = G.freq; h[j].unit = G.unit_qk; h[j].eps = G.eps; }
  h[2].src = w.av; h[2].ld_src = a.ldv; h[2].dst = a.vc; h[2].ld_dst = a.ldvc; h[2].heads = G.kv_heads; h[2].dim = G.vdim;
  for (int j = 1; j < 3; ++j) { h[j].dst_at_pos = true; h[j].cap = a.cap; }
  CK(k_head_rows(ctx, s, T, h, 3, c->pos, d->f32));
  if (!plain_route(m) && T > kMaxRows && grouped_flash_ok(G, a)) return k_grouped_flash(ctx, s, G, a);
  return k_grouped_plain(ctx, s, G, a, d->f32);
}
// the decayed state over rows; result in w.lo
int decay_rows(orn_model* m, orn_cache* c, Scratch& w, int i, int T, bool keep_all) {
  orn_ctx* ctx = m->ctx;
  cudaStream_t s = ctx->stream;
  orn_decoder* d = m->dec;
  const DecayedDims& D = d->spec.layers[i].lin;
  const DecayedArgs a = decayed_args(m, c, w, i, T, keep_all);
  if (D.rot_dims > 0) {
    HeadRows h[2];
    h[0].src = h[0].dst = w.lq;
    h[1].src = h[1].dst = w.lk;
    for (int j = 0; j < 2; ++j) { h[j].ld_src = h[j].ld_dst = d->ldlq; h[j].heads = D.heads; h[j].dim = D.dim; h[j].rot_dims = D.rot_dims; h[j].freq = D.freq; }
    CK(k_head_rows(ctx, s, T, h, 2, c->pos, d->f32));
  }
  if (!plain_route(m) && T > kMaxRows && w.chunk != nullptr && decayed_chunk_ok(D, a)) return k_decayed_chunk(ctx, s, D, a, w.chunk);
  return k_decayed_plain(ctx, s, D, a, d->f32);
}

// ------------------------------------------------------------------ rows route (prompt chunks, control path)
// one layer whose residual is normed after its sum
int post_norm_layer(orn_model* m, orn_cache* c, Scratch& w, int i, int T, bool capture) {
  orn_ctx* ctx = m->ctx;
  cudaStream_t s = ctx->stream;
  orn_decoder* d = m->dec;
  const LayerSpec& ly = d->spec.layers[i];
  const int ld = d->ldD;
  void* act = d->f32 ? nullptr : w.xa;
  DenseJob jobs[kInputJobs];
  CK(products(m, w.xa, ld, T, jobs, input_jobs(m, w, i, jobs)));
  if (ly.attends()) {
    CK(attend_grouped(m, c, w, i, T));
    DenseJob oj = o_job(m, w, i);
    CK(products(m, w.att, d->ldatt, T, &oj, 1));
  }
  CK(decay_rows(m, c, w, i, T, capture));
  CK(k_group_gate_rows(ctx, s, T, lin_gate(m, w, i), w.la, d->ldlv, d->f32));
  DenseJob oj = lin_o_job(m, w, i);
  CK(products(m, w.la, d->ldlv, T, &oj, 1));
  PostNormStep r = post_norm(m, w, i, 1);
  r.x_in = w.x; r.x_out = w.x; r.act_out = act;
  CK(k_post_norm_rows(ctx, s, T, r, d->f32));
  if (ly.ff == 0) return ORN_OK;
  DenseJob gj, uj;
  gj.lin = d->w[i].gate; gj.y = w.ug; gj.ldy = d->ldu; gj.out_f32 = d->f32; gj.act.kind = ACT_GELU_TANH;
  uj.lin = d->w[i].up; uj.y = w.u; uj.ldy = d->ldu; uj.out_f32 = d->f32; uj.mul = w.ug;
  CK(products(m, w.xa, ld, T, &gj, 1));
  CK(products(m, w.xa, ld, T, &uj, 1));  // multiplies by the first on its way out
  DenseJob dj = down_job(m, w, i);
  CK(products(m, w.u, d->ldu, T, &dj, 1));
  r = post_norm(m, w, i, 2);
  r.x_in = w.x; r.x_out = w.x; r.act_out = act;
  return k_post_norm_rows(ctx, s, T, r, d->f32);
}
int final_norm_rows(orn_model* m, const float* x, int T, void* out) {
  orn_decoder* d = m->dec;
  const Spec& s = d->spec;
  if (s.form == RES_POST_NORM) return k_rms_norm_rows(m->ctx, m->ctx->stream, x, T, s.width, d->ldD, d->final_norm, s.w_add, s.eps, out, d->f32);
  return k_layer_norm_rows(m->ctx, m->ctx->stream, x, T, s.width, d->ldD, d->final_norm, s.eps, out, d->f32);
}

int rows_forward(orn_model* m, orn_cache* c, Scratch& w, const uint32_t* dev_ids, int T, bool capture, void* normed_out) {
  orn_ctx* ctx = m->ctx;
  cudaStream_t s = ctx->stream;
  orn_decoder* d = m->dec;
  const Spec& sp = d->spec;
  const int D = sp.width, ld = d->ldD, L = (int)sp.layers.size();
  void* act = d->f32 ? nullptr : w.xa;  // float32: the stream is its own activation
  CK(k_embed_rows(ctx, s, m->embed, dev_ids, T, D, ld, sp.embed_scale, w.x, w.streams, act, d->f32));
  DenseJob jobs[kInputJobs];
  for (int i = 0; i < L; ++i) {
    const LayerSpec& ly = sp.layers[i];
    if (sp.form == RES_POST_NORM) {
      CK(post_norm_layer(m, c, w, i, T, capture));
      CK(copy_tap(m, i, w.x, T));
      continue;
    }
    CK(products(m, w.xa, ld, T, jobs, input_jobs(m, w, i, jobs)));
    if (expand_layer(m, i, T)) CK(attend_expanded(m, c, w, i, T));
    else CK(attend_absorbed(m, c, w, i, T, StreamSum()));
    DenseJob oj = o_job(m, w, i);
    CK(products(m, w.att, d->ldatt, T, &oj, 1));
    ResidualStep r = residual(m, w, i, 1, ly.ff == 0);
    r.x_in = w.x; r.x_out = w.x; r.act_out = act;
    CK(k_residual_rows(ctx, s, T, r, d->f32));
    if (ly.ff > 0) {
      CK(products(m, w.xa, ld, T, jobs, ff_jobs(m, w, i, jobs)));
      DenseJob dj = down_job(m, w, i);
      CK(products(m, w.u, d->ldu, T, &dj, 1));
      r = residual(m, w, i, 2, true);
      r.x_in = w.x; r.x_out = w.x; r.act_out = act;
      CK(k_residual_rows(ctx, s, T, r, d->f32));
    }
    CK(copy_tap(m, i, w.x, T));
  }
  return normed_out != nullptr ? final_norm_rows(m, w.x, T, normed_out) : ORN_OK;
}

// ------------------------------------------------------------------ windows of 1..4 rows, fused
bool window_fits(const orn_model* m, int T) {
  const orn_decoder* d = m->dec;
  DecodePrologue p;
  p.mode = DRO_RESIDUAL;  // the other residual form stages as much
  p.K = d->spec.width;
  DecodePrologue q;
  q.K = std::max(d->ldu, d->ldatt);
  for (const LayerSpec& ly : d->spec.layers) {
    if (!ly.decays()) continue;
    DecodePrologue g;
    g.mode = DRO_GATED;
    g.K = ly.attends() ? ly.att.heads * ly.att.vdim : 0;
    g.gg.n = ly.lin.heads * ly.lin.vdim;
    g.gg.group = ly.lin_group;
    if (!decode_dense_fits(g, T)) return false;
  }
  return decode_dense_fits(p, T) && decode_dense_fits(q, T);
}

// One layer whose residual is normed after its sum: `p` ends the layer before and comes back as what ends this one.
int post_norm_window(orn_model* m, orn_cache* c, Scratch& w, int i, int T, bool capture, DecodePrologue* p) {
  orn_ctx* ctx = m->ctx;
  cudaStream_t s = ctx->stream;
  orn_decoder* d = m->dec;
  const LayerSpec& ly = d->spec.layers[i];
  const LayerW& W = d->w[i];
  DenseJob jobs[kInputJobs];
  CK(f_decode_dense(ctx, s, T, *p, jobs, input_jobs(m, w, i, jobs)));
  if (i > 0) CK(copy_tap(m, i - 1, w.x, T));
  const DecayedArgs la = decayed_args(m, c, w, i, T, capture);
  const bool lin_fast = decayed_window_ok(ly.lin, la);
  bool lin_done = false;
  if (ly.attends()) {
    const GroupedArgs ga = grouped_args(m, c, w, i, T);
    if (grouped_window_ok(ctx, ly.att, ga)) {
      CK(k_grouped_window(ctx, s, ly.att, ga, d->window_scratch, lin_fast ? &ly.lin : nullptr, lin_fast ? &la : nullptr));
      lin_done = lin_fast;
    } else {
      CK(attend_grouped(m, c, w, i, T));
    }
  }
  if (!lin_done) {
    if (lin_fast) CK(k_decayed_window(ctx, s, ly.lin, la));
    else CK(decay_rows(m, c, w, i, T, capture));
  }
  DecodePrologue g;
  g.mode = DRO_GATED;
  g.gg = lin_gate(m, w, i);
  int n = 0;
  if (ly.attends()) {
    g.K = ly.att.heads * ly.att.vdim;
    g.rows = reinterpret_cast<const bf16_t*>(w.att);
    g.ldx = d->ldatt;
    jobs[n++] = o_job(m, w, i);
  }
  jobs[n] = lin_o_job(m, w, i);
  jobs[n++].x0 = pad8(g.K);
  CK(f_decode_dense(ctx, s, T, g, jobs, n));
  *p = DecodePrologue();
  p->mode = DRO_POSTNORM; p->K = d->spec.width; p->pn = post_norm(m, w, i, 1); p->pn.x_in = w.x; p->x_out = w.xm;
  if (ly.ff > 0) {
    DenseJob uj;
    uj.lin = W.gate; uj.lin2 = W.up; uj.act.kind = ACT_GELU_TANH; uj.y = w.u; uj.ldy = d->ldu; uj.out_f32 = false;
    CK(f_decode_dense(ctx, s, T, *p, &uj, 1));
    DecodePrologue q;
    q.rows = reinterpret_cast<const bf16_t*>(w.u); q.ldx = d->ldu; q.K = ly.ff;
    DenseJob dj = down_job(m, w, i);
    CK(f_decode_dense(ctx, s, T, q, &dj, 1));
    p->pn = post_norm(m, w, i, 2); p->pn.x_in = w.xm; p->x_out = w.x;
  } else {
    std::swap(w.x, w.xm);  // the stream is always in w.x when a layer starts
  }
  return ORN_OK;
}

int window_forward(orn_model* m, orn_cache* c, Scratch& w, const uint32_t* dev_ids, int T, bool capture, void* normed_out, float* logits) {
  orn_ctx* ctx = m->ctx;
  cudaStream_t s = ctx->stream;
  orn_decoder* d = m->dec;
  const Spec& sp = d->spec;
  const int D = sp.width, ld = d->ldD, L = (int)sp.layers.size();
  DenseJob jobs[kInputJobs];
  DecodePrologue p;
  p.mode = DRO_EMBED; p.K = D; p.table = m->embed; p.ids = dev_ids; p.embed_scale = sp.embed_scale; p.x_out = w.x; p.stream_out = w.streams;
  auto rows_of = [&](const void* x, int ldx, int K) {
    DecodePrologue q;
    q.mode = DRO_ROWS; q.rows = reinterpret_cast<const bf16_t*>(x); q.ldx = ldx; q.K = K;
    return q;
  };
  for (int i = 0; i < L; ++i) {
    const LayerSpec& ly = sp.layers[i];
    if (sp.form == RES_POST_NORM) {
      CK(post_norm_window(m, c, w, i, T, capture, &p));
      continue;
    }
    std::swap(w.rg, w.rg_prev);  // p still reads the last gates
    CK(f_decode_dense(ctx, s, T, p, jobs, input_jobs(m, w, i, jobs)));
    if (i > 0) CK(copy_tap(m, i - 1, w.x, T));
    StreamSum sum;  // the streams up to this layer's input enter its average
    sum.n = i + 1; sum.a = d->w[i].dwa; sum.streams = w.streams; sum.stride = w.stream_stride; sum.out = w.part; sum.count = T * ld;
    CK(attend_absorbed(m, c, w, i, T, sum));
    DenseJob oj = o_job(m, w, i);
    CK(f_decode_dense(ctx, s, T, rows_of(w.att, d->ldatt, ly.mix.heads * ly.mix.vdim), &oj, 1));
    const float* x_in = w.x;
    if (ly.ff > 0) {
      p = DecodePrologue();
      p.mode = DRO_RESIDUAL; p.K = D; p.r = residual(m, w, i, 1, false); p.r.x_in = w.x; p.x_out = w.xm;
      std::swap(w.rg, w.rg_prev);
      CK(f_decode_dense(ctx, s, T, p, jobs, ff_jobs(m, w, i, jobs)));
      DenseJob dj = down_job(m, w, i);
      CK(f_decode_dense(ctx, s, T, rows_of(w.u, d->ldu, ly.ff), &dj, 1));
      x_in = w.xm;
    }
    // the layer's last add and its average are the prologue of what comes next
    p = DecodePrologue();
    p.mode = DRO_RESIDUAL; p.K = D; p.r = residual(m, w, i, ly.ff > 0 ? 2 : 1, true); p.r.x_in = x_in; p.part = w.part;
    p.x_out = x_in == w.x ? w.xm : w.x;
    p.stream_out = w.streams + (size_t)(i + 1) * w.stream_stride;
    if (p.x_out == w.xm) std::swap(w.x, w.xm);  // the stream is always in w.x when a layer starts
  }
  if (logits != nullptr) {
    p.w2 = d->final_norm;
    p.normed_out = reinterpret_cast<bf16_t*>(normed_out);
    DenseJob hj = head_job(m, logits);
    CK(f_decode_dense(ctx, s, T, p, &hj, 1));
  } else if (normed_out != nullptr || m->tap != nullptr) {  // rows without the head
    if (sp.form == RES_POST_NORM) {
      PostNormStep r = p.pn;
      r.x_out = p.x_out;
      CK(k_post_norm_rows(ctx, s, T, r, false));
    } else {
      ResidualStep r = p.r;
      r.x_out = p.x_out;
      CK(k_residual_rows(ctx, s, T, r, false));
    }
    if (normed_out != nullptr) CK(final_norm_rows(m, w.x, T, normed_out));
  }
  return copy_tap(m, L - 1, w.x, T);
}

int commit_rows(orn_cache* c, int T) { return orn_cache_commit(c, T, 1); }

int window(orn_model* m, orn_cache* c, const uint32_t* dev_ids, int T, bool capture, void* normed_out, float* logits) {
  orn_ctx* ctx = m->ctx;
  if (T < 1 || T > kMaxRows) ORN_FAIL(ctx, ORN_ERR_ARG, "forward: 1..4 rows per call");
  if (c->h_pos + T > m->cfg.max_ctx) ORN_FAIL(ctx, ORN_ERR_STATE, "forward: context exceeds max_ctx");
  orn_decoder* d = m->dec;
  if (!plain_route(m) && window_fits(m, T)) {
    CK(window_forward(m, c, d->win, dev_ids, T, capture, normed_out, logits));
  } else {
    void* rows = normed_out ? normed_out : d->win.normed;
    CK(rows_forward(m, c, d->win, dev_ids, T, capture, rows));
    if (logits) {
      DenseJob hj = head_job(m, logits);
      CK(products(m, rows, d->ldD, T, &hj, 1));
    }
  }
  if (capture) c->cap_T = T;
  else CK(commit_rows(c, T));
  return ORN_OK;
}

int decoder_forward(orn_model* m, orn_cache* c, const uint32_t* dev_ids, int T, bool capture, void* normed_out, void* pre_norm_out) {
  if (pre_norm_out != nullptr) ORN_FAIL(m->ctx, ORN_ERR_ARG, "forward: this architecture hands out rows after the final norm only");
  return window(m, c, dev_ids, T, capture, normed_out, nullptr);
}
int decoder_forward_greedy(orn_model* m, orn_cache* c, const uint32_t* dev_ids, int T, bool capture, void* normed_out, uint32_t* dev_tokens) {
  orn_decoder* d = m->dec;
  CK(window(m, c, dev_ids, T, capture, normed_out, d->logits));
  return k_greedy_f32(m->ctx, m->ctx->stream, d->logits, T, d->spec.vocab, dev_tokens, m->ws.greedy_scratch);
}

bool decoder_chunked(const orn_model*) { return true; }
int decoder_chunk(orn_model* m, orn_cache* c, const uint32_t* host_ids, int T, void* normed_out) {
  orn_ctx* ctx = m->ctx;
  orn_decoder* d = m->dec;
  if (c->h_pos + T > m->cfg.max_ctx) ORN_FAIL(ctx, ORN_ERR_STATE, "forward: context exceeds max_ctx");
  CK(reserve(m, d->wide, std::max(T, std::min(m->cfg.max_ctx, 256))));
  bool expand = false;
  for (size_t i = 0; i < d->spec.layers.size(); ++i) expand = expand || expand_layer(m, (int)i, T);
  if (expand) CK(reserve_expanded(m, c->h_pos + T));
  ORN_CHECK_CUDA(ctx, cudaMemcpyAsync(d->wide.ids, host_ids, sizeof(uint32_t) * (size_t)T, cudaMemcpyHostToDevice, ctx->stream));
  CK(rows_forward(m, c, d->wide, d->wide.ids, T, false, normed_out));
  return commit_rows(c, T);
}

int decoder_logits(orn_model* m, const void* rows, int T, float* dev_out) {
  DenseJob hj = head_job(m, dev_out);
  return products(m, rows, m->dec->ldD, T, &hj, 1);
}
int decoder_head_greedy(orn_model* m, const void* rows, int T, uint32_t* dev_tokens, void* dev_logits) {
  orn_decoder* d = m->dec;
  float* lg = dev_logits ? reinterpret_cast<float*>(dev_logits) : d->logits;
  DenseJob hj = head_job(m, lg);
  if (!plain_route(m) && window_fits(m, T)) {
    DecodePrologue p;
    p.mode = DRO_ROWS; p.rows = reinterpret_cast<const bf16_t*>(rows); p.ldx = d->ldD; p.K = d->spec.width;
    CK(f_decode_dense(m->ctx, m->ctx->stream, T, p, &hj, 1));
  } else {
    CK(products(m, rows, d->ldD, T, &hj, 1));
  }
  return k_greedy_f32(m->ctx, m->ctx->stream, lg, T, d->spec.vocab, dev_tokens, m->ws.greedy_scratch);
}
bool decoder_graphs(const orn_model* m) { return !plain_route(m) && m->tap == nullptr; }

}  // namespace

const orn_arch kArchPeratar = {
    "Peratar",          peratar_load,         peratar_create,        decoder_finalize,     decoder_init_random, decoder_release,
    decoder_cache_init, decoder_cache_reset,  decoder_cache_release, decoder_forward,      decoder_forward_greedy,
    kMaxRows + 1,       8192,                 decoder_chunked,       decoder_chunk,        decoder_logits,      decoder_head_greedy,
    decoder_graphs,
};
const orn_arch kArchDokulorn = {
    "Dokulorn",         dokulorn_load,        dokulorn_create,       decoder_finalize,     decoder_init_random, decoder_release,
    decoder_cache_init, decoder_cache_reset,  decoder_cache_release, decoder_forward,      decoder_forward_greedy,
    kMaxRows + 1,       8192,                 decoder_chunked,       decoder_chunk,        decoder_logits,      decoder_head_greedy,
    decoder_graphs,
};
