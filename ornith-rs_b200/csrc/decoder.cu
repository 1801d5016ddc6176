// The Peratar decoder: latent attention and dense feed-forwards around a float32 residual stream.
//
//   y = mixer(x) or ff(x)              a sublayer reads the stream itself
//   x <- x + norm(y * sigmoid(W x + b))   its result is gated from the same input, then normed
//   X_(i+1) = the stream after layer i;  what goes on is sum_j a_ij X_j over all of them so far
//   logits = cap * tanh(head(norm(x)) / cap)
//
// Three routes through the same layers, equal to rounding:
//   * windows of 1..4 rows (decoding): seven kernels a layer (dense.cu, latent.cu), programmatic
//     dependents, capturable into CUDA graphs: every position-dependent size is read on the device;
//   * prompt chunks: tensor-core products with bias and activation in their epilogue, absorbed
//     attention for short chunks, expanded attention for long ones, one row kernel per sublayer;
//   * the control route, one plain kernel per operation: models loaded in float32, and ORN_UNFUSED=1.
#include <algorithm>
#include <cmath>
#include <cstring>
#include <memory>
#include <string>
#include <vector>

#include "arch.h"
#include "dense.h"
#include "fused.h"
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
struct LayerSpec {
  LatentDims mix;
  double rot_base = 1.0;
  int kv_from = -1;  // the layer whose cache this one reads, -1: its own
  int ff = 0;        // 0: no feed-forward
};
struct Spec {
  int width = 0, vocab = 0;
  float eps = 0.f, softcap = 0.f;
  std::vector<LayerSpec> layers;
};
struct LayerW {
  orn_linear *q = nullptr, *dkv = nullptr, *uk = nullptr, *uv = nullptr, *g = nullptr, *o = nullptr;
  orn_linear *rg1 = nullptr, *rg2 = nullptr, *up = nullptr, *down = nullptr;
  bf16_t *norm1 = nullptr, *norm2 = nullptr, *dkv_norm = nullptr, *rg1_b = nullptr, *rg2_b = nullptr;
  bf16_t *up_b = nullptr, *down_b = nullptr, *act = nullptr, *dwa = nullptr;
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
  size_t stream_stride = 0;
};
}  // namespace

struct orn_decoder {
  Spec spec;
  std::vector<LayerW> w;
  bf16_t* final_norm = nullptr;
  orn_linear* head = nullptr;
  std::vector<float*> freq;  // per layer
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
bool is_null(const JVal* v) { return v == nullptr || v->type == JVal::Null; }

Spec parse_spec(const JVal& c) {
  Spec s;
  s.width = need_int(&c, "width", "config", 1);
  s.vocab = need_int(&c, "vocab", "config", 1);
  s.eps = (float)need_num(c.get("norm"), "eps", "norm");
  if (!is_null(c.get("logit_softcap"))) s.softcap = (float)need_num(&c, "logit_softcap", "config");
  const JVal* ls = c.get("layers");
  if (!ls || ls->type != JVal::Arr || ls->arr.empty()) throw FieldError{"layers is missing or empty"};
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
    const JVal* f = l.get("mlp");
    if (!is_null(f)) {
      const JVal* k = f->get("kind");
      if (!k || k->str != "dense") throw FieldError{at + ".mlp.kind is not a feed-forward of this architecture"};
      L.ff = need_int(f, "ff", at + ".mlp", 1);
    }
    s.layers.push_back(L);
  }
  return s;
}

// Every weight by name and shape; K == 0: a vector of O entries.
struct WeightDesc {
  std::string name;
  int O, K;
};
std::vector<WeightDesc> weight_table(const Spec& s) {
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
int peratar_create(orn_ctx* ctx, const JVal& cfg, int max_ctx, int dtype, orn_model** out) {
  if (dtype != ORN_DT_BF16 && dtype != ORN_DT_F32) ORN_FAIL(ctx, ORN_ERR_ARG, "model: unknown data type");
  if (max_ctx < 1) ORN_FAIL(ctx, ORN_ERR_ARG, "model: max_ctx must be positive");
  std::unique_ptr<orn_decoder> d(new orn_decoder());
  try {
    d->spec = parse_spec(cfg);
  } catch (const FieldError& e) {
    ORN_FAIL(ctx, ORN_ERR_ARG, "config.json: " + e.what);
  }
  d->f32 = dtype == ORN_DT_F32;
  orn_model* m = new orn_model();
  m->ctx = ctx;
  m->arch = &kArchPeratar;
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

int peratar_load(orn_ctx* ctx, const std::string& dir, const JVal& cfg, int max_ctx, int dtype, orn_model** out) {
  Store st;
  std::string err;
  if (!open_shards(dir, &st, &err)) ORN_FAIL(ctx, ORN_ERR_IO, err);
  orn_model* m = nullptr;
  CK(peratar_create(ctx, cfg, max_ctx, dtype, &m));
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

uint64_t mix64(uint64_t x) {
  x += 0x9e3779b97f4a7c15ull;
  x = (x ^ (x >> 30)) * 0xbf58476d1ce4e5b9ull;
  x = (x ^ (x >> 27)) * 0x94d049bb133111ebull;
  return x ^ (x >> 31);
}

// seeded synthetic weights: matrices ~ 1 / sqrt(K), norms near 1, each average mostly its newest stream
int peratar_init_random(orn_model* m, uint64_t seed) {
  orn_ctx* ctx = m->ctx;
  uint64_t n = 0;
  for (const WeightDesc& w : weight_table(m->dec->spec)) {
    const uint64_t sd = mix64(seed + (++n));
    if (w.K) {
      if (w.K % 8) ORN_FAIL(ctx, ORN_ERR_ARG, "init_random: row lengths must be multiples of 8");
      orn_linear* L = nullptr;
      const float std = w.name == "embed" ? 1.0f : 1.0f / std::sqrt((float)w.K);
      CK(orn_linear_create_random(ctx, ORN_BF16, 1, w.O, w.K, sd, std, &L));
      CK(orn_model_set_linear(m, w.name.c_str(), L));
    } else {
      const bool norm = w.name.find("norm") != std::string::npos;
      const bool dwa = ends_with(w.name, ".dwa");
      void* d = nullptr;
      CK(orn_alloc(ctx, (size_t)w.O * 2, &d));
      int rc = k_fill_bf16(ctx, ctx->stream, (bf16_t*)d, w.O, sd, norm ? 1.0f : 0.0f, norm ? 0.05f : dwa ? 0.1f : 0.3f);
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
  return !plain_route(m) && T > kAbsorbMaxRows && latent_flash_ok(d->spec.layers[i].mix, d->ldq);
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
  w.stream_stride = R * D;
  take(&w.ids, R * 4);
  take(&w.streams, (L + 1) * w.stream_stride * 4);
  take(&w.x, R * D * 4); take(&w.xm, R * D * 4); take(&w.part, R * D * 4); take(&w.y, R * D * 4); take(&w.rg, R * D * 4); take(&w.rg_prev, R * D * 4);
  take(&w.kv, R * d->ldkv * 4); take(&w.g, R * d->ldg * 4);
  take(&w.q, R * d->ldq * A); take(&w.att, R * d->ldatt * A); take(&w.u, R * d->ldu * A); take(&w.normed, R * D * A);
  if (d->f32) w.xa = reinterpret_cast<uint8_t*>(w.x);
  else take(&w.xa, R * D * A);
  // absorbed attention: queries, partial sums
  size_t qa = 0, part = 0, ml = 0;
  for (size_t i = 0; i < L; ++i) {
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

int peratar_finalize(orn_model* m) {
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
  m->lm_head = d->head = lin("head");
  d->final_norm = ten("final.norm");
  d->w.assign(s.layers.size(), LayerW());
  for (float* p : d->freq) cudaFree(p);
  d->freq.clear();
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
    LatentDims& M = L.mix;
    d->ldq = std::max(d->ldq, pad8(M.heads * M.qk()));
    d->ldkv = std::max(d->ldkv, pad8(M.kv_rank + M.rot_dim));
    d->ldg = std::max(d->ldg, pad8(M.heads));
    d->ldatt = std::max(d->ldatt, pad8(M.heads * M.vdim));
    d->ldu = std::max(d->ldu, pad8(L.ff));
    d->ldkx = std::max(d->ldkx, pad8(M.heads * M.dim));
    d->ldvx = std::max(d->ldvx, pad8(M.heads * M.vdim));
    std::vector<float> f(std::max(1, M.rot_dims / 2));
    for (int e = 0; e < M.rot_dims / 2; ++e) f[e] = (float)std::pow(L.rot_base, -2.0 * e / M.rot_dims);
    float* df = nullptr;
    CK(orn_alloc(ctx, f.size() * 4, (void**)&df));
    d->freq.push_back(df);
    CK(orn_upload(ctx, df, f.data(), f.size() * 4));
    M.freq = df;
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
  CK(reserve(m, d->win, kMaxRows));
  for (int i = 0; i < 4; ++i) ORN_CHECK_CUDA(ctx, cudaEventCreate(&m->ev[i]));
  m->finalized = true;
  return ORN_OK;
}

void peratar_release(orn_model* m) {
  orn_decoder* d = m->dec;
  if (!d) return;
  release_scratch(d->win);
  release_scratch(d->wide);
  for (float* p : d->freq) cudaFree(p);
  cudaFree(d->kx);
  cudaFree(d->vx);
  delete d;
  m->dec = nullptr;
}

// ------------------------------------------------------------------ cache: one row per position and owning layer
int peratar_cache_init(orn_cache* c) {
  orn_model* m = c->m;
  const Spec& s = m->dec->spec;
  c->latent.assign(s.layers.size(), nullptr);
  for (size_t i = 0; i < s.layers.size(); ++i) {
    if (s.layers[i].kv_from >= 0) continue;
    const size_t bytes = (size_t)m->cfg.max_ctx * s.layers[i].mix.row() * act_bytes(m->dec);
    CK(orn_alloc(m->ctx, bytes, &c->latent[i]));
    CK(orn_memset(m->ctx, c->latent[i], 0, bytes));
  }
  for (size_t i = 0; i < s.layers.size(); ++i)
    if (s.layers[i].kv_from >= 0) c->latent[i] = c->latent[s.layers[i].kv_from];
  return ORN_OK;
}
int peratar_cache_reset(orn_cache*) { return ORN_OK; }  // rows beyond the position are never read
void peratar_cache_release(orn_cache* c) {
  const Spec& s = c->m->dec->spec;
  for (size_t i = 0; i < c->latent.size(); ++i)
    if (s.layers[i].kv_from < 0) cudaFree(c->latent[i]);
  c->latent.clear();
}

// ------------------------------------------------------------------ products
// y_j = act(x W_j^T + b) of up to four matrices over the same rows
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
  const orn_linear* Ls[4];
  void* ys[4];
  int ldys[4];
  QGemmEpi epi[4];
  for (int j = 0; j < n; ++j) {
    Ls[j] = jobs[j].lin; ys[j] = jobs[j].y; ldys[j] = jobs[j].ldy;
    epi[j].bias = jobs[j].bias; epi[j].act = jobs[j].act; epi[j].out_f32 = jobs[j].out_f32;
  }
  return f_qgemm_multi(ctx, ctx->stream, Ls, ys, ldys, n, reinterpret_cast<const bf16_t*>(x), T, nullptr, nullptr, 0, 0, epi, ldx);
}

// the products that read a layer's input, into the scratch; returns how many
int input_jobs(orn_model* m, Scratch& w, int i, DenseJob* j) {
  orn_decoder* d = m->dec;
  const LayerW& W = d->w[i];
  int n = 0;
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

// ------------------------------------------------------------------ rows route (prompt chunks, control path)
int rows_forward(orn_model* m, orn_cache* c, Scratch& w, const uint32_t* dev_ids, int T, void* normed_out) {
  orn_ctx* ctx = m->ctx;
  cudaStream_t s = ctx->stream;
  orn_decoder* d = m->dec;
  const Spec& sp = d->spec;
  const int D = sp.width, ld = d->ldD, L = (int)sp.layers.size();
  void* act = d->f32 ? nullptr : w.xa;  // float32: the stream is its own activation
  CK(k_embed_rows(ctx, s, m->embed, dev_ids, T, D, ld, w.x, w.streams, act, d->f32));
  DenseJob jobs[4];
  for (int i = 0; i < L; ++i) {
    const LayerSpec& ly = sp.layers[i];
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
  if (normed_out != nullptr) CK(k_layer_norm_rows(ctx, s, w.x, T, D, ld, d->final_norm, sp.eps, normed_out, d->f32));
  return ORN_OK;
}

// ------------------------------------------------------------------ windows of 1..4 rows, fused
bool window_fits(const orn_model* m, int T) {
  const orn_decoder* d = m->dec;
  DecodePrologue p;
  p.mode = DRO_RESIDUAL;
  p.K = d->spec.width;
  DecodePrologue q;
  q.K = std::max(d->ldu, d->ldatt);
  return decode_dense_fits(p, T) && decode_dense_fits(q, T);
}

int window_forward(orn_model* m, orn_cache* c, Scratch& w, const uint32_t* dev_ids, int T, void* normed_out, float* logits) {
  orn_ctx* ctx = m->ctx;
  cudaStream_t s = ctx->stream;
  orn_decoder* d = m->dec;
  const Spec& sp = d->spec;
  const int D = sp.width, ld = d->ldD, L = (int)sp.layers.size();
  DenseJob jobs[4];
  DecodePrologue p;
  p.mode = DRO_EMBED; p.K = D; p.table = m->embed; p.ids = dev_ids; p.x_out = w.x; p.stream_out = w.streams;
  auto rows_of = [&](const void* x, int ldx, int K) {
    DecodePrologue q;
    q.mode = DRO_ROWS; q.rows = reinterpret_cast<const bf16_t*>(x); q.ldx = ldx; q.K = K;
    return q;
  };
  for (int i = 0; i < L; ++i) {
    const LayerSpec& ly = sp.layers[i];
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
    ResidualStep r = p.r;
    r.x_out = p.x_out;
    CK(k_residual_rows(ctx, s, T, r, false));
    if (normed_out != nullptr) CK(k_layer_norm_rows(ctx, s, w.x, T, D, ld, d->final_norm, sp.eps, normed_out, false));
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
    CK(window_forward(m, c, d->win, dev_ids, T, normed_out, logits));
  } else {
    void* rows = normed_out ? normed_out : d->win.normed;
    CK(rows_forward(m, c, d->win, dev_ids, T, rows));
    if (logits) {
      DenseJob hj = head_job(m, logits);
      CK(products(m, rows, d->ldD, T, &hj, 1));
    }
  }
  if (capture) c->cap_T = T;
  else CK(commit_rows(c, T));
  return ORN_OK;
}

int peratar_forward(orn_model* m, orn_cache* c, const uint32_t* dev_ids, int T, bool capture, void* normed_out, void* pre_norm_out) {
  if (pre_norm_out != nullptr) ORN_FAIL(m->ctx, ORN_ERR_ARG, "forward: this architecture hands out rows after the final norm only");
  return window(m, c, dev_ids, T, capture, normed_out, nullptr);
}
int peratar_forward_greedy(orn_model* m, orn_cache* c, const uint32_t* dev_ids, int T, bool capture, void* normed_out, uint32_t* dev_tokens) {
  orn_decoder* d = m->dec;
  CK(window(m, c, dev_ids, T, capture, normed_out, d->logits));
  return k_greedy_f32(m->ctx, m->ctx->stream, d->logits, T, d->spec.vocab, dev_tokens, m->ws.greedy_scratch);
}

bool peratar_chunked(const orn_model*) { return true; }
int peratar_chunk(orn_model* m, orn_cache* c, const uint32_t* host_ids, int T, void* normed_out) {
  orn_ctx* ctx = m->ctx;
  orn_decoder* d = m->dec;
  if (c->h_pos + T > m->cfg.max_ctx) ORN_FAIL(ctx, ORN_ERR_STATE, "forward: context exceeds max_ctx");
  CK(reserve(m, d->wide, std::max(T, std::min(m->cfg.max_ctx, 256))));
  bool expand = false;
  for (size_t i = 0; i < d->spec.layers.size(); ++i) expand = expand || expand_layer(m, (int)i, T);
  if (expand) CK(reserve_expanded(m, c->h_pos + T));
  ORN_CHECK_CUDA(ctx, cudaMemcpyAsync(d->wide.ids, host_ids, sizeof(uint32_t) * (size_t)T, cudaMemcpyHostToDevice, ctx->stream));
  CK(rows_forward(m, c, d->wide, d->wide.ids, T, normed_out));
  return commit_rows(c, T);
}

int peratar_logits(orn_model* m, const void* rows, int T, float* dev_out) {
  DenseJob hj = head_job(m, dev_out);
  return products(m, rows, m->dec->ldD, T, &hj, 1);
}
int peratar_head_greedy(orn_model* m, const void* rows, int T, uint32_t* dev_tokens, void* dev_logits) {
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
bool peratar_graphs(const orn_model* m) { return !plain_route(m) && m->tap == nullptr; }

}  // namespace

const orn_arch kArchPeratar = {
    "Peratar",          peratar_load,         peratar_create,      peratar_finalize,       peratar_init_random, peratar_release,
    peratar_cache_init, peratar_cache_reset,  peratar_cache_release, peratar_forward,      peratar_forward_greedy,
    kMaxRows + 1,       8192,                 peratar_chunked,     peratar_chunk,          peratar_logits,      peratar_head_greedy,
    peratar_graphs,
};
