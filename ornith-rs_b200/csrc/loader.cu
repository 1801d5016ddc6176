// Artifact loader: config.json + safetensors shards -> orn_model.
//
// Follows src/safetensors.rs:189-308 (8-byte little-endian header length, JSON
// header, raw tensor bytes; shards listed by model.safetensors.index.json),
// src/weights.rs:41-279 (per-module quantisation from config.json, the
// three-tensor k-quant modules `.weight/.scales/.dm`, affine modules
// `.weight/.scales/.biases`, numbered MTP experts stacked at load) and
// src/model/config.rs:44-158 (text_config fields).
#include "artifact.h"
#include "arch.h"
#include "model_types.h"
#include "orn_internal.h"

using namespace orna;

namespace {

// per-module quantisation of config.json (src/weights.rs:41-98): a default {group_size, bits, mode}
// and overrides keyed by module path
struct QSpec {
  int group = 0, bits = 0;
  std::string mode;  // "affine", "q4k", "q6k", "nvfp4", ...
  bool present = false;
};

}  // namespace

// the Qwen3.5-MoE artifact (the registry's entry for config.json without an "architecture" of ours)
int qwen35_load(orn_ctx* ctx, const std::string& dir, const JVal& cfgj, int max_ctx, int dtype, orn_model** out) {
  if (dtype != ORN_DT_BF16) ORN_FAIL(ctx, ORN_ERR_ARG, "this architecture runs in bfloat16 only");
  const JVal* t = cfgj.get("text_config");
  if (!t) t = &cfgj;
  bool missing = false;
  std::string missing_key;
  auto u = [&](const char* k) -> int {
    const JVal* v = t->get(k);
    if (!v || v->type != JVal::Num) { if (!missing) missing_key = k; missing = true; return 0; }
    return (int)v->num;
  };
  auto f = [&](const char* k, float d) -> float {
    const JVal* v = t->get(k);
    return (v && v->type == JVal::Num) ? (float)v->num : d;
  };
  orn_config c{};
  c.hidden = u("hidden_size");
  c.n_layers = u("num_hidden_layers");
  c.n_heads = u("num_attention_heads");
  c.n_kv_heads = u("num_key_value_heads");
  { const JVal* v = t->get("head_dim"); c.head_dim = v ? (int)v->num : (c.n_heads ? c.hidden / c.n_heads : 0); }
  { const JVal* v = t->get("full_attention_interval"); c.full_attn_interval = v ? (int)v->num : 4; }
  const JVal* rope = t->get("rope_parameters");
  float theta = f("rope_theta", 100000.0f), prf = f("partial_rotary_factor", 0.25f);
  if (rope) {
    if (const JVal* v = rope->get("rope_theta")) theta = (float)v->num;
    if (const JVal* v = rope->get("partial_rotary_factor")) prf = (float)v->num;
  }
  c.rope_theta = theta;
  c.rope_dims = (int)((float)c.head_dim * prf);
  c.gdn_k_heads = u("linear_num_key_heads");
  c.gdn_v_heads = u("linear_num_value_heads");
  c.gdn_head_dim = u("linear_key_head_dim");
  c.gdn_conv_kernel = u("linear_conv_kernel_dim");
  c.n_experts = u("num_experts");
  c.top_k = u("num_experts_per_tok");
  c.expert_inter = u("moe_intermediate_size");
  c.shared_inter = u("shared_expert_intermediate_size");
  { const JVal* v = t->get("norm_topk_prob"); c.norm_topk_prob = (!v || v->type != JVal::Bool) ? 1 : (v->b ? 1 : 0); }
  c.vocab = u("vocab_size");
  c.rms_eps = f("rms_norm_eps", 1e-6f);
  c.max_ctx = max_ctx;
  if (missing) ORN_FAIL(ctx, ORN_ERR_IO, "config.json: missing " + missing_key);
  if (u("linear_value_head_dim") != c.gdn_head_dim) ORN_FAIL(ctx, ORN_ERR_ARG, "config.json: key and value head dims differ");

  // ---- quantization block (src/weights.rs:49-79); absent in hand-made artifacts: formats then follow the tensors
  QSpec qdef;
  std::map<std::string, QSpec> qmods;
  if (const JVal* q = cfgj.get("quantization")) {
    if (q->type != JVal::Obj) ORN_FAIL(ctx, ORN_ERR_IO, "config.json: quantization is not an object");
    const JVal* g = q->get("group_size");
    const JVal* b = q->get("bits");
    if (!g || !b || g->type != JVal::Num || b->type != JVal::Num) ORN_FAIL(ctx, ORN_ERR_IO, "config.json: quantization.group_size / bits");
    qdef.group = (int)g->num; qdef.bits = (int)b->num; qdef.present = true;
    const JVal* md = q->get("mode");
    qdef.mode = (md && md->type == JVal::Str) ? md->str : "affine";  // older artifacts carry no mode (weights.rs:52-53)
    for (auto& kv : q->obj) {
      if (kv.second.type != JVal::Obj) continue;
      QSpec sp = qdef;
      if (const JVal* v = kv.second.get("group_size")) sp.group = (int)v->num;
      if (const JVal* v = kv.second.get("bits")) sp.bits = (int)v->num;
      if (const JVal* v = kv.second.get("mode")) if (v->type == JVal::Str) sp.mode = v->str;
      qmods[kv.first] = sp;
    }
  }
  auto spec_of = [&](const std::string& mod) -> QSpec {
    auto it = qmods.find(mod);
    return it == qmods.end() ? qdef : it->second;
  };

  // ---- shards (src/safetensors.rs:296-308) and the MTP sidecar (mtp.rs:270-279)
  Store st;
  std::string err;
  if (!open_shards(dir, &st, &err)) ORN_FAIL(ctx, ORN_ERR_IO, err);
  {
    std::string rel = "mtp/weights.safetensors";
    if (const JVal* x = cfgj.get("mlx_lm_extra_tensors"))
      if (const JVal* mf = x->get("mtp_file")) rel = mf->str;
    struct stat sb;
    if (stat((dir + "/" + rel).c_str(), &sb) == 0)
      if (!open_shard(dir + "/" + rel, &st, &err)) ORN_FAIL(ctx, ORN_ERR_IO, err);
  }

  orn_model* m = nullptr;
  int rc = orn_model_create(ctx, &c, &m);
  if (rc != ORN_OK) return rc;
  auto fail = [&](int code, const std::string& msg) {
    orn_model_destroy(m);
    ctx->err = msg;
    return code;
  };

  // ---- classify and upload
  const std::string mtp_moe = "mtp.layers.0.mlp.";
  const std::string mtp_exp = "mtp.layers.0.mlp.experts.";
  std::map<std::string, bool> stacked_done;
  for (auto& kv : st.tensors) {
    const std::string& name = kv.first;
    const TInfo& ti = kv.second;
    if (ends_with(name, ".scales") || ends_with(name, ".biases") || ends_with(name, ".dm")) continue;
    if (name.find("visual") != std::string::npos || name.find("vision") != std::string::npos) continue;
    // numbered MTP experts: stack 0..E-1 into one [E, O, K] bf16 matrix (weights.rs:237-279)
    if (name.rfind(mtp_exp, 0) == 0) {
      size_t dot = name.find('.', mtp_exp.size());
      if (dot == std::string::npos) continue;
      std::string proj = name.substr(dot + 1);  // gate_proj.weight
      if (stacked_done[proj]) continue;
      stacked_done[proj] = true;
      if (ti.dtype != "BF16" || ti.shape.size() != 2 || !bytes_match(ti, 2))
        return fail(ORN_ERR_ARG, "mtp expert tensor is not 2-D bf16 of its declared size: " + name);
      const int O = (int)ti.shape[0], K = (int)ti.shape[1];
      std::vector<uint8_t> buf((size_t)c.n_experts * O * K * 2);
      for (int e = 0; e < c.n_experts; ++e) {
        auto it = st.tensors.find(mtp_exp + std::to_string(e) + "." + proj);
        if (it == st.tensors.end() || it->second.nbytes != (size_t)O * K * 2)
          return fail(ORN_ERR_IO, "missing MTP expert " + std::to_string(e) + " " + proj);
        memcpy(buf.data() + (size_t)e * O * K * 2, it->second.data, (size_t)O * K * 2);
      }
      orn_linear* L = nullptr;
      rc = orn_linear_create(ctx, ORN_BF16, c.n_experts, O, K, buf.data(), nullptr, nullptr, &L);
      if (rc != ORN_OK) { orn_model_destroy(m); return rc; }
      std::string mod = proj.substr(0, proj.size() - strlen(".weight"));
      orn_model_set_linear(m, (mtp_moe + "switch_mlp." + mod).c_str(), L);
      continue;
    }
    if (ends_with(name, ".weight")) {
      const std::string mod = name.substr(0, name.size() - strlen(".weight"));
      auto sc = st.tensors.find(mod + ".scales");
      if (sc != st.tensors.end()) {
        auto dmq = st.tensors.find(mod + ".dm");
        auto bia = st.tensors.find(mod + ".biases");
        int kind;
        const TInfo* third;
        // leading expert axis, then [O, packed K]
        if (ti.shape.size() < 2 || sc->second.shape.empty()) return fail(ORN_ERR_ARG, "quantised weight is not a matrix: " + name);
        const int E = ti.shape.size() == 3 ? (int)ti.shape[0] : 1;
        const int O = (int)ti.shape[ti.shape.size() - 2];
        const int64_t packed = ti.shape.back();  // u32 words per row
        const int64_t scols = sc->second.shape.back();
        if (packed <= 0 || scols <= 0 || O <= 0 || E <= 0) return fail(ORN_ERR_ARG, "empty quantised tensor: " + mod);
        const QSpec sp = spec_of(mod);
        int K;
        const bool as_kquant = sp.present ? (sp.mode == "q4k" || sp.mode == "q6k") : dmq != st.tensors.end();
        if (sp.present && sp.mode != "affine" && !as_kquant)
          return fail(ORN_ERR_ARG, "quantization mode '" + sp.mode + "' is not on this path: " + mod);
        if (as_kquant) {
          // kquant_matrix (src/weights.rs:199-227): .weight/.scales/.dm, never .biases, super-blocks of 256
          if (dmq == st.tensors.end() || bia != st.tensors.end())
            return fail(ORN_ERR_ARG, "k-quant module must carry .dm and no .biases: " + mod);
          if (sp.present && sp.group != 256) return fail(ORN_ERR_ARG, "k-quant group_size must be 256: " + mod);
          third = &dmq->second;
          if (third->shape.empty()) return fail(ORN_ERR_ARG, "k-quant .dm has no shape: " + mod);
          const int64_t last = third->shape.back();
          const bool q4 = sp.present ? sp.mode == "q4k" : last == 2;
          if (q4 && last == 2) { kind = ORN_Q4K; K = (int)(packed * 8); }
          else if (!q4 && last == 1) { kind = ORN_Q6K; K = (int)(packed * 16 / 3); }
          else return fail(ORN_ERR_ARG, "k-quant .dm width does not match the module's mode: " + mod);
        } else {
          // quant_matrix (src/weights.rs:132-172): mlx affine, bits and group size from config.json
          if (bia == st.tensors.end() || dmq != st.tensors.end())
            return fail(ORN_ERR_ARG, "affine module must carry .biases and no .dm: " + mod);
          third = &bia->second;
          int bits = sp.bits, group = sp.group;
          if (!sp.present) {  // no quantization block: the 8-bit group-64 layout is the only one that can be assumed
            bits = 8; group = 64;
          }
          if (bits == 8 && group == 64) kind = ORN_A8;
          else if (bits == 4 && group == 32) kind = ORN_A4;
          else return fail(ORN_ERR_ARG, "affine module is neither 8-bit group-64 nor 4-bit group-32 (unsupported on this path): " + mod);
          K = (int)(packed * 32 / bits);
          if (scols * group != K) return fail(ORN_ERR_ARG, "affine module's scales do not match its bits and group size: " + mod);
        }
        size_t aw, as, ab;
        linear_artifact_sizes(kind, E, O, K, &aw, &as, &ab);
        if (ti.nbytes != aw || sc->second.nbytes != as || third->nbytes != ab)
          return fail(ORN_ERR_ARG, "tensor sizes do not match the declared shapes: " + mod);
        orn_linear* L = nullptr;
        rc = orn_linear_create(ctx, kind, E, O, K, ti.data, sc->second.data, third->data, &L);
        if (rc != ORN_OK) { orn_model_destroy(m); return rc; }
        orn_model_set_linear(m, mod.c_str(), L);
        continue;
      }
      if (ti.dtype == "BF16" && ti.shape.size() == 2) {
        if (!bytes_match(ti, 2)) return fail(ORN_ERR_ARG, "tensor bytes do not match its shape: " + name);
        orn_linear* L = nullptr;
        rc = orn_linear_create(ctx, ORN_BF16, 1, (int)ti.shape[0], (int)ti.shape[1], ti.data, nullptr, nullptr, &L);
        if (rc != ORN_OK) { orn_model_destroy(m); return rc; }
        // the MTP head's MoE matrices are addressed by module name
        std::string reg = (name.rfind(mtp_moe, 0) == 0) ? mod : name;
        orn_model_set_linear(m, reg.c_str(), L);
        continue;
      }
    }
    if (ti.dtype == "BF16") {
      if (!bytes_match(ti, 2)) return fail(ORN_ERR_ARG, "tensor bytes do not match its shape: " + name);
      rc = orn_model_set_tensor(m, name.c_str(), (const uint16_t*)ti.data, (size_t)numel(ti));
      if (rc != ORN_OK) { orn_model_destroy(m); return rc; }
    }
    // other dtypes (e.g. vision tensors in float) are not on this path
  }
  *out = m;
  return ORN_OK;
}

// config.json names the architecture; its registry entry reads the rest (src/model/config.rs:44-158
// and src/weights.rs:41-279 for the reference's own)
extern "C" int32_t orn_model_load_as(orn_ctx* ctx, const char* dir_c, int32_t max_ctx, int32_t dtype, orn_model** out) {
  if (!ctx || !dir_c || !out) return ORN_ERR_ARG;
  *out = nullptr;
  const std::string dir(dir_c);
  std::string raw;
  if (!read_file(dir + "/config.json", &raw)) ORN_FAIL(ctx, ORN_ERR_IO, "config.json: cannot read");
  JVal cfgj;
  if (!parse_json(raw.data(), raw.size(), &cfgj)) ORN_FAIL(ctx, ORN_ERR_IO, "config.json: parse error");
  const orn_arch* arch = orn_arch_of_config(cfgj);
  if (arch == nullptr) ORN_FAIL(ctx, ORN_ERR_ARG, "config.json: unknown architecture");
  return arch->load(ctx, dir, cfgj, max_ctx, dtype, out);
}

extern "C" int32_t orn_model_load(orn_ctx* ctx, const char* dir, int32_t max_ctx, orn_model** out) {
  return orn_model_load_as(ctx, dir, max_ctx, ORN_DT_BF16, out);
}

// a model from its configuration alone: weights follow by orn_model_init_random or one by one
extern "C" int32_t orn_model_create_json(orn_ctx* ctx, const char* json, int32_t max_ctx, int32_t dtype, orn_model** out) {
  if (!ctx || !json || !out) return ORN_ERR_ARG;
  *out = nullptr;
  JVal cfgj;
  if (!parse_json(json, strlen(json), &cfgj)) ORN_FAIL(ctx, ORN_ERR_ARG, "model configuration: parse error");
  const orn_arch* arch = orn_arch_of_config(cfgj);
  if (arch == nullptr || arch->create == nullptr)
    ORN_FAIL(ctx, ORN_ERR_ARG, "model configuration: unknown architecture (or one that orn_model_create builds)");
  return arch->create(ctx, cfgj, max_ctx, dtype, out);
}
