// The model registry: one entry per architecture, and what the generic entry points (loading,
// caches, prompt, windows, greedy generation, logits) call on it.  orn_model_load reads config.json
// once, finds the entry by it and hands the rest over.
#pragma once

#include "artifact.h"
#include "orn_internal.h"

struct orn_arch {
  const char* name;
  // config.json + safetensors in `dir` -> model
  int (*load)(orn_ctx* ctx, const std::string& dir, const orna::JVal& cfg, int max_ctx, int dtype, orn_model** out);
  // nullable: a model of this configuration without weights
  int (*create)(orn_ctx* ctx, const orna::JVal& cfg, int max_ctx, int dtype, orn_model** out);
  int (*finalize)(orn_model* m);  // resolve every weight the forward pass needs, build the scratch (idempotent)
  int (*init_random)(orn_model* m, uint64_t seed);
  void (*release)(orn_model* m);  // what finalize and create added besides lins, tensors and ws_allocs
  int (*cache_init)(orn_cache* c);
  int (*cache_reset)(orn_cache* c);
  void (*cache_release)(orn_cache* c);
  // 1..kMaxRows rows whose ids are on the device; capture: the caller commits (orn_cache_rewind)
  int (*forward)(orn_model* m, orn_cache* c, const uint32_t* dev_ids, int T, bool capture, void* normed_out, void* pre_norm_out);
  int (*forward_greedy)(orn_model* m, orn_cache* c, const uint32_t* dev_ids, int T, bool capture, void* normed_out,
                        uint32_t* dev_tokens);
  // one prompt chunk of chunk_min..chunk_max rows, committed; normed_out (nullable): rows after the final norm
  int chunk_min, chunk_max;
  bool (*chunked)(const orn_model* m);  // whether prompts go through `chunk` at all
  int (*chunk)(orn_model* m, orn_cache* c, const uint32_t* host_ids, int T, void* normed_out);
  // float32 logits of T normed rows
  int (*logits)(orn_model* m, const void* rows, int T, float* dev_out);
  // greedy tokens of T <= kMaxRows normed rows; dev_logits (nullable) in the architecture's logit type
  int (*head_greedy)(orn_model* m, const void* rows, int T, uint32_t* dev_tokens, void* dev_logits);
  bool (*graphs)(const orn_model* m);  // the window steps may be captured into CUDA graphs
};

const orn_arch* orn_arch_of_config(const orna::JVal& cfg);

// loader.cu
int qwen35_load(orn_ctx* ctx, const std::string& dir, const orna::JVal& cfg, int max_ctx, int dtype, orn_model** out);
// decoder.cu
extern const orn_arch kArchPeratar;
extern const orn_arch kArchDokulorn;
