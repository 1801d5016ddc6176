// Launchers of grouped-query softmax attention with unit-norm queries and keys, a capped score, a sink
// per head and an element-wise output gate (grouped.cu).
#pragma once

#include "decayed.h"

struct GroupedDims {
  int heads = 0, kv_heads = 0, dim = 0, vdim = 0;
  int rot_dims = 0;              // entries (i, i + rot_dims / 2) of q and k turn by position * freq[i]
  const double* freq = nullptr;  // device [rot_dims / 2]
  bool unit_qk = true;           // after turning, q and k over their root mean square
  float eps = 0.f;               // of that
  float scale = 1.f;
  float softcap = 0.f;           // score <- cap * tanh(score / cap); 0: none
  const bf16_t* sink = nullptr;  // device [heads], nullable: exp(sink) joins the denominator
};
struct GroupedArgs {
  int T = 0;
  const void *q = nullptr, *k = nullptr, *v = nullptr;  // [T][ld*], the activation type; k and v: window form only
  int ldq = 0, ldk = 0, ldv = 0;
  void *kc = nullptr, *vc = nullptr;  // caches [cap][ldkc], [cap][ldvc]: all kv heads of a position, turned and normed keys
  int ldkc = 0, ldvc = 0, cap = 0;
  const int* pos = nullptr;
  const void* gate = nullptr;    // [T][ldg] logits, nullable: out *= sigmoid(gate)
  int ldg = 0;
  void* att = nullptr;           // [T][ldatt]
  int ldatt = 0;
};
// windows of 1..4 bf16 rows: queries and keys are turned and normed inside and the keys appended; with
// `lin` a decayed state's window runs beside it in the same launch
bool grouped_window_ok(const orn_ctx* ctx, const GroupedDims& D, const GroupedArgs& A);
size_t grouped_window_scratch(const orn_ctx* ctx, const GroupedDims& D);  // bytes for windows of up to 4 rows, zeroed once
int k_grouped_window(orn_ctx* ctx, cudaStream_t s, const GroupedDims& D, const GroupedArgs& A, void* scratch, const DecayedDims* lin_dims,
                     const DecayedArgs* lin);
// many rows or any sizes: q is already turned and normed, the rows' keys and values are in the cache
bool grouped_flash_ok(const GroupedDims& D, const GroupedArgs& A);
int k_grouped_flash(orn_ctx* ctx, cudaStream_t s, const GroupedDims& D, const GroupedArgs& A);
int k_grouped_plain(orn_ctx* ctx, cudaStream_t s, const GroupedDims& D, const GroupedArgs& A, bool act_f32);
