// Launchers of the linear attention with a fixed decay per head (decayed.cu):
//   S_t = g S_(t-1) + c k_t v_t^T,   o_t = S_t^T q_t
#pragma once

#include "orn_internal.h"

constexpr int kDecayChunk = 256;  // tokens between two kept states of a prompt chunk

struct DecayedDims {
  int heads = 0, dim = 0, vdim = 0;
  float k_scale = 1.f;           // c
  int rot_dims = 0;              // entries (i, i + rot_dims / 2) of q and k turn by position * freq[i]
  const double* freq = nullptr;  // device [rot_dims / 2]
  const float* gpow = nullptr;   // device [heads][kDecayChunk + 1]: g^0, g^1, ...
  ORN_HD size_t state() const { return (size_t)heads * dim * vdim; }  // floats per state: [heads][dim][vdim]
};
struct DecayedArgs {
  int T = 0;
  const void *q = nullptr, *k = nullptr, *v = nullptr;  // [T][ld*], the activation type
  int ldq = 0, ldk = 0, ldv = 0;
  float* ring = nullptr;         // [nring][state()]: slot *cur % nring goes in
  int nring = 1;
  const int* cur = nullptr;
  bool keep_all = false;         // the state after row t to slot *cur + 1 + t; else the last one to *cur + 1
  const int* pos = nullptr;      // the first row's position
  float* o = nullptr;            // [T][ldo]
  int ldo = 0;
};
// windows of 1..4 bf16 rows, q and k rotated inside; one launch of its own (grouped.h has it beside attention)
bool decayed_window_ok(const DecayedDims& D, const DecayedArgs& A);
int k_decayed_window(orn_ctx* ctx, cudaStream_t s, const DecayedDims& D, const DecayedArgs& A);
// token by token, any sizes: the control route.  q and k are already rotated.
int k_decayed_plain(orn_ctx* ctx, cudaStream_t s, const DecayedDims& D, const DecayedArgs& A, bool act_f32);
// prompt chunks on the tensor cores, bf16 rows.  q and k are already rotated.
bool decayed_chunk_ok(const DecayedDims& D, const DecayedArgs& A);
size_t decayed_chunk_scratch(const DecayedDims& D, int T);
int k_decayed_chunk(orn_ctx* ctx, cudaStream_t s, const DecayedDims& D, const DecayedArgs& A, void* scratch);
