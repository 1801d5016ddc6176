// Launchers of the latent-attention kernels (latent.cu).
#pragma once

#include "orn_internal.h"

// Sizes and constants of one latent-attention mixer, and the layout of its cache rows: the normed
// latent (kv_rank entries, padded to a multiple of 8 with zeros), then the rotated key part all heads
// share (rot_dim entries, padded likewise).
struct LatentDims {
  int heads = 0, dim = 0, rot_dim = 0, vdim = 0, kv_rank = 0;
  int rot_dims = 0;         // leading entries of the rotated part that turn, in neighbouring pairs
  float scale = 1.f;
  float eps = 0.f;          // of the latent's RMS norm
  const float* freq = nullptr;  // device [rot_dims / 2]: base^(-2i / rot_dims)
  ORN_HD int rp() const { return (kv_rank + 7) & ~7; }
  ORN_HD int row() const { return rp() + ((rot_dim + 7) & ~7); }  // elements per cache row
  ORN_HD int qk() const { return dim + rot_dim; }
};

// Append: cache row *pos + t = [rms_norm(kv[t][0..R)) * norm_w | rotate(kv[t][R..R + rot_dim))].
// kv null: nothing is appended (the layer reads another layer's cache).  rotate_q: the rotated parts
// of q [T][ldq] turn in place (the expanded form reads q directly).
int k_latent_rows(orn_ctx* ctx, cudaStream_t s, const LatentDims& D, int T, const float* kv, int ldkv, const bf16_t* norm_w,
                  void* cache, int cap, const int* pos, void* q, int ldq, bool rotate_q, bool act_f32);

// The depth average's older streams, summed beside the kernel's own work: out = sum_{j < n} a[j] streams_j
struct StreamSum {
  int n = 0;
  const bf16_t* a = nullptr;
  const float* streams = nullptr;
  size_t stride = 0;
  float* out = nullptr;
  int count = 0;  // floats per stream
};
// Absorbed form: qa[t][h] = [W_uk[h]^T q_unrot | rotate(q_rot)] in cache-row layout, plus the append
// above (kv nullable) and the stream sum.
int k_latent_absorb(orn_ctx* ctx, cudaStream_t s, const LatentDims& D, int T, const void* q, int ldq, const orn_linear* uk,
                    const float* kv, int ldkv, const bf16_t* norm_w, void* cache, int cap, const int* pos, void* qa,
                    const StreamSum& sum, bool act_f32);
// how the keys of a window are split over CTAs: fixed per (rows, heads), so that a captured step
// serves every context length
int latent_splits(const orn_ctx* ctx, const LatentDims& D, int T, bool plain);
bool latent_attn_tensor_ok(const LatentDims& D);  // the tensor-core form takes these sizes
// partial[t*H + h][split] = {unnormalised sum_j p_j c_j [R]}, ml = {max, sum} (base 2 exponents)
int k_latent_attn(orn_ctx* ctx, cudaStream_t s, const LatentDims& D, int T, const void* qa, const void* cache, int cap,
                  const int* pos, int splits, float* partial, float* ml, bool plain, bool act_f32);
// att[t][h*vdim + i] = (W_uv[h] merged latent)_i * sigmoid(gate[t][h])
int k_latent_out(orn_ctx* ctx, cudaStream_t s, const LatentDims& D, int T, const orn_linear* uv, const float* partial,
                 const float* ml, int splits, const int* pos, const float* gate, int ldgate, void* att, int ldatt, bool plain,
                 bool act_f32);
// Expanded form (bf16, many rows): per-head keys kx [n][ldk] (dim per head) and values vx [n][ldv] of
// all n = *pos + T cached positions, q already rotated; the output gate is applied on the way out.
bool latent_flash_ok(const LatentDims& D, int ldq);
int k_latent_flash(orn_ctx* ctx, cudaStream_t s, const LatentDims& D, int T, const bf16_t* q, int ldq, const bf16_t* kx, int ldk,
                   const bf16_t* vx, int ldv, const bf16_t* cache, int cap, const int* pos, const float* gate, int ldgate,
                   bf16_t* att, int ldatt);
