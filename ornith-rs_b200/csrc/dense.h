// Launchers of the dense-layer kernels (dense.cu): products with bf16 weights in their plain and
// mat-vec forms, and the row kernels between the products (the forms of the residual, norms, gates).
#pragma once

#include "act.cuh"
#include "orn_internal.h"

static inline int pad8(int n) { return (n + 7) & ~7; }

// One matrix of a launch over shared input rows: y[m][0..O) = act(x[m] W^T + bias) * mul[m].  y is
// float32 (out_f32) or the activation type; row stride ldy.
struct DenseJob {
  const orn_linear* lin = nullptr;
  void* y = nullptr;
  int ldy = 0;
  bool out_f32 = true;
  const bf16_t* bias = nullptr;
  ActParams act;
  const void* mul = nullptr;         // [rows][ldy] in the activation type, nullable; not in decode windows
  const orn_linear* lin2 = nullptr;  // decode windows: y = act(x W^T) * (x W2^T), without a bias
  int x0 = 0;                        // decode windows: the staged row's entry the matrix starts at
};

// x + LN(y * sigmoid(r + b)) * w, then (stream_out != null) the depth average over the streams so far:
//   r_out = x_in + norm(y * sigmoid(gate + gate_b)) * w
//   avg:    stream n_avg - 1 = r_out,  x = sum_{j < n_avg} a[j] stream_j
struct ResidualStep {
  const float* x_in = nullptr;    // [rows][ld]
  const float* y = nullptr;       // sublayer result [rows][ld]
  const float* gate = nullptr;    // gate logits before the bias [rows][ld], nullable: no gate
  const bf16_t* gate_b = nullptr; // [width]
  const bf16_t* w = nullptr;      // norm weight [width]
  int width = 0, ld = 0;
  float eps = 0.f;
  float* x_out = nullptr;         // [rows][ld]
  void* act_out = nullptr;        // x_out in the activation type [rows][ld] (nullable)
  // depth average
  int n_avg = 0;                  // 0: none
  const bf16_t* a = nullptr;      // [n_avg]
  float* streams = nullptr;       // [n_avg][stream_stride]
  size_t stream_stride = 0;
};
// The residual that is normed after its sum, over the result of one sublayer or of two side by side:
//   y      = y,  or (y / rms(y) * wl + y2 / rms(y2) * wr) / 2
//   x_out  = v / rms(v) * (w_add + w),  v = alpha x_in + y
struct PostNormStep {
  const float* x_in = nullptr;    // [rows][ld]
  const float* y = nullptr;       // [rows][ld]
  const float* y2 = nullptr;      // [rows][ld], nullable
  const bf16_t *wl = nullptr, *wr = nullptr;  // [width], with y2
  const bf16_t* w = nullptr;      // [width]
  float w_add = 0.f, alpha = 1.f, eps = 0.f;
  int width = 0, ld = 0;
  float* x_out = nullptr;         // [rows][ld]
  void* act_out = nullptr;        // x_out in the activation type (nullable)
};
int k_post_norm_rows(orn_ctx* ctx, cudaStream_t s, int rows, const PostNormStep& r, bool act_f32);
// out = x / rms(x) * (w_add + w) in the activation type, row stride ld (pads zero)
int k_rms_norm_rows(orn_ctx* ctx, cudaStream_t s, const float* x, int rows, int width, int ld, const bf16_t* w, float w_add, float eps,
                    void* out, bool act_f32);

// A mixer's heads on their way to the output product: every group of `group` neighbouring entries over
// its root mean square, times w (nullable), times act(gate).
struct GroupGate {
  const float* o = nullptr;       // [rows][ldo]
  const void* gate = nullptr;     // [rows][ldg], the activation type
  int ldo = 0, ldg = 0;           // multiples of 8
  int n = 0, group = 1;           // n entries, n % group == 0
  const bf16_t* w = nullptr;      // [n]
  int act = ACT_SIGMOID;          // or ACT_SILU
  float eps = 0.f;
};
int k_group_gate_rows(orn_ctx* ctx, cudaStream_t s, int rows, const GroupGate& g, void* out, int ldout, bool act_f32);
int k_residual_rows(orn_ctx* ctx, cudaStream_t s, int rows, const ResidualStep& r, bool act_f32);
// out = LN(x) * w in the activation type, row stride ld (pads zero)
int k_layer_norm_rows(orn_ctx* ctx, cudaStream_t s, const float* x, int rows, int width, int ld, const bf16_t* w, float eps,
                      void* out, bool act_f32);
// x = scale * table row in float32 (both copies; stream0 nullable), act = the same in the activation type
int k_embed_rows(orn_ctx* ctx, cudaStream_t s, const orn_linear* table, const uint32_t* ids, int rows, int width, int ld, float scale,
                 float* x, float* stream0, void* act, bool act_f32);
int k_gather_act_rows(orn_ctx* ctx, cudaStream_t s, const void* src, const int* idx, int n, int ld, void* dst, bool act_f32);
// the control path's product: one thread per output tile element, float32 accumulation in k order
int k_linear_plain(orn_ctx* ctx, cudaStream_t s, const orn_linear* L, const void* x, bool x_f32, int ldx, int rows,
                   const DenseJob& job);

// ---- decode windows (1..4 rows, bfloat16 activations): prologue + up to eight mat-vecs in one kernel
constexpr int kDecJobs = 8;
enum { DRO_ROWS = 0, DRO_EMBED = 1, DRO_RESIDUAL = 2, DRO_POSTNORM = 3, DRO_GATED = 4 };
struct DecodePrologue {
  int mode = DRO_ROWS;
  int K = 0;                      // input width (DRO_GATED: of the plain entries, may be 0)
  // DRO_ROWS, DRO_GATED
  const bf16_t* rows = nullptr;   // [M][ldx]
  int ldx = 0;
  // DRO_EMBED
  const orn_linear* table = nullptr;
  const uint32_t* ids = nullptr;
  float embed_scale = 1.f;
  // DRO_POSTNORM (its x_out and act_out stay empty)
  PostNormStep pn;
  // DRO_GATED: the staged row is [K plain entries, padded to 8 | the gated heads, padded to 8]
  GroupGate gg;
  // DRO_RESIDUAL: r as above; with r.n_avg the streams below the newest are already in `part`
  ResidualStep r;
  const float* part = nullptr;    // [M][ld]: sum_{j < n_avg - 1} a[j] stream_j
  // the stream this kernel hands on: x (and its newest stream copy), written by CTA 0
  float* x_out = nullptr;
  float* stream_out = nullptr;
  // a last norm before the products (the head): staged rows = LN(x) * w2; after DRO_POSTNORM
  // x / rms(x) * (pn.w_add + w2)
  const bf16_t* w2 = nullptr;
  bf16_t* normed_out = nullptr;   // [M][ld], by CTA 0
};
// false: the rows do not fit the kernel's shared memory (the caller takes the wide path)
bool decode_dense_fits(const DecodePrologue& p, int M);
int f_decode_dense(orn_ctx* ctx, cudaStream_t s, int M, const DecodePrologue& p, const DenseJob* jobs, int njobs);
