// Dense layers with bf16 weights around a float32 residual stream.
//
// Three forms of a product y = act(x W^T + bias):
//   * k_linear_plain: float32 accumulation in k order on CUDA cores, float32 or bf16 activations: the
//     control path, and the only path of a model that runs in float32;
//   * f_decode_dense: windows of 1..4 rows.  One kernel rebuilds its input rows in shared memory
//     (embedding lookup; the previous sublayer's residual step in one of its forms; the norm and gate
//     of a mixer's heads; or a plain load) and multiplies up to eight matrices by them, weights streamed
//     once with 16-byte loads whose first batch is requested before the kernel waits for its predecessor;
//   * many rows: the tensor-core product of gemm.cu, with the row kernels below between the products.
#include <algorithm>
#include <set>
#include <string>

#include "dense.h"

namespace {

// sum over the block; every thread gets it.  red: 33 floats.
template <int THREADS>
ORN_D float block_sum(float v, float* red) {
  v = warp_sum(v);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  __syncthreads();
  if (lane == 0) red[warp] = v;
  __syncthreads();
  float t = 0.f;
#pragma unroll
  for (int i = 0; i < THREADS / 32; ++i) t += red[i];
  return t;
}

ORN_D void store_act4(float* p, const float* v) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
ORN_D void store_act4(bf16_t* p, const float* v) {
  uint2 u;
  u.x = (uint32_t)f2bf(v[0]) | ((uint32_t)f2bf(v[1]) << 16);
  u.y = (uint32_t)f2bf(v[2]) | ((uint32_t)f2bf(v[3]) << 16);
  *reinterpret_cast<uint2*>(p) = u;
}
ORN_D void load_bf4(const bf16_t* p, int d, int width, float* v) {
  if (d + 3 < width && (reinterpret_cast<uintptr_t>(p + d) & 7) == 0) {
    const uint2 u = __ldg(reinterpret_cast<const uint2*>(p + d));
    v[0] = bf2f((bf16_t)(u.x & 0xffff)); v[1] = bf2f((bf16_t)(u.x >> 16));
    v[2] = bf2f((bf16_t)(u.y & 0xffff)); v[3] = bf2f((bf16_t)(u.y >> 16));
  } else {
#pragma unroll
    for (int e = 0; e < 4; ++e) v[e] = d + e < width ? bf2f(p[d + e]) : 0.f;
  }
}
ORN_D void unpack4(const float4& f, float* v) { v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w; }

// two sums over the block at once; red: 2 * THREADS / 32 floats
template <int THREADS>
ORN_D float2 block_sum2(float a, float b, float* red) {
  a = warp_sum(a);
  b = warp_sum(b);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  __syncthreads();
  if (lane == 0) { red[2 * warp] = a; red[2 * warp + 1] = b; }
  __syncthreads();
  float2 t = make_float2(0.f, 0.f);
#pragma unroll
  for (int i = 0; i < THREADS / 32; ++i) { t.x += red[2 * i]; t.y += red[2 * i + 1]; }
  return t;
}
// entries d .. d + 3 of a row of n (zeros beyond), one request when vec
ORN_D void load_row4(const float* p, int d, int n, bool vec, float* v) {
  if (vec && d + 3 < n) { unpack4(__ldcg(reinterpret_cast<const float4*>(p + d)), v); return; }
#pragma unroll
  for (int e = 0; e < 4; ++e) v[e] = d + e < n ? __ldcg(p + d + e) : 0.f;
}
ORN_D void load_row4(const bf16_t* p, int d, int n, bool vec, float* v) {
  if (vec && d + 3 < n) {
    const uint2 u = __ldcg(reinterpret_cast<const uint2*>(p + d));
    v[0] = bf2f((bf16_t)(u.x & 0xffff)); v[1] = bf2f((bf16_t)(u.x >> 16));
    v[2] = bf2f((bf16_t)(u.y & 0xffff)); v[3] = bf2f((bf16_t)(u.y >> 16));
    return;
  }
#pragma unroll
  for (int e = 0; e < 4; ++e) v[e] = d + e < n ? bf2f(__ldcg(p + d + e)) : 0.f;
}

// the gate of a mixer's heads: sigmoid(z) or, for ACT_SILU, z sigmoid(z)
ORN_D float head_gate(int act, float z) {
  const float s = sigmoid_f32(z);
  return act == ACT_SILU ? z * s : s;
}
// An activation as a call: decode kernels run once through their code, which should be short.
__device__ __noinline__ float act_apply_call(int kind, float z, float a, float b) { return act_apply(kind, z, a, b); }

// Row m of a mixer's heads under their group norm and gate.  A warp per group while a group fits its
// registers, the whole block otherwise.  stash: group_gate_stash() floats; red: as block_sum.
constexpr int kGgRegs = 4;  // groups of up to kGgRegs * 128 entries stay in a warp's registers
ORN_HD bool group_gate_warp(const GroupGate& G) { return G.group <= kGgRegs * 128; }
template <int THREADS, typename TA>
ORN_D void group_gate_row(const GroupGate& G, int m, TA* out, float* stash, float* red) {
  const float* o = G.o + (size_t)m * G.ldo;
  const TA* gate = reinterpret_cast<const TA*>(G.gate) + (size_t)m * G.ldg;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const bool vec = G.group % 4 == 0;  // row strides are multiples of 8
  const float inv = 1.0f / (float)G.group;
  auto put = [&](int at, int d, const float* v) {
    if (vec) { store_act4(out + at, v); return; }
#pragma unroll
    for (int e = 0; e < 4; ++e)
      if (d + e < G.group) out[at + e] = to_act<TA>(v[e]);
  };
  if (vec && G.group <= 128) {  // four groups at a time, all requested before the first is used
    constexpr int kAhead = 4;
    const int step = (THREADS / 32) * G.group, d = 4 * lane;
    for (int g0 = warp * G.group; g0 < G.n; g0 += kAhead * step) {
      float v[kAhead][4], z[kAhead][4], w[kAhead][4];
#pragma unroll
      for (int k = 0; k < kAhead; ++k) {
        const int at = g0 + k * step, n = at < G.n ? G.group : 0;
        load_row4(o + at, d, n, true, v[k]);
        load_row4(gate + at, d, n, true, z[k]);
#pragma unroll
        for (int e = 0; e < 4; ++e) w[k][e] = 1.f;
        if (G.w != nullptr) load_bf4(G.w + at, d, n, w[k]);
      }
#pragma unroll
      for (int k = 0; k < kAhead; ++k) {
        const int at = g0 + k * step;
        if (at >= G.n) break;  // warp-uniform
        float sq = 0.f;
#pragma unroll
        for (int e = 0; e < 4; ++e) sq = fmaf(v[k][e], v[k][e], sq);
        const float rstd = 1.0f / sqrtf(warp_sum(sq) * inv + G.eps);
        if (d < G.group) {
#pragma unroll
          for (int e = 0; e < 4; ++e) v[k][e] = v[k][e] * rstd * w[k][e] * head_gate(G.act, z[k][e]);
          store_act4(out + at + d, v[k]);
        }
      }
    }
    return;
  }
  if (group_gate_warp(G)) {
    for (int g0 = warp * G.group; g0 < G.n; g0 += (THREADS / 32) * G.group) {
      float v[kGgRegs][4], z[kGgRegs][4], sq = 0.f;
#pragma unroll
      for (int it = 0; it < kGgRegs; ++it) {
        const int d = 4 * (lane + 32 * it);
        if (d < G.group) {
          load_row4(o + g0, d, G.group, vec, v[it]);
          load_row4(gate + g0, d, G.group, vec, z[it]);
#pragma unroll
          for (int e = 0; e < 4; ++e) sq = fmaf(v[it][e], v[it][e], sq);
        }
      }
      const float rstd = 1.0f / sqrtf(warp_sum(sq) * inv + G.eps);
#pragma unroll
      for (int it = 0; it < kGgRegs; ++it) {
        const int d = 4 * (lane + 32 * it);
        if (d < G.group) {
          float w[4] = {1.f, 1.f, 1.f, 1.f};
          if (G.w != nullptr) load_bf4(G.w + g0, d, G.group, w);
#pragma unroll
          for (int e = 0; e < 4; ++e) v[it][e] = v[it][e] * rstd * w[e] * head_gate(G.act, z[it][e]);
          put(g0 + d, d, v[it]);
        }
      }
    }
    return;
  }
  for (int g0 = 0; g0 < G.n; g0 += G.group) {
    float sq = 0.f;
    for (int d = 4 * threadIdx.x; d < G.group; d += 4 * THREADS) {
      float v[4], z[4], w[4] = {1.f, 1.f, 1.f, 1.f};
      load_row4(o + g0, d, G.group, vec, v);
      load_row4(gate + g0, d, G.group, vec, z);
      if (G.w != nullptr) load_bf4(G.w + g0, d, G.group, w);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        sq = fmaf(v[e], v[e], sq);
        if (d + e < G.group) stash[d + e] = v[e] * w[e] * head_gate(G.act, z[e]);
      }
    }
    const float rstd = 1.0f / sqrtf(block_sum<THREADS>(sq, red) * inv + G.eps);
    for (int d = 4 * threadIdx.x; d < G.group; d += 4 * THREADS) {  // a thread's own entries
      float v[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) v[e] = d + e < G.group ? stash[d + e] * rstd : 0.f;
      put(g0 + d, d, v);
    }
  }
}
size_t group_gate_stash(const GroupGate& G) { return group_gate_warp(G) ? 0 : (size_t)G.group; }

ORN_D float bflo(uint32_t u) { return __uint_as_float(u << 16); }
ORN_D float bfhi(uint32_t u) { return __uint_as_float(u & 0xffff0000u); }

// ------------------------------------------------------------------ row kernels
constexpr int kRowThreads = 256;

// One CTA per row; the row's gated result waits in shared memory between the passes.  Rows are padded
// to a multiple of 8 with zeros, so every pass moves four elements at a time.
template <typename TA>
__global__ void __launch_bounds__(kRowThreads) residual_rows_kernel(ResidualStep R, TA* __restrict__ act_out) {
  extern __shared__ float s_row[];  // [ld]
  __shared__ float red[33];
  const size_t base = (size_t)blockIdx.x * R.ld;
  float sum = 0.f;
  for (int d = 4 * threadIdx.x; d < R.ld; d += 4 * kRowThreads) {
    float z[4], g[4], b[4];
    unpack4(__ldg(reinterpret_cast<const float4*>(R.y + base + d)), z);
    if (R.gate != nullptr) {
      unpack4(__ldg(reinterpret_cast<const float4*>(R.gate + base + d)), g);
      load_bf4(R.gate_b, d, R.width, b);
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      if (R.gate != nullptr) z[e] *= sigmoid_f32(g[e] + b[e]);
      if (d + e >= R.width) z[e] = 0.f;
      sum += z[e];
    }
    *reinterpret_cast<float4*>(s_row + d) = make_float4(z[0], z[1], z[2], z[3]);
  }
  const float mean = block_sum<kRowThreads>(sum, red) / (float)R.width;
  float sq = 0.f;
  for (int d = 4 * threadIdx.x; d < R.ld; d += 4 * kRowThreads)
#pragma unroll
    for (int e = 0; e < 4; ++e)
      if (d + e < R.width) {
        const float c = s_row[d + e] - mean;
        sq = fmaf(c, c, sq);
      }
  const float rstd = 1.0f / sqrtf(block_sum<kRowThreads>(sq, red) / (float)R.width + R.eps);
  for (int d = 4 * threadIdx.x; d < R.ld; d += 4 * kRowThreads) {
    float w[4], x[4];
    load_bf4(R.w, d, R.width, w);
    unpack4(*reinterpret_cast<const float4*>(R.x_in + base + d), x);
#pragma unroll
    for (int e = 0; e < 4; ++e) x[e] = d + e < R.width ? fmaf((s_row[d + e] - mean) * rstd, w[e], x[e]) : 0.f;
    if (R.n_avg > 0) {
      const int last = R.n_avg - 1;
      *reinterpret_cast<float4*>(R.streams + last * R.stream_stride + base + d) = make_float4(x[0], x[1], x[2], x[3]);
      const float al = bf2f(R.a[last]);
      float acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 4
      for (int j = 0; j < last; ++j) {
        const float aj = bf2f(R.a[j]);
        float v[4];
        unpack4(__ldg(reinterpret_cast<const float4*>(R.streams + j * R.stream_stride + base + d)), v);
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[e] = fmaf(aj, v[e], acc[e]);
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) x[e] = fmaf(al, x[e], acc[e]);
    }
    *reinterpret_cast<float4*>(R.x_out + base + d) = make_float4(x[0], x[1], x[2], x[3]);
    if (act_out != nullptr) store_act4(act_out + base + d, x);
  }
}

// One CTA per row; the weighted sum waits in shared memory for its norm.
template <typename TA>
__global__ void __launch_bounds__(kRowThreads) post_norm_rows_kernel(PostNormStep R, TA* __restrict__ act_out) {
  extern __shared__ float s_row[];  // [ld]
  __shared__ float red[kRowThreads / 16];
  const size_t base = (size_t)blockIdx.x * R.ld;
  const float inv = 1.0f / (float)R.width;
  float ra = 0.f, rb = 0.f;
  if (R.y2 != nullptr) {
    float a = 0.f, b = 0.f;
    for (int d = 4 * threadIdx.x; d < R.ld; d += 4 * kRowThreads) {
      float u[4], v[4];
      unpack4(__ldg(reinterpret_cast<const float4*>(R.y + base + d)), u);
      unpack4(__ldg(reinterpret_cast<const float4*>(R.y2 + base + d)), v);
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (d + e < R.width) { a = fmaf(u[e], u[e], a); b = fmaf(v[e], v[e], b); }
    }
    const float2 s2 = block_sum2<kRowThreads>(a, b, red);
    ra = 0.5f / sqrtf(s2.x * inv + R.eps);
    rb = 0.5f / sqrtf(s2.y * inv + R.eps);
  }
  float sq = 0.f;
  for (int d = 4 * threadIdx.x; d < R.ld; d += 4 * kRowThreads) {
    float x[4], y[4];
    unpack4(*reinterpret_cast<const float4*>(R.x_in + base + d), x);
    unpack4(__ldg(reinterpret_cast<const float4*>(R.y + base + d)), y);
    if (R.y2 != nullptr) {
      float v[4], wl[4], wr[4];
      unpack4(__ldg(reinterpret_cast<const float4*>(R.y2 + base + d)), v);
      load_bf4(R.wl, d, R.width, wl);
      load_bf4(R.wr, d, R.width, wr);
#pragma unroll
      for (int e = 0; e < 4; ++e) y[e] = fmaf(y[e] * ra, wl[e], v[e] * rb * wr[e]);
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      x[e] = d + e < R.width ? fmaf(R.alpha, x[e], y[e]) : 0.f;
      sq = fmaf(x[e], x[e], sq);
    }
    *reinterpret_cast<float4*>(s_row + d) = make_float4(x[0], x[1], x[2], x[3]);
  }
  const float rstd = 1.0f / sqrtf(block_sum<kRowThreads>(sq, red) * inv + R.eps);
  for (int d = 4 * threadIdx.x; d < R.ld; d += 4 * kRowThreads) {
    float w[4], x[4];
    load_bf4(R.w, d, R.width, w);
    unpack4(*reinterpret_cast<const float4*>(s_row + d), x);
#pragma unroll
    for (int e = 0; e < 4; ++e) x[e] = x[e] * rstd * (R.w_add + w[e]);
    *reinterpret_cast<float4*>(R.x_out + base + d) = make_float4(x[0], x[1], x[2], x[3]);
    if (act_out != nullptr) store_act4(act_out + base + d, x);
  }
}

template <typename TA>
__global__ void __launch_bounds__(kRowThreads) rms_norm_rows_kernel(const float* __restrict__ x, int width, int ld, const bf16_t* __restrict__ w,
                                                                    float w_add, float eps, TA* __restrict__ out) {
  __shared__ float red[kRowThreads / 32];
  const float* xr = x + (size_t)blockIdx.x * ld;
  float sq = 0.f;
  for (int d = threadIdx.x; d < width; d += kRowThreads) sq = fmaf(xr[d], xr[d], sq);
  const float rstd = 1.0f / sqrtf(block_sum<kRowThreads>(sq, red) / (float)width + eps);
  for (int d = threadIdx.x; d < ld; d += kRowThreads)
    out[(size_t)blockIdx.x * ld + d] = to_act<TA>(d < width ? xr[d] * rstd * (w_add + bf2f(w[d])) : 0.f);
}

template <typename TA>
__global__ void __launch_bounds__(kRowThreads) group_gate_rows_kernel(GroupGate G, TA* __restrict__ out, int ldout) {
  extern __shared__ float s_row[];
  __shared__ float red[kRowThreads / 32];
  group_gate_row<kRowThreads, TA>(G, blockIdx.x, out + (size_t)blockIdx.x * ldout, s_row, red);
}

template <typename TA>
__global__ void __launch_bounds__(kRowThreads) layer_norm_rows_kernel(const float* __restrict__ x, int width, int ld,
                                                                      const bf16_t* __restrict__ w, float eps, TA* __restrict__ out) {
  __shared__ float red[33];
  const float* xr = x + (size_t)blockIdx.x * ld;
  float sum = 0.f;
  for (int d = threadIdx.x; d < width; d += kRowThreads) sum += xr[d];
  const float mean = block_sum<kRowThreads>(sum, red) / (float)width;
  float sq = 0.f;
  for (int d = threadIdx.x; d < width; d += kRowThreads) { const float c = xr[d] - mean; sq = fmaf(c, c, sq); }
  const float rstd = 1.0f / sqrtf(block_sum<kRowThreads>(sq, red) / (float)width + eps);
  for (int d = threadIdx.x; d < ld; d += kRowThreads)
    out[(size_t)blockIdx.x * ld + d] = to_act<TA>(d < width ? (xr[d] - mean) * rstd * bf2f(w[d]) : 0.f);
}

template <typename TA>
__global__ void __launch_bounds__(kRowThreads) embed_rows_kernel(LinDev E, const uint32_t* __restrict__ ids, int width, int ld, float scale,
                                                                 float* __restrict__ x, float* __restrict__ stream0, TA* __restrict__ act) {
  const uint32_t id = min(ids[blockIdx.x], (uint32_t)(E.O - 1));
  const bf16_t* row = reinterpret_cast<const bf16_t*>(E.w + (size_t)id * E.rec);
  const size_t base = (size_t)blockIdx.x * ld;
  for (int d = threadIdx.x; d < ld; d += kRowThreads) {
    const float v = d < width ? scale * bf2f(row[d]) : 0.f;
    x[base + d] = v;
    if (stream0 != nullptr) stream0[base + d] = v;
    if (act != nullptr) act[base + d] = to_act<TA>(v);
  }
}

__global__ void gather_rows16_kernel(const uint4* __restrict__ src, const int* __restrict__ idx, int n16, uint4* __restrict__ dst) {
  const uint4* s = src + (size_t)idx[blockIdx.x] * n16;
  for (int i = threadIdx.x; i < n16; i += blockDim.x) dst[(size_t)blockIdx.x * n16 + i] = s[i];
}

// ------------------------------------------------------------------ plain product
constexpr int kPlTile = 64, kPlK = 16;

template <typename TA, typename TY>
__global__ void __launch_bounds__(256) linear_plain_kernel(LinDev L, const TA* __restrict__ x, int ldx, int rows, TY* __restrict__ y,
                                                           int ldy, const bf16_t* __restrict__ bias, ActParams act,
                                                           const TA* __restrict__ mul) {
  __shared__ float sx[kPlK][kPlTile + 1], sw[kPlK][kPlTile + 1];
  const int m0 = blockIdx.y * kPlTile, o0 = blockIdx.x * kPlTile;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < L.K; k0 += kPlK) {
    for (int i = threadIdx.x; i < kPlTile * kPlK; i += 256) {
      const int r = i / kPlK, k = i % kPlK;
      const bool kin = k0 + k < L.K;
      sx[k][r] = kin && m0 + r < rows ? from_act(x[(size_t)(m0 + r) * ldx + k0 + k]) : 0.f;
      sw[k][r] = kin && o0 + r < L.O ? bf2f(reinterpret_cast<const bf16_t*>(L.w + (size_t)(o0 + r) * L.rec)[k0 + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kPlK; ++k) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { a[i] = sx[k][ty + 16 * i]; b[i] = sw[k][tx + 16 * i]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    __syncthreads();
  }
  float pa, pb;
  act_prepare(act, pa, pb);
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int m = m0 + ty + 16 * i, o = o0 + tx + 16 * j;
      if (m < rows && o < L.O) {
        const float v = act_apply(act.kind, acc[i][j] + (bias != nullptr ? bf2f(bias[o]) : 0.f), pa, pb);
        y[(size_t)m * ldy + o] = to_act<TY>(mul != nullptr ? v * from_act(mul[(size_t)m * ldy + o]) : v);
      }
    }
}

// ------------------------------------------------------------------ decode windows
constexpr int kDecThreads = 256;
constexpr int kDecWarps = kDecThreads / 32;
constexpr size_t kDecSmemMax = 200 * 1024;
constexpr int kDecRegs = 4;  // a residual row of up to kDecRegs * 1024 entries stays in registers

struct DecJobDev {
  const uint8_t* w;
  const uint8_t* w2;  // a gated pair's second matrix (a task is then one row of each), or null
  uint32_t rec;
  int O, task0, step; // rows of w per task
  int n16, x0;        // 16-byte pieces per row, first entry of the staged row
  void* y;
  int ldy, out_f32;
  const bf16_t* bias;
  ActParams act;
};
struct DecParams {
  DecodePrologue p;
  LinDev table;
  int njobs, tasks, Kp;  // Kp: entries per staged row, a multiple of 8
  DecJobDev job[kDecJobs];
};

// M rows staged as bf16 [M][Kp]: plain entries, then heads under their norm and gate.
template <int M>
ORN_D void decode_prologue_gated(const DecParams& P, bf16_t* s_x, float* f, float* red) {
  const DecodePrologue& p = P.p;
  const int Kp = P.Kp, Kr = (p.K + 7) & ~7;
  for (int i = threadIdx.x; i < M * (Kr / 8); i += kDecThreads) {
    const int m = i / (Kr / 8), c = i - m * (Kr / 8);
    *reinterpret_cast<uint4*>(s_x + (size_t)m * Kp + 8 * c) = __ldcg(reinterpret_cast<const uint4*>(p.rows + (size_t)m * p.ldx) + c);
  }
#pragma unroll 1
  for (int m = 0; m < M; ++m) {
    bf16_t* xs = s_x + (size_t)m * Kp + Kr;
    group_gate_row<kDecThreads, bf16_t>(p.gg, m, xs, f, red);
    if ((int)threadIdx.x < Kp - Kr - p.gg.n) xs[p.gg.n + threadIdx.x] = 0;
    if (!group_gate_warp(p.gg)) __syncthreads();  // the stash is reused by the next row
  }
  __syncthreads();
}
// M rows staged as bf16 [M][Kp]: the residual normed after its sum.
template <int M>
ORN_D void decode_prologue_post(const DecParams& P, bf16_t* s_x, float* f, float* red) {
  const DecodePrologue& p = P.p;
  const int Kp = P.Kp, K = p.K;
  const bool lead = blockIdx.x == 0;
  const PostNormStep& Q = p.pn;
  const float inv = 1.0f / (float)K;
  const bool pair = Q.y2 != nullptr;
  // a row of up to kDecRegs * 1024 entries stays in registers, a longer one waits in f
  const bool in_regs = Kp <= kDecRegs * 4 * kDecThreads;
#pragma unroll 1
  for (int m = 0; m < M; ++m) {
    bf16_t* xs = s_x + (size_t)m * Kp;
    const size_t base = (size_t)m * Q.ld;
    float v[kDecRegs][4], rstd;
    if (in_regs) {
      float y[kDecRegs][4], z[kDecRegs][4], a = 0.f, b = 0.f;
#pragma unroll
      for (int it = 0; it < kDecRegs; ++it) {
        const int d = 4 * (threadIdx.x + it * kDecThreads);
        const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
        const bool in = d < Kp;
        const float4 x4 = in ? __ldcg(reinterpret_cast<const float4*>(Q.x_in + base + d)) : zero;
        const float4 y4 = in ? __ldcg(reinterpret_cast<const float4*>(Q.y + base + d)) : zero;
        const float4 z4 = in && pair ? __ldcg(reinterpret_cast<const float4*>(Q.y2 + base + d)) : zero;
        unpack4(x4, v[it]); unpack4(y4, y[it]); unpack4(z4, z[it]);
#pragma unroll
        for (int e = 0; e < 4; ++e) { a = fmaf(y[it][e], y[it][e], a); b = fmaf(z[it][e], z[it][e], b); }  // pads are zeros
      }
      if (pair) {
        const float2 s2 = block_sum2<kDecThreads>(a, b, red);
        const float ra = 0.5f / sqrtf(s2.x * inv + Q.eps), rb = 0.5f / sqrtf(s2.y * inv + Q.eps);
#pragma unroll
        for (int it = 0; it < kDecRegs; ++it) {
          const int d = 4 * (threadIdx.x + it * kDecThreads);
          if (d < Kp) {
            float wl[4], wr[4];
            load_bf4(Q.wl, d, K, wl);
            load_bf4(Q.wr, d, K, wr);
#pragma unroll
            for (int e = 0; e < 4; ++e) y[it][e] = fmaf(y[it][e] * ra, wl[e], z[it][e] * rb * wr[e]);
          }
        }
      }
      float sq = 0.f;
#pragma unroll
      for (int it = 0; it < kDecRegs; ++it)
#pragma unroll
        for (int e = 0; e < 4; ++e) { v[it][e] = fmaf(Q.alpha, v[it][e], y[it][e]); sq = fmaf(v[it][e], v[it][e], sq); }
      rstd = 1.0f / sqrtf(block_sum<kDecThreads>(sq, red) * inv + Q.eps);
    } else {
      float ra = 0.f, rb = 0.f;
      if (pair) {
        float a = 0.f, b = 0.f;
        for (int d = threadIdx.x; d < K; d += kDecThreads) {
          const float y = __ldcg(Q.y + base + d), z = __ldcg(Q.y2 + base + d);
          a = fmaf(y, y, a); b = fmaf(z, z, b);
        }
        const float2 s2 = block_sum2<kDecThreads>(a, b, red);
        ra = 0.5f / sqrtf(s2.x * inv + Q.eps); rb = 0.5f / sqrtf(s2.y * inv + Q.eps);
      }
      float sq = 0.f;
      for (int d = 4 * threadIdx.x; d < Kp; d += 4 * kDecThreads) {
        float x[4], y[4];
        unpack4(__ldcg(reinterpret_cast<const float4*>(Q.x_in + base + d)), x);
        unpack4(__ldcg(reinterpret_cast<const float4*>(Q.y + base + d)), y);
        if (pair) {
          float z[4], wl[4], wr[4];
          unpack4(__ldcg(reinterpret_cast<const float4*>(Q.y2 + base + d)), z);
          load_bf4(Q.wl, d, K, wl);
          load_bf4(Q.wr, d, K, wr);
#pragma unroll
          for (int e = 0; e < 4; ++e) y[e] = fmaf(y[e] * ra, wl[e], z[e] * rb * wr[e]);
        }
#pragma unroll
        for (int e = 0; e < 4; ++e) { x[e] = fmaf(Q.alpha, x[e], y[e]); sq = fmaf(x[e], x[e], sq); }
        *reinterpret_cast<float4*>(f + d) = make_float4(x[0], x[1], x[2], x[3]);
      }
      rstd = 1.0f / sqrtf(block_sum<kDecThreads>(sq, red) * inv + Q.eps);
    }
    float sq2 = 0.f;
    auto finish = [&](int d, float* x) {  // the thread's own entries in both forms
      float w[4];
      load_bf4(Q.w, d, K, w);
#pragma unroll
      for (int e = 0; e < 4; ++e) { x[e] = x[e] * rstd * (Q.w_add + w[e]); sq2 = fmaf(x[e], x[e], sq2); }
      if (lead) *reinterpret_cast<float4*>(p.x_out + base + d) = make_float4(x[0], x[1], x[2], x[3]);
      if (p.w2 != nullptr) *reinterpret_cast<float4*>(f + d) = make_float4(x[0], x[1], x[2], x[3]);
      else store_act4(xs + d, x);
    };
    if (in_regs) {
#pragma unroll
      for (int it = 0; it < kDecRegs; ++it) {
        const int d = 4 * (threadIdx.x + it * kDecThreads);
        if (d < Kp) finish(d, v[it]);
      }
    } else {
      for (int d = 4 * threadIdx.x; d < Kp; d += 4 * kDecThreads) {
        float x[4];
        unpack4(*reinterpret_cast<const float4*>(f + d), x);
        finish(d, x);
      }
    }
    if (p.w2 != nullptr) {  // the norm in front of the head
      const float r2 = 1.0f / sqrtf(block_sum<kDecThreads>(sq2, red) * inv + Q.eps);
      for (int d = 4 * threadIdx.x; d < Kp; d += 4 * kDecThreads) {
        float x[4], w[4];
        unpack4(*reinterpret_cast<const float4*>(f + d), x);
        load_bf4(p.w2, d, K, w);
#pragma unroll
        for (int e = 0; e < 4; ++e) x[e] = d + e < K ? x[e] * r2 * (Q.w_add + w[e]) : 0.f;
        store_act4(xs + d, x);
        if (lead && p.normed_out != nullptr) store_act4(p.normed_out + base + d, x);
      }
    }
    __syncthreads();  // f and red are reused by the next row
  }
}

// M rows staged as bf16 [M][Kp]; LN steps work on float rows behind them.
template <int M>
ORN_D void decode_prologue(const DecParams& P, bf16_t* s_x, float* s_f, float* red) {
  const DecodePrologue& p = P.p;
  const int Kp = P.Kp, K = p.K;
  const bool lead = blockIdx.x == 0;
  if (p.mode == DRO_ROWS) {
    for (int i = threadIdx.x; i < M * (Kp / 8); i += kDecThreads) {
      const int m = i / (Kp / 8), c = i - m * (Kp / 8);
      *reinterpret_cast<uint4*>(s_x + (size_t)m * Kp + 8 * c) = __ldcg(reinterpret_cast<const uint4*>(p.rows + (size_t)m * p.ldx) + c);
    }
    __syncthreads();
    return;
  }
  const ResidualStep& R = p.r;
#pragma unroll 1
  for (int m = 0; m < M; ++m) {
    float* f = s_f;
    bf16_t* xs = s_x + (size_t)m * Kp;
    if (p.mode == DRO_EMBED) {
      const uint32_t id = min(p.ids[m], (uint32_t)(P.table.O - 1));
      const uint8_t* row = P.table.w + (size_t)id * P.table.rec;  // padded with zeros to Kp
      for (int c = threadIdx.x; c < Kp / 8; c += kDecThreads) {
        const uint4 u = ldg128(row + 16 * (size_t)c);
        const float sc = p.embed_scale;
        const float lo4[4] = {sc * bflo(u.x), sc * bfhi(u.x), sc * bflo(u.y), sc * bfhi(u.y)};
        const float hi4[4] = {sc * bflo(u.z), sc * bfhi(u.z), sc * bflo(u.w), sc * bfhi(u.w)};
        const float4 lo = make_float4(lo4[0], lo4[1], lo4[2], lo4[3]), hi = make_float4(hi4[0], hi4[1], hi4[2], hi4[3]);
        const size_t at = (size_t)m * Kp + 8 * c;
        store_act4(xs + 8 * c, lo4);
        store_act4(xs + 8 * c + 4, hi4);
        *reinterpret_cast<float4*>(f + 8 * c) = lo;
        *reinterpret_cast<float4*>(f + 8 * c + 4) = hi;
        if (lead) {
          *reinterpret_cast<float4*>(p.x_out + at) = lo;
          *reinterpret_cast<float4*>(p.x_out + at + 4) = hi;
          if (p.stream_out != nullptr) {
            *reinterpret_cast<float4*>(p.stream_out + at) = lo;
            *reinterpret_cast<float4*>(p.stream_out + at + 4) = hi;
          }
        }
      }
    } else if (Kp <= kDecRegs * 4 * kDecThreads) {
      // everything the row needs is requested at once and stays in registers
      const size_t base = (size_t)m * R.ld;
      float z[kDecRegs][4], x[kDecRegs][4], pt[kDecRegs][4];
      const float al = R.n_avg > 0 ? bf2f(R.a[R.n_avg - 1]) : 0.f;
      uint32_t wq[kDecRegs][2];
#pragma unroll
      for (int it = 0; it < kDecRegs; ++it) {
        const int d = 4 * (threadIdx.x + it * kDecThreads);
        const bool in = d < Kp;
        const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
        const float4 y4 = in ? __ldcg(reinterpret_cast<const float4*>(R.y + base + d)) : zero;
        const float4 g4 = in && R.gate != nullptr ? __ldcg(reinterpret_cast<const float4*>(R.gate + base + d)) : zero;
        const float4 x4 = in ? __ldcg(reinterpret_cast<const float4*>(R.x_in + base + d)) : zero;
        const float4 p4 = in && R.n_avg > 0 ? __ldcg(reinterpret_cast<const float4*>(p.part + base + d)) : zero;
        float b[4] = {0.f, 0.f, 0.f, 0.f}, w[4] = {0.f, 0.f, 0.f, 0.f}, g[4];
        if (in && R.gate != nullptr) load_bf4(R.gate_b, d, K, b);
        if (in) load_bf4(R.w, d, K, w);
        unpack4(y4, z[it]); unpack4(g4, g); unpack4(x4, x[it]); unpack4(p4, pt[it]);
        wq[it][0] = (uint32_t)f2bf(w[0]) | ((uint32_t)f2bf(w[1]) << 16);  // exact: they are bf16
        wq[it][1] = (uint32_t)f2bf(w[2]) | ((uint32_t)f2bf(w[3]) << 16);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          if (R.gate != nullptr) z[it][e] *= sigmoid_f32(g[e] + b[e]);
          if (d + e >= K) z[it][e] = 0.f;
        }
      }
      float sum = 0.f;
#pragma unroll
      for (int it = 0; it < kDecRegs; ++it)
#pragma unroll
        for (int e = 0; e < 4; ++e) sum += z[it][e];
      const float mean = block_sum<kDecThreads>(sum, red) / (float)K;
      float sq = 0.f;
#pragma unroll
      for (int it = 0; it < kDecRegs; ++it)
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (4 * (int)(threadIdx.x + it * kDecThreads) + e < K) { const float c = z[it][e] - mean; sq = fmaf(c, c, sq); }
      const float rstd = 1.0f / sqrtf(block_sum<kDecThreads>(sq, red) / (float)K + R.eps);
#pragma unroll
      for (int it = 0; it < kDecRegs; ++it) {
        const int d = 4 * (threadIdx.x + it * kDecThreads);
        if (d >= Kp) break;
        const float w[4] = {__uint_as_float(wq[it][0] << 16), __uint_as_float(wq[it][0] & 0xffff0000u), __uint_as_float(wq[it][1] << 16),
                            __uint_as_float(wq[it][1] & 0xffff0000u)};
        float v[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) v[e] = d + e < K ? fmaf((z[it][e] - mean) * rstd, w[e], x[it][e]) : 0.f;
        if (R.n_avg > 0) {
          if (lead) *reinterpret_cast<float4*>(p.stream_out + base + d) = make_float4(v[0], v[1], v[2], v[3]);
#pragma unroll
          for (int e = 0; e < 4; ++e) v[e] = fmaf(al, v[e], pt[it][e]);
        }
        if (lead) *reinterpret_cast<float4*>(p.x_out + base + d) = make_float4(v[0], v[1], v[2], v[3]);
        if (p.w2 != nullptr) *reinterpret_cast<float4*>(f + d) = make_float4(v[0], v[1], v[2], v[3]);
        store_act4(xs + d, v);
      }
    } else {
      const size_t base = (size_t)m * R.ld;
      float sum = 0.f;
      for (int d = 4 * threadIdx.x; d < Kp; d += 4 * kDecThreads) {
        float z[4], g[4], b[4];
        unpack4(__ldcg(reinterpret_cast<const float4*>(R.y + base + d)), z);
        if (R.gate != nullptr) {
          unpack4(__ldcg(reinterpret_cast<const float4*>(R.gate + base + d)), g);
          load_bf4(R.gate_b, d, K, b);
        }
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          if (R.gate != nullptr) z[e] *= sigmoid_f32(g[e] + b[e]);
          if (d + e >= K) z[e] = 0.f;
          sum += z[e];
        }
        *reinterpret_cast<float4*>(f + d) = make_float4(z[0], z[1], z[2], z[3]);
      }
      const float mean = block_sum<kDecThreads>(sum, red) / (float)K;
      float sq = 0.f;
      for (int d = 4 * threadIdx.x; d < Kp; d += 4 * kDecThreads)
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (d + e < K) { const float c = f[d + e] - mean; sq = fmaf(c, c, sq); }
      const float rstd = 1.0f / sqrtf(block_sum<kDecThreads>(sq, red) / (float)K + R.eps);
      const float al = R.n_avg > 0 ? bf2f(R.a[R.n_avg - 1]) : 0.f;
      for (int d = 4 * threadIdx.x; d < Kp; d += 4 * kDecThreads) {
        float w[4], x[4];
        load_bf4(R.w, d, K, w);
        unpack4(__ldcg(reinterpret_cast<const float4*>(R.x_in + base + d)), x);
#pragma unroll
        for (int e = 0; e < 4; ++e) x[e] = d + e < K ? fmaf((f[d + e] - mean) * rstd, w[e], x[e]) : 0.f;
        if (R.n_avg > 0) {
          if (lead) *reinterpret_cast<float4*>(p.stream_out + base + d) = make_float4(x[0], x[1], x[2], x[3]);
          float a[4];
          unpack4(__ldcg(reinterpret_cast<const float4*>(p.part + base + d)), a);
#pragma unroll
          for (int e = 0; e < 4; ++e) x[e] = fmaf(al, x[e], a[e]);
        }
        if (lead) *reinterpret_cast<float4*>(p.x_out + base + d) = make_float4(x[0], x[1], x[2], x[3]);
        *reinterpret_cast<float4*>(f + d) = make_float4(x[0], x[1], x[2], x[3]);
        store_act4(xs + d, x);
      }
    }
    if (p.w2 != nullptr) {  // the norm in front of the head
      __syncthreads();  // a thread reads what other threads wrote
      float sum = 0.f;
      for (int d = threadIdx.x; d < K; d += kDecThreads) sum += f[d];
      const float mean = block_sum<kDecThreads>(sum, red) / (float)K;
      float sq = 0.f;
      for (int d = threadIdx.x; d < K; d += kDecThreads) { const float c = f[d] - mean; sq = fmaf(c, c, sq); }
      const float rstd = 1.0f / sqrtf(block_sum<kDecThreads>(sq, red) / (float)K + R.eps);
      for (int d = threadIdx.x; d < Kp; d += kDecThreads) {
        const bf16_t v = d < K ? f2bf((f[d] - mean) * rstd * bf2f(p.w2[d])) : (bf16_t)0;
        xs[d] = v;
        if (lead && p.normed_out != nullptr) p.normed_out[(size_t)m * Kp + d] = v;
      }
    }
    __syncthreads();  // f is reused by the next row
  }
}

// A warp takes R consecutive rows of one matrix: 32 lanes x 16 bytes per step and row, U steps in flight.
// One instance per family of prologues: an instance holds the code of its own only.
enum { PF_STREAM = 0, PF_POSTNORM = 1, PF_GATED = 2 };
template <int M, int R, int U, int PF>
__global__ void __launch_bounds__(kDecThreads) decode_dense_kernel(const __grid_constant__ DecParams P) {
  extern __shared__ __align__(16) uint8_t s_raw[];
  __shared__ float red[33], s_act[kDecJobs][2];
  bf16_t* s_x = reinterpret_cast<bf16_t*>(s_raw);
  float* s_f = reinterpret_cast<float*>(s_raw + (((size_t)M * P.Kp * 2 + 15) & ~(size_t)15));
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  int task = blockIdx.x * kDecWarps + warp;
  const int stride = gridDim.x * kDecWarps;
  uint4 buf[R][U];
  int j = 0, o0 = 0;
  auto locate = [&](int t) {
    j = 0;
    while (j + 1 < P.njobs && t >= P.job[j + 1].task0) ++j;
    o0 = (t - P.job[j].task0) * P.job[j].step;
  };
  auto load = [&](int c0) {
    const int n16 = P.job[j].n16;
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const uint8_t* row = r == 1 && P.job[j].w2 != nullptr ? P.job[j].w2 + (size_t)o0 * P.job[j].rec
                                                           : P.job[j].w + (size_t)min(o0 + r, P.job[j].O - 1) * P.job[j].rec;
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int c = c0 + 32 * u + lane;
        buf[r][u] = c < n16 ? ldg128_stream(row + 16 * (size_t)c) : make_uint4(0, 0, 0, 0);
      }
    }
  };
  if (task < P.tasks) {  // weights do not depend on the kernel before this one
    locate(task);
    load(0);
  }
  if (threadIdx.x < P.njobs) act_prepare(P.job[threadIdx.x].act, s_act[threadIdx.x][0], s_act[threadIdx.x][1]);
  pdl_wait();
  pdl_trigger();
  if (PF == PF_POSTNORM) decode_prologue_post<M>(P, s_x, s_f, red);
  else if (PF == PF_GATED) decode_prologue_gated<M>(P, s_x, s_f, red);
  else decode_prologue<M>(P, s_x, s_f, red);
  for (; task < P.tasks; task += stride) {
    float acc[R][M];
#pragma unroll
    for (int r = 0; r < R; ++r)
#pragma unroll
      for (int m = 0; m < M; ++m) acc[r][m] = 0.f;
    const int n16 = P.job[j].n16;
    const bf16_t* s_xj = s_x + P.job[j].x0;
    for (int c0 = 0; c0 < n16; c0 += 32 * U) {
      if (c0 > 0) load(c0);
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int c = c0 + 32 * u + lane;
        const int cs = min(c, n16 - 1);  // weights beyond the row are zeros
#pragma unroll
        for (int m = 0; m < M; ++m) {
          const uint4 xv = *reinterpret_cast<const uint4*>(s_xj + (size_t)m * P.Kp + 8 * cs);
          const float x0 = bflo(xv.x), x1 = bfhi(xv.x), x2 = bflo(xv.y), x3 = bfhi(xv.y);
          const float x4 = bflo(xv.z), x5 = bfhi(xv.z), x6 = bflo(xv.w), x7 = bfhi(xv.w);
#pragma unroll
          for (int r = 0; r < R; ++r) {
            const uint4 w = buf[r][u];
            float a = acc[r][m];
            a = fmaf(bflo(w.x), x0, a); a = fmaf(bfhi(w.x), x1, a);
            a = fmaf(bflo(w.y), x2, a); a = fmaf(bfhi(w.y), x3, a);
            a = fmaf(bflo(w.z), x4, a); a = fmaf(bfhi(w.z), x5, a);
            a = fmaf(bflo(w.w), x6, a); a = fmaf(bfhi(w.w), x7, a);
            acc[r][m] = a;
          }
        }
      }
    }
    const int jj = j, oo = o0;
    if (task + stride < P.tasks) {  // the next task's first batch flies during the reduction
      locate(task + stride);
      load(0);
    }
    const DecJobDev& J = P.job[jj];
#pragma unroll
    for (int r = 0; r < R; ++r)
#pragma unroll
      for (int m = 0; m < M; ++m) acc[r][m] = warp_sum(acc[r][m]);
    if (R == 2 && J.w2 != nullptr) {
#pragma unroll
      for (int m = 0; m < M; ++m)
        if (lane == m) {
          const float v = act_apply_call(J.act.kind, acc[0][m], s_act[jj][0], s_act[jj][1]) * acc[R - 1][m];
          if (J.out_f32) reinterpret_cast<float*>(J.y)[(size_t)m * J.ldy + oo] = v;
          else reinterpret_cast<bf16_t*>(J.y)[(size_t)m * J.ldy + oo] = f2bf(v);
        }
      continue;
    }
    float mine = 0.f;
    int mr = 0, mm = 0;
#pragma unroll
    for (int r = 0; r < R; ++r)
#pragma unroll
      for (int m = 0; m < M; ++m)
        if (lane == r * M + m) { mine = acc[r][m]; mr = r; mm = m; }
    if (lane < R * M && oo + mr < J.O) {
      const int o = oo + mr;
      float v = mine + (J.bias != nullptr ? bf2f(J.bias[o]) : 0.f);
      if (J.act.kind != ACT_NONE) v = act_apply_call(J.act.kind, v, s_act[jj][0], s_act[jj][1]);
      if (J.out_f32) reinterpret_cast<float*>(J.y)[(size_t)mm * J.ldy + o] = v;
      else reinterpret_cast<bf16_t*>(J.y)[(size_t)mm * J.ldy + o] = f2bf(v);
    }
  }
}

int decode_row(const DecodePrologue& p) { return pad8(p.K) + (p.mode == DRO_GATED ? pad8(p.gg.n) : 0); }
size_t decode_smem(const DecodePrologue& p, int M) {
  const size_t Kp = decode_row(p);
  const size_t floats = p.mode == DRO_ROWS ? 0 : p.mode == DRO_GATED ? group_gate_stash(p.gg) : Kp;
  return (((size_t)M * Kp * 2 + 15) & ~(size_t)15) + floats * 4;
}

template <int M, int R, int U, int PF>
int launch_decode(orn_ctx* ctx, cudaStream_t s, const DecParams& P, int grid, size_t smem, const char* label) {
  if (smem > 48 * 1024) {
    const int rc = orn_grant_smem(ctx, reinterpret_cast<const void*>(decode_dense_kernel<M, R, U, PF>), kDecSmemMax);
    if (rc != ORN_OK) return rc;
  }
  ORN_CHECK_CUDA(ctx, orn_launch_dependent(ctx, s, 0, decode_dense_kernel<M, R, U, PF>, dim3(grid), dim3(kDecThreads), smem, P));
  return orn_launch_check(ctx, label);
}

}  // namespace

int k_residual_rows(orn_ctx* ctx, cudaStream_t s, int rows, const ResidualStep& r, bool act_f32) {
  const size_t smem = sizeof(float) * (size_t)r.ld;
  if (smem > kDecSmemMax) ORN_FAIL(ctx, ORN_ERR_ARG, "residual: width above 51200");
  if (act_f32) {
    if (smem > 48 * 1024) { int rc = orn_grant_smem(ctx, (const void*)residual_rows_kernel<float>, kDecSmemMax); if (rc) return rc; }
    residual_rows_kernel<float><<<rows, kRowThreads, smem, s>>>(r, reinterpret_cast<float*>(r.act_out));
  } else {
    if (smem > 48 * 1024) { int rc = orn_grant_smem(ctx, (const void*)residual_rows_kernel<bf16_t>, kDecSmemMax); if (rc) return rc; }
    residual_rows_kernel<bf16_t><<<rows, kRowThreads, smem, s>>>(r, reinterpret_cast<bf16_t*>(r.act_out));
  }
  return orn_launch_check(ctx, r.n_avg > 0 ? "residual_rows avg" : "residual_rows");
}

int k_post_norm_rows(orn_ctx* ctx, cudaStream_t s, int rows, const PostNormStep& r, bool act_f32) {
  const size_t smem = sizeof(float) * (size_t)r.ld;
  if (smem > kDecSmemMax) ORN_FAIL(ctx, ORN_ERR_ARG, "residual: width above 51200");
  if (act_f32) {
    if (smem > 48 * 1024) { int rc = orn_grant_smem(ctx, (const void*)post_norm_rows_kernel<float>, kDecSmemMax); if (rc) return rc; }
    post_norm_rows_kernel<float><<<rows, kRowThreads, smem, s>>>(r, reinterpret_cast<float*>(r.act_out));
  } else {
    if (smem > 48 * 1024) { int rc = orn_grant_smem(ctx, (const void*)post_norm_rows_kernel<bf16_t>, kDecSmemMax); if (rc) return rc; }
    post_norm_rows_kernel<bf16_t><<<rows, kRowThreads, smem, s>>>(r, reinterpret_cast<bf16_t*>(r.act_out));
  }
  return orn_launch_check(ctx, r.y2 != nullptr ? "post_norm_rows pair" : "post_norm_rows");
}

int k_rms_norm_rows(orn_ctx* ctx, cudaStream_t s, const float* x, int rows, int width, int ld, const bf16_t* w, float w_add, float eps,
                    void* out, bool act_f32) {
  if (act_f32) rms_norm_rows_kernel<float><<<rows, kRowThreads, 0, s>>>(x, width, ld, w, w_add, eps, reinterpret_cast<float*>(out));
  else rms_norm_rows_kernel<bf16_t><<<rows, kRowThreads, 0, s>>>(x, width, ld, w, w_add, eps, reinterpret_cast<bf16_t*>(out));
  return orn_launch_check(ctx, "rms_norm_rows");
}

int k_group_gate_rows(orn_ctx* ctx, cudaStream_t s, int rows, const GroupGate& g, void* out, int ldout, bool act_f32) {
  if (g.group < 1 || g.n % g.group || (g.act != ACT_SILU && g.act != ACT_SIGMOID)) ORN_FAIL(ctx, ORN_ERR_ARG, "group gate: whole groups, sigmoid or SiLU");
  if (g.ldo % 8 || g.ldg % 8 || ldout % 8) ORN_FAIL(ctx, ORN_ERR_ARG, "group gate: row strides must be multiples of 8");
  const size_t smem = sizeof(float) * group_gate_stash(g);
  if (smem > kDecSmemMax) ORN_FAIL(ctx, ORN_ERR_ARG, "group gate: a group above 51200 entries");
  if (act_f32) {
    if (smem > 48 * 1024) { int rc = orn_grant_smem(ctx, (const void*)group_gate_rows_kernel<float>, kDecSmemMax); if (rc) return rc; }
    group_gate_rows_kernel<float><<<rows, kRowThreads, smem, s>>>(g, reinterpret_cast<float*>(out), ldout);
  } else {
    if (smem > 48 * 1024) { int rc = orn_grant_smem(ctx, (const void*)group_gate_rows_kernel<bf16_t>, kDecSmemMax); if (rc) return rc; }
    group_gate_rows_kernel<bf16_t><<<rows, kRowThreads, smem, s>>>(g, reinterpret_cast<bf16_t*>(out), ldout);
  }
  return orn_launch_check(ctx, "group_gate_rows");
}

int k_layer_norm_rows(orn_ctx* ctx, cudaStream_t s, const float* x, int rows, int width, int ld, const bf16_t* w, float eps, void* out,
                      bool act_f32) {
  if (act_f32) layer_norm_rows_kernel<float><<<rows, kRowThreads, 0, s>>>(x, width, ld, w, eps, reinterpret_cast<float*>(out));
  else layer_norm_rows_kernel<bf16_t><<<rows, kRowThreads, 0, s>>>(x, width, ld, w, eps, reinterpret_cast<bf16_t*>(out));
  return orn_launch_check(ctx, "layer_norm_rows");
}

int k_embed_rows(orn_ctx* ctx, cudaStream_t s, const orn_linear* table, const uint32_t* ids, int rows, int width, int ld, float scale,
                 float* x, float* stream0, void* act, bool act_f32) {
  if (act_f32)
    embed_rows_kernel<float><<<rows, kRowThreads, 0, s>>>(lin_dev(table), ids, width, ld, scale, x, stream0, reinterpret_cast<float*>(act));
  else
    embed_rows_kernel<bf16_t><<<rows, kRowThreads, 0, s>>>(lin_dev(table), ids, width, ld, scale, x, stream0, reinterpret_cast<bf16_t*>(act));
  return orn_launch_check(ctx, "embed_rows");
}

int k_gather_act_rows(orn_ctx* ctx, cudaStream_t s, const void* src, const int* idx, int n, int ld, void* dst, bool act_f32) {
  const int n16 = ld * (act_f32 ? 4 : 2) / 16;
  gather_rows16_kernel<<<n, 128, 0, s>>>(reinterpret_cast<const uint4*>(src), idx, n16, reinterpret_cast<uint4*>(dst));
  return orn_launch_check(ctx, "gather_rows16");
}

int k_linear_plain(orn_ctx* ctx, cudaStream_t s, const orn_linear* L, const void* x, bool x_f32, int ldx, int rows, const DenseJob& j) {
  if (L->kind != ORN_BF16 || L->E != 1) ORN_FAIL(ctx, ORN_ERR_ARG, "plain product: dense bf16 weights only");
  const int gx = (L->O + kPlTile - 1) / kPlTile;
  for (int r0 = 0; r0 < rows; r0 += kPlTile * 32768) {  // the grid's second axis is 16-bit
    const int n = std::min(rows - r0, kPlTile * 32768);
    const dim3 grid(gx, (n + kPlTile - 1) / kPlTile);
    const LinDev D = lin_dev(L);
    const float* xf = reinterpret_cast<const float*>(x) + (size_t)r0 * ldx;
    const bf16_t* xb = reinterpret_cast<const bf16_t*>(x) + (size_t)r0 * ldx;
    float* yf = reinterpret_cast<float*>(j.y) + (size_t)r0 * j.ldy;
    bf16_t* yb = reinterpret_cast<bf16_t*>(j.y) + (size_t)r0 * j.ldy;
    const float* mf = j.mul ? reinterpret_cast<const float*>(j.mul) + (size_t)r0 * j.ldy : nullptr;
    const bf16_t* mb = j.mul ? reinterpret_cast<const bf16_t*>(j.mul) + (size_t)r0 * j.ldy : nullptr;
    if (x_f32) {
      linear_plain_kernel<float, float><<<grid, 256, 0, s>>>(D, xf, ldx, n, yf, j.ldy, j.bias, j.act, mf);
    } else if (j.out_f32) {
      linear_plain_kernel<bf16_t, float><<<grid, 256, 0, s>>>(D, xb, ldx, n, yf, j.ldy, j.bias, j.act, mb);
    } else {
      linear_plain_kernel<bf16_t, bf16_t><<<grid, 256, 0, s>>>(D, xb, ldx, n, yb, j.ldy, j.bias, j.act, mb);
    }
    const int rc = orn_launch_check(ctx, "linear_plain");
    if (rc != ORN_OK) return rc;
  }
  return ORN_OK;
}

bool decode_dense_fits(const DecodePrologue& p, int M) { return decode_smem(p, M) <= kDecSmemMax; }

int f_decode_dense(orn_ctx* ctx, cudaStream_t s, int M, const DecodePrologue& p, const DenseJob* jobs, int njobs) {
  if (M < 1 || M > 4 || njobs < 1 || njobs > kDecJobs) ORN_FAIL(ctx, ORN_ERR_ARG, "decode product: 1..4 rows, 1..8 matrices");
  const size_t smem = decode_smem(p, M);
  if (smem > kDecSmemMax) ORN_FAIL(ctx, ORN_ERR_ARG, "decode product: rows do not fit shared memory");
  DecParams P;
  P.p = p;
  P.Kp = decode_row(p);
  P.njobs = njobs;
  if (p.mode == DRO_EMBED) P.table = lin_dev(p.table);
  if (p.mode == DRO_ROWS && (p.ldx % 8 || p.ldx < P.Kp)) ORN_FAIL(ctx, ORN_ERR_ARG, "decode product: row stride");
  if (p.mode == DRO_RESIDUAL && p.r.ld != P.Kp) ORN_FAIL(ctx, ORN_ERR_ARG, "decode product: residual stride");
  if (p.mode == DRO_POSTNORM && p.pn.ld != P.Kp) ORN_FAIL(ctx, ORN_ERR_ARG, "decode product: residual stride");
  if (p.mode == DRO_GATED && (p.gg.group < 1 || p.gg.n % p.gg.group || (p.gg.act != ACT_SILU && p.gg.act != ACT_SIGMOID) || p.gg.ldo % 8 || p.gg.ldg % 8 || (p.K > 0 && (p.ldx % 8 || p.ldx < pad8(p.K)))))
    ORN_FAIL(ctx, ORN_ERR_ARG, "decode product: gated rows");
  long total = 0;
  bool pairs = false;
  for (int j = 0; j < njobs; ++j) {
    const orn_linear* L = jobs[j].lin;
    const bool whole = p.mode != DRO_GATED;  // every matrix takes the whole staged row
    if (L->kind != ORN_BF16 || L->E != 1 || jobs[j].x0 % 8 || (whole ? L->K != P.Kp || jobs[j].x0 != 0 : L->K % 8 || jobs[j].x0 + L->K > P.Kp))
      ORN_FAIL(ctx, ORN_ERR_ARG, "decode product: bf16 matrices over the staged rows");
    const orn_linear* L2 = jobs[j].lin2;
    if (L2 != nullptr && (L2->kind != ORN_BF16 || L2->E != 1 || L2->K != L->K || L2->O != L->O || L2->rec != L->rec))
      ORN_FAIL(ctx, ORN_ERR_ARG, "decode product: a gated pair's matrices differ in shape");
    pairs = pairs || L2 != nullptr;
    total += L2 != nullptr ? 2 * (long)L->O : L->O;
  }
  const int fit = (int)std::max<size_t>(1, std::min<size_t>(2, (220 * 1024) / (smem + 2048)));
  // rows per warp: two where that costs no extra round over the GPU's warps
  const long warps = (long)fit * ctx->sm_count * kDecWarps;
  const int R = pairs || 2 * ((total + 2 * warps - 1) / (2 * warps)) <= (total + warps - 1) / warps ? 2 : 1;
  P.tasks = 0;
  for (int j = 0; j < njobs; ++j) {
    DecJobDev& D = P.job[j];
    const orn_linear* L = jobs[j].lin;
    D.w2 = jobs[j].lin2 != nullptr ? jobs[j].lin2->w : nullptr;
    D.step = D.w2 != nullptr ? 1 : R; D.n16 = L->K / 8; D.x0 = jobs[j].x0;
    D.w = L->w; D.rec = L->rec; D.O = L->O; D.task0 = P.tasks; D.y = jobs[j].y; D.ldy = jobs[j].ldy;
    D.out_f32 = jobs[j].out_f32 ? 1 : 0; D.bias = jobs[j].bias; D.act = jobs[j].act;
    P.tasks += (L->O + D.step - 1) / D.step;
  }
  const int grid = std::min((P.tasks + kDecWarps - 1) / kDecWarps, fit * ctx->sm_count);
  const char* label = "decode_dense";
  if (ctx->kt != nullptr) {  // per-kernel timing: one label per shape
    static std::mutex mu;
    static std::set<std::string> pool;
    std::string t = "decode_dense M=" + std::to_string(M) + " kind=3 " + std::to_string(total) + "x" + std::to_string(jobs[0].lin->K);
    std::lock_guard<std::mutex> lock(mu);
    label = pool.insert(t).first->c_str();
  }
#define ORN_DEC_PF(M_, PF_)                                                       \
  return R == 2 ? launch_decode<M_, 2, 4, PF_>(ctx, s, P, grid, smem, label)      \
                : launch_decode<M_, 1, 8, PF_>(ctx, s, P, grid, smem, label)
#define ORN_DEC(M_)                                                               \
  case M_:                                                                        \
    if (p.mode == DRO_POSTNORM) ORN_DEC_PF(M_, PF_POSTNORM);                      \
    if (p.mode == DRO_GATED) ORN_DEC_PF(M_, PF_GATED);                            \
    ORN_DEC_PF(M_, PF_STREAM)
  switch (M) {
    ORN_DEC(1);
    ORN_DEC(2);
    ORN_DEC(3);
    ORN_DEC(4);
  }
#undef ORN_DEC
#undef ORN_DEC_PF
  return ORN_ERR_ARG;
}
