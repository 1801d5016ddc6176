// Dense layers with bf16 weights around a float32 residual stream.
//
// Three forms of a product y = act(x W^T + bias):
//   * k_linear_plain: float32 accumulation in k order on CUDA cores, float32 or bf16 activations: the
//     control path, and the only path of a model that runs in float32;
//   * f_decode_dense: windows of 1..4 rows.  One kernel rebuilds its input rows in shared memory
//     (embedding lookup; or the previous sublayer's gate, norm, residual add and depth average; or a
//     plain load) and multiplies up to four matrices by them, weights streamed once with 16-byte
//     loads whose first batch is requested before the kernel waits for its predecessor;
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
__global__ void __launch_bounds__(kRowThreads) embed_rows_kernel(LinDev E, const uint32_t* __restrict__ ids, int width, int ld,
                                                                 float* __restrict__ x, float* __restrict__ stream0, TA* __restrict__ act) {
  const uint32_t id = min(ids[blockIdx.x], (uint32_t)(E.O - 1));
  const bf16_t* row = reinterpret_cast<const bf16_t*>(E.w + (size_t)id * E.rec);
  const size_t base = (size_t)blockIdx.x * ld;
  for (int d = threadIdx.x; d < ld; d += kRowThreads) {
    const float v = d < width ? bf2f(row[d]) : 0.f;
    x[base + d] = v;
    stream0[base + d] = v;
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
                                                           int ldy, const bf16_t* __restrict__ bias, ActParams act) {
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
      if (m < rows && o < L.O)
        y[(size_t)m * ldy + o] = to_act<TY>(act_apply(act.kind, acc[i][j] + (bias != nullptr ? bf2f(bias[o]) : 0.f), pa, pb));
    }
}

// ------------------------------------------------------------------ decode windows
constexpr int kDecThreads = 256;
constexpr int kDecWarps = kDecThreads / 32;
constexpr size_t kDecSmemMax = 200 * 1024;
constexpr int kDecRegs = 4;  // a residual row of up to kDecRegs * 1024 entries stays in registers

struct DecJobDev {
  const uint8_t* w;
  uint32_t rec;
  int O, task0;
  void* y;
  int ldy, out_f32;
  const bf16_t* bias;
  ActParams act;
};
struct DecParams {
  DecodePrologue p;
  LinDev table;
  int njobs, tasks, Kp;  // Kp: K rounded up to 8
  DecJobDev job[4];
};

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
        const float4 lo = make_float4(bflo(u.x), bfhi(u.x), bflo(u.y), bfhi(u.y)), hi = make_float4(bflo(u.z), bfhi(u.z), bflo(u.w), bfhi(u.w));
        const size_t at = (size_t)m * Kp + 8 * c;
        *reinterpret_cast<uint4*>(xs + 8 * c) = u;
        *reinterpret_cast<float4*>(f + 8 * c) = lo;
        *reinterpret_cast<float4*>(f + 8 * c + 4) = hi;
        if (lead) {
          *reinterpret_cast<float4*>(p.x_out + at) = lo;
          *reinterpret_cast<float4*>(p.x_out + at + 4) = hi;
          *reinterpret_cast<float4*>(p.stream_out + at) = lo;
          *reinterpret_cast<float4*>(p.stream_out + at + 4) = hi;
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
template <int M, int R, int U>
__global__ void __launch_bounds__(kDecThreads) decode_dense_kernel(const __grid_constant__ DecParams P) {
  extern __shared__ __align__(16) uint8_t s_raw[];
  __shared__ float red[33], s_act[4][2];
  bf16_t* s_x = reinterpret_cast<bf16_t*>(s_raw);
  float* s_f = reinterpret_cast<float*>(s_raw + (((size_t)M * P.Kp * 2 + 15) & ~(size_t)15));
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int n16 = P.Kp / 8;  // 16-byte pieces per row
  int task = blockIdx.x * kDecWarps + warp;
  const int stride = gridDim.x * kDecWarps;
  uint4 buf[R][U];
  int j = 0, o0 = 0;
  auto locate = [&](int t) {
    j = 0;
    while (j + 1 < P.njobs && t >= P.job[j + 1].task0) ++j;
    o0 = (t - P.job[j].task0) * R;
  };
  auto load = [&](int c0) {
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const uint8_t* row = P.job[j].w + (size_t)min(o0 + r, P.job[j].O - 1) * P.job[j].rec;
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
  decode_prologue<M>(P, s_x, s_f, red);
  for (; task < P.tasks; task += stride) {
    float acc[R][M];
#pragma unroll
    for (int r = 0; r < R; ++r)
#pragma unroll
      for (int m = 0; m < M; ++m) acc[r][m] = 0.f;
    for (int c0 = 0; c0 < n16; c0 += 32 * U) {
      if (c0 > 0) load(c0);
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int c = c0 + 32 * u + lane;
        const int cs = min(c, n16 - 1);  // weights beyond the row are zeros
#pragma unroll
        for (int m = 0; m < M; ++m) {
          const uint4 xv = *reinterpret_cast<const uint4*>(s_x + (size_t)m * P.Kp + 8 * cs);
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
    float mine = 0.f;
    int mr = 0, mm = 0;
#pragma unroll
    for (int r = 0; r < R; ++r)
#pragma unroll
      for (int m = 0; m < M; ++m)
        if (lane == r * M + m) { mine = acc[r][m]; mr = r; mm = m; }
    if (lane < R * M && oo + mr < J.O) {
      const int o = oo + mr;
      const float v = act_apply(J.act.kind, mine + (J.bias != nullptr ? bf2f(J.bias[o]) : 0.f), s_act[jj][0], s_act[jj][1]);
      if (J.out_f32) reinterpret_cast<float*>(J.y)[(size_t)mm * J.ldy + o] = v;
      else reinterpret_cast<bf16_t*>(J.y)[(size_t)mm * J.ldy + o] = f2bf(v);
    }
  }
}

size_t decode_smem(const DecodePrologue& p, int M) {
  const size_t Kp = pad8(p.K);
  return (((size_t)M * Kp * 2 + 15) & ~(size_t)15) + (p.mode == DRO_ROWS ? 0 : Kp * 4);
}

template <int M, int R, int U>
int launch_decode(orn_ctx* ctx, cudaStream_t s, const DecParams& P, int grid, size_t smem, const char* label) {
  if (smem > 48 * 1024) {
    const int rc = orn_grant_smem(ctx, reinterpret_cast<const void*>(decode_dense_kernel<M, R, U>), kDecSmemMax);
    if (rc != ORN_OK) return rc;
  }
  ORN_CHECK_CUDA(ctx, orn_launch_dependent(ctx, s, 0, decode_dense_kernel<M, R, U>, dim3(grid), dim3(kDecThreads), smem, P));
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

int k_layer_norm_rows(orn_ctx* ctx, cudaStream_t s, const float* x, int rows, int width, int ld, const bf16_t* w, float eps, void* out,
                      bool act_f32) {
  if (act_f32) layer_norm_rows_kernel<float><<<rows, kRowThreads, 0, s>>>(x, width, ld, w, eps, reinterpret_cast<float*>(out));
  else layer_norm_rows_kernel<bf16_t><<<rows, kRowThreads, 0, s>>>(x, width, ld, w, eps, reinterpret_cast<bf16_t*>(out));
  return orn_launch_check(ctx, "layer_norm_rows");
}

int k_embed_rows(orn_ctx* ctx, cudaStream_t s, const orn_linear* table, const uint32_t* ids, int rows, int width, int ld, float* x,
                 float* stream0, void* act, bool act_f32) {
  if (act_f32)
    embed_rows_kernel<float><<<rows, kRowThreads, 0, s>>>(lin_dev(table), ids, width, ld, x, stream0, reinterpret_cast<float*>(act));
  else
    embed_rows_kernel<bf16_t><<<rows, kRowThreads, 0, s>>>(lin_dev(table), ids, width, ld, x, stream0, reinterpret_cast<bf16_t*>(act));
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
    if (x_f32) {
      linear_plain_kernel<float, float><<<grid, 256, 0, s>>>(D, xf, ldx, n, yf, j.ldy, j.bias, j.act);
    } else if (j.out_f32) {
      linear_plain_kernel<bf16_t, float><<<grid, 256, 0, s>>>(D, xb, ldx, n, yf, j.ldy, j.bias, j.act);
    } else {
      linear_plain_kernel<bf16_t, bf16_t><<<grid, 256, 0, s>>>(D, xb, ldx, n, yb, j.ldy, j.bias, j.act);
    }
    const int rc = orn_launch_check(ctx, "linear_plain");
    if (rc != ORN_OK) return rc;
  }
  return ORN_OK;
}

bool decode_dense_fits(const DecodePrologue& p, int M) { return decode_smem(p, M) <= kDecSmemMax; }

int f_decode_dense(orn_ctx* ctx, cudaStream_t s, int M, const DecodePrologue& p, const DenseJob* jobs, int njobs) {
  if (M < 1 || M > 4 || njobs < 1 || njobs > 4) ORN_FAIL(ctx, ORN_ERR_ARG, "decode product: 1..4 rows, 1..4 matrices");
  const size_t smem = decode_smem(p, M);
  if (smem > kDecSmemMax) ORN_FAIL(ctx, ORN_ERR_ARG, "decode product: rows do not fit shared memory");
  DecParams P;
  P.p = p;
  P.Kp = pad8(p.K);
  P.njobs = njobs;
  if (p.mode == DRO_EMBED) P.table = lin_dev(p.table);
  if (p.mode == DRO_ROWS && (p.ldx % 8 || p.ldx < P.Kp)) ORN_FAIL(ctx, ORN_ERR_ARG, "decode product: row stride");
  if (p.mode == DRO_RESIDUAL && p.r.ld != P.Kp) ORN_FAIL(ctx, ORN_ERR_ARG, "decode product: residual stride");
  long total = 0;
  for (int j = 0; j < njobs; ++j) {
    const orn_linear* L = jobs[j].lin;
    if (L->kind != ORN_BF16 || L->E != 1 || L->K != P.Kp) ORN_FAIL(ctx, ORN_ERR_ARG, "decode product: bf16 matrices over the staged rows");
    total += L->O;
  }
  const int fit = (int)std::max<size_t>(1, std::min<size_t>(2, (220 * 1024) / (smem + 2048)));
  // rows per warp: two where that costs no extra round over the GPU's warps
  const long warps = (long)fit * ctx->sm_count * kDecWarps;
  const int R = 2 * ((total + 2 * warps - 1) / (2 * warps)) <= (total + warps - 1) / warps ? 2 : 1;
  P.tasks = 0;
  for (int j = 0; j < njobs; ++j) {
    DecJobDev& D = P.job[j];
    const orn_linear* L = jobs[j].lin;
    D.w = L->w; D.rec = L->rec; D.O = L->O; D.task0 = P.tasks; D.y = jobs[j].y; D.ldy = jobs[j].ldy;
    D.out_f32 = jobs[j].out_f32 ? 1 : 0; D.bias = jobs[j].bias; D.act = jobs[j].act;
    P.tasks += (L->O + R - 1) / R;
  }
  const int grid = std::min((P.tasks + kDecWarps - 1) / kDecWarps, fit * ctx->sm_count);
  const char* label = "decode_dense";
  if (ctx->kt != nullptr) {  // per-kernel timing: one label per shape
    static std::mutex mu;
    static std::set<std::string> pool;
    std::string t = "decode_dense M=" + std::to_string(M) + " kind=3 " + std::to_string(total) + "x" + std::to_string(p.K);
    std::lock_guard<std::mutex> lock(mu);
    label = pool.insert(t).first->c_str();
  }
#define ORN_DEC(M_)                                                              \
  case M_:                                                                       \
    return R == 2 ? launch_decode<M_, 2, 4>(ctx, s, P, grid, smem, label)        \
                  : launch_decode<M_, 1, 8>(ctx, s, P, grid, smem, label)
  switch (M) {
    ORN_DEC(1);
    ORN_DEC(2);
    ORN_DEC(3);
    ORN_DEC(4);
  }
#undef ORN_DEC
  return ORN_ERR_ARG;
}
