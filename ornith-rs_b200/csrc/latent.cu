// Latent attention: keys and values are linear images of one small latent per position, so the cache
// holds the latent c (RMS-normed) and one rotated key part that all heads share.
//
//   score(t, j, h) = (q_u[t,h] . W_uk[h] c_j + q_r[t,h] . k_r[j]) * scale
//   out(t, h)      = W_uv[h] (sum_j softmax_j c_j) * sigmoid(gate[t,h])
//
// Two forms, equal to rounding:
//   * absorbed: W_uk[h]^T q_u is taken first; all heads then attend to the cache rows [c | k_r] as to
//     one shared key, whose leading part is also the value.  A position costs its cache row once for all
//     heads: decode windows and short portions.  Scores and sums run on the tensor cores with the
//     (row, head) pairs as the M side and the keys split over CTAs, or in a plain kernel (the control
//     path, float32 models, sizes the tensor form does not take);
//   * expanded: keys and values of every cached position are multiplied out by the tensor-core product
//     and attended to head by head with an online softmax: prompt chunks.
#include <algorithm>

#include "latent.h"
#include "mma_bf16.cuh"
#include "act.cuh"

namespace {

constexpr float kLog2e = 1.4426950408889634f;

// entry i of a rotated vector v of n entries, the first `dims` in neighbouring pairs
template <typename F>
ORN_D float rotated(int i, int dims, float position, const float* freq, F v) {
  if (i >= dims) return v(i);
  float sn, cs;
  sincosf(position * freq[i >> 1], &sn, &cs);
  const float u = v(i & ~1), w = v(i | 1);
  return (i & 1) ? fmaf(w, cs, u * sn) : fmaf(u, cs, -(w * sn));
}

constexpr int kLrThreads = 128;

ORN_D float block_sum_lr(float v, float* red) {
  v = warp_sum(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  return red[0] + red[1] + red[2] + red[3];
}

template <typename TA>
ORN_D void append_row(const LatentDims& D, const float* __restrict__ y, const bf16_t* __restrict__ norm_w, int position, TA* row, float* red) {
  const int R = D.kv_rank, RP = D.rp(), ROW = D.row();
  float sq = 0.f;
  for (int i = threadIdx.x; i < R; i += kLrThreads) { const float v = __ldcg(y + i); sq = fmaf(v, v, sq); }
  const float rstd = 1.0f / sqrtf(block_sum_lr(sq, red) / (float)R + D.eps);
  for (int i = threadIdx.x; i < RP; i += kLrThreads) row[i] = to_act<TA>(i < R ? __ldcg(y + i) * rstd * bf2f(norm_w[i]) : 0.f);
  for (int i = threadIdx.x; i < ROW - RP; i += kLrThreads)
    row[RP + i] = to_act<TA>(i < D.rot_dim ? rotated(i, D.rot_dims, (float)position, D.freq, [&](int e) { return __ldcg(y + R + e); }) : 0.f);
}

// grid (T): append the row, rotate its q
template <typename TA>
__global__ void __launch_bounds__(kLrThreads) latent_rows_kernel(LatentDims D, const float* __restrict__ kv, int ldkv,
                                                                 const bf16_t* __restrict__ norm_w, TA* __restrict__ cache, int cap,
                                                                 const int* __restrict__ pos, TA* __restrict__ q, int ldq, int rotate_q) {
  __shared__ float red[4];
  const int t = blockIdx.x, p = *pos + t;
  if (kv != nullptr && p < cap) append_row<TA>(D, kv + (size_t)t * ldkv, norm_w, p, cache + (size_t)p * D.row(), red);
  if (!rotate_q) return;
  const int half = D.rot_dims / 2;
  for (int i = threadIdx.x; i < D.heads * half; i += kLrThreads) {
    const int h = i / half, e = i - h * half;
    TA* v = q + (size_t)t * ldq + h * D.qk() + D.dim + 2 * e;
    float sn, cs;
    sincosf((float)p * D.freq[e], &sn, &cs);
    const float a = from_act(v[0]), b = from_act(v[1]);
    v[0] = to_act<TA>(fmaf(a, cs, -(b * sn)));
    v[1] = to_act<TA>(fmaf(b, cs, a * sn));
  }
}

// ------------------------------------------------------------------ absorbed form: queries
// CTAs [0, T*H*chunks): (t, h, 128 latent entries); then T appends (kv != null); then the stream sum.
constexpr int kAbCols = 128;

template <typename TA>
__global__ void __launch_bounds__(kLrThreads) latent_absorb_kernel(LatentDims D, int T, int chunks, const TA* __restrict__ q, int ldq, LinDev uk,
                                                                   const float* __restrict__ kv, int ldkv,
                                                                   const bf16_t* __restrict__ norm_w, TA* __restrict__ cache, int cap,
                                                                   const int* __restrict__ pos, TA* __restrict__ qa, StreamSum S) {
  extern __shared__ float s_q[];  // [dim]
  __shared__ float s_part[4][kAbCols];
  __shared__ float red[4];
  const int nq = T * D.heads * chunks;
  int b = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  // the head's first rows do not depend on the kernel before this one
  constexpr int kPre = 16;
  uint2 pre[kPre];
  if (b < nq) {
    const int h = (b / chunks) % D.heads, r0 = (b % chunks) * kAbCols + 4 * lane;
#pragma unroll
    for (int k = 0; k < kPre; ++k) {
      const int i = warp + 4 * k;
      pre[k] = i < D.dim && r0 < D.rp() ? __ldg(reinterpret_cast<const uint2*>(uk.w + (size_t)(h * D.dim + i) * uk.rec + 2 * (size_t)r0)) : make_uint2(0, 0);
    }
  }
  pdl_wait();
  pdl_trigger();
  if (b < nq) {
    const int c = b % chunks, h = (b / chunks) % D.heads, t = b / (chunks * D.heads);
    const TA* qr = q + (size_t)t * ldq + (size_t)h * D.qk();
    TA* out = qa + ((size_t)t * D.heads + h) * D.row();
    for (int i = threadIdx.x; i < D.dim; i += kLrThreads) s_q[i] = from_act(__ldcg(qr + i));
    if (c == 0) {
      const int RP = D.rp(), n = D.row() - RP;
      const float p = (float)(*pos + t);
      for (int i = threadIdx.x; i < n; i += kLrThreads)
        out[RP + i] = to_act<TA>(i < D.rot_dim ? rotated(i, D.rot_dims, p, D.freq, [&](int e) { return from_act(__ldcg(qr + D.dim + e)); }) : 0.f);
    }
    __syncthreads();
    const int r0 = c * kAbCols + 4 * lane;  // four latent entries per lane, a quarter of the head's rows per warp
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    if (r0 < D.rp()) {
      const uint8_t* w = uk.w + (size_t)(h * D.dim) * uk.rec + 2 * (size_t)r0;
      auto add = [&](const uint2& u, float x) {
        acc[0] = fmaf(x, __uint_as_float(u.x << 16), acc[0]);
        acc[1] = fmaf(x, __uint_as_float(u.x & 0xffff0000u), acc[1]);
        acc[2] = fmaf(x, __uint_as_float(u.y << 16), acc[2]);
        acc[3] = fmaf(x, __uint_as_float(u.y & 0xffff0000u), acc[3]);
      };
      uint2 nxt[kPre];  // the rows after those, all in flight before the first is used
#pragma unroll
      for (int k = 0; k < kPre; ++k) {
        const int i = warp + 4 * (kPre + k);
        nxt[k] = i < D.dim ? __ldg(reinterpret_cast<const uint2*>(w + (size_t)i * uk.rec)) : make_uint2(0, 0);
      }
#pragma unroll
      for (int k = 0; k < kPre; ++k)
        if (warp + 4 * k < D.dim) add(pre[k], s_q[warp + 4 * k]);
#pragma unroll
      for (int k = 0; k < kPre; ++k)
        if (warp + 4 * (kPre + k) < D.dim) add(nxt[k], s_q[warp + 4 * (kPre + k)]);
#pragma unroll 8
      for (int i = warp + 8 * kPre; i < D.dim; i += 4) {
        const uint2 u = __ldg(reinterpret_cast<const uint2*>(w + (size_t)i * uk.rec));
        add(u, s_q[i]);
      }
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) s_part[warp][4 * lane + e] = acc[e];
    __syncthreads();
    const int r = c * kAbCols + threadIdx.x;
    if (r < D.rp()) out[r] = to_act<TA>((s_part[0][threadIdx.x] + s_part[1][threadIdx.x]) + (s_part[2][threadIdx.x] + s_part[3][threadIdx.x]));
    return;
  }
  b -= nq;
  if (kv != nullptr) {
    if (b < T) {
      const int p = *pos + b;
      if (p < cap) append_row<TA>(D, kv + (size_t)b * ldkv, norm_w, p, cache + (size_t)p * D.row(), red);
      return;
    }
    b -= T;
  }
  const int i = 4 * (b * kLrThreads + threadIdx.x);
  if (i < S.count) {
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
    for (int j = 0; j < S.n; ++j) {
      const float a = bf2f(S.a[j]);
      const float4 v = __ldcg(reinterpret_cast<const float4*>(S.streams + j * S.stride + i));
      acc.x = fmaf(a, v.x, acc.x); acc.y = fmaf(a, v.y, acc.y); acc.z = fmaf(a, v.z, acc.z); acc.w = fmaf(a, v.w, acc.w);
    }
    *reinterpret_cast<float4*>(S.out + i) = acc;
  }
}

// ------------------------------------------------------------------ absorbed form: attention
// keys [k0, k1) of split sp, for n visible positions
ORN_D int split_keys(int n, int splits) { return max(64, (((n + splits - 1) / splits) + 63) & ~63); }

// control path: one CTA per (row, head), all keys; scores of a tile, then every thread its share of c
constexpr int kPaThreads = 256, kPaTile = 256;
template <typename TA>
__global__ void __launch_bounds__(kPaThreads) latent_attn_plain_kernel(LatentDims D, const TA* __restrict__ qa, const TA* __restrict__ cache,
                                                                       int cap, const int* __restrict__ pos, float* __restrict__ partial,
                                                                       float* __restrict__ ml) {
  extern __shared__ float s_mem[];  // q [row], o [kv_rank], p [tile]
  __shared__ float red[kPaThreads / 32];
  const int ROW = D.row(), R = D.kv_rank;
  float *s_q = s_mem, *s_o = s_mem + ROW, *s_p = s_o + R;
  const int rh = blockIdx.x, t = rh / D.heads;
  const int n = min(cap, *pos + t + 1);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  for (int i = threadIdx.x; i < ROW; i += kPaThreads) s_q[i] = from_act(qa[(size_t)rh * ROW + i]);
  for (int i = threadIdx.x; i < R; i += kPaThreads) s_o[i] = 0.f;
  float m = -INFINITY, l = 0.f;
  for (int k0 = 0; k0 < n; k0 += kPaTile) {
    __syncthreads();
    for (int k = warp; k < kPaTile; k += kPaThreads / 32) {  // one warp per key
      float s = 0.f;
      if (k0 + k < n) {
        const TA* row = cache + (size_t)(k0 + k) * ROW;
        for (int i = lane; i < ROW; i += 32) s = fmaf(s_q[i], from_act(row[i]), s);
      }
      s = warp_sum(s);
      if (lane == 0) s_p[k] = k0 + k < n ? s * D.scale * kLog2e : -INFINITY;
    }
    __syncthreads();
    const float mine = s_p[threadIdx.x];
    float x = warp_max(mine);
    if (lane == 0) red[warp] = x;
    __syncthreads();
    x = red[0];
#pragma unroll
    for (int i = 1; i < kPaThreads / 32; ++i) x = fmaxf(x, red[i]);
    const float mn = fmaxf(m, x), c = exp2f(m - mn), p = exp2f(mine - mn);
    float ps = warp_sum(p);
    __syncthreads();
    s_p[threadIdx.x] = p;
    if (lane == 0) red[warp] = ps;
    __syncthreads();
    ps = 0.f;
#pragma unroll
    for (int i = 0; i < kPaThreads / 32; ++i) ps += red[i];
    l = fmaf(l, c, ps);
    m = mn;
    const int kn = min(kPaTile, n - k0);
    for (int i = threadIdx.x; i < R; i += kPaThreads) {
      float o = s_o[i] * c;
      for (int k = 0; k < kn; ++k) o = fmaf(s_p[k], from_act(cache[(size_t)(k0 + k) * ROW + i]), o);
      s_o[i] = o;
    }
  }
  for (int i = threadIdx.x; i < R; i += kPaThreads) partial[(size_t)rh * R + i] = s_o[i];
  if (threadIdx.x == 0) { ml[2 * rh] = m; ml[2 * rh + 1] = l; }
}

// tensor-core form: a CTA takes 16 (row, head) pairs and one range of keys; 8 warps.
// Per tile of 64 keys: warp w scores keys 8w..8w+7 over the whole row, the warps agree on the new row
// maxima through shared memory, and each adds its 16-column groups of sum_j p_j c_j.
constexpr int kLaWarps = 8, kLaKeys = 64;
template <int NG>  // 16-column groups of the latent per warp
__global__ void __launch_bounds__(kLaWarps * 32) latent_attn_kernel(LatentDims D, int T, const bf16_t* __restrict__ qa,
                                                                    const bf16_t* __restrict__ cache, int cap,
                                                                    const int* __restrict__ pos, int splits,
                                                                    float* __restrict__ partial, float* __restrict__ ml) {
  extern __shared__ __align__(128) uint8_t lsm[];
  __shared__ float s_max[kLaWarps][16], s_sum[kLaWarps][16];
  pdl_wait();
  pdl_trigger();
  const int ROW = D.row(), KD = (ROW + 31) & ~31, rowB = 2 * (KD + 8), pieces = KD / 8;
  const int rows = T * D.heads, r0 = blockIdx.x * 16;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, qd = lane & 3;
  const int p0 = *pos, n = min(cap, p0 + T);
  const int kps = split_keys(n, splits);
  const int k0 = blockIdx.y * kps, k1 = min(n, k0 + kps);
  if (k0 >= k1) return;
  const int tiles = (k1 - k0 + kLaKeys - 1) / kLaKeys;
  const uint32_t q_s = smem_u32(lsm), p_s = q_s + 16 * rowB, c_s = p_s + 16 * (2 * (kLaKeys + 8));
  constexpr int pB = 2 * (kLaKeys + 8);
  for (int i = threadIdx.x; i < 16 * pieces; i += blockDim.x) {
    const int r = i / pieces, c = i - r * pieces;
    const bool ok = r0 + r < rows && 8 * c < ROW;
    cp_async16(q_s + r * rowB + 16 * c, qa + (ok ? (size_t)(r0 + r) * ROW + 8 * c : 0), ok ? 16 : 0);
  }
  auto issue = [&](int i) {
    const uint32_t dst = c_s + (i & 1) * kLaKeys * rowB;
    for (int it = threadIdx.x; it < kLaKeys * pieces; it += blockDim.x) {
      const int r = it / pieces, c = it - r * pieces;
      const int key = k0 + i * kLaKeys + r;
      const bool ok = key < k1 && 8 * c < ROW;
      cp_async16(dst + r * rowB + 16 * c, cache + (ok ? (size_t)key * ROW + 8 * c : 0), ok ? 16 : 0);
    }
    cp_async_commit();
  };
  issue(0);
  float o[2 * NG][4];
#pragma unroll
  for (int i = 0; i < 2 * NG; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;
  const float sc2 = D.scale * kLog2e;
  const int ra = r0 + g, rb = ra + 8;
  const int lim0 = ra < rows ? p0 + ra / D.heads + 1 : 0, lim1 = rb < rows ? p0 + rb / D.heads + 1 : 0;  // keys below are visible
  const uint32_t a_off = ((lane & 7) + 8 * ((lane >> 3) & 1)) * rowB + 16 * (lane >> 4);
  const uint32_t k_off = (8 * warp + (lane & 7)) * rowB + 16 * (lane >> 3);   // x4: four 8-wide k pieces of 8 keys
  const uint32_t pa_off = ((lane & 7) + 8 * ((lane >> 3) & 1)) * pB + 16 * (lane >> 4);
  const uint32_t v_off = ((lane & 7) + 8 * ((lane >> 3) & 1)) * rowB + 16 * (lane >> 4);
  const int groups = (D.kv_rank + 15) / 16;
  for (int i = 0; i < tiles; ++i) {
    if (i + 1 < tiles) {
      issue(i + 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const uint32_t ct = c_s + (i & 1) * kLaKeys * rowB;
    float sa[4] = {0.f, 0.f, 0.f, 0.f}, sb[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 4
    for (int kk = 0; kk < KD / 32; ++kk) {
      uint32_t a[4], b[4];
      ldsm4(ct + k_off + 64 * kk, b);
      ldsm4(q_s + a_off + 64 * kk, a);
      mma16816(sa, a, b[0], b[1]);
      ldsm4(q_s + a_off + 64 * kk + 32, a);
      mma16816(sb, a, b[2], b[3]);
    }
    const int key = k0 + i * kLaKeys + 8 * warp + 2 * qd;
    float s[4];
#pragma unroll
    for (int c = 0; c < 4; ++c) {
      const int kc = key + (c & 1);
      s[c] = (kc < k1 && kc < (c < 2 ? lim0 : lim1)) ? (sa[c] + sb[c]) * sc2 : -INFINITY;
    }
    float x0 = fmaxf(s[0], s[1]), x1 = fmaxf(s[2], s[3]);
    x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, 1)); x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, 2));
    x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, 1)); x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, 2));
    if (qd == 0) { s_max[warp][g] = x0; s_max[warp][g + 8] = x1; }
    __syncthreads();
    float n0 = m0, n1 = m1;
#pragma unroll
    for (int w = 0; w < kLaWarps; ++w) { n0 = fmaxf(n0, s_max[w][g]); n1 = fmaxf(n1, s_max[w][g + 8]); }
    const float u0 = n0 == -INFINITY ? 0.f : n0, u1 = n1 == -INFINITY ? 0.f : n1;
    const float c0 = exp2f(m0 - u0), c1 = exp2f(m1 - u1);
    m0 = n0; m1 = n1;
    const float e0 = exp2f(s[0] - u0), e1 = exp2f(s[1] - u0), e2 = exp2f(s[2] - u1), e3 = exp2f(s[3] - u1);
    l0 = fmaf(l0, c0, e0 + e1);
    l1 = fmaf(l1, c1, e2 + e3);
    {
      uint8_t* pp = lsm + (p_s - q_s) + 2 * (8 * warp + 2 * qd);
      *reinterpret_cast<uint32_t*>(pp + g * pB) = pack_bf16x2(e0, e1);
      *reinterpret_cast<uint32_t*>(pp + (g + 8) * pB) = pack_bf16x2(e2, e3);
    }
#pragma unroll
    for (int j = 0; j < 2 * NG; ++j) { o[j][0] *= c0; o[j][1] *= c0; o[j][2] *= c1; o[j][3] *= c1; }
    __syncthreads();
#pragma unroll
    for (int ks = 0; ks < kLaKeys / 16; ++ks) {
      uint32_t a[4];
      ldsm4(p_s + pa_off + 32 * ks, a);
#pragma unroll
      for (int j = 0; j < NG; ++j) {
        const int gr = warp + kLaWarps * j;
        if (gr < groups) {  // warp-uniform
          uint32_t b[4];
          ldsm4t(ct + v_off + ks * 16 * rowB + 32 * gr, b);
          mma16816(o[2 * j], a, b[0], b[1]);
          mma16816(o[2 * j + 1], a, b[2], b[3]);
        }
      }
    }
    __syncthreads();  // the tile and P are refilled next
  }
  l0 += __shfl_xor_sync(0xffffffffu, l0, 1); l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
  l1 += __shfl_xor_sync(0xffffffffu, l1, 1); l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
  if (qd == 0) { s_sum[warp][g] = l0; s_sum[warp][g + 8] = l1; }
  __syncthreads();
  const int R = D.kv_rank;
#pragma unroll
  for (int j = 0; j < NG; ++j) {
    const int gr = warp + kLaWarps * j;
    if (gr >= groups) continue;
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      const int col = 16 * gr + 8 * hf + 2 * qd;
      if (col >= R) continue;
      const float* v = o[2 * j + hf];
      float* da = partial + ((size_t)ra * splits + blockIdx.y) * R + col;
      float* db = partial + ((size_t)rb * splits + blockIdx.y) * R + col;
      if (ra < rows) { da[0] = v[0]; if (col + 1 < R) da[1] = v[1]; }
      if (rb < rows) { db[0] = v[2]; if (col + 1 < R) db[1] = v[3]; }
    }
  }
  if (warp == 0 && qd == 0) {
    float t0 = 0.f, t1 = 0.f;
#pragma unroll
    for (int w = 0; w < kLaWarps; ++w) { t0 += s_sum[w][g]; t1 += s_sum[w][g + 8]; }
    if (ra < rows) { ml[2 * ((size_t)ra * splits + blockIdx.y)] = m0; ml[2 * ((size_t)ra * splits + blockIdx.y) + 1] = t0; }
    if (rb < rows) { ml[2 * ((size_t)rb * splits + blockIdx.y)] = m1; ml[2 * ((size_t)rb * splits + blockIdx.y) + 1] = t1; }
  }
}

// ------------------------------------------------------------------ absorbed form: output
constexpr int kLoThreads = 256, kLoRows = 32;  // value rows per CTA
constexpr int kLoCols = 512;                   // latent columns per merge pass
template <typename TA>
__global__ void __launch_bounds__(kLoThreads) latent_out_kernel(LatentDims D, int T, LinDev uv, const float* __restrict__ partial,
                                                                const float* __restrict__ ml, int splits, int plain,
                                                                const int* __restrict__ pos, const float* __restrict__ gate, int ldgate,
                                                                TA* __restrict__ att, int ldatt) {
  extern __shared__ float s_c[];  // [rp] merged latent, [splits] weights, [warps][kLoCols] partial sums of a merge pass
  __shared__ float s_tot;
  const int R = D.kv_rank, RP = D.rp();
  const int rh = blockIdx.x, t = rh / D.heads, h = rh - t * D.heads;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int row0 = blockIdx.y * kLoRows + warp, row1 = min(D.vdim, (int)(blockIdx.y + 1) * kLoRows);
  // the first pieces of this warp's value rows do not depend on the kernel before this one
  constexpr int kPre = kLoRows / (kLoThreads / 32);
  uint4 pre[kPre][2];
#pragma unroll
  for (int i = 0; i < kPre; ++i)
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int r = row0 + i * (kLoThreads / 32), c = lane + 32 * u;
      pre[i][u] = r < row1 && c < RP / 8 ? ldg128(uv.w + (size_t)(h * D.vdim + r) * uv.rec + 16 * (size_t)c) : make_uint4(0, 0, 0, 0);
    }
  pdl_wait();
  pdl_trigger();
  float *s_w = s_c + RP, *s_m = s_w + ((splits + 3) & ~3);
  int used = 1;
  if (!plain) {
    const int n = *pos + T;
    const int kps = split_keys(n, splits);
    used = min(splits, (n + kps - 1) / kps);
  }
  const float* mlr = ml + 2 * (size_t)rh * splits;
  if (warp == 0) {
    float m = -INFINITY;
    for (int i = lane; i < used; i += 32) m = fmaxf(m, __ldcg(mlr + 2 * i));
    m = warp_max(m);
    float tot = 0.f;
    for (int i = lane; i < used; i += 32) {
      const float w = exp2f(__ldcg(mlr + 2 * i) - m);
      s_w[i] = w;
      tot = fmaf(w, __ldcg(mlr + 2 * i + 1), tot);
    }
    tot = warp_sum(tot);
    if (lane == 0) s_tot = tot;
  }
  __syncthreads();
  const float inv = 1.0f / s_tot;
  // 512 columns per pass, the splits dealt to the warps; a fixed order of additions
  const float* pr = partial + (size_t)rh * splits * R;
  for (int c0 = 0; c0 < RP; c0 += kLoCols) {
    float a[4][4] = {};
    if ((R & 3) == 0) {
#pragma unroll 4
      for (int sp = warp; sp < used; sp += kLoThreads / 32) {
        const float w = s_w[sp];
        float4 v[4];
#pragma unroll
        for (int g = 0; g < 4; ++g) {
          const int i = c0 + 128 * g + 4 * lane;
          v[g] = i < R ? __ldcg(reinterpret_cast<const float4*>(pr + (size_t)sp * R + i)) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
#pragma unroll
        for (int g = 0; g < 4; ++g) {
          a[g][0] = fmaf(w, v[g].x, a[g][0]); a[g][1] = fmaf(w, v[g].y, a[g][1]);
          a[g][2] = fmaf(w, v[g].z, a[g][2]); a[g][3] = fmaf(w, v[g].w, a[g][3]);
        }
      }
    } else {
      for (int sp = warp; sp < used; sp += kLoThreads / 32)
#pragma unroll
        for (int g = 0; g < 4; ++g)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int i = c0 + 128 * g + 4 * lane + e;
            if (i < R) a[g][e] = fmaf(s_w[sp], __ldcg(pr + (size_t)sp * R + i), a[g][e]);
          }
    }
#pragma unroll
    for (int g = 0; g < 4; ++g)
      *reinterpret_cast<float4*>(s_m + kLoCols * warp + 128 * g + 4 * lane) = make_float4(a[g][0], a[g][1], a[g][2], a[g][3]);
    __syncthreads();
    for (int i = threadIdx.x; i < kLoCols && c0 + i < RP; i += kLoThreads) {
      float v = 0.f;
#pragma unroll
      for (int w = 0; w < kLoThreads / 32; ++w) v += s_m[kLoCols * w + i];
      s_c[c0 + i] = c0 + i < R ? v * inv : 0.f;
    }
    __syncthreads();
  }
  const float gt = sigmoid_f32(__ldcg(gate + (size_t)t * ldgate + h));
#pragma unroll
  for (int k = 0; k < kPre; ++k) {
    const int i = row0 + k * (kLoThreads / 32);
    if (i >= row1) break;  // warp-uniform
    const uint8_t* w = uv.w + (size_t)(h * D.vdim + i) * uv.rec;
    float a = 0.f;
    for (int c = lane, u = 0; c < RP / 8; c += 32, ++u) {
      const uint4 v = u == 0 ? pre[k][0] : u == 1 ? pre[k][1] : ldg128(w + 16 * (size_t)c);
      const float4 x = *reinterpret_cast<const float4*>(s_c + 8 * c), y = *reinterpret_cast<const float4*>(s_c + 8 * c + 4);
      a = fmaf(__uint_as_float(v.x << 16), x.x, a); a = fmaf(__uint_as_float(v.x & 0xffff0000u), x.y, a);
      a = fmaf(__uint_as_float(v.y << 16), x.z, a); a = fmaf(__uint_as_float(v.y & 0xffff0000u), x.w, a);
      a = fmaf(__uint_as_float(v.z << 16), y.x, a); a = fmaf(__uint_as_float(v.z & 0xffff0000u), y.y, a);
      a = fmaf(__uint_as_float(v.w << 16), y.z, a); a = fmaf(__uint_as_float(v.w & 0xffff0000u), y.w, a);
    }
    a = warp_sum(a);
    if (lane == 0) att[(size_t)t * ldatt + (size_t)h * D.vdim + i] = to_act<TA>(a * gt);
  }
}

// ------------------------------------------------------------------ expanded form
constexpr int kLfWarps = 4, kLfRows = 16 * kLfWarps, kLfKeys = 32;
constexpr int kLfTiles = kLfKeys / 8;  // 8-key accumulator tiles per stage

struct FlashArgs {
  const bf16_t *q, *kx, *vx, *cache;
  int ldq, ldk, ldv, cap, T;
  const int* pos;
  const float* gate;
  int ldgate;
  bf16_t* att;
  int ldatt;
  int kd, vd;  // padded widths of the staged key and value rows
};

template <int NV>  // 16-column groups of the value
__global__ void __launch_bounds__(kLfWarps * 32, NV <= 8 ? 3 : 2) latent_flash_kernel(LatentDims D, FlashArgs A) {
  extern __shared__ __align__(128) uint8_t fsm[];
  const int qt = gridDim.x - 1 - blockIdx.x;  // the tiles with the most keys start first
  const int h = blockIdx.y;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, qd = lane & 3;
  const int p0 = *A.pos, r0 = qt * kLfRows, T = A.T;
  const int n = min(A.cap, p0 + min(r0 + kLfRows, T));  // keys any row of this tile sees
  const int tiles = (n + kLfKeys - 1) / kLfKeys;
  const int kB = 2 * (A.kd + 8), vB = 2 * (A.vd + 8);
  const int kp = A.kd / 8, vp = A.vd / 8, dp = D.dim / 8, qkp = D.qk() / 8, vv = D.vdim / 8, RP = D.rp(), ROW = D.row();
  const uint32_t q_s = smem_u32(fsm), st_s = q_s + kLfRows * kB, stage = kLfKeys * (kB + vB);
  for (int i = threadIdx.x; i < kLfRows * kp; i += blockDim.x) {
    const int r = i / kp, c = i - r * kp;
    const bool ok = r0 + r < T && c < qkp;
    cp_async16(q_s + r * kB + 16 * c, A.q + (ok ? (size_t)(r0 + r) * A.ldq + (size_t)h * D.qk() + 8 * c : 0), ok ? 16 : 0);
  }
  auto issue = [&](int i) {
    const uint32_t kt = st_s + (i & 1) * stage, vt = kt + kLfKeys * kB;
    for (int it = threadIdx.x; it < kLfKeys * kp; it += blockDim.x) {
      const int r = it / kp, c = it - r * kp, key = i * kLfKeys + r;
      const bool ok = key < n && c < qkp;
      const bf16_t* src = !ok ? A.kx : c < dp ? A.kx + (size_t)key * A.ldk + (size_t)h * D.dim + 8 * c : A.cache + (size_t)key * ROW + RP + 8 * (c - dp);
      cp_async16(kt + r * kB + 16 * c, src, ok ? 16 : 0);
    }
    for (int it = threadIdx.x; it < kLfKeys * vp; it += blockDim.x) {
      const int r = it / vp, c = it - r * vp, key = i * kLfKeys + r;
      const bool ok = key < n && c < vv;
      cp_async16(vt + r * vB + 16 * c, A.vx + (ok ? (size_t)key * A.ldv + (size_t)h * D.vdim + 8 * c : 0), ok ? 16 : 0);
    }
    cp_async_commit();
  };
  issue(0);
  float o[2 * NV][4];
#pragma unroll
  for (int j = 0; j < 2 * NV; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
  float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;
  const float sc2 = D.scale * kLog2e;
  const int wrow = r0 + 16 * warp;
  const int lim0 = p0 + wrow + g + 1, lim1 = lim0 + 8;
  const int wlast = p0 + wrow + 15;
  const uint32_t a_off = (16 * warp + (lane & 7) + 8 * ((lane >> 3) & 1)) * kB + 16 * (lane >> 4);
  const uint32_t k_off = ((lane & 7) + 8 * (lane >> 4)) * kB + 16 * ((lane >> 3) & 1);
  const uint32_t v_off = ((lane & 7) + 8 * ((lane >> 3) & 1)) * vB + 16 * (lane >> 4);
  for (int i = 0; i < tiles; ++i) {
    if (i + 1 < tiles) {
      issue(i + 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const uint32_t kt = st_s + (i & 1) * stage, vt = kt + kLfKeys * kB;
    const int n0 = i * kLfKeys;
    if (n0 <= wlast) {  // warp-uniform: otherwise every key of this tile is in the future of every row
      float s[kLfTiles][4];
#pragma unroll
      for (int j = 0; j < kLfTiles; ++j) s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.f;
#pragma unroll 4
      for (int kk = 0; kk < A.kd / 16; ++kk) {
        uint32_t a[4];
        ldsm4(q_s + a_off + 32 * kk, a);
#pragma unroll
        for (int j = 0; j < kLfTiles / 2; ++j) {
          uint32_t b[4];
          ldsm4(kt + k_off + j * 16 * kB + 32 * kk, b);
          mma16816(s[2 * j], a, b[0], b[1]);
          mma16816(s[2 * j + 1], a, b[2], b[3]);
        }
      }
      const bool all_visible = n0 + kLfKeys <= p0 + wrow + 1 && n0 + kLfKeys <= n;
      if (!all_visible) {
#pragma unroll
        for (int j = 0; j < kLfTiles; ++j)
#pragma unroll
          for (int c = 0; c < 4; ++c)
            if (n0 + 8 * j + 2 * qd + (c & 1) >= min(n, c < 2 ? lim0 : lim1)) s[j][c] = -INFINITY;
      }
      float x0 = -INFINITY, x1 = -INFINITY;
#pragma unroll
      for (int j = 0; j < kLfTiles; ++j) {
        x0 = fmaxf(x0, fmaxf(s[j][0], s[j][1]));
        x1 = fmaxf(x1, fmaxf(s[j][2], s[j][3]));
      }
      x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, 1)); x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, 2));
      x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, 1)); x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, 2));
      // maxima in the scaled domain (the scale is positive here)
      const float a0 = fmaxf(m0, x0 * sc2), a1 = fmaxf(m1, x1 * sc2);
      const float u0 = a0 == -INFINITY ? 0.f : a0, u1 = a1 == -INFINITY ? 0.f : a1;
      const float c0 = exp2f(m0 - u0), c1 = exp2f(m1 - u1);
      m0 = a0; m1 = a1;
      float t0 = 0.f, t1 = 0.f;
#pragma unroll
      for (int j = 0; j < kLfTiles; ++j) {
        s[j][0] = exp2f(fmaf(s[j][0], sc2, -u0)); s[j][1] = exp2f(fmaf(s[j][1], sc2, -u0));
        s[j][2] = exp2f(fmaf(s[j][2], sc2, -u1)); s[j][3] = exp2f(fmaf(s[j][3], sc2, -u1));
        t0 += s[j][0] + s[j][1];
        t1 += s[j][2] + s[j][3];
      }
      l0 = fmaf(l0, c0, t0);
      l1 = fmaf(l1, c1, t1);
      if (__any_sync(0xffffffffu, c0 != 1.f || c1 != 1.f)) {
#pragma unroll
        for (int j = 0; j < 2 * NV; ++j) { o[j][0] *= c0; o[j][1] *= c0; o[j][2] *= c1; o[j][3] *= c1; }
      }
#pragma unroll
      for (int ks = 0; ks < kLfKeys / 16; ++ks) {
        const uint32_t pa[4] = {pack_bf16x2(s[2 * ks][0], s[2 * ks][1]), pack_bf16x2(s[2 * ks][2], s[2 * ks][3]),
                                pack_bf16x2(s[2 * ks + 1][0], s[2 * ks + 1][1]), pack_bf16x2(s[2 * ks + 1][2], s[2 * ks + 1][3])};
#pragma unroll
        for (int j = 0; j < NV; ++j) {
          uint32_t b[4];
          ldsm4t(vt + v_off + ks * 16 * vB + 32 * j, b);
          mma16816(o[2 * j], pa, b[0], b[1]);
          mma16816(o[2 * j + 1], pa, b[2], b[3]);
        }
      }
    }
    __syncthreads();
  }
  l0 += __shfl_xor_sync(0xffffffffu, l0, 1); l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
  l1 += __shfl_xor_sync(0xffffffffu, l1, 1); l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
  const int ra = wrow + g, rb = ra + 8;
  const float i0 = ra < T ? sigmoid_f32(A.gate[(size_t)ra * A.ldgate + h]) / l0 : 0.f;
  const float i1 = rb < T ? sigmoid_f32(A.gate[(size_t)rb * A.ldgate + h]) / l1 : 0.f;
#pragma unroll
  for (int j = 0; j < 2 * NV; ++j) {
    const int d = 8 * j + 2 * qd;
    if (d >= D.vdim) continue;  // vdim is a multiple of 8
    if (ra < T) *reinterpret_cast<uint32_t*>(A.att + (size_t)ra * A.ldatt + (size_t)h * D.vdim + d) = pack_bf16x2(o[j][0] * i0, o[j][1] * i0);
    if (rb < T) *reinterpret_cast<uint32_t*>(A.att + (size_t)rb * A.ldatt + (size_t)h * D.vdim + d) = pack_bf16x2(o[j][2] * i1, o[j][3] * i1);
  }
}

size_t latent_attn_smem(const LatentDims& D) {
  const size_t KD = (D.row() + 31) & ~31, rowB = 2 * (KD + 8);
  return 16 * rowB + 16 * (2 * (kLaKeys + 8)) + 2 * (size_t)kLaKeys * rowB;
}
size_t latent_flash_smem(const LatentDims& D, int kd, int vd) {
  return (size_t)kLfRows * 2 * (kd + 8) + 2 * (size_t)kLfKeys * (2 * (kd + 8) + 2 * (vd + 8));
}
constexpr size_t kSmemMax = 224 * 1024;

template <int NG>
int launch_attn(orn_ctx* ctx, cudaStream_t s, dim3 grid, size_t smem, const LatentDims& D, int T, const bf16_t* qa, const bf16_t* cache, int cap,
                const int* pos, int splits, float* partial, float* ml) {
  const int rc = orn_grant_smem(ctx, reinterpret_cast<const void*>(latent_attn_kernel<NG>), kSmemMax);
  if (rc != ORN_OK) return rc;
  ORN_CHECK_CUDA(ctx, orn_launch_dependent(ctx, s, 4, latent_attn_kernel<NG>, grid, dim3(kLaWarps * 32), smem, D, T, qa, cache, cap, pos, splits, partial, ml));
  return orn_launch_check(ctx, "latent_attn");
}
template <int NV>
int launch_flash(orn_ctx* ctx, cudaStream_t s, dim3 grid, size_t smem, const LatentDims& D, const FlashArgs& A) {
  const int rc = orn_grant_smem(ctx, reinterpret_cast<const void*>(latent_flash_kernel<NV>), kSmemMax);
  if (rc != ORN_OK) return rc;
  latent_flash_kernel<NV><<<grid, kLfWarps * 32, smem, s>>>(D, A);
  return orn_launch_check(ctx, "latent_flash");
}

}  // namespace

int k_latent_rows(orn_ctx* ctx, cudaStream_t s, const LatentDims& D, int T, const float* kv, int ldkv, const bf16_t* norm_w, void* cache,
                  int cap, const int* pos, void* q, int ldq, bool rotate_q, bool act_f32) {
  if (act_f32)
    latent_rows_kernel<float><<<T, kLrThreads, 0, s>>>(D, kv, ldkv, norm_w, (float*)cache, cap, pos, (float*)q, ldq, rotate_q ? 1 : 0);
  else
    latent_rows_kernel<bf16_t><<<T, kLrThreads, 0, s>>>(D, kv, ldkv, norm_w, (bf16_t*)cache, cap, pos, (bf16_t*)q, ldq, rotate_q ? 1 : 0);
  return orn_launch_check(ctx, "latent_rows");
}

int k_latent_absorb(orn_ctx* ctx, cudaStream_t s, const LatentDims& D, int T, const void* q, int ldq, const orn_linear* uk, const float* kv,
                    int ldkv, const bf16_t* norm_w, void* cache, int cap, const int* pos, void* qa, const StreamSum& sum, bool act_f32) {
  const int chunks = (D.rp() + kAbCols - 1) / kAbCols;
  const int extra = sum.n > 0 ? (sum.count + 4 * kLrThreads - 1) / (4 * kLrThreads) : 0;
  const dim3 grid(T * D.heads * chunks + (kv != nullptr ? T : 0) + extra);
  StreamSum S = sum;
  if (S.n == 0) S.count = 0;
  const size_t smem = sizeof(float) * (size_t)D.dim;
  if (smem > 40 * 1024) ORN_FAIL(ctx, ORN_ERR_ARG, "latent attention: more than 10240 unrotated dimensions per head");
  if (act_f32)
    ORN_CHECK_CUDA(ctx, orn_launch_dependent(ctx, s, 0, latent_absorb_kernel<float>, grid, dim3(kLrThreads), smem, D, T, chunks, (const float*)q, ldq,
                                             lin_dev(uk), kv, ldkv, norm_w, (float*)cache, cap, pos, (float*)qa, S));
  else
    ORN_CHECK_CUDA(ctx, orn_launch_dependent(ctx, s, 0, latent_absorb_kernel<bf16_t>, grid, dim3(kLrThreads), smem, D, T, chunks, (const bf16_t*)q, ldq,
                                             lin_dev(uk), kv, ldkv, norm_w, (bf16_t*)cache, cap, pos, (bf16_t*)qa, S));
  return orn_launch_check(ctx, "latent_absorb");
}

bool latent_attn_tensor_ok(const LatentDims& D) {
  return D.kv_rank % 8 == 0 && (D.kv_rank + 15) / 16 <= 8 * kLaWarps && latent_attn_smem(D) <= kSmemMax;
}

int latent_splits(const orn_ctx* ctx, const LatentDims& D, int T, bool plain) {
  if (plain) return 1;
  const int tiles = (T * D.heads + 15) / 16;
  const int per_sm = latent_attn_smem(D) <= 110 * 1024 ? 2 : 1;
  return std::max(1, std::min(128, per_sm * ctx->sm_count / tiles));
}

int k_latent_attn(orn_ctx* ctx, cudaStream_t s, const LatentDims& D, int T, const void* qa, const void* cache, int cap, const int* pos,
                  int splits, float* partial, float* ml, bool plain, bool act_f32) {
  if (plain) {
    const size_t smem = sizeof(float) * (size_t)(D.row() + D.kv_rank + kPaTile);
    if (smem > kSmemMax) ORN_FAIL(ctx, ORN_ERR_ARG, "latent attention: the latent row does not fit shared memory");
    if (act_f32) {
      if (smem > 48 * 1024) { int rc = orn_grant_smem(ctx, (const void*)latent_attn_plain_kernel<float>, kSmemMax); if (rc) return rc; }
      latent_attn_plain_kernel<float><<<T * D.heads, kPaThreads, smem, s>>>(D, (const float*)qa, (const float*)cache, cap, pos, partial, ml);
    } else {
      if (smem > 48 * 1024) { int rc = orn_grant_smem(ctx, (const void*)latent_attn_plain_kernel<bf16_t>, kSmemMax); if (rc) return rc; }
      latent_attn_plain_kernel<bf16_t><<<T * D.heads, kPaThreads, smem, s>>>(D, (const bf16_t*)qa, (const bf16_t*)cache, cap, pos, partial, ml);
    }
    return orn_launch_check(ctx, "latent_attn_plain");
  }
  const dim3 grid((T * D.heads + 15) / 16, splits);
  const size_t smem = latent_attn_smem(D);
  const int per_warp = ((D.kv_rank + 15) / 16 + kLaWarps - 1) / kLaWarps;
  const bf16_t *q = (const bf16_t*)qa, *c = (const bf16_t*)cache;
  if (per_warp <= 1) return launch_attn<1>(ctx, s, grid, smem, D, T, q, c, cap, pos, splits, partial, ml);
  if (per_warp <= 2) return launch_attn<2>(ctx, s, grid, smem, D, T, q, c, cap, pos, splits, partial, ml);
  if (per_warp <= 4) return launch_attn<4>(ctx, s, grid, smem, D, T, q, c, cap, pos, splits, partial, ml);
  return launch_attn<8>(ctx, s, grid, smem, D, T, q, c, cap, pos, splits, partial, ml);
}

int k_latent_out(orn_ctx* ctx, cudaStream_t s, const LatentDims& D, int T, const orn_linear* uv, const float* partial, const float* ml,
                 int splits, const int* pos, const float* gate, int ldgate, void* att, int ldatt, bool plain, bool act_f32) {
  const dim3 grid(T * D.heads, (D.vdim + kLoRows - 1) / kLoRows);
  const size_t smem = sizeof(float) * (size_t)(D.rp() + ((splits + 3) & ~3) + kLoCols * (kLoThreads / 32));
  if (smem > 48 * 1024) ORN_FAIL(ctx, ORN_ERR_ARG, "latent attention: latent above 8000 entries");
  if (act_f32)
    ORN_CHECK_CUDA(ctx, orn_launch_dependent(ctx, s, 0, latent_out_kernel<float>, grid, dim3(kLoThreads), smem, D, T, lin_dev(uv), partial, ml, splits,
                                             plain ? 1 : 0, pos, gate, ldgate, (float*)att, ldatt));
  else
    ORN_CHECK_CUDA(ctx, orn_launch_dependent(ctx, s, 0, latent_out_kernel<bf16_t>, grid, dim3(kLoThreads), smem, D, T, lin_dev(uv), partial, ml, splits,
                                             plain ? 1 : 0, pos, gate, ldgate, (bf16_t*)att, ldatt));
  return orn_launch_check(ctx, "latent_out");
}

bool latent_flash_ok(const LatentDims& D, int ldq) {
  const int kd = (D.qk() + 15) & ~15, vd = (D.vdim + 15) & ~15;
  return D.scale > 0.f && D.dim % 8 == 0 && D.rot_dim % 8 == 0 && D.vdim % 8 == 0 && ldq % 8 == 0 && D.vdim <= 256 && latent_flash_smem(D, kd, vd) <= kSmemMax;
}

int k_latent_flash(orn_ctx* ctx, cudaStream_t s, const LatentDims& D, int T, const bf16_t* q, int ldq, const bf16_t* kx, int ldk, const bf16_t* vx,
                   int ldv, const bf16_t* cache, int cap, const int* pos, const float* gate, int ldgate, bf16_t* att, int ldatt) {
  FlashArgs A{q, kx, vx, cache, ldq, ldk, ldv, cap, T, pos, gate, ldgate, att, ldatt, (D.qk() + 15) & ~15, (D.vdim + 15) & ~15};
  const dim3 grid((T + kLfRows - 1) / kLfRows, D.heads);
  const int nv = A.vd / 16;
  // the staged value rows are as wide as the instance reads them
  auto width = [&](int groups) { A.vd = 16 * groups; return latent_flash_smem(D, A.kd, A.vd); };
  if (nv <= 2) return launch_flash<2>(ctx, s, grid, width(2), D, A);
  if (nv <= 4) return launch_flash<4>(ctx, s, grid, width(4), D, A);
  if (nv <= 6) return launch_flash<6>(ctx, s, grid, width(6), D, A);
  if (nv <= 8) return launch_flash<8>(ctx, s, grid, width(8), D, A);
  if (nv <= 12) return launch_flash<12>(ctx, s, grid, width(12), D, A);
  return launch_flash<16>(ctx, s, grid, width(16), D, A);
}
