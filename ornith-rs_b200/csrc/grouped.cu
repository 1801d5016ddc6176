// Grouped-query softmax attention: H query heads over G key/value heads, query head h with key/value head
// h / (H / G).
//
//   q, k <- turned, then over their root mean square
//   s_j  = cap * tanh((q . k_j) * scale / cap)
//   out  = sum_j e^(s_j) v_j / (sum_j e^(s_j) + e^sink) * sigmoid(gate)
//
// The sink is the first thing a row's running maximum and sum see; it has no value.
// Three forms, equal to rounding:
//   * windows of 1..4 rows: the (row, head) pairs that share a key head are the M side of mma.sync, the
//     keys are split over CTAs, the last CTA of a key head to finish merges the ranges.  Every size that
//     depends on the position is read on the device, so a captured step serves every context length;
//   * prompt chunks: 64 rows of one query head per CTA, online softmax over tiles of 32 keys;
//   * plain: one CTA per (row, head), for the control route, float32 models and other sizes.
#include <algorithm>

#include "act.cuh"
#include "decayed.cuh"
#include "grouped.h"
#include "heads.h"
#include "mma_bf16.cuh"

namespace {

constexpr float kLog2e = 1.4426950408889634f;

// scores in the base-2 domain.  tanh x = 1 - 2 / (1 + e^2x): absolute error a few float32 ulps of one
struct ScoreMap {
  float a, cap2;  // s -> a s without a cap; cap2 tanh(a s / 2 in base 2) with one
};
ORN_D ScoreMap score_map(const GroupedDims& D) {
  ScoreMap m;
  m.cap2 = D.softcap > 0.f ? D.softcap * kLog2e : 0.f;
  m.a = D.softcap > 0.f ? 2.f * kLog2e * D.scale / D.softcap : D.scale * kLog2e;
  return m;
}
ORN_D float map_score(const ScoreMap& m, float s) {
  const float z = s * m.a;
  if (m.cap2 == 0.f) return z;
  return m.cap2 * (1.f - __fdividef(2.f, 1.f + exp2f(z)));
}

// ------------------------------------------------------------------ plain
constexpr int kGpThreads = 256, kGpTile = 256;
template <typename TA>
__global__ void __launch_bounds__(kGpThreads) grouped_plain_kernel(GroupedDims D, GroupedArgs A) {
  extern __shared__ float s_mem[];  // q [dim], o [vdim], p [tile]
  __shared__ float red[kGpThreads / 32];
  float *s_q = s_mem, *s_o = s_q + D.dim, *s_p = s_o + D.vdim;
  const int t = blockIdx.x / D.heads, h = blockIdx.x - t * D.heads, j = h / (D.heads / D.kv_heads);
  const int n = min(A.cap, *A.pos + t + 1);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const TA *kc = reinterpret_cast<const TA*>(A.kc) + (size_t)j * D.dim, *vc = reinterpret_cast<const TA*>(A.vc) + (size_t)j * D.vdim;
  for (int i = threadIdx.x; i < D.dim; i += kGpThreads) s_q[i] = from_act(reinterpret_cast<const TA*>(A.q)[(size_t)t * A.ldq + (size_t)h * D.dim + i]);
  for (int i = threadIdx.x; i < D.vdim; i += kGpThreads) s_o[i] = 0.f;
  float m = D.sink != nullptr ? bf2f(D.sink[h]) : -INFINITY, l = D.sink != nullptr ? 1.f : 0.f;
  for (int k0 = 0; k0 < n; k0 += kGpTile) {
    __syncthreads();
    for (int k = warp; k < kGpTile; k += kGpThreads / 32) {  // one warp per key
      float s = 0.f;
      if (k0 + k < n) {
        const TA* row = kc + (size_t)(k0 + k) * A.ldkc;
        for (int i = lane; i < D.dim; i += 32) s = fmaf(s_q[i], from_act(row[i]), s);
      }
      s = warp_sum(s) * D.scale;
      if (D.softcap > 0.f) s = D.softcap * tanhf(s / D.softcap);
      if (lane == 0) s_p[k] = k0 + k < n ? s : -INFINITY;
    }
    __syncthreads();
    const float mine = s_p[threadIdx.x];
    float x = warp_max(mine);
    if (lane == 0) red[warp] = x;
    __syncthreads();
    x = red[0];
#pragma unroll
    for (int i = 1; i < kGpThreads / 32; ++i) x = fmaxf(x, red[i]);
    const float mn = fmaxf(m, x), c = expf(m - mn), p = expf(mine - mn);
    float ps = warp_sum(p);
    __syncthreads();
    s_p[threadIdx.x] = p;
    if (lane == 0) red[warp] = ps;
    __syncthreads();
    ps = 0.f;
#pragma unroll
    for (int i = 0; i < kGpThreads / 32; ++i) ps += red[i];
    l = fmaf(l, c, ps);
    m = mn;
    const int kn = min(kGpTile, n - k0);
    for (int i = threadIdx.x; i < D.vdim; i += kGpThreads) {
      float o = s_o[i] * c;
      for (int k = 0; k < kn; ++k) o = fmaf(s_p[k], from_act(vc[(size_t)(k0 + k) * A.ldvc + i]), o);
      s_o[i] = o;
    }
  }
  const float inv = 1.0f / l;
  for (int i = threadIdx.x; i < D.vdim; i += kGpThreads) {
    const size_t at = (size_t)h * D.vdim + i;
    float o = s_o[i] * inv;
    if (A.gate != nullptr) o *= sigmoid_f32(from_act(reinterpret_cast<const TA*>(A.gate)[(size_t)t * A.ldg + at]));
    reinterpret_cast<TA*>(A.att)[(size_t)t * A.ldatt + at] = to_act<TA>(o);
  }
}

// ------------------------------------------------------------------ decode windows
constexpr int kGwWarps = 8, kGwThreads = 32 * kGwWarps, kGwKeys = 64, kGwMaxSplits = 64, kGwMaxRows = 4, kGwTeams = 8;
static_assert(kGwThreads == kDwThreads, "attention and decayed state share a launch");
struct WindowArgs {
  GroupedArgs a;
  int splits, mtiles, ctas;  // ctas of the attention; the decayed state's come after them
  float *partial, *ml;       // [kv head][row tile][split][16][vdim], [..][16][2]
  int* arrivals;             // [kv head][row tile], zero between launches
};
// keys of one range for n visible positions
ORN_D int range_keys(int n, int splits) { return max(kGwKeys, ((n + splits - 1) / splits + kGwKeys - 1) / kGwKeys * kGwKeys); }

struct WindowLayout {  // bytes in shared memory
  int rowB, vB;
  int q, p, tiles, stage, cs, nk, nv, w, end;
};
ORN_HD WindowLayout window_layout(const GroupedDims& D, int T) {
  WindowLayout L;
  L.rowB = 2 * (((D.dim + 31) & ~31) + 8);
  L.vB = 2 * (((D.vdim + 15) & ~15) + 8);
  L.q = 0;
  L.p = L.q + 16 * L.rowB;
  L.tiles = L.p + 16 * 2 * (kGwKeys + 8);
  L.stage = kGwKeys * (L.rowB + L.vB);
  L.cs = L.tiles + 2 * L.stage;
  L.nk = L.cs + T * (D.rot_dims / 2) * 8;
  L.nk = (L.nk + 15) & ~15;
  L.nv = L.nk + T * D.dim * 2;
  L.w = L.nv + T * D.vdim * 2;
  L.end = L.w + 16 * (kGwMaxSplits + 1) * 4;
  return L;
}

template <int NG>  // 16-column groups of the value per warp
ORN_D void grouped_window_cta(const GroupedDims& D, const WindowArgs& W, uint8_t* smem) {
  const GroupedArgs& A = W.a;
  __shared__ float s_max[kGwWarps][16], s_sum[kGwWarps][16];
  __shared__ int s_last;
  const int T = A.T, rep = D.heads / D.kv_heads, rows = T * rep;
  const int split = blockIdx.x % W.splits, jm = blockIdx.x / W.splits, j = jm / W.mtiles, r0 = (jm - j * W.mtiles) * 16;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, qd = lane & 3;
  const WindowLayout L = window_layout(D, T);
  const int KD = (D.dim + 31) & ~31, kp = KD / 8, dp = D.dim / 8, groups = (D.vdim + 15) / 16, vp = 2 * groups, vv = D.vdim / 8;
  const int p0 = *A.pos, n = min(A.cap, p0 + T), kps = range_keys(n, W.splits);
  const int k0 = split * kps, k1 = min(n, k0 + kps);
  if (k0 >= k1) return;
  const int tiles = (k1 - k0 + kGwKeys - 1) / kGwKeys, used = (n + kps - 1) / kps;
  bf16_t *kc = reinterpret_cast<bf16_t*>(A.kc) + (size_t)j * D.dim, *vc = reinterpret_cast<bf16_t*>(A.vc) + (size_t)j * D.vdim;
  const uint32_t sm = smem_u32(smem), q_s = sm + L.q, p_s = sm + L.p;
  // cached keys by cp.async; the window's own rows (key >= p0) are put in by hand
  auto issue = [&](int i) {
    const uint32_t kt = sm + L.tiles + (i & 1) * L.stage, vt = kt + kGwKeys * L.rowB;
    for (int it = threadIdx.x; it < kGwKeys * kp; it += kGwThreads) {
      const int r = it / kp, c = it - r * kp, key = k0 + i * kGwKeys + r;
      if (key >= p0 && key < k1) continue;
      const bool ok = key < k1 && c < dp;
      cp_async16(kt + r * L.rowB + 16 * c, kc + (ok ? (size_t)key * A.ldkc + 8 * c : 0), ok ? 16 : 0);
    }
    for (int it = threadIdx.x; it < kGwKeys * vp; it += kGwThreads) {
      const int r = it / vp, c = it - r * vp, key = k0 + i * kGwKeys + r;
      if (key >= p0 && key < k1) continue;
      const bool ok = key < k1 && c < vv;
      cp_async16(vt + r * L.vB + 16 * c, vc + (ok ? (size_t)key * A.ldvc + 8 * c : 0), ok ? 16 : 0);
    }
    cp_async_commit();
  };
  issue(0);  // rows of earlier steps: they do not depend on the kernel before this one
  float2* s_cs = reinterpret_cast<float2*>(smem + L.cs);
  const int half = D.rot_dims / 2;
  for (int i = threadIdx.x; i < T * half; i += kGwThreads) {
    const int t = i / half;
    float2 r;
    head_rotation(p0 + t, D.freq[i - t * half], r.x, r.y);
    s_cs[i] = r;
  }
  pdl_wait();
  pdl_trigger();
  __syncthreads();
  // the rows as they come wait in the second tile buffer, which is not in use yet: one request each
  uint8_t* raw = smem + L.tiles + L.stage;
  auto fetch = [&](int slot, const bf16_t* src) {
    for (int c = lane; c < dp; c += 32) *reinterpret_cast<uint4*>(raw + slot * L.rowB + 16 * c) = __ldcg(reinterpret_cast<const uint4*>(src) + c);
  };
  auto norm_of = [&](const bf16_t* src) {
    if (!D.unit_qk) return 1.0f;
    float sq = 0.f;
    for (int d = lane; d < D.dim; d += 32) { const float v = bf2f(src[d]); sq = fmaf(v, v, sq); }
    return 1.0f / sqrtf(warp_sum(sq) / (float)D.dim + D.eps);  // turning keeps the length
  };
  for (int r = warp; r < 16 && r0 + r < rows; r += kGwWarps) {
    const int t = (r0 + r) / rep, h = j * rep + r0 + r - t * rep;
    fetch(r, reinterpret_cast<const bf16_t*>(A.q) + (size_t)t * A.ldq + (size_t)h * D.dim);
  }
  for (int t = kGwWarps - 1 - warp; t < T; t += kGwWarps)
    if (p0 + t >= k0 && p0 + t < k1) fetch(16 + t, reinterpret_cast<const bf16_t*>(A.k) + (size_t)t * A.ldk + (size_t)j * D.dim);
  __syncwarp();  // a warp reads what it fetched
  for (int r = warp; r < 16; r += kGwWarps) {
    bf16_t* dst = reinterpret_cast<bf16_t*>(smem + L.q + r * L.rowB);
    const int row = r0 + r;
    if (row < rows) {
      const int t = row / rep;
      const bf16_t* src = reinterpret_cast<const bf16_t*>(raw + r * L.rowB);
      const float rn = norm_of(src);
      for (int d = lane; d < KD; d += 32)
        dst[d] = d < D.dim ? f2bf(rn * rotated_half(d, half, s_cs + t * half, [&](int e) { return bf2f(src[e]); })) : (bf16_t)0;
    } else {
      for (int d = lane; d < KD; d += 32) dst[d] = 0;
    }
  }
  for (int t = kGwWarps - 1 - warp; t < T; t += kGwWarps) {
    const int key = p0 + t;
    if (key < k0 || key >= k1) continue;  // warp-uniform
    const bf16_t* src = reinterpret_cast<const bf16_t*>(raw + (16 + t) * L.rowB);
    bf16_t *nk = reinterpret_cast<bf16_t*>(smem + L.nk) + t * D.dim, *nv = reinterpret_cast<bf16_t*>(smem + L.nv) + t * D.vdim;
    const float rn = norm_of(src);
    for (int d = lane; d < D.dim; d += 32) {
      const bf16_t v = f2bf(rn * rotated_half(d, half, s_cs + t * half, [&](int e) { return bf2f(src[e]); }));
      nk[d] = v;
      if (r0 == 0) kc[(size_t)key * A.ldkc + d] = v;
    }
    for (int d = lane; d < D.vdim; d += 32) {
      const bf16_t v = __ldcg(reinterpret_cast<const bf16_t*>(A.v) + (size_t)t * A.ldv + (size_t)j * D.vdim + d);
      nv[d] = v;
      if (r0 == 0) vc[(size_t)key * A.ldvc + d] = v;
    }
  }
  __syncthreads();
  const ScoreMap map = score_map(D);
  float o[2 * NG][4];
#pragma unroll
  for (int i = 0; i < 2 * NG; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  const int ra = r0 + g, rb = ra + 8;
  float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;
  if (split == 0 && D.sink != nullptr) {
    if (ra < rows) { m0 = bf2f(D.sink[j * rep + ra % rep]) * kLog2e; l0 = warp == 0 && qd == 0 ? 1.f : 0.f; }
    if (rb < rows) { m1 = bf2f(D.sink[j * rep + rb % rep]) * kLog2e; l1 = warp == 0 && qd == 0 ? 1.f : 0.f; }
  }
  const int lim0 = ra < rows ? p0 + ra / rep + 1 : 0, lim1 = rb < rows ? p0 + rb / rep + 1 : 0;  // keys below are visible
  constexpr int pB = 2 * (kGwKeys + 8);
  const uint32_t a_off = ((lane & 7) + 8 * ((lane >> 3) & 1)) * L.rowB + 16 * (lane >> 4);
  const uint32_t k_off = (8 * warp + (lane & 7)) * L.rowB + 16 * (lane >> 3);  // x4: four 8-wide k pieces of 8 keys
  const uint32_t pa_off = ((lane & 7) + 8 * ((lane >> 3) & 1)) * pB + 16 * (lane >> 4);
  const uint32_t v_off = ((lane & 7) + 8 * ((lane >> 3) & 1)) * L.vB + 16 * (lane >> 4);
  for (int i = 0; i < tiles; ++i) {
    if (i + 1 < tiles) {
      issue(i + 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    const int t_off = L.tiles + (i & 1) * L.stage;
    for (int key = max(p0, k0 + i * kGwKeys); key < min(k1, k0 + (i + 1) * kGwKeys); ++key) {
      const int r = key - k0 - i * kGwKeys, t = key - p0;
      const uint4 zero = make_uint4(0, 0, 0, 0);
      const uint4 *nk = reinterpret_cast<const uint4*>(smem + L.nk) + t * dp, *nv = reinterpret_cast<const uint4*>(smem + L.nv) + t * vv;
      for (int c = threadIdx.x; c < kp + vp; c += kGwThreads) {
        if (c < kp) *reinterpret_cast<uint4*>(smem + t_off + r * L.rowB + 16 * c) = c < dp ? nk[c] : zero;
        else *reinterpret_cast<uint4*>(smem + t_off + kGwKeys * L.rowB + r * L.vB + 16 * (c - kp)) = c - kp < vv ? nv[c - kp] : zero;
      }
    }
    __syncthreads();
    const uint32_t kt = sm + t_off, vt = kt + kGwKeys * L.rowB;
    float sa[4] = {0.f, 0.f, 0.f, 0.f}, sb[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 4
    for (int kk = 0; kk < KD / 32; ++kk) {
      uint32_t a[4], b[4];
      ldsm4(kt + k_off + 64 * kk, b);
      ldsm4(q_s + a_off + 64 * kk, a);
      mma16816(sa, a, b[0], b[1]);
      ldsm4(q_s + a_off + 64 * kk + 32, a);
      mma16816(sb, a, b[2], b[3]);
    }
    const int key = k0 + i * kGwKeys + 8 * warp + 2 * qd;
    float s[4];
#pragma unroll
    for (int c = 0; c < 4; ++c) {
      const int kc_ = key + (c & 1);
      s[c] = (kc_ < k1 && kc_ < (c < 2 ? lim0 : lim1)) ? map_score(map, sa[c] + sb[c]) : -INFINITY;
    }
    float x0 = fmaxf(s[0], s[1]), x1 = fmaxf(s[2], s[3]);
    x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, 1)); x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, 2));
    x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, 1)); x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, 2));
    if (qd == 0) { s_max[warp][g] = x0; s_max[warp][g + 8] = x1; }
    __syncthreads();
    float n0 = m0, n1 = m1;
#pragma unroll
    for (int w = 0; w < kGwWarps; ++w) { n0 = fmaxf(n0, s_max[w][g]); n1 = fmaxf(n1, s_max[w][g + 8]); }
    const float u0 = n0 == -INFINITY ? 0.f : n0, u1 = n1 == -INFINITY ? 0.f : n1;
    const float c0 = exp2f(m0 - u0), c1 = exp2f(m1 - u1);
    m0 = n0; m1 = n1;
    const float e0 = exp2f(s[0] - u0), e1 = exp2f(s[1] - u0), e2 = exp2f(s[2] - u1), e3 = exp2f(s[3] - u1);
    l0 = fmaf(l0, c0, e0 + e1);
    l1 = fmaf(l1, c1, e2 + e3);
    {
      uint8_t* pp = smem + L.p + 2 * (8 * warp + 2 * qd);
      *reinterpret_cast<uint32_t*>(pp + g * pB) = pack_bf16x2(e0, e1);
      *reinterpret_cast<uint32_t*>(pp + (g + 8) * pB) = pack_bf16x2(e2, e3);
    }
#pragma unroll
    for (int c = 0; c < 2 * NG; ++c) { o[c][0] *= c0; o[c][1] *= c0; o[c][2] *= c1; o[c][3] *= c1; }
    __syncthreads();
#pragma unroll
    for (int ks = 0; ks < kGwKeys / 16; ++ks) {
      uint32_t a[4];
      ldsm4(p_s + pa_off + 32 * ks, a);
#pragma unroll
      for (int c = 0; c < NG; ++c) {
        const int gr = warp + kGwWarps * c;
        if (gr < groups) {  // warp-uniform
          uint32_t b[4];
          ldsm4t(vt + v_off + ks * 16 * L.vB + 32 * gr, b);
          mma16816(o[2 * c], a, b[0], b[1]);
          mma16816(o[2 * c + 1], a, b[2], b[3]);
        }
      }
    }
    __syncthreads();  // the tile and P are refilled next
  }
  l0 += __shfl_xor_sync(0xffffffffu, l0, 1); l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
  l1 += __shfl_xor_sync(0xffffffffu, l1, 1); l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
  if (qd == 0) { s_sum[warp][g] = l0; s_sum[warp][g + 8] = l1; }
  __syncthreads();
  float t0 = 0.f, t1 = 0.f;
#pragma unroll
  for (int w = 0; w < kGwWarps; ++w) { t0 += s_sum[w][g]; t1 += s_sum[w][g + 8]; }
  bf16_t* att = reinterpret_cast<bf16_t*>(A.att);
  const bf16_t* gate = reinterpret_cast<const bf16_t*>(A.gate);
  auto put = [&](int row, int col, float v) {
    const int t = row / rep;
    const size_t at = (size_t)(j * rep + row - t * rep) * D.vdim + col;
    if (gate != nullptr) v *= sigmoid_f32(bf2f(__ldcg(gate + (size_t)t * A.ldg + at)));
    att[(size_t)t * A.ldatt + at] = f2bf(v);
  };
  float* part = W.partial + ((size_t)jm * W.splits + split) * 16 * D.vdim;
  const float i0 = 1.0f / t0, i1 = 1.0f / t1;
#pragma unroll
  for (int c = 0; c < NG; ++c) {
    const int gr = warp + kGwWarps * c;
    if (gr >= groups) continue;
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      const int col = 16 * gr + 8 * hf + 2 * qd;
      if (col >= D.vdim) continue;  // vdim is a multiple of 8
      const float* v = o[2 * c + hf];
      if (used == 1) {
        if (ra < rows) { put(ra, col, v[0] * i0); put(ra, col + 1, v[1] * i0); }
        if (rb < rows) { put(rb, col, v[2] * i1); put(rb, col + 1, v[3] * i1); }
      } else {
        if (ra < rows) *reinterpret_cast<float2*>(part + g * D.vdim + col) = make_float2(v[0], v[1]);
        if (rb < rows) *reinterpret_cast<float2*>(part + (g + 8) * D.vdim + col) = make_float2(v[2], v[3]);
      }
    }
  }
  if (used == 1) return;
  float* ml = W.ml + ((size_t)jm * W.splits + split) * 32;
  if (warp == 0 && qd == 0) {
    ml[2 * g] = m0; ml[2 * g + 1] = t0;
    ml[2 * (g + 8)] = m1; ml[2 * (g + 8) + 1] = t1;
  }
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) s_last = atomicAdd(W.arrivals + jm, 1) == used - 1 ? 1 : 0;
  __syncthreads();
  if (!s_last) return;
  __threadfence();
  // the last CTA of this key head and row tile merges the ranges in their order
  const int nr = min(16, rows - r0);
  float *s_w = reinterpret_cast<float*>(smem + L.w), *s_inv = s_w + 16 * kGwMaxSplits;
  const float* mls = W.ml + (size_t)jm * W.splits * 32;
  for (int r = warp; r < nr; r += kGwWarps) {
    float m = -INFINITY, tot = 0.f;
    for (int i = lane; i < used; i += 32) m = fmaxf(m, __ldcg(mls + 32 * i + 2 * r));
    m = warp_max(m);
    for (int i = lane; i < used; i += 32) {
      const float mi = __ldcg(mls + 32 * i + 2 * r), w = mi == -INFINITY ? 0.f : exp2f(mi - m);
      s_w[r * kGwMaxSplits + i] = w;
      tot = fmaf(w, __ldcg(mls + 32 * i + 2 * r + 1), tot);
    }
    tot = warp_sum(tot);
    if (lane == 0) s_inv[r] = 1.0f / tot;
  }
  __syncthreads();
  const float* ps = W.partial + (size_t)jm * W.splits * 16 * D.vdim;
  // four columns per thread; where that leaves threads over, they share the ranges
  const int units = nr * D.vdim / 4, teams = max(1, min(kGwTeams, kGwThreads / units));
  float4* s_acc = reinterpret_cast<float4*>(smem + L.tiles);
  for (int u0 = 0; u0 < units; u0 += kGwThreads) {
    const int team = teams > 1 ? threadIdx.x / units : 0, u = teams > 1 ? threadIdx.x - team * units : u0 + threadIdx.x;
    const bool on = u < units && team < teams;
    const int r = 4 * u / D.vdim;
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
    if (on) {
#pragma unroll 8
      for (int sp = team; sp < used; sp += teams) {
        const float w = s_w[r * kGwMaxSplits + sp];
        const float4 v = __ldcg(reinterpret_cast<const float4*>(ps + (size_t)sp * 16 * D.vdim) + u);
        a.x = fmaf(w, v.x, a.x); a.y = fmaf(w, v.y, a.y); a.z = fmaf(w, v.z, a.z); a.w = fmaf(w, v.w, a.w);
      }
    }
    if (teams > 1) {  // one round: the same for every thread
      if (on) s_acc[team * units + u] = a;
      __syncthreads();
      if (on && team == 0)
        for (int k = 1; k < teams; ++k) {
          const float4 v = s_acc[k * units + u];
          a.x += v.x; a.y += v.y; a.z += v.z; a.w += v.w;
        }
    }
    if (on && team == 0) {
      const int col = 4 * u - r * D.vdim;
      const float inv = s_inv[r];
      put(r0 + r, col, a.x * inv); put(r0 + r, col + 1, a.y * inv); put(r0 + r, col + 2, a.z * inv); put(r0 + r, col + 3, a.w * inv);
    }
  }
  if (threadIdx.x == 0) W.arrivals[jm] = 0;  // ready for the next launch
}

template <int NG>
__global__ void __launch_bounds__(kGwThreads, 2) grouped_window_kernel(GroupedDims D, WindowArgs W, DecayedDims LD, DecayedArgs LA) {
  extern __shared__ __align__(128) uint8_t gsm[];
  if ((int)blockIdx.x < W.ctas) grouped_window_cta<NG>(D, W, gsm);
  else decayed_window_any(LD, LA, blockIdx.x - W.ctas, gsm);
}

// ------------------------------------------------------------------ prompt chunks
constexpr int kGfWarps = 4, kGfRows = 16 * kGfWarps, kGfKeys = 32, kGfTiles = kGfKeys / 8;

template <int NV>  // 16-column groups of the value
__global__ void __launch_bounds__(kGfWarps * 32, NV <= 8 ? 3 : 2) grouped_flash_kernel(GroupedDims D, GroupedArgs A) {
  extern __shared__ __align__(128) uint8_t fsm[];
  const int qt = gridDim.x - 1 - blockIdx.x;  // the tiles with the most keys start first
  const int h = blockIdx.y, j = h / (D.heads / D.kv_heads);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, qd = lane & 3;
  const int p0 = *A.pos, r0 = qt * kGfRows, T = A.T;
  const int n = min(A.cap, p0 + min(r0 + kGfRows, T));  // keys any row of this tile sees
  const int tiles = (n + kGfKeys - 1) / kGfKeys;
  const int KD = (D.dim + 15) & ~15, kB = 2 * (KD + 8), vB = 2 * (16 * NV + 8), kp = KD / 8, dp = D.dim / 8, vp = 2 * NV, vv = D.vdim / 8;
  const uint32_t q_s = smem_u32(fsm), st_s = q_s + kGfRows * kB, stage = kGfKeys * (kB + vB);
  const bf16_t* q = reinterpret_cast<const bf16_t*>(A.q) + (size_t)h * D.dim;
  const bf16_t *kc = reinterpret_cast<const bf16_t*>(A.kc) + (size_t)j * D.dim, *vc = reinterpret_cast<const bf16_t*>(A.vc) + (size_t)j * D.vdim;
  for (int i = threadIdx.x; i < kGfRows * kp; i += blockDim.x) {
    const int r = i / kp, c = i - r * kp;
    const bool ok = r0 + r < T && c < dp;
    cp_async16(q_s + r * kB + 16 * c, q + (ok ? (size_t)(r0 + r) * A.ldq + 8 * c : 0), ok ? 16 : 0);
  }
  auto issue = [&](int i) {
    const uint32_t kt = st_s + (i & 1) * stage, vt = kt + kGfKeys * kB;
    for (int it = threadIdx.x; it < kGfKeys * kp; it += blockDim.x) {
      const int r = it / kp, c = it - r * kp, key = i * kGfKeys + r;
      const bool ok = key < n && c < dp;
      cp_async16(kt + r * kB + 16 * c, kc + (ok ? (size_t)key * A.ldkc + 8 * c : 0), ok ? 16 : 0);
    }
    for (int it = threadIdx.x; it < kGfKeys * vp; it += blockDim.x) {
      const int r = it / vp, c = it - r * vp, key = i * kGfKeys + r;
      const bool ok = key < n && c < vv;
      cp_async16(vt + r * vB + 16 * c, vc + (ok ? (size_t)key * A.ldvc + 8 * c : 0), ok ? 16 : 0);
    }
    cp_async_commit();
  };
  issue(0);
  float o[2 * NV][4];
#pragma unroll
  for (int c = 0; c < 2 * NV; ++c) o[c][0] = o[c][1] = o[c][2] = o[c][3] = 0.f;
  float m0 = -INFINITY, l0 = 0.f;
  if (D.sink != nullptr) { m0 = bf2f(D.sink[h]) * kLog2e; l0 = qd == 0 ? 1.f : 0.f; }
  float m1 = m0, l1 = l0;
  const ScoreMap map = score_map(D);
  const int wrow = r0 + 16 * warp;
  const int lim0 = p0 + wrow + g + 1, lim1 = lim0 + 8, wlast = p0 + wrow + 15;
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
    const uint32_t kt = st_s + (i & 1) * stage, vt = kt + kGfKeys * kB;
    const int n0 = i * kGfKeys;
    if (n0 <= wlast) {  // warp-uniform: otherwise every key of this tile is in the future of every row
      float s[kGfTiles][4];
#pragma unroll
      for (int c = 0; c < kGfTiles; ++c) s[c][0] = s[c][1] = s[c][2] = s[c][3] = 0.f;
#pragma unroll 4
      for (int kk = 0; kk < KD / 16; ++kk) {
        uint32_t a[4];
        ldsm4(q_s + a_off + 32 * kk, a);
#pragma unroll
        for (int c = 0; c < kGfTiles / 2; ++c) {
          uint32_t b[4];
          ldsm4(kt + k_off + c * 16 * kB + 32 * kk, b);
          mma16816(s[2 * c], a, b[0], b[1]);
          mma16816(s[2 * c + 1], a, b[2], b[3]);
        }
      }
#pragma unroll
      for (int c = 0; c < kGfTiles; ++c)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[c][e] = map_score(map, s[c][e]);
      if (!(n0 + kGfKeys <= p0 + wrow + 1 && n0 + kGfKeys <= n)) {
#pragma unroll
        for (int c = 0; c < kGfTiles; ++c)
#pragma unroll
          for (int e = 0; e < 4; ++e)
            if (n0 + 8 * c + 2 * qd + (e & 1) >= min(n, e < 2 ? lim0 : lim1)) s[c][e] = -INFINITY;
      }
      float x0 = m0, x1 = m1;
#pragma unroll
      for (int c = 0; c < kGfTiles; ++c) {
        x0 = fmaxf(x0, fmaxf(s[c][0], s[c][1]));
        x1 = fmaxf(x1, fmaxf(s[c][2], s[c][3]));
      }
      x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, 1)); x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, 2));
      x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, 1)); x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, 2));
      const float u0 = x0 == -INFINITY ? 0.f : x0, u1 = x1 == -INFINITY ? 0.f : x1;
      const float c0 = exp2f(m0 - u0), c1 = exp2f(m1 - u1);
      m0 = x0; m1 = x1;
      float t0 = 0.f, t1 = 0.f;
#pragma unroll
      for (int c = 0; c < kGfTiles; ++c) {
        s[c][0] = exp2f(s[c][0] - u0); s[c][1] = exp2f(s[c][1] - u0);
        s[c][2] = exp2f(s[c][2] - u1); s[c][3] = exp2f(s[c][3] - u1);
        t0 += s[c][0] + s[c][1];
        t1 += s[c][2] + s[c][3];
      }
      l0 = fmaf(l0, c0, t0);
      l1 = fmaf(l1, c1, t1);
      if (__any_sync(0xffffffffu, c0 != 1.f || c1 != 1.f)) {
#pragma unroll
        for (int c = 0; c < 2 * NV; ++c) { o[c][0] *= c0; o[c][1] *= c0; o[c][2] *= c1; o[c][3] *= c1; }
      }
#pragma unroll
      for (int ks = 0; ks < kGfKeys / 16; ++ks) {
        const uint32_t pa[4] = {pack_bf16x2(s[2 * ks][0], s[2 * ks][1]), pack_bf16x2(s[2 * ks][2], s[2 * ks][3]),
                                pack_bf16x2(s[2 * ks + 1][0], s[2 * ks + 1][1]), pack_bf16x2(s[2 * ks + 1][2], s[2 * ks + 1][3])};
#pragma unroll
        for (int c = 0; c < NV; ++c) {
          uint32_t b[4];
          ldsm4t(vt + v_off + ks * 16 * vB + 32 * c, b);
          mma16816(o[2 * c], pa, b[0], b[1]);
          mma16816(o[2 * c + 1], pa, b[2], b[3]);
        }
      }
    }
    __syncthreads();
  }
  l0 += __shfl_xor_sync(0xffffffffu, l0, 1); l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
  l1 += __shfl_xor_sync(0xffffffffu, l1, 1); l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
  const int ra = wrow + g, rb = ra + 8;
  const float i0 = 1.0f / l0, i1 = 1.0f / l1;
  auto put = [&](int row, int d, float a, float b) {
    const size_t at = (size_t)h * D.vdim + d;
    if (A.gate != nullptr) {
      const uint32_t z = __ldg(reinterpret_cast<const uint32_t*>(reinterpret_cast<const bf16_t*>(A.gate) + (size_t)row * A.ldg + at));
      a *= sigmoid_f32(__uint_as_float(z << 16));
      b *= sigmoid_f32(__uint_as_float(z & 0xffff0000u));
    }
    *reinterpret_cast<uint32_t*>(reinterpret_cast<bf16_t*>(A.att) + (size_t)row * A.ldatt + at) = pack_bf16x2(a, b);
  };
#pragma unroll
  for (int c = 0; c < 2 * NV; ++c) {
    const int d = 8 * c + 2 * qd;
    if (d >= D.vdim) continue;  // vdim is a multiple of 8
    if (ra < T) put(ra, d, o[c][0] * i0, o[c][1] * i0);
    if (rb < T) put(rb, d, o[c][2] * i1, o[c][3] * i1);
  }
}

constexpr size_t kGSmemMax = 220 * 1024;
size_t flash_smem(const GroupedDims& D, int nv) {
  const size_t kB = 2 * (((D.dim + 15) & ~15) + 8), vB = 2 * (16 * nv + 8);
  return kGfRows * kB + 2 * kGfKeys * (kB + vB);
}
template <int NV>
int launch_flash(orn_ctx* ctx, cudaStream_t s, const GroupedDims& D, const GroupedArgs& A) {
  const int rc = orn_grant_smem(ctx, reinterpret_cast<const void*>(grouped_flash_kernel<NV>), kGSmemMax);
  if (rc != ORN_OK) return rc;
  grouped_flash_kernel<NV><<<dim3((A.T + kGfRows - 1) / kGfRows, D.heads), kGfWarps * 32, flash_smem(D, NV), s>>>(D, A);
  return orn_launch_check(ctx, "grouped_flash");
}
template <int NG>
int launch_window(orn_ctx* ctx, cudaStream_t s, int ctas, size_t smem, const GroupedDims& D, const WindowArgs& W, const DecayedDims& LD, const DecayedArgs& LA) {
  const int rc = orn_grant_smem(ctx, reinterpret_cast<const void*>(grouped_window_kernel<NG>), kGSmemMax);
  if (rc != ORN_OK) return rc;
  ORN_CHECK_CUDA(ctx, orn_launch_dependent(ctx, s, 4, grouped_window_kernel<NG>, dim3(ctas), dim3(kGwThreads), smem, D, W, LD, LA));
  return orn_launch_check(ctx, LA.T > 0 ? "grouped_window + decayed" : "grouped_window");
}

int row_tiles(const GroupedDims& D, int T) { return (T * (D.heads / D.kv_heads) + 15) / 16; }
int window_splits(const orn_ctx* ctx, const GroupedDims& D, int T) {
  const int per_sm = window_layout(D, T).end <= 110 * 1024 ? 2 : 1;
  return std::max(1, std::min(kGwMaxSplits, per_sm * ctx->sm_count / (D.kv_heads * row_tiles(D, T))));
}

}  // namespace

bool grouped_window_ok(const orn_ctx*, const GroupedDims& D, const GroupedArgs& A) {
  return A.T >= 1 && A.T <= kGwMaxRows && D.dim % 8 == 0 && D.vdim % 8 == 0 && D.vdim <= 256 && A.ldkc % 8 == 0 && A.ldvc % 8 == 0 &&
         window_layout(D, kGwMaxRows).end <= (int)kGSmemMax;
}
size_t grouped_window_scratch(const orn_ctx* ctx, const GroupedDims& D) {
  size_t units = 0, tiles = 0;
  for (int T = 1; T <= kGwMaxRows; ++T) {
    tiles = std::max(tiles, (size_t)D.kv_heads * row_tiles(D, T));
    units = std::max(units, (size_t)D.kv_heads * row_tiles(D, T) * window_splits(ctx, D, T));
  }
  return ((tiles * 4 + 255) & ~(size_t)255) + units * 16 * (D.vdim + 2) * 4;
}
int k_grouped_window(orn_ctx* ctx, cudaStream_t s, const GroupedDims& D, const GroupedArgs& A, void* scratch, const DecayedDims* lin_dims,
                     const DecayedArgs* lin) {
  if (!grouped_window_ok(ctx, D, A)) ORN_FAIL(ctx, ORN_ERR_ARG, "grouped attention: sizes of the window form");
  if (lin != nullptr && !decayed_window_ok(*lin_dims, *lin)) ORN_FAIL(ctx, ORN_ERR_ARG, "decayed state: sizes of the window form");
  WindowArgs W;
  W.a = A;
  W.mtiles = row_tiles(D, A.T);
  W.splits = window_splits(ctx, D, A.T);
  W.ctas = D.kv_heads * W.mtiles * W.splits;
  size_t tiles = 0;
  for (int T = 1; T <= kGwMaxRows; ++T) tiles = std::max(tiles, (size_t)D.kv_heads * row_tiles(D, T));
  W.arrivals = reinterpret_cast<int*>(scratch);
  W.ml = reinterpret_cast<float*>(reinterpret_cast<uint8_t*>(scratch) + ((tiles * 4 + 255) & ~(size_t)255));
  W.partial = W.ml + (size_t)W.ctas * 32;
  size_t smem = window_layout(D, A.T).end;
  int ctas = W.ctas;
  DecayedDims LD;
  DecayedArgs LA;
  if (lin != nullptr) {
    LD = *lin_dims;
    LA = *lin;
    ctas += LD.heads * decayed_slices(LD);
    smem = std::max(smem, kDwSmem);
  }
  if (D.vdim <= 128) return launch_window<1>(ctx, s, ctas, smem, D, W, LD, LA);
  return launch_window<2>(ctx, s, ctas, smem, D, W, LD, LA);
}

bool grouped_flash_ok(const GroupedDims& D, const GroupedArgs& A) {
  return D.dim % 8 == 0 && D.vdim % 8 == 0 && D.vdim <= 256 && A.ldq % 8 == 0 && A.ldkc % 8 == 0 && A.ldvc % 8 == 0 && A.ldg % 2 == 0 && A.ldatt % 2 == 0 &&
         flash_smem(D, 16) <= kGSmemMax;
}
int k_grouped_flash(orn_ctx* ctx, cudaStream_t s, const GroupedDims& D, const GroupedArgs& A) {
  if (!grouped_flash_ok(D, A)) ORN_FAIL(ctx, ORN_ERR_ARG, "grouped attention: sizes of the tensor form");
  const int nv = (D.vdim + 15) / 16;
  if (nv <= 2) return launch_flash<2>(ctx, s, D, A);
  if (nv <= 4) return launch_flash<4>(ctx, s, D, A);
  if (nv <= 6) return launch_flash<6>(ctx, s, D, A);
  if (nv <= 8) return launch_flash<8>(ctx, s, D, A);
  if (nv <= 12) return launch_flash<12>(ctx, s, D, A);
  return launch_flash<16>(ctx, s, D, A);
}

int k_grouped_plain(orn_ctx* ctx, cudaStream_t s, const GroupedDims& D, const GroupedArgs& A, bool act_f32) {
  const size_t smem = sizeof(float) * (size_t)(D.dim + D.vdim + kGpTile);
  if (smem > kGSmemMax) ORN_FAIL(ctx, ORN_ERR_ARG, "grouped attention: heads do not fit shared memory");
  if (act_f32) {
    if (smem > 48 * 1024) { int rc = orn_grant_smem(ctx, (const void*)grouped_plain_kernel<float>, kGSmemMax); if (rc) return rc; }
    grouped_plain_kernel<float><<<A.T * D.heads, kGpThreads, smem, s>>>(D, A);
  } else {
    if (smem > 48 * 1024) { int rc = orn_grant_smem(ctx, (const void*)grouped_plain_kernel<bf16_t>, kGSmemMax); if (rc) return rc; }
    grouped_plain_kernel<bf16_t><<<A.T * D.heads, kGpThreads, smem, s>>>(D, A);
  }
  return orn_launch_check(ctx, "grouped_plain");
}
