// Linear attention with a fixed decay g per head: S_t = g S_(t-1) + c k_t v_t^T, o_t = S_t^T q_t, the
// state in float32 and carried from call to call in a ring of slots.
//
// Three forms, equal to rounding:
//   * windows of 1..4 rows (decayed.cuh): the state passes through registers once;
//   * token by token with the state in shared memory: the control route, float32 models, odd sizes;
//   * prompt chunks.  With states kept every C tokens and i, j counted from the last kept one,
//       o_i     = g^(i+1) S^T q_i + sum_(j <= i) c g^(i-j) (q_i . k_j) v_j
//       S_next  = g^n S + sum_j c g^(n-1-j) k_j v_j^T          (n tokens, n <= C)
//     so one kernel folds every C tokens on their own, a second carries the state across (element by
//     element), and a third makes all rows at once.  Every power is of a whole number of tokens and at
//     most one: nothing overflows, whatever the decay.  The products run on mma.sync with bf16 operands;
//     the weighted keys and the state go in as a bf16 value and its bf16 remainder.
#include <algorithm>

#include "decayed.cuh"
#include "mma_bf16.cuh"

namespace {

__global__ void __launch_bounds__(kDwThreads) decayed_window_kernel(DecayedDims D, DecayedArgs A) {
  extern __shared__ __align__(16) uint8_t dsm[];
  decayed_window_any(D, A, blockIdx.x, dsm);
}

// ------------------------------------------------------------------ token by token
constexpr int kDpThreads = 256, kDpCols = 32;
constexpr size_t kDpSmemMax = 220 * 1024;
template <typename TA>
__global__ void __launch_bounds__(kDpThreads) decayed_plain_kernel(DecayedDims D, DecayedArgs A) {
  extern __shared__ float s_mem[];  // S [dim][kDpCols], q [dim], k [dim], partial sums [warps][kDpCols]
  float *s_S = s_mem, *s_q = s_S + (size_t)D.dim * kDpCols, *s_k = s_q + D.dim, *s_red = s_k + D.dim;
  const int h = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int c = blockIdx.x * kDpCols + lane;  // a lane's column; the rows are dealt to the warps
  const bool mine = c < D.vdim;
  const size_t ssz = D.state(), at = (size_t)h * D.dim * D.vdim + c;
  const int cur = *A.cur;
  const float g = D.gpow[(size_t)h * (kDecayChunk + 1) + 1];
  for (int r = warp; r < D.dim; r += kDpThreads / 32)
    s_S[r * kDpCols + lane] = mine ? A.ring[(size_t)(cur % A.nring) * ssz + at + (size_t)r * D.vdim] : 0.f;
  const TA *q = reinterpret_cast<const TA*>(A.q) + (size_t)h * D.dim, *k = reinterpret_cast<const TA*>(A.k) + (size_t)h * D.dim;
  for (int t = 0; t < A.T; ++t) {
    for (int d = threadIdx.x; d < D.dim; d += kDpThreads) {
      s_q[d] = from_act(q[(size_t)t * A.ldq + d]);
      s_k[d] = from_act(k[(size_t)t * A.ldk + d]) * D.k_scale;
    }
    __syncthreads();
    const float v = mine ? from_act(reinterpret_cast<const TA*>(A.v)[(size_t)t * A.ldv + (size_t)h * D.vdim + c]) : 0.f;
    float* sout = nullptr;
    if (A.keep_all) sout = A.ring + (size_t)((cur + 1 + t) % A.nring) * ssz + at;
    else if (t + 1 == A.T) sout = A.ring + (size_t)((cur + 1) % A.nring) * ssz + at;
    float o = 0.f;
    for (int r = warp; r < D.dim; r += kDpThreads / 32) {
      const float S = fmaf(s_k[r], v, g * s_S[r * kDpCols + lane]);
      s_S[r * kDpCols + lane] = S;
      o = fmaf(s_q[r], S, o);
      if (sout != nullptr && mine) sout[(size_t)r * D.vdim] = S;
    }
    s_red[warp * kDpCols + lane] = o;
    __syncthreads();
    if (warp == 0 && mine) {
      float s = 0.f;
#pragma unroll
      for (int w = 0; w < kDpThreads / 32; ++w) s += s_red[w * kDpCols + lane];
      A.o[(size_t)t * A.ldo + (size_t)h * D.vdim + c] = s;
    }
    __syncthreads();  // q, k and the partial sums are replaced next
  }
}

// ------------------------------------------------------------------ prompt chunks
// fold: one CTA per (C tokens, head, 64 x 64 block of the state)
constexpr int kFoTok = 64, kFoPitch = 2 * (64 + 8), kFoStage = 2 * kFoTok * kFoPitch;
__global__ void __launch_bounds__(128) decayed_fold_kernel(DecayedDims D, DecayedArgs A, float* __restrict__ U) {
  __shared__ __align__(128) uint8_t fsm[2 * kFoStage];
  __shared__ float s_g[kDecayChunk + 1];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, gr = lane >> 2, qd = lane & 3;
  const int h = blockIdx.y, vb = (D.vdim + 63) / 64, m0 = (blockIdx.z / vb) * 64, n0 = (blockIdx.z % vb) * 64;
  const int t0 = blockIdx.x * kDecayChunk, n = min(kDecayChunk, A.T - t0), tiles = (n + kFoTok - 1) / kFoTok;
  const bf16_t *k = reinterpret_cast<const bf16_t*>(A.k) + (size_t)t0 * A.ldk + (size_t)h * D.dim + m0;
  const bf16_t *v = reinterpret_cast<const bf16_t*>(A.v) + (size_t)t0 * A.ldv + (size_t)h * D.vdim + n0;
  const int kw = min(64, D.dim - m0) / 8, vw = min(64, D.vdim - n0) / 8;  // 16-byte pieces
  const uint32_t base = smem_u32(fsm);
  auto issue = [&](int i) {
    const uint32_t kt = base + (i & 1) * kFoStage, vt = kt + kFoTok * kFoPitch;
    for (int it = threadIdx.x; it < kFoTok * 8; it += 128) {
      const int r = it >> 3, c = it & 7, t = i * kFoTok + r;
      const bool ko = t < n && c < kw, vo = t < n && c < vw;
      cp_async16(kt + r * kFoPitch + 16 * c, k + (ko ? (size_t)t * A.ldk + 8 * c : 0), ko ? 16 : 0);
      cp_async16(vt + r * kFoPitch + 16 * c, v + (vo ? (size_t)t * A.ldv + 8 * c : 0), vo ? 16 : 0);
    }
    cp_async_commit();
  };
  issue(0);
  for (int i = threadIdx.x; i <= kDecayChunk; i += 128) s_g[i] = D.gpow[(size_t)h * (kDecayChunk + 1) + i];
  float acc[8][4];
#pragma unroll
  for (int j = 0; j < 8; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
  const uint32_t a_off = ((lane & 7) + 8 * (lane >> 4)) * kFoPitch + 2 * (16 * warp + 8 * ((lane >> 3) & 1));
  const uint32_t b_off = ((lane & 7) + 8 * ((lane >> 3) & 1)) * kFoPitch + 16 * (lane >> 4);
  for (int i = 0; i < tiles; ++i) {
    if (i + 1 < tiles) { issue(i + 1); cp_async_wait<1>(); }
    else cp_async_wait<0>();
    __syncthreads();
    const uint32_t kt = base + (i & 1) * kFoStage, vt = kt + kFoTok * kFoPitch;
#pragma unroll
    for (int ks = 0; ks < kFoTok / 16; ++ks) {
      uint32_t a[4], hi[4], lo[4];
      ldsm4t(kt + a_off + ks * 16 * kFoPitch, a);
      const int j0 = n - 1 - (i * kFoTok + 16 * ks + 2 * qd);  // tokens from this one to the last
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int j = j0 - 8 * (e >> 1);
        const float x = __uint_as_float(a[e] << 16) * (D.k_scale * s_g[max(j, 0)]);  // beyond the end the keys are zeros
        const float y = __uint_as_float(a[e] & 0xffff0000u) * (D.k_scale * s_g[max(j - 1, 0)]);
        hi[e] = pack_bf16x2(x, y);
        lo[e] = pack_bf16x2(x - __uint_as_float(hi[e] << 16), y - __uint_as_float(hi[e] & 0xffff0000u));
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        uint32_t b[4];
        ldsm4t(vt + b_off + ks * 16 * kFoPitch + 32 * j, b);
        mma16816(acc[2 * j], hi, b[0], b[1]);
        mma16816(acc[2 * j + 1], hi, b[2], b[3]);
        mma16816(acc[2 * j], lo, b[0], b[1]);
        mma16816(acc[2 * j + 1], lo, b[2], b[3]);
      }
    }
    __syncthreads();
  }
  float* out = U + (size_t)blockIdx.x * D.state() + (size_t)h * D.dim * D.vdim;
#pragma unroll
  for (int j = 0; j < 8; ++j) {
    const int c = n0 + 8 * j + 2 * qd, r = m0 + 16 * warp + gr;
    if (c >= D.vdim) continue;  // sizes are multiples of 8
    if (r < D.dim) *reinterpret_cast<float2*>(out + (size_t)r * D.vdim + c) = make_float2(acc[j][0], acc[j][1]);
    if (r + 8 < D.dim) *reinterpret_cast<float2*>(out + (size_t)(r + 8) * D.vdim + c) = make_float2(acc[j][2], acc[j][3]);
  }
}

// carry: the state before every C tokens as [chunk][head][value, remainder][dim][vdim] bf16, the last one into the ring
constexpr int kCaAhead = 8;
__global__ void __launch_bounds__(128) decayed_carry_kernel(DecayedDims D, DecayedArgs A, const float* __restrict__ U, bf16_t* __restrict__ S2) {
  const size_t per = (size_t)D.dim * D.vdim, ssz = D.state();
  const size_t i = 4 * ((size_t)blockIdx.x * 128 + threadIdx.x);
  if (i >= ssz) return;
  const int h = (int)(i / per), chunks = (A.T + kDecayChunk - 1) / kDecayChunk;
  const float* gp = D.gpow + (size_t)h * (kDecayChunk + 1);
  const float g_full = gp[kDecayChunk], g_last = gp[A.T - (chunks - 1) * kDecayChunk];
  const int cur = *A.cur;
  float4 S = *reinterpret_cast<const float4*>(A.ring + (size_t)(cur % A.nring) * ssz + i);
  bf16_t* out = S2 + 2 * (size_t)h * per + (i - (size_t)h * per);
  for (int c0 = 0; c0 < chunks; c0 += kCaAhead) {
    float4 u[kCaAhead];
#pragma unroll
    for (int c = 0; c < kCaAhead; ++c)
      u[c] = c0 + c < chunks ? __ldcg(reinterpret_cast<const float4*>(U + (size_t)(c0 + c) * ssz + i)) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int c = 0; c < kCaAhead; ++c) {
      if (c0 + c >= chunks) break;
      uint2 hi, lo;
      hi.x = pack_bf16x2(S.x, S.y); hi.y = pack_bf16x2(S.z, S.w);
      lo.x = pack_bf16x2(S.x - __uint_as_float(hi.x << 16), S.y - __uint_as_float(hi.x & 0xffff0000u));
      lo.y = pack_bf16x2(S.z - __uint_as_float(hi.y << 16), S.w - __uint_as_float(hi.y & 0xffff0000u));
      bf16_t* o = out + (size_t)(c0 + c) * 2 * ssz;
      *reinterpret_cast<uint2*>(o) = hi;
      *reinterpret_cast<uint2*>(o + per) = lo;
      const float g = c0 + c + 1 < chunks ? g_full : g_last;
      S.x = fmaf(g, S.x, u[c].x); S.y = fmaf(g, S.y, u[c].y); S.z = fmaf(g, S.z, u[c].z); S.w = fmaf(g, S.w, u[c].w);
    }
  }
  *reinterpret_cast<float4*>(A.ring + (size_t)((cur + 1) % A.nring) * ssz + i) = S;
}

// rows: one CTA per (64 rows, head); first the kept state's tiles, then the keys since then up to the row
constexpr int kDrWarps = 4, kDrRows = 16 * kDrWarps, kDrKeys = 32;
template <int NV>  // 16-column groups of the value
__global__ void __launch_bounds__(kDrWarps * 32, NV <= 8 ? 3 : 2) decayed_rows_kernel(DecayedDims D, DecayedArgs A, const bf16_t* __restrict__ S2) {
  extern __shared__ __align__(128) uint8_t rsm[];
  __shared__ float s_g[kDecayChunk + 1];
  const int h = blockIdx.y, r0 = blockIdx.x * kDrRows, T = A.T;
  const int chunk = r0 / kDecayChunk, t0 = chunk * kDecayChunk, i0 = r0 - t0;  // rows from the kept state
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, gr = lane >> 2, qd = lane & 3;
  const int KD = (D.dim + 31) & ~31, kB = 2 * (KD + 8), vB = 2 * (16 * NV + 8), kp = KD / 8, dp = D.dim / 8, vp = 2 * NV, vv = D.vdim / 8;
  const int s_tiles = KD / kDrKeys, keys = min(i0 + kDrRows, T - t0), tiles = 2 * s_tiles + (keys + kDrKeys - 1) / kDrKeys;
  const uint32_t q_s = smem_u32(rsm), st_s = q_s + kDrRows * kB, stage = kDrKeys * (kB + vB);
  const bf16_t *q = reinterpret_cast<const bf16_t*>(A.q) + (size_t)r0 * A.ldq + (size_t)h * D.dim;
  const bf16_t *k = reinterpret_cast<const bf16_t*>(A.k) + (size_t)t0 * A.ldk + (size_t)h * D.dim;
  const bf16_t *v = reinterpret_cast<const bf16_t*>(A.v) + (size_t)t0 * A.ldv + (size_t)h * D.vdim;
  const size_t per = (size_t)D.dim * D.vdim;
  const bf16_t* S = S2 + (size_t)chunk * 2 * D.state() + 2 * (size_t)h * per;
  for (int i = threadIdx.x; i < kDrRows * kp; i += kDrWarps * 32) {
    const int r = i / kp, c = i - r * kp;
    const bool ok = r0 + r < T && c < dp;
    cp_async16(q_s + r * kB + 16 * c, q + (ok ? (size_t)r * A.ldq + 8 * c : 0), ok ? 16 : 0);
  }
  auto issue = [&](int i) {
    const uint32_t kt = st_s + (i & 1) * stage, vt = kt + kDrKeys * kB;
    if (i < 2 * s_tiles) {
      const int part = i >= s_tiles ? 1 : 0, d0 = (i - part * s_tiles) * kDrKeys;
      for (int it = threadIdx.x; it < kDrKeys * vp; it += kDrWarps * 32) {
        const int r = it / vp, c = it - r * vp;
        const bool ok = d0 + r < D.dim && c < vv;
        cp_async16(vt + r * vB + 16 * c, S + (ok ? part * per + (size_t)(d0 + r) * D.vdim + 8 * c : 0), ok ? 16 : 0);
      }
    } else {
      const int j0 = (i - 2 * s_tiles) * kDrKeys;
      for (int it = threadIdx.x; it < kDrKeys * kp; it += kDrWarps * 32) {
        const int r = it / kp, c = it - r * kp;
        const bool ok = j0 + r < keys && c < dp;
        cp_async16(kt + r * kB + 16 * c, k + (ok ? (size_t)(j0 + r) * A.ldk + 8 * c : 0), ok ? 16 : 0);
      }
      for (int it = threadIdx.x; it < kDrKeys * vp; it += kDrWarps * 32) {
        const int r = it / vp, c = it - r * vp;
        const bool ok = j0 + r < keys && c < vv;
        cp_async16(vt + r * vB + 16 * c, v + (ok ? (size_t)(j0 + r) * A.ldv + 8 * c : 0), ok ? 16 : 0);
      }
    }
    cp_async_commit();
  };
  issue(0);
  for (int i = threadIdx.x; i <= kDecayChunk; i += kDrWarps * 32) s_g[i] = D.gpow[(size_t)h * (kDecayChunk + 1) + i];
  float o[2 * NV][4];
#pragma unroll
  for (int j = 0; j < 2 * NV; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
  const int ia = i0 + 16 * warp + gr, ib = ia + 8, wlast = i0 + 16 * warp + 15;
  const uint32_t a_off = (16 * warp + (lane & 7) + 8 * ((lane >> 3) & 1)) * kB + 16 * (lane >> 4);
  const uint32_t k_off = ((lane & 7) + 8 * (lane >> 4)) * kB + 16 * ((lane >> 3) & 1);
  const uint32_t v_off = ((lane & 7) + 8 * ((lane >> 3) & 1)) * vB + 16 * (lane >> 4);
  for (int i = 0; i < tiles; ++i) {
    if (i + 1 < tiles) { issue(i + 1); cp_async_wait<1>(); }
    else cp_async_wait<0>();
    __syncthreads();
    const uint32_t kt = st_s + (i & 1) * stage, vt = kt + kDrKeys * kB;
    if (i < 2 * s_tiles) {
      const int d0 = (i >= s_tiles ? i - s_tiles : i) * kDrKeys;
#pragma unroll
      for (int ks = 0; ks < kDrKeys / 16; ++ks) {
        uint32_t a[4];
        ldsm4(q_s + a_off + 2 * (d0 + 16 * ks), a);
#pragma unroll
        for (int j = 0; j < NV; ++j) {
          uint32_t b[4];
          ldsm4t(vt + v_off + ks * 16 * vB + 32 * j, b);
          mma16816(o[2 * j], a, b[0], b[1]);
          mma16816(o[2 * j + 1], a, b[2], b[3]);
        }
      }
      if (i + 1 == 2 * s_tiles) {
        const float fa = s_g[ia + 1], fb = s_g[ib + 1];
#pragma unroll
        for (int j = 0; j < 2 * NV; ++j) { o[j][0] *= fa; o[j][1] *= fa; o[j][2] *= fb; o[j][3] *= fb; }
      }
    } else if ((i - 2 * s_tiles) * kDrKeys <= wlast) {  // warp-uniform: some row of the warp sees a key of the tile
      const int j0 = (i - 2 * s_tiles) * kDrKeys;
      float s[4][4];
#pragma unroll
      for (int j = 0; j < 4; ++j) s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.f;
#pragma unroll 4
      for (int kk = 0; kk < KD / 16; ++kk) {
        uint32_t a[4];
        ldsm4(q_s + a_off + 32 * kk, a);
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          uint32_t b[4];
          ldsm4(kt + k_off + j * 16 * kB + 32 * kk, b);
          mma16816(s[2 * j], a, b[0], b[1]);
          mma16816(s[2 * j + 1], a, b[2], b[3]);
        }
      }
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          const int back = (c < 2 ? ia : ib) - (j0 + 8 * j + 2 * qd + (c & 1));
          s[j][c] = back >= 0 ? s[j][c] * D.k_scale * s_g[back] : 0.f;
        }
#pragma unroll
      for (int ks = 0; ks < 2; ++ks) {
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
  const int ra = r0 + 16 * warp + gr, rb = ra + 8;
#pragma unroll
  for (int j = 0; j < 2 * NV; ++j) {
    const int d = 8 * j + 2 * qd;
    if (d >= D.vdim) continue;  // vdim is a multiple of 8
    if (ra < T) *reinterpret_cast<float2*>(A.o + (size_t)ra * A.ldo + (size_t)h * D.vdim + d) = make_float2(o[j][0], o[j][1]);
    if (rb < T) *reinterpret_cast<float2*>(A.o + (size_t)rb * A.ldo + (size_t)h * D.vdim + d) = make_float2(o[j][2], o[j][3]);
  }
}

size_t rows_smem(const DecayedDims& D, int nv) {
  const size_t kB = 2 * (((D.dim + 31) & ~31) + 8), vB = 2 * (16 * nv + 8);
  return kDrRows * kB + 2 * kDrKeys * (kB + vB);
}
constexpr size_t kDrSmemMax = 200 * 1024;
template <int NV>
int launch_rows(orn_ctx* ctx, cudaStream_t s, const DecayedDims& D, const DecayedArgs& A, const bf16_t* S2) {
  const int rc = orn_grant_smem(ctx, reinterpret_cast<const void*>(decayed_rows_kernel<NV>), kDrSmemMax);
  if (rc != ORN_OK) return rc;
  decayed_rows_kernel<NV><<<dim3((A.T + kDrRows - 1) / kDrRows, D.heads), kDrWarps * 32, rows_smem(D, NV), s>>>(D, A, S2);
  return orn_launch_check(ctx, "decayed_rows");
}

}  // namespace

bool decayed_window_ok(const DecayedDims& D, const DecayedArgs& A) {
  return A.T >= 1 && A.T <= kDwMaxRows && D.dim <= kDwMaxDim && D.vdim % 4 == 0 && A.ldv % 4 == 0 && A.nring > (A.keep_all ? A.T : 1);
}
int k_decayed_window(orn_ctx* ctx, cudaStream_t s, const DecayedDims& D, const DecayedArgs& A) {
  if (!decayed_window_ok(D, A)) ORN_FAIL(ctx, ORN_ERR_ARG, "decayed state: sizes of the window form");
  ORN_CHECK_CUDA(ctx, orn_launch_dependent(ctx, s, 3, decayed_window_kernel, dim3(D.heads * decayed_slices(D)), dim3(kDwThreads), kDwSmem, D, A));
  return orn_launch_check(ctx, "decayed_window");
}

int k_decayed_plain(orn_ctx* ctx, cudaStream_t s, const DecayedDims& D, const DecayedArgs& A, bool act_f32) {
  if (A.nring < 2 || (A.keep_all && A.T >= A.nring)) ORN_FAIL(ctx, ORN_ERR_ARG, "decayed state: window wider than the ring");
  const size_t smem = sizeof(float) * ((size_t)D.dim * (kDpCols + 2) + (kDpThreads / 32) * kDpCols);
  if (smem > kDpSmemMax) ORN_FAIL(ctx, ORN_ERR_ARG, "decayed state: more than 1600 dimensions per head");
  const dim3 grid((D.vdim + kDpCols - 1) / kDpCols, D.heads);
  if (act_f32) {
    if (smem > 48 * 1024) { int rc = orn_grant_smem(ctx, (const void*)decayed_plain_kernel<float>, kDpSmemMax); if (rc) return rc; }
    decayed_plain_kernel<float><<<grid, kDpThreads, smem, s>>>(D, A);
  } else {
    if (smem > 48 * 1024) { int rc = orn_grant_smem(ctx, (const void*)decayed_plain_kernel<bf16_t>, kDpSmemMax); if (rc) return rc; }
    decayed_plain_kernel<bf16_t><<<grid, kDpThreads, smem, s>>>(D, A);
  }
  return orn_launch_check(ctx, "decayed_plain");
}

bool decayed_chunk_ok(const DecayedDims& D, const DecayedArgs& A) {
  return D.dim % 8 == 0 && D.vdim % 8 == 0 && D.vdim <= 256 && A.ldq % 8 == 0 && A.ldk % 8 == 0 && A.ldv % 8 == 0 && A.ldo % 2 == 0 &&
         A.nring >= 2 && !A.keep_all && rows_smem(D, 16) <= kDrSmemMax;
}
size_t decayed_chunk_scratch(const DecayedDims& D, int T) {
  return ((size_t)T + kDecayChunk - 1) / kDecayChunk * D.state() * 8;  // folded chunks; states as bf16 value and remainder
}
int k_decayed_chunk(orn_ctx* ctx, cudaStream_t s, const DecayedDims& D, const DecayedArgs& A, void* scratch) {
  if (!decayed_chunk_ok(D, A)) ORN_FAIL(ctx, ORN_ERR_ARG, "decayed state: sizes of the chunk form");
  const int chunks = (A.T + kDecayChunk - 1) / kDecayChunk;
  float* U = reinterpret_cast<float*>(scratch);
  bf16_t* S2 = reinterpret_cast<bf16_t*>(U + (size_t)chunks * D.state());
  decayed_fold_kernel<<<dim3(chunks, D.heads, ((D.dim + 63) / 64) * ((D.vdim + 63) / 64)), 128, 0, s>>>(D, A, U);
  int rc = orn_launch_check(ctx, "decayed_fold");
  if (rc != ORN_OK) return rc;
  decayed_carry_kernel<<<(unsigned)((D.state() / 4 + 127) / 128), 128, 0, s>>>(D, A, U, S2);
  rc = orn_launch_check(ctx, "decayed_carry");
  if (rc != ORN_OK) return rc;
  const int nv = (D.vdim + 15) / 16;
  if (nv <= 2) return launch_rows<2>(ctx, s, D, A, S2);
  if (nv <= 4) return launch_rows<4>(ctx, s, D, A, S2);
  if (nv <= 6) return launch_rows<6>(ctx, s, D, A, S2);
  if (nv <= 8) return launch_rows<8>(ctx, s, D, A, S2);
  if (nv <= 12) return launch_rows<12>(ctx, s, D, A, S2);
  return launch_rows<16>(ctx, s, D, A, S2);
}
