// Device side of the decayed state over a decode window: one CTA's share, for the kernels that run it.
#pragma once

#include "act.cuh"
#include "decayed.h"
#include "heads.h"

constexpr int kDwThreads = 256, kDwCols = 16, kDwMaxDim = 256, kDwMaxRows = 4;
constexpr size_t kDwSmem = sizeof(float) * (2 * kDwMaxRows * kDwMaxDim + kDwMaxRows * (kDwThreads / 32) * kDwCols) + sizeof(float2) * kDwMaxRows * (kDwMaxDim / 2);
ORN_HD int decayed_slices(const DecayedDims& D) { return (D.vdim + kDwCols - 1) / kDwCols; }

// A CTA owns 16 value columns of one head; a thread four of them in every 64th state row, in registers.
// The state does not depend on the kernel before this one, so it is requested before the wait.
template <int NP>  // 64-row passes: dim <= 64 NP
ORN_D void decayed_window_cta(const DecayedDims& D, const DecayedArgs& A, int cta, uint8_t* smem) {
  float* s_q = reinterpret_cast<float*>(smem);
  float* s_k = s_q + kDwMaxRows * kDwMaxDim;
  float* s_red = s_k + kDwMaxRows * kDwMaxDim;
  float2* s_cs = reinterpret_cast<float2*>(s_red + kDwMaxRows * (kDwThreads / 32) * kDwCols);
  const int slices = decayed_slices(D), h = cta / slices;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int col = (cta - h * slices) * kDwCols + 4 * (threadIdx.x & 3), row0 = threadIdx.x >> 2;
  const size_t ssz = D.state(), at = ((size_t)h * D.dim) * D.vdim + col;
  const bool mine = col < D.vdim;  // vdim is a multiple of 4
  const int cur = *A.cur;
  const float* sin = A.ring + (size_t)(cur % A.nring) * ssz + at;
  float4 S[NP];
#pragma unroll
  for (int i = 0; i < NP; ++i) {
    const int r = row0 + 64 * i;
    S[i] = mine && r < D.dim ? __ldcg(reinterpret_cast<const float4*>(sin + (size_t)r * D.vdim)) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  const float g = __ldg(D.gpow + (size_t)h * (kDecayChunk + 1) + 1);
  const int half = D.rot_dims / 2, T = A.T;
  const int p0 = *A.pos;
  for (int i = threadIdx.x; i < T * half; i += kDwThreads) {
    const int t = i / half, e = i - t * half;
    float2 r;
    head_rotation(p0 + t, D.freq[e], r.x, r.y);
    s_cs[i] = r;
  }
  pdl_wait();
  pdl_trigger();
  __syncthreads();
  const bf16_t *q = reinterpret_cast<const bf16_t*>(A.q) + (size_t)h * D.dim, *k = reinterpret_cast<const bf16_t*>(A.k) + (size_t)h * D.dim;
  for (int i = threadIdx.x; i < T * D.dim; i += kDwThreads) {
    const int t = i / D.dim, d = i - t * D.dim;
    s_q[t * kDwMaxDim + d] = rotated_half(d, half, s_cs + t * half, [&](int e) { return bf2f(__ldcg(q + (size_t)t * A.ldq + e)); });
    s_k[t * kDwMaxDim + d] = D.k_scale * rotated_half(d, half, s_cs + t * half, [&](int e) { return bf2f(__ldcg(k + (size_t)t * A.ldk + e)); });
  }
  __syncthreads();
  for (int t = 0; t < T; ++t) {
    float v[4] = {0.f, 0.f, 0.f, 0.f}, o[4] = {0.f, 0.f, 0.f, 0.f};
    if (mine) {
      const uint2 u = __ldcg(reinterpret_cast<const uint2*>(reinterpret_cast<const bf16_t*>(A.v) + (size_t)t * A.ldv + (size_t)h * D.vdim + col));
      v[0] = __uint_as_float(u.x << 16); v[1] = __uint_as_float(u.x & 0xffff0000u);
      v[2] = __uint_as_float(u.y << 16); v[3] = __uint_as_float(u.y & 0xffff0000u);
    }
    float* sout = nullptr;
    if (A.keep_all) sout = A.ring + (size_t)((cur + 1 + t) % A.nring) * ssz + at;
    else if (t + 1 == T) sout = A.ring + (size_t)((cur + 1) % A.nring) * ssz + at;
#pragma unroll
    for (int i = 0; i < NP; ++i) {
      const int r = row0 + 64 * i;
      if (r < D.dim) {
        const float kk = s_k[t * kDwMaxDim + r], qq = s_q[t * kDwMaxDim + r];
        S[i].x = fmaf(kk, v[0], g * S[i].x); S[i].y = fmaf(kk, v[1], g * S[i].y);
        S[i].z = fmaf(kk, v[2], g * S[i].z); S[i].w = fmaf(kk, v[3], g * S[i].w);
        o[0] = fmaf(qq, S[i].x, o[0]); o[1] = fmaf(qq, S[i].y, o[1]);
        o[2] = fmaf(qq, S[i].z, o[2]); o[3] = fmaf(qq, S[i].w, o[3]);
        if (mine && sout != nullptr) *reinterpret_cast<float4*>(sout + (size_t)r * D.vdim) = S[i];
      }
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) {  // over the warp's eight rows
      o[e] += __shfl_xor_sync(0xffffffffu, o[e], 4);
      o[e] += __shfl_xor_sync(0xffffffffu, o[e], 8);
      o[e] += __shfl_xor_sync(0xffffffffu, o[e], 16);
    }
    if (lane < 4) *reinterpret_cast<float4*>(s_red + (t * (kDwThreads / 32) + warp) * kDwCols + 4 * lane) = make_float4(o[0], o[1], o[2], o[3]);
  }
  __syncthreads();
  if (threadIdx.x < T * kDwCols) {
    const int t = threadIdx.x / kDwCols, c = threadIdx.x % kDwCols, gc = (cta - h * slices) * kDwCols + c;
    float s = 0.f;
#pragma unroll
    for (int w = 0; w < kDwThreads / 32; ++w) s += s_red[(t * (kDwThreads / 32) + w) * kDwCols + c];
    if (gc < D.vdim) A.o[(size_t)t * A.ldo + (size_t)h * D.vdim + gc] = s;
  }
}
ORN_D void decayed_window_any(const DecayedDims& D, const DecayedArgs& A, int cta, uint8_t* smem) {
  if (D.dim <= 64) decayed_window_cta<1>(D, A, cta, smem);
  else if (D.dim <= 128) decayed_window_cta<2>(D, A, cta, smem);
  else decayed_window_cta<4>(D, A, cta, smem);
}
