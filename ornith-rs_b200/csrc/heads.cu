// Rotation in halves, unit norm and cache append of a projection's heads, for prompt chunks and the
// control route (decode windows do the same inside their mixers' kernels).
#include <algorithm>

#include "act.cuh"
#include "heads.h"

namespace {

constexpr int kHrThreads = 256, kHrWarps = kHrThreads / 32;
constexpr size_t kHrSmemMax = 200 * 1024;

struct HeadRowsArgs {
  HeadRows job[3];
  int n, half, max_dim, cs_job;
};

// One CTA per row: the row's angles once, then a warp per head.
template <typename TA>
__global__ void __launch_bounds__(kHrThreads) head_rows_kernel(HeadRowsArgs A, const int* __restrict__ pos) {
  extern __shared__ __align__(16) uint8_t hsm[];
  float2* s_cs = reinterpret_cast<float2*>(hsm);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  float* s_v = reinterpret_cast<float*>(s_cs + A.half) + (size_t)warp * A.max_dim;
  const int t = blockIdx.x, p = *pos + t;
  for (int i = threadIdx.x; i < A.half; i += kHrThreads) {
    float2 r;
    head_rotation(p, A.job[A.cs_job].freq[i], r.x, r.y);
    s_cs[i] = r;
  }
  __syncthreads();
  int first = 0;  // heads of all projections are dealt to the warps in turn
  for (int j = 0; j < A.n; ++j) {
    const HeadRows& J = A.job[j];
    const int row = J.dst_at_pos ? p : t;
    if (!J.dst_at_pos || p < J.cap) {
      const TA* src = reinterpret_cast<const TA*>(J.src) + (size_t)t * J.ld_src;
      TA* dst = reinterpret_cast<TA*>(J.dst) + (size_t)row * J.ld_dst;
      for (int h = (warp + kHrWarps - first % kHrWarps) % kHrWarps; h < J.heads; h += kHrWarps) {
        float sq = 0.f;
        for (int d = lane; d < J.dim; d += 32) {
          const float v = from_act(src[(size_t)h * J.dim + d]);
          s_v[d] = v;
          sq = fmaf(v, v, sq);
        }
        __syncwarp();
        const float r = J.unit ? 1.0f / sqrtf(warp_sum(sq) / (float)J.dim + J.eps) : 1.0f;  // turning keeps the length
        const int half = J.rot_dims / 2;
        for (int d = lane; d < J.dim; d += 32)
          dst[(size_t)h * J.dim + d] = to_act<TA>(rotated_half(d, half, s_cs, [&](int e) { return s_v[e]; }) * r);
        __syncwarp();
      }
    }
    first += J.heads;
  }
}

}  // namespace

int k_head_rows(orn_ctx* ctx, cudaStream_t s, int T, const HeadRows* jobs, int n, const int* pos, bool act_f32) {
  if (n < 1 || n > 3) ORN_FAIL(ctx, ORN_ERR_ARG, "head rows: 1..3 projections");
  HeadRowsArgs A{};
  A.n = n;
  for (int j = 0; j < n; ++j) {
    const HeadRows& J = jobs[j];
    A.job[j] = J;
    A.max_dim = std::max(A.max_dim, J.dim);
    if (J.rot_dims > 0) {
      if (J.rot_dims % 2 || J.rot_dims > J.dim || (A.half > 0 && (A.half != J.rot_dims / 2 || A.job[A.cs_job].freq != J.freq)))
        ORN_FAIL(ctx, ORN_ERR_ARG, "head rows: the projections of one launch share their rotation");
      A.half = J.rot_dims / 2;
      A.cs_job = j;
    }
  }
  const size_t smem = sizeof(float2) * (size_t)A.half + sizeof(float) * (size_t)A.max_dim * kHrWarps;
  if (smem > kHrSmemMax) ORN_FAIL(ctx, ORN_ERR_ARG, "head rows: heads do not fit shared memory");
  if (act_f32) {
    if (smem > 48 * 1024) { int rc = orn_grant_smem(ctx, (const void*)head_rows_kernel<float>, kHrSmemMax); if (rc) return rc; }
    head_rows_kernel<float><<<T, kHrThreads, smem, s>>>(A, pos);
  } else {
    if (smem > 48 * 1024) { int rc = orn_grant_smem(ctx, (const void*)head_rows_kernel<bf16_t>, kHrSmemMax); if (rc) return rc; }
    head_rows_kernel<bf16_t><<<T, kHrThreads, smem, s>>>(A, pos);
  }
  return orn_launch_check(ctx, "head_rows");
}
