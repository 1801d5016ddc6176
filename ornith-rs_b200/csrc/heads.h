// Row-wise work on the heads of a projection: rotation in halves, unit norm, append to a cache.
#pragma once

#include "orn_internal.h"

// One projection of a launch.  Row t, head h is src[t][h * dim ..]; it goes to row t (dst_at_pos: row
// *pos + t, dropped from row `cap` on) of dst with the same layout.  dst may be src.
struct HeadRows {
  void* src = nullptr;
  int ld_src = 0;
  void* dst = nullptr;
  int ld_dst = 0;
  bool dst_at_pos = false;
  int cap = 0;
  int heads = 0, dim = 0;
  int rot_dims = 0;              // entries (i, i + rot_dims / 2) turn by position * freq[i], the rest pass
  const double* freq = nullptr;  // device [rot_dims / 2]
  bool unit = false;             // then every head over its root mean square
  float eps = 0.f;
};
// up to three projections that share a rotation; row t is at position *pos + t
int k_head_rows(orn_ctx* ctx, cudaStream_t s, int T, const HeadRows* jobs, int n, const int* pos, bool act_f32);

#ifdef __CUDACC__
// sine and cosine of position * f, the whole turns taken off in float64 so that far positions keep
// float32 accuracy
ORN_D void head_rotation(int position, double f, float& sn, float& cs) {
  constexpr double kTurn = 6.283185307179586;
  double a = (double)position * f;
  a = a - kTurn * rint(a / kTurn);
  sincosf((float)a, &sn, &cs);
}
// entry d of a vector v (a callable) whose first 2 * half entries turn in halves; cs: [half] {sine, cosine}
template <typename F>
ORN_D float rotated_half(int d, int half, const float2* cs, F v) {
  if (d >= 2 * half) return v(d);
  const float2 r = cs[d < half ? d : d - half];
  return d < half ? fmaf(v(d), r.y, -(v(d + half) * r.x)) : fmaf(v(d), r.y, v(d - half) * r.x);
}
#endif
