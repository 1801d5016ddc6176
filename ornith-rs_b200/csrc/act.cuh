// Activations that kernels apply to a float32 product before it is stored.
#pragma once

#include "orn_common.cuh"

enum { ACT_NONE = 0, ACT_XIELU = 1, ACT_SOFTCAP = 2, ACT_SILU = 3, ACT_SIGMOID = 4, ACT_GELU_TANH = 5 };

// xIELU with the two learned numbers (p, q): a = softplus(p) scales the square above zero,
// b = 1/2 + softplus(q) the exponential below; the slope at zero is 1/2 on both sides.
struct ActParams {
  int kind = ACT_NONE;
  const bf16_t* pq = nullptr;  // ACT_XIELU: device array of two
  float cap = 0.f;             // ACT_SOFTCAP: cap * tanh(z / cap)
};

#ifdef __CUDACC__
// the activation type of a model: float32 or bfloat16
template <typename T> __device__ __forceinline__ T to_act(float v);
template <> __device__ __forceinline__ float to_act<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16_t to_act<bf16_t>(float v) { return f2bf(v); }
ORN_D float from_act(float v) { return v; }
ORN_D float from_act(bf16_t v) { return bf2f(v); }

ORN_D float act_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
// the two scalars an activation needs, once per thread
ORN_D void act_prepare(const ActParams& A, float& a, float& b) {
  a = A.cap; b = 0.f;
  if (A.kind == ACT_XIELU) {
    a = act_softplus(bf2f(A.pq[0]));
    b = 0.5f + act_softplus(bf2f(A.pq[1]));
  }
}
ORN_D float sigmoid_f32(float z) { return 1.0f / (1.0f + expf(-z)); }
// z / 2 (1 + tanh u), u = sqrt(2 / pi) (z + 0.044715 z^3)
ORN_D float gelu_tanh_f32(float z) { return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * fmaf(0.044715f * z * z, z, z))); }
ORN_D float act_apply(int kind, float z, float a, float b) {
  if (kind == ACT_XIELU) return z > 0.f ? fmaf(a * z, z, 0.5f * z) : fmaf(b, expm1f(z) - z, 0.5f * z);
  if (kind == ACT_SOFTCAP) return a * tanhf(z / a);
  if (kind == ACT_SILU) return z * sigmoid_f32(z);
  if (kind == ACT_SIGMOID) return sigmoid_f32(z);
  if (kind == ACT_GELU_TANH) return gelu_tanh_f32(z);
  return z;
}
// N values at once: the kind is looked at once, and an unrolled caller holds every activation's code
// N times in a row instead of all of them between any two values
template <int N> ORN_D void act_apply_n(int kind, float* z, float a, float b) {
#define ORN_ACT_CASE(K)                                       \
  case K:                                                     \
    _Pragma("unroll") for (int i = 0; i < N; ++i) z[i] = act_apply(K, z[i], a, b); \
    break
  switch (kind) {
    ORN_ACT_CASE(ACT_XIELU);
    ORN_ACT_CASE(ACT_SOFTCAP);
    ORN_ACT_CASE(ACT_SILU);
    ORN_ACT_CASE(ACT_SIGMOID);
    ORN_ACT_CASE(ACT_GELU_TANH);
    default: break;
  }
#undef ORN_ACT_CASE
}
#endif
