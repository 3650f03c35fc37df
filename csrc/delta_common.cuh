// Pieces shared by the portion kernels of the delta rules (delta_rule.cu, channel_delta.cu).
#pragma once
#include "typed.cuh"

namespace ats {

constexpr int DC = 8;  // tokens per group

// exp(rate softplus(a)), rate < 0.  The bf16 form uses the fast functions and, where exp(a) is small, the series of log(1 + x), so that a
// slow decay keeps its digits.
template <typename T>
__device__ __forceinline__ float decay_of(float a, float rate) {
  if constexpr (sizeof(T) == 4) {
    return expf(rate * (a > 20.f ? a : log1pf(expf(a))));
  } else {
    const float x = __expf(fminf(a, 20.f));
    const float l = x < 0.02f ? x * (1.f - x * (0.5f - x * (0.33333333f - 0.25f * x))) : __logf(1.f + x);
    return __expf(rate * (a > 20.f ? a : l));
  }
}

__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) { return __ffma2_rn(a, b, c); }  // one packed instruction
// Keeps the compiler from requesting the shared-memory rows of more tokens than registers can hold.
__device__ __forceinline__ void pace() { asm volatile("" ::: "memory"); }

// One step of a transposing reduction over lanes: of the pair (lo, hi) this lane keeps hi when its bit `s` is set, else lo, and adds
// what the lane across sends.
__device__ __forceinline__ float keep_add(float lo, float hi, int lane, int s) {
  const bool up = (lane & s) != 0;
  return (up ? hi : lo) + __shfl_xor_sync(0xffffffffu, up ? lo : hi, s);
}

template <int BYTES> struct Bits;
template <> struct Bits<4> { using type = uint32_t; };
template <> struct Bits<8> { using type = uint2; };
template <> struct Bits<16> { using type = uint4; };

// Column c of (1 + M)^-1 for the unit lower triangular system M_ij = beta_i kk[i][j], j < i, by forward substitution.
template <typename KK>
__device__ __forceinline__ void inverse_column(const float (&beta)[DC], const KK& kk, int c, float (&y)[DC]) {
#pragma unroll
  for (int i = 0; i < DC; ++i) {
    float acc = i == c ? 1.f : 0.f;
#pragma unroll
    for (int j = i - 1; j >= 0; --j) acc -= beta[i] * kk[i][j] * y[j];
    y[i] = acc;
  }
}

}  // namespace ats
