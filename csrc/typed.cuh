// Helpers for kernels that exist in two element types: bf16 (serving) and fp32 (everything in true 32-bit).  Arithmetic is fp32 in
// both; the fp32 form uses the accurate math functions, the bf16 form the fast ones (their error is far below a bf16 rounding).
// Sources that include this file are compiled without --use_fast_math.
#pragma once
#include "common.cuh"

namespace ats {

template <typename T> struct Typed;
template <> struct Typed<float> {
  static __device__ __forceinline__ float load(const float* p) { return *p; }
  static __device__ __forceinline__ void store(float* p, float v) { *p = v; }
  static __device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
  static __device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
  // eight values, 16-byte aligned; Raw8: as they lie in memory
  static __device__ __forceinline__ void load8(const float* p, float (&v)[8]) {
    *reinterpret_cast<float4*>(v) = *reinterpret_cast<const float4*>(p);
    *reinterpret_cast<float4*>(v + 4) = *reinterpret_cast<const float4*>(p + 4);
  }
  struct Raw8 { float4 a, b; };
  static __device__ __forceinline__ Raw8 raw8(const float* p) { return {*reinterpret_cast<const float4*>(p), *reinterpret_cast<const float4*>(p + 4)}; }
  static __device__ __forceinline__ void unpack8(const Raw8& r, float (&v)[8]) {
    v[0] = r.a.x; v[1] = r.a.y; v[2] = r.a.z; v[3] = r.a.w;
    v[4] = r.b.x; v[5] = r.b.y; v[6] = r.b.z; v[7] = r.b.w;
  }
  static __device__ __forceinline__ Raw8 pack8(const float (&v)[8]) { return {make_float4(v[0], v[1], v[2], v[3]), make_float4(v[4], v[5], v[6], v[7])}; }
  static __device__ __forceinline__ void store_raw8(float* p, const Raw8& r) {
    *reinterpret_cast<float4*>(p) = r.a;
    *reinterpret_cast<float4*>(p + 4) = r.b;
  }
  static __device__ __forceinline__ void store8(float* p, const float (&v)[8]) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
  }
  static __device__ __forceinline__ float exp_(float x) { return expf(x); }
  static __device__ __forceinline__ float tanh_(float x) { return tanhf(x); }
  static __device__ __forceinline__ float sigmoid_(float x) { return 1.f / (1.f + expf(-x)); }
};
template <> struct Typed<__nv_bfloat16> {
  static __device__ __forceinline__ float load(const __nv_bfloat16* p) { return __bfloat162float(*p); }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }
  static __device__ __forceinline__ float4 load4(const __nv_bfloat16* p) {  // 8-byte aligned
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y);
    return make_float4(a.x, a.y, b.x, b.y);
  }
  static __device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
  }
  using Raw8 = uint4;
  static __device__ __forceinline__ Raw8 raw8(const __nv_bfloat16* p) { return *reinterpret_cast<const uint4*>(p); }
  static __device__ __forceinline__ void load8(const __nv_bfloat16* p, float (&v)[8]) { unpack8(raw8(p), v); }
  static __device__ __forceinline__ void unpack8(const Raw8& u, float (&v)[8]) {
    const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y), c = unpack_bf16x2(u.z), d = unpack_bf16x2(u.w);
    v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y; v[4] = c.x; v[5] = c.y; v[6] = d.x; v[7] = d.y;
  }
  static __device__ __forceinline__ Raw8 pack8(const float (&v)[8]) {
    return make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]), pack_bf16x2(v[6], v[7]));
  }
  static __device__ __forceinline__ void store_raw8(__nv_bfloat16* p, const Raw8& r) { *reinterpret_cast<uint4*>(p) = r; }
  static __device__ __forceinline__ void store8(__nv_bfloat16* p, const float (&v)[8]) { store_raw8(p, pack8(v)); }
  static __device__ __forceinline__ float exp_(float x) { return __expf(x); }
  static __device__ __forceinline__ float tanh_(float x) { return tanh_fast(x); }
  static __device__ __forceinline__ float sigmoid_(float x) { return __fdividef(1.f, 1.f + __expf(-x)); }
};

// tanh form of gelu
template <typename T>
__device__ __forceinline__ float gelu_tanh_f(float z) {
  return 0.5f * z * (1.f + Typed<T>::tanh_(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

}  // namespace ats
