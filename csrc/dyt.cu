// Element-wise steps of blocks whose norm is Dynamic Tanh: dyt(x) = tanh(alpha x) w + b, no mean and no variance, so a whole
// "sublayer output -> output norm -> layer scale -> residual add -> next sublayer's input norm" chain is one element-wise function
//
//   x <- x + tanh(a1 (y + bias)) w1 + b1        (w1, b1: output norm times layer scale, in fp32)
//   h <- tanh(a2 x) w2 + b2
//
// The residual x is fp32.  For bf16 products the chain runs in the epilogue of the GEMM (gemm_tcgen05.cu); the kernels here serve
// the token embedding, fp32 products and the fold of split reductions.
#include "typed.cuh"

namespace ats {

struct DytVectors {  // all [N]
  const float* w1; const float* b1; float a1;
  const float* w2; const float* b2; float a2;
};

// y: `splits` fp32 blocks [rows, N], `split_stride` elements apart, summed; bias optional.  One thread per four columns.
template <typename T>
__global__ void __launch_bounds__(256) fold_dyt_kernel(const float* __restrict__ y, int splits, long long split_stride, const float* __restrict__ bias,
                                                       float* __restrict__ x, const DytVectors v, T* __restrict__ h, long long rows, int N) {
  pdl_prologue();
  const int quads = N >> 2;
  const long long total = rows * quads;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const int c = int(i % quads) << 2;
    const long long at = (i / quads) * N + c;
    float4 s = bias ? *reinterpret_cast<const float4*>(bias + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    for (int k = 0; k < splits; ++k) {
      const float4 t = *reinterpret_cast<const float4*>(y + k * split_stride + at);
      s.x += t.x; s.y += t.y; s.z += t.z; s.w += t.w;
    }
    const float4 w1 = *reinterpret_cast<const float4*>(v.w1 + c), b1 = *reinterpret_cast<const float4*>(v.b1 + c);
    float4 r = *reinterpret_cast<const float4*>(x + at);
    r.x += Typed<T>::tanh_(v.a1 * s.x) * w1.x + b1.x;
    r.y += Typed<T>::tanh_(v.a1 * s.y) * w1.y + b1.y;
    r.z += Typed<T>::tanh_(v.a1 * s.z) * w1.z + b1.z;
    r.w += Typed<T>::tanh_(v.a1 * s.w) * w1.w + b1.w;
    *reinterpret_cast<float4*>(x + at) = r;
    const float4 w2 = *reinterpret_cast<const float4*>(v.w2 + c), b2 = *reinterpret_cast<const float4*>(v.b2 + c);
    Typed<T>::store4(h + at, make_float4(Typed<T>::tanh_(v.a2 * r.x) * w2.x + b2.x, Typed<T>::tanh_(v.a2 * r.y) * w2.y + b2.y,
                                         Typed<T>::tanh_(v.a2 * r.z) * w2.z + b2.z, Typed<T>::tanh_(v.a2 * r.w) * w2.w + b2.w));
  }
}

// out = gelu_tanh(sum of the splits + bias)
template <typename T>
__global__ void __launch_bounds__(256) fold_gelu_kernel(const float* __restrict__ y, int splits, long long split_stride, const float* __restrict__ bias,
                                                        T* __restrict__ out, long long rows, int N) {
  pdl_prologue();
  const int quads = N >> 2;
  const long long total = rows * quads;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const int c = int(i % quads) << 2;
    const long long at = (i / quads) * N + c;
    float4 s = bias ? *reinterpret_cast<const float4*>(bias + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    for (int k = 0; k < splits; ++k) {
      const float4 t = *reinterpret_cast<const float4*>(y + k * split_stride + at);
      s.x += t.x; s.y += t.y; s.z += t.z; s.w += t.w;
    }
    Typed<T>::store4(out + at, make_float4(gelu_tanh_f<T>(s.x), gelu_tanh_f<T>(s.y), gelu_tanh_f<T>(s.z), gelu_tanh_f<T>(s.w)));
  }
}

// x = table[id] (+ add), h = dyt2(x).  Ids outside the table are clamped, as in the other embedding kernel.
template <typename T>
__global__ void __launch_bounds__(256) embed_dyt_kernel(const long long* __restrict__ ids, const T* __restrict__ table, int vocab,
                                                        const float* __restrict__ add, float* __restrict__ x, const float* __restrict__ w2,
                                                        const float* __restrict__ b2, float a2, T* __restrict__ h, long long rows, int N) {
  pdl_prologue();
  const int quads = N >> 2;
  const long long total = rows * quads;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const int c = int(i % quads) << 2;
    const long long r = i / quads, at = r * N + c;
    long long id = ids[r];
    id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
    float4 s = Typed<T>::load4(table + id * N + c);
    if (add) {
      const float4 t = *reinterpret_cast<const float4*>(add + c);
      s.x += t.x; s.y += t.y; s.z += t.z; s.w += t.w;
    }
    *reinterpret_cast<float4*>(x + at) = s;
    const float4 w = *reinterpret_cast<const float4*>(w2 + c), b = *reinterpret_cast<const float4*>(b2 + c);
    Typed<T>::store4(h + at, make_float4(Typed<T>::tanh_(a2 * s.x) * w.x + b.x, Typed<T>::tanh_(a2 * s.y) * w.y + b.y,
                                         Typed<T>::tanh_(a2 * s.z) * w.z + b.z, Typed<T>::tanh_(a2 * s.w) * w.w + b.w));
  }
}

static inline int elementwise_grid(long long threads) {
  const long long b = (threads + 255) / 256;
  return int(b < 1 ? 1 : (b > 148 * 16 ? 148 * 16 : b));
}

}  // namespace ats

using namespace ats;

ATS_API int ats_fold_dyt(const void* y, int splits, long long split_stride, const void* bias, void* x, const void* w1, const void* b1, float a1,
                         const void* w2, const void* b2, float a2, void* h, int h_fp32, long long rows, int N, void* stream) {
  if ((N & 7) || splits < 1) return 1003;
  if (rows <= 0) return 0;
  DytVectors v{static_cast<const float*>(w1), static_cast<const float*>(b1), a1, static_cast<const float*>(w2), static_cast<const float*>(b2), a2};
  const dim3 grid(elementwise_grid(rows * (N >> 2)));
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (h_fp32)
    launch_pdl(fold_dyt_kernel<float>, grid, dim3(256), 0, s, static_cast<const float*>(y), splits, split_stride, static_cast<const float*>(bias),
               static_cast<float*>(x), v, static_cast<float*>(h), rows, N);
  else
    launch_pdl(fold_dyt_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, static_cast<const float*>(y), splits, split_stride,
               static_cast<const float*>(bias), static_cast<float*>(x), v, static_cast<__nv_bfloat16*>(h), rows, N);
  return int(cudaGetLastError());
}

ATS_API int ats_fold_gelu(const void* y, int splits, long long split_stride, const void* bias, void* out, int out_fp32, long long rows, int N, void* stream) {
  if ((N & 7) || splits < 1) return 1003;
  if (rows <= 0) return 0;
  const dim3 grid(elementwise_grid(rows * (N >> 2)));
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (out_fp32)
    launch_pdl(fold_gelu_kernel<float>, grid, dim3(256), 0, s, static_cast<const float*>(y), splits, split_stride, static_cast<const float*>(bias),
               static_cast<float*>(out), rows, N);
  else
    launch_pdl(fold_gelu_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, static_cast<const float*>(y), splits, split_stride,
               static_cast<const float*>(bias), static_cast<__nv_bfloat16*>(out), rows, N);
  return int(cudaGetLastError());
}

ATS_API int ats_embed_dyt(const void* ids, const void* table, int table_fp32, int vocab, const void* add, void* x, const void* w2, const void* b2,
                          float a2, void* h, long long rows, int N, void* stream) {
  if ((N & 7) || vocab < 1) return 1003;
  if (rows <= 0) return 0;
  const dim3 grid(elementwise_grid(rows * (N >> 2)));
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (table_fp32)
    launch_pdl(embed_dyt_kernel<float>, grid, dim3(256), 0, s, static_cast<const long long*>(ids), static_cast<const float*>(table), vocab,
               static_cast<const float*>(add), static_cast<float*>(x), static_cast<const float*>(w2), static_cast<const float*>(b2), a2,
               static_cast<float*>(h), rows, N);
  else
    launch_pdl(embed_dyt_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, static_cast<const long long*>(ids), static_cast<const __nv_bfloat16*>(table),
               vocab, static_cast<const float*>(add), static_cast<float*>(x), static_cast<const float*>(w2), static_cast<const float*>(b2), a2,
               static_cast<__nv_bfloat16*>(h), rows, N);
  return int(cudaGetLastError());
}
