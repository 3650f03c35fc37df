// Steps of blocks whose norm follows the residual sum (post-norm): x <- rms(alpha x + y) w, rms(z) = z / sqrt(mean(z^2) + eps).
//
// * embed_rows: x = table[id] in fp32, h = the same in the element type of the products.
// * fold_postnorm: the residual step after a product whose fp32 result arrives as `splits` partial blocks (a decode-sized product
//   splits its reduction): one CTA per row sums the blocks, adds alpha x, normalises, writes the fp32 residual and the next product's
//   input h.  With w2 (the model's last norm) h is rms(x) w2 instead of x.
// * fold_silu: the sum of the blocks in the element type, silu on the first act_cols columns (the GEMM's own epilogue does the same
//   when the reduction is not split).
// * norm_gate: out = rms(o) w sigmoid(gate) over whole rows (all heads of a recurrence together).
// * softcap: z <- cap tanh(z / cap) in place.
//
// Rows are padded to multiples of 8 columns; padded columns hold zeros and the mean runs over the real width.
#include "typed.cuh"

namespace ats {

template <typename T>
__global__ void __launch_bounds__(256) embed_rows_kernel(const long long* __restrict__ ids, const T* __restrict__ table, int V, float* __restrict__ x,
                                                         T* __restrict__ h, long long rows, int N) {
  pdl_prologue();
  const int quads = N >> 2;
  const long long total = rows * quads;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long row = i / quads;
    const int c = int(i % quads) << 2;
    long long id = ids[row];
    id = id < 0 ? 0 : (id >= V ? V - 1 : id);
    const float4 v = Typed<T>::load4(table + id * N + c);
    *reinterpret_cast<float4*>(x + row * N + c) = v;
    if (h) Typed<T>::store4(h + row * N + c, v);
  }
}

struct PostNormArgs {
  const float* y;        // `splits` blocks [rows, N], split_stride elements apart
  int splits;
  long long split_stride;
  float* x;              // [rows, N]
  float alpha;
  const float* w;        // [N], zero in padded columns
  const float* w2;       // [N] or null: norm of the result, for h only
  float eps;
  void* h;               // [rows, N] or null
  long long rows;
  int N, width;
};

// QPT quads per thread stay in registers between the passes (N <= 4 * 256 * QPT); QPT = 0: rows of any length go through x.
template <typename T, int QPT>
__global__ void __launch_bounds__(256) fold_postnorm_kernel(const PostNormArgs p) {
  pdl_prologue();
  __shared__ float red[40];
  const long long row = blockIdx.x;
  const int quads = p.N >> 2, tid = threadIdx.x;
  float* x = p.x + row * p.N;
  const float* y = p.y + row * p.N;
  T* h = p.h ? static_cast<T*>(p.h) + row * p.N : nullptr;
  auto sum = [&](int q) {
    float4 z = *reinterpret_cast<const float4*>(x + 4 * q);
    z.x *= p.alpha; z.y *= p.alpha; z.z *= p.alpha; z.w *= p.alpha;
    for (int s = 0; s < p.splits; ++s) {
      const float4 t = *reinterpret_cast<const float4*>(y + s * p.split_stride + 4 * q);
      z.x += t.x; z.y += t.y; z.z += t.z; z.w += t.w;
    }
    return z;
  };
  auto sq = [](const float4& z) { return z.x * z.x + z.y * z.y + z.z * z.z + z.w * z.w; };
  auto scaled = [](const float4& z, const float* w, float r) {
    const float4 g = *reinterpret_cast<const float4*>(w);
    return make_float4(z.x * r * g.x, z.y * r * g.y, z.z * r * g.z, z.w * r * g.w);
  };
  constexpr int R = QPT > 0 ? QPT : 1;
  float4 z[R];
  float ss = 0.f;
  if constexpr (QPT > 0) {
#pragma unroll
    for (int i = 0; i < QPT; ++i) {
      const int q = tid + i * 256;
      z[i] = q < quads ? sum(q) : make_float4(0.f, 0.f, 0.f, 0.f);
      ss += sq(z[i]);
    }
  } else {
    for (int q = tid; q < quads; q += 256) {
      const float4 t = sum(q);
      *reinterpret_cast<float4*>(x + 4 * q) = t;  // read back by this thread
      ss += sq(t);
    }
  }
  const float r = 1.f / sqrtf(block_sum(ss, red) / float(p.width) + p.eps);
  float s2 = 0.f;
  auto finish = [&](int q, float4 t) {
    t = scaled(t, p.w + 4 * q, r);
    *reinterpret_cast<float4*>(x + 4 * q) = t;
    if (p.w2) s2 += sq(t);
    else if (h) Typed<T>::store4(h + 4 * q, t);
    return t;
  };
  if constexpr (QPT > 0) {
#pragma unroll
    for (int i = 0; i < QPT; ++i)
      if (tid + i * 256 < quads) z[i] = finish(tid + i * 256, z[i]);
  } else {
    for (int q = tid; q < quads; q += 256) finish(q, *reinterpret_cast<const float4*>(x + 4 * q));
  }
  if (!p.w2) return;  // the whole grid agrees
  const float r2 = 1.f / sqrtf(block_sum(s2, red) / float(p.width) + p.eps);
  if constexpr (QPT > 0) {
#pragma unroll
    for (int i = 0; i < QPT; ++i)
      if (tid + i * 256 < quads) Typed<T>::store4(h + 4 * (tid + i * 256), scaled(z[i], p.w2 + 4 * (tid + i * 256), r2));
  } else {
    for (int q = tid; q < quads; q += 256) Typed<T>::store4(h + 4 * q, scaled(*reinterpret_cast<const float4*>(x + 4 * q), p.w2 + 4 * q, r2));
  }
}

template <typename T>
__global__ void __launch_bounds__(256) fold_silu_kernel(const float* __restrict__ y, int splits, long long split_stride, T* __restrict__ out, long long rows,
                                                        int N, int act_cols) {
  pdl_prologue();
  const int quads = N >> 2;
  const long long total = rows * quads;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const int c = int(i % quads) << 2;
    float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int k = 0; k < splits; ++k) {
      const float4 t = *reinterpret_cast<const float4*>(y + k * split_stride + 4 * i);
      s.x += t.x; s.y += t.y; s.z += t.z; s.w += t.w;
    }
    if (c < act_cols) {  // act_cols is a multiple of 8
      s.x *= Typed<T>::sigmoid_(s.x); s.y *= Typed<T>::sigmoid_(s.y); s.z *= Typed<T>::sigmoid_(s.z); s.w *= Typed<T>::sigmoid_(s.w);
    }
    Typed<T>::store4(out + 4 * i, s);
  }
}

struct NormGateArgs {
  const void* o;         // [rows, ldo]
  long long ldo;
  const void* gate;      // [rows, ldg]
  long long ldg;
  const float* w;        // [width]
  float eps;
  void* out;             // [rows, ldout]; columns width .. ldout are zeroed
  long long ldout;
  long long rows;
  int width, vec;        // vec: every row starts at a multiple of 16 bytes and width is a multiple of 8
};

// OPT octets per thread stay in registers (width <= 8 * 256 * OPT); OPT = 0: any width, element by element.
template <typename T, int OPT>
__global__ void __launch_bounds__(256) norm_gate_kernel(const NormGateArgs p) {
  pdl_prologue();
  __shared__ float red[40];
  const long long row = blockIdx.x;
  const T* o = static_cast<const T*>(p.o) + row * p.ldo;
  const T* g = static_cast<const T*>(p.gate) + row * p.ldg;
  T* out = static_cast<T*>(p.out) + row * p.ldout;
  const int tid = threadIdx.x;
  float ss = 0.f;
  if constexpr (OPT > 0) {
    float v[OPT][8];
#pragma unroll
    for (int i = 0; i < OPT; ++i) {
      const int c = 8 * (tid + i * 256);
      if (c < p.width) {
        Typed<T>::load8(o + c, v[i]);
#pragma unroll
        for (int e = 0; e < 8; ++e) ss += v[i][e] * v[i][e];
      }
    }
    const float r = 1.f / sqrtf(block_sum(ss, red) / float(p.width) + p.eps);
#pragma unroll
    for (int i = 0; i < OPT; ++i) {
      const int c = 8 * (tid + i * 256);
      if (c >= p.width) continue;
      float z[8], w[8];
      Typed<T>::load8(g + c, z);
      Typed<float>::load8(p.w + c, w);
#pragma unroll
      for (int e = 0; e < 8; ++e) v[i][e] *= r * w[e] * Typed<T>::sigmoid_(z[e]);
      Typed<T>::store8(out + c, v[i]);
    }
  } else {
    for (int c = tid; c < p.width; c += 256) {
      const float v = Typed<T>::load(o + c);
      ss += v * v;
    }
    const float r = 1.f / sqrtf(block_sum(ss, red) / float(p.width) + p.eps);
    for (int c = tid; c < p.width; c += 256) Typed<T>::store(out + c, Typed<T>::load(o + c) * r * p.w[c] * Typed<T>::sigmoid_(Typed<T>::load(g + c)));
  }
  for (int c = p.width + tid; c < p.ldout; c += 256) Typed<T>::store(out + c, 0.f);
}

template <bool FAST>
__global__ void __launch_bounds__(256) softcap_kernel(float* __restrict__ z, long long quads, float cap) {
  pdl_prologue();
  const float inv = 1.f / cap;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < quads; i += (long long)gridDim.x * blockDim.x) {
    float4 v = reinterpret_cast<float4*>(z)[i];
    if constexpr (FAST) v = make_float4(cap * tanh_fast(v.x * inv), cap * tanh_fast(v.y * inv), cap * tanh_fast(v.z * inv), cap * tanh_fast(v.w * inv));
    else v = make_float4(cap * tanhf(v.x / cap), cap * tanhf(v.y / cap), cap * tanhf(v.z / cap), cap * tanhf(v.w / cap));
    reinterpret_cast<float4*>(z)[i] = v;
  }
}

static unsigned grid_for(long long n) {
  long long b = (n + 255) / 256;
  return unsigned(b < 1 ? 1 : b > 148 * 16 ? 148 * 16 : b);
}

template <typename T>
static int launch_postnorm(const PostNormArgs& p, cudaStream_t s) {
  const int q = (p.N / 4 + 255) / 256;
  const dim3 grid{unsigned(p.rows)}, block(256);
  if (q <= 1) launch_pdl(fold_postnorm_kernel<T, 1>, grid, block, 0, s, p);
  else if (q <= 2) launch_pdl(fold_postnorm_kernel<T, 2>, grid, block, 0, s, p);
  else if (q <= 4) launch_pdl(fold_postnorm_kernel<T, 4>, grid, block, 0, s, p);
  else if (q <= 8) launch_pdl(fold_postnorm_kernel<T, 8>, grid, block, 0, s, p);
  else launch_pdl(fold_postnorm_kernel<T, 0>, grid, block, 0, s, p);
  return int(cudaGetLastError());
}

template <typename T>
static int launch_norm_gate(const NormGateArgs& p, cudaStream_t s) {
  const int o = (p.width / 8 + 255) / 256;
  const dim3 grid{unsigned(p.rows)}, block(256);
  if (!p.vec || o > 4) launch_pdl(norm_gate_kernel<T, 0>, grid, block, 0, s, p);
  else if (o <= 1) launch_pdl(norm_gate_kernel<T, 1>, grid, block, 0, s, p);
  else if (o <= 2) launch_pdl(norm_gate_kernel<T, 2>, grid, block, 0, s, p);
  else launch_pdl(norm_gate_kernel<T, 4>, grid, block, 0, s, p);
  return int(cudaGetLastError());
}

}  // namespace ats

using namespace ats;

ATS_API int ats_embed_rows(const void* ids, const void* table, int fp32, int V, float* x, void* h, long long rows, int N, void* stream) {
  if (rows <= 0) return 0;
  if ((N & 3) || V < 1) return 1003;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const dim3 grid(grid_for(rows * (N / 4)));
  const long long* i = static_cast<const long long*>(ids);
  if (fp32) launch_pdl(embed_rows_kernel<float>, grid, dim3(256), 0, s, i, static_cast<const float*>(table), V, x, static_cast<float*>(h), rows, N);
  else launch_pdl(embed_rows_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, i, static_cast<const __nv_bfloat16*>(table), V, x, static_cast<__nv_bfloat16*>(h), rows, N);
  return int(cudaGetLastError());
}

// Argument structs are passed by address (ctypes mirrors in ops/postnorm.py); `fp32` selects the element type.
ATS_API int ats_fold_postnorm(const PostNormArgs* p, int fp32, void* stream) {
  if (p->rows <= 0) return 0;
  if ((p->N & 3) || p->width < 1 || p->width > p->N || p->splits < 1 || (p->w2 && !p->h)) return 1003;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return fp32 ? launch_postnorm<float>(*p, s) : launch_postnorm<__nv_bfloat16>(*p, s);
}

ATS_API int ats_norm_gate(const NormGateArgs* p, int fp32, void* stream) {
  if (p->rows <= 0) return 0;
  if (p->width < 1 || (p->vec && (p->width & 7))) return 1003;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return fp32 ? launch_norm_gate<float>(*p, s) : launch_norm_gate<__nv_bfloat16>(*p, s);
}

ATS_API int ats_fold_silu(const float* y, int splits, long long split_stride, void* out, int fp32, long long rows, int N, int act_cols, void* stream) {
  if (rows <= 0) return 0;
  if ((N & 3) || (act_cols & 7) || splits < 1) return 1003;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const dim3 grid(grid_for(rows * (N / 4)));
  if (fp32) launch_pdl(fold_silu_kernel<float>, grid, dim3(256), 0, s, y, splits, split_stride, static_cast<float*>(out), rows, N, act_cols);
  else launch_pdl(fold_silu_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, y, splits, split_stride, static_cast<__nv_bfloat16*>(out), rows, N, act_cols);
  return int(cudaGetLastError());
}

// z: n fp32 values (a multiple of 4); `fast`: one exponential per value (absolute error a few 1e-7 cap) instead of tanhf.
ATS_API int ats_softcap(float* z, long long n, float cap, int fast, void* stream) {
  if (n <= 0) return 0;
  if ((n & 3) || !(cap > 0.f)) return 1003;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (fast) launch_pdl(softcap_kernel<true>, dim3(grid_for(n / 4)), dim3(256), 0, s, z, n / 4, cap);
  else launch_pdl(softcap_kernel<false>, dim3(grid_for(n / 4)), dim3(256), 0, s, z, n / 4, cap);
  return int(cudaGetLastError());
}
