// Grouped-query attention over a full key / value cache with normed queries and keys, partial interleaved rotation, capped scores and
// one output gate per head (each of these a parameter; cap = 0 and gate = null switch theirs off):
//
//   q, k <- rotate(rms over all heads together)       (2 i and 2 i + 1 turn by position * f_i, i < dims / 2; the rest passes)
//   out[i, h] = sigmoid(gate[i, h]) softmax_{j <= i}( cap tanh(scale q_i . k_j / cap) ) v_j,   key head h / (H / G)
//
// The cache holds k [B, max_len, ldk] as the scores use it (normed and rotated) and v [B, max_len, ldv]; a layer that shares another
// layer's keys and values reads that layer's cache and prepares only its queries.
//
// * gqa_prepare: norm, rotation, cache append; a warp (few tokens: a CTA) for a token's queries and one for its key and value.
// * gqa_portion: L queries of a prompt at positions pos0 .. against the cache, any sizes, bf16 and fp32 (gqa_attention_tcgen05.cu is the
//   tensor-core form).
// * gqa_decode + gqa_merge: one query token per sequence, any sizes (decode_attn_mma_kernel in inference.cu serves bf16 heads of 64 and 128).
#include "typed.cuh"

namespace ats {

template <typename T> struct Cap;
template <> struct Cap<float> {
  static __device__ __forceinline__ float apply(float s, float cap) { return cap > 0.f ? cap * tanhf(s / cap) : s; }
};
template <> struct Cap<__nv_bfloat16> {
  static __device__ __forceinline__ float apply(float s, float cap) { return cap > 0.f ? cap * tanh_fast(__fdividef(s, cap)) : s; }
};

struct GqaPrepArgs {
  const void* proj;        // [B * L, ld]: q at column 0, k and v at the columns below (k_col < 0: queries only)
  long long ld;
  int k_col, v_col;
  const float* q_w;        // [H * dim] norm weights
  const float* k_w;        // [G * dim]
  float eps;
  const float* cos;        // [positions, dims / 2]
  const float* sin;
  int dims;
  void* q;                 // [B * L, ldq]
  long long ldq;
  void* k;                 // [B, max_len, ldk]
  void* v;                 // [B, max_len, ldv]
  long long k_bs, v_bs, ldk, ldv;
  int B, L, H, G, dim, vdim, max_len, pos0;
  const int* lengths;      // decoding: position per sequence
  const int* active;       // decoding: rows with 0 leave the cache alone
};

// Normed and rotated value c of a row of heads (c counts over all heads).
template <typename T>
__device__ __forceinline__ float rotated(const T* in, const float* w, float r, int c, int dim, int dims, const float* cos, const float* sin) {
  const int d = c % dim;
  const float x = Typed<T>::load(in + c) * r * w[c];
  if (d >= dims) return x;
  const int m = d >> 1, other = (d & 1) ? c - 1 : c + 1;
  const float y = Typed<T>::load(in + other) * r * w[other];
  return (d & 1) ? x * cos[m] + y * sin[m] : x * cos[m] - y * sin[m];
}

// One row of n values by `threads` threads: out = rotate(in r w).  VEC: dim, dims multiples of 8, so that eight consecutive values belong to one
// head and are rotated or pass as a whole.
template <typename T, bool VEC>
__device__ __forceinline__ void norm_rotate_row(const T* in, const float* w, float r, int n, int dim, int dims, const float* cos, const float* sin, T* out,
                                                int id, int threads) {
  if constexpr (VEC) {
#pragma unroll 4
    for (int c = id * 8; c < n; c += 8 * threads) {
      float v[8], g[8];
      Typed<T>::load8(in + c, v);
      Typed<float>::load8(w + c, g);
#pragma unroll
      for (int e = 0; e < 8; ++e) v[e] *= r * g[e];
      const unsigned d = unsigned(c) % unsigned(dim);
      if (d < unsigned(dims)) {
        const float4 cs = *reinterpret_cast<const float4*>(cos + (d >> 1)), sn = *reinterpret_cast<const float4*>(sin + (d >> 1));
        const float c4[4] = {cs.x, cs.y, cs.z, cs.w}, s4[4] = {sn.x, sn.y, sn.z, sn.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float a = v[2 * e], b = v[2 * e + 1];
          v[2 * e] = a * c4[e] - b * s4[e];
          v[2 * e + 1] = b * c4[e] + a * s4[e];
        }
      }
      Typed<T>::store8(out + c, v);
    }
  } else {
    for (int c = id; c < n; c += threads) Typed<T>::store(out + c, rotated<T>(in, w, r, c, dim, dims, cos, sin));
  }
}

template <typename T, bool VEC>
__device__ __forceinline__ float row_square_sum(const T* in, int n, int id, int threads) {
  float ss = 0.f;
  if constexpr (VEC) {
#pragma unroll 4
    for (int c = id * 8; c < n; c += 8 * threads) {
      float v[8];
      Typed<T>::load8(in + c, v);
#pragma unroll
      for (int e = 0; e < 8; ++e) ss += v[e] * v[e];
    }
  } else {
    for (int c = id; c < n; c += threads) {
      const float v = Typed<T>::load(in + c);
      ss += v * v;
    }
  }
  return ss;
}

// One warp (WPR = 1) or one CTA of four (WPR = 4, for a handful of tokens) per (token, part): queries, or key and value.
template <typename T, bool VEC, int WPR>
__global__ void __launch_bounds__(128) gqa_prepare_kernel(const GqaPrepArgs p) {
  pdl_prologue();
  __shared__ float red[40];
  constexpr int threads = 32 * WPR;
  const int parts = p.k_col >= 0 ? 2 : 1, id = threadIdx.x % threads;
  const long long w = WPR == 4 ? blockIdx.x : blockIdx.x * 4ll + (threadIdx.x >> 5);
  if (w >= (long long)p.B * p.L * parts) return;  // whole warp, or whole CTA
  auto sum = [&](float v) {
    if constexpr (WPR == 4) return block_sum(v, red);
    else return warp_sum(v);
  };
  const long long row = w / parts;
  const int b = int(row / p.L), t = int(row % p.L), pos = p.lengths ? p.lengths[b] : p.pos0 + t;
  const T* in = static_cast<const T*>(p.proj) + row * p.ld;
  const float* cs = p.cos + (long long)pos * (p.dims >> 1);
  const float* sn = p.sin + (long long)pos * (p.dims >> 1);
  if (w % parts == 0) {
    const int nq = p.H * p.dim;
    const float rq = 1.f / sqrtf(sum(row_square_sum<T, VEC>(in, nq, id, threads)) / float(nq) + p.eps);
    T* q = static_cast<T*>(p.q) + row * p.ldq;
    norm_rotate_row<T, VEC>(in, p.q_w, rq, nq, p.dim, p.dims, cs, sn, q, id, threads);
    for (int c = nq + id; c < p.ldq; c += threads) Typed<T>::store(q + c, 0.f);
    return;
  }
  if (pos >= p.max_len || (p.active && !p.active[b])) return;
  const int nk = p.G * p.dim, nv = p.G * p.vdim;
  T* v = static_cast<T*>(p.v) + (long long)b * p.v_bs + pos * p.ldv;
  if constexpr (VEC) {
    for (int c = id * 8; c < nv; c += 8 * threads) Typed<T>::store_raw8(v + c, Typed<T>::raw8(in + p.v_col + c));
  } else {
    for (int c = id; c < nv; c += threads) v[c] = in[p.v_col + c];
  }
  const float rk = 1.f / sqrtf(sum(row_square_sum<T, VEC>(in + p.k_col, nk, id, threads)) / float(nk) + p.eps);
  norm_rotate_row<T, VEC>(in + p.k_col, p.k_w, rk, nk, p.dim, p.dims, cs, sn, static_cast<T*>(p.k) + (long long)b * p.k_bs + pos * p.ldk, id, threads);
}

struct GqaArgs {
  const void* q;           // [B * L, ldq], head h at h * dim
  long long ldq;
  const void* k;
  const void* v;
  long long k_bs, v_bs, ldk, ldv;
  const void* gate;        // [B * L, ldg] + h, or null
  long long ldg;
  void* out;               // [B * L, ldo], head h at h * vdim; columns H * vdim .. ldo are zeroed
  long long ldo;
  int B, L, H, G, dim, vdim, pos0, max_len;
  float scale, cap;
  const int* lengths;      // decoding: position per sequence (its key is in the cache already)
  int chunk, n_chunks;     // decoding: keys per CTA
  float* part_o;           // [B, H, n_chunks, vdim]
  float* part_ml;          // [B, H, n_chunks, 2]
};

constexpr int GA_MAX_V = 16;  // value dimensions per lane: heads of up to 512

// One warp per (query, head), 32 keys at a time.
template <typename T>
__global__ void __launch_bounds__(256) gqa_portion_kernel(const GqaArgs p) {
  pdl_prologue();
  extern __shared__ float s_q[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, t = blockIdx.x * 8 + warp, h = blockIdx.y, b = blockIdx.z, g = h / (p.H / p.G);
  if (t >= p.L) return;  // whole warp; no CTA barrier below
  const long long row = (long long)b * p.L + t;
  float* q = s_q + warp * p.dim;
  const T* qg = static_cast<const T*>(p.q) + row * p.ldq + (long long)h * p.dim;
  for (int c = lane; c < p.dim; c += 32) q[c] = Typed<T>::load(qg + c) * p.scale;
  __syncwarp();
  const T* kbase = static_cast<const T*>(p.k) + (long long)b * p.k_bs + (long long)g * p.dim;
  const T* vbase = static_cast<const T*>(p.v) + (long long)b * p.v_bs + (long long)g * p.vdim;
  const int hi = p.pos0 + t;
  float m = -INFINITY, l = 0.f, o[GA_MAX_V];
#pragma unroll
  for (int e = 0; e < GA_MAX_V; ++e) o[e] = 0.f;
  const bool vec = (p.dim & 3) == 0 && (p.ldk & 3) == 0;  // rows and heads start at multiples of four elements
  for (int k0 = 0; k0 <= hi; k0 += 32) {
    const int key = k0 + lane;
    float s = -INFINITY;
    if (key <= hi) {
      const T* kk = kbase + key * p.ldk;
      float acc = 0.f;
      if (vec) {
        for (int c = 0; c < p.dim; c += 4) {
          const float4 x = Typed<T>::load4(kk + c), y = *reinterpret_cast<const float4*>(q + c);
          acc += y.x * x.x + y.y * x.y + y.z * x.z + y.w * x.w;
        }
      } else {
        for (int c = 0; c < p.dim; ++c) acc += q[c] * Typed<T>::load(kk + c);
      }
      s = Cap<T>::apply(acc, p.cap);
    }
    const float mn = fmaxf(m, warp_max(s)), f = Typed<T>::exp_(m - mn);
    const float pr = key <= hi ? Typed<T>::exp_(s - mn) : 0.f;
    m = mn;
    l = l * f + pr;  // per lane; summed at the end
#pragma unroll
    for (int e = 0; e < GA_MAX_V; ++e) o[e] *= f;
    const int n = min(32, hi - k0 + 1);
    for (int j = 0; j < n; ++j) {
      const float pj = __shfl_sync(0xffffffffu, pr, j);
      const T* vv = vbase + (k0 + j) * p.ldv;
#pragma unroll
      for (int e = 0; e < GA_MAX_V; ++e)
        if (e * 32 + lane < p.vdim) o[e] += pj * Typed<T>::load(vv + e * 32 + lane);
    }
  }
  float inv = 1.f / warp_sum(l);
  if (p.gate) inv *= Typed<T>::sigmoid_(Typed<T>::load(static_cast<const T*>(p.gate) + row * p.ldg + h));
  T* out = static_cast<T*>(p.out) + row * p.ldo;
#pragma unroll
  for (int e = 0; e < GA_MAX_V; ++e) {
    const int c = e * 32 + lane;
    if (c < p.vdim) Typed<T>::store(out + (long long)h * p.vdim + c, o[e] * inv);
  }
  if (h == 0)
    for (int c = p.H * p.vdim + lane; c < p.ldo; c += 32) Typed<T>::store(out + c, 0.f);
}

constexpr int GD_R = 8;  // query heads per pass

// CTA (chunk of keys, key head, sequence): scores of up to eight query heads of the group, their soft-max inside the chunk, weighted values.
template <typename T>
__global__ void __launch_bounds__(128) gqa_decode_kernel(const GqaArgs p) {
  pdl_prologue();
  extern __shared__ __align__(16) float gsm[];
  const int chunk = blockIdx.x, g = blockIdx.y, b = blockIdx.z, rep = p.H / p.G, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int n_tot = min(p.lengths[b] + 1, p.max_len), k0 = chunk * p.chunk, n = min(p.chunk, n_tot - k0);
  const int dq = (p.dim + 3) & ~3;
  float* s_q = gsm;                 // [GD_R][dq]
  float* s_s = gsm + GD_R * dq;     // [GD_R][chunk]
  if (n <= 0) {
    for (int r = tid; r < rep; r += 128) {
      float* ml = p.part_ml + (((long long)b * p.H + g * rep + r) * p.n_chunks + chunk) * 2;
      ml[0] = -INFINITY;
      ml[1] = 0.f;
    }
    return;
  }
  const T* kbase = static_cast<const T*>(p.k) + (long long)b * p.k_bs + k0 * p.ldk + (long long)g * p.dim;
  const T* vbase = static_cast<const T*>(p.v) + (long long)b * p.v_bs + k0 * p.ldv + (long long)g * p.vdim;
  const bool vec = (p.dim & 3) == 0 && (p.ldk & 3) == 0;
  for (int r0 = 0; r0 < rep; r0 += GD_R) {
    const int nr = min(GD_R, rep - r0);
    for (int i = tid; i < nr * p.dim; i += 128)
      s_q[(i / p.dim) * dq + i % p.dim] = Typed<T>::load(static_cast<const T*>(p.q) + (long long)b * p.ldq + (long long)(g * rep + r0) * p.dim + i) * p.scale;
    __syncthreads();
    for (int j = tid; j < n; j += 128) {
      const T* kk = kbase + j * p.ldk;
      float acc[GD_R];
#pragma unroll
      for (int r = 0; r < GD_R; ++r) acc[r] = 0.f;
      if (vec) {
        for (int c = 0; c < p.dim; c += 4) {
          const float4 x = Typed<T>::load4(kk + c);
#pragma unroll
          for (int r = 0; r < GD_R; ++r) {
            if (r >= nr) break;
            const float4 y = *reinterpret_cast<const float4*>(s_q + r * dq + c);
            acc[r] += y.x * x.x + y.y * x.y + y.z * x.z + y.w * x.w;
          }
        }
      } else {
        for (int c = 0; c < p.dim; ++c) {
          const float x = Typed<T>::load(kk + c);
#pragma unroll
          for (int r = 0; r < GD_R; ++r)
            if (r < nr) acc[r] += s_q[r * dq + c] * x;
        }
      }
#pragma unroll
      for (int r = 0; r < GD_R; ++r)
        if (r < nr) s_s[r * p.chunk + j] = Cap<T>::apply(acc[r], p.cap);
    }
    __syncthreads();
    for (int r = warp; r < nr; r += 4) {
      float m = -INFINITY, l = 0.f;
      for (int j = lane; j < n; j += 32) m = fmaxf(m, s_s[r * p.chunk + j]);
      m = warp_max(m);
      for (int j = lane; j < n; j += 32) {
        const float e = Typed<T>::exp_(s_s[r * p.chunk + j] - m);
        s_s[r * p.chunk + j] = e;
        l += e;
      }
      l = warp_sum(l);
      if (lane == 0) {
        float* ml = p.part_ml + (((long long)b * p.H + g * rep + r0 + r) * p.n_chunks + chunk) * 2;
        ml[0] = m;
        ml[1] = l;
      }
    }
    __syncthreads();
    for (int c = tid; c < p.vdim; c += 128) {
      float o[GD_R];
#pragma unroll
      for (int r = 0; r < GD_R; ++r) o[r] = 0.f;
      for (int j = 0; j < n; ++j) {
        const float x = Typed<T>::load(vbase + j * p.ldv + c);
#pragma unroll
        for (int r = 0; r < GD_R; ++r)
          if (r < nr) o[r] += s_s[r * p.chunk + j] * x;
      }
#pragma unroll
      for (int r = 0; r < GD_R; ++r)
        if (r < nr) p.part_o[(((long long)b * p.H + g * rep + r0 + r) * p.n_chunks + chunk) * p.vdim + c] = o[r];
    }
    __syncthreads();
  }
}

// One warp per (sequence, head).
template <typename T>
__global__ void __launch_bounds__(256) gqa_merge_kernel(const GqaArgs p) {
  pdl_prologue();
  const int w = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (w >= p.B * p.H) return;
  const int b = w / p.H, h = w % p.H;
  const int used = min(p.n_chunks, p.lengths[b] / p.chunk + 1);
  const float* ml = p.part_ml + (long long)w * p.n_chunks * 2;
  float m = -INFINITY, l = 0.f;
  for (int c = 0; c < used; ++c) m = fmaxf(m, ml[2 * c]);
  for (int c = 0; c < used; ++c) l += ml[2 * c + 1] * Typed<T>::exp_(ml[2 * c] - m);
  float inv = 1.f / l;
  if (p.gate) inv *= Typed<T>::sigmoid_(Typed<T>::load(static_cast<const T*>(p.gate) + (long long)b * p.ldg + h));
  T* out = static_cast<T*>(p.out) + (long long)b * p.ldo;
  for (int d = lane; d < p.vdim; d += 32) {
    float t = 0.f;
    for (int c = 0; c < used; ++c) t += p.part_o[((long long)w * p.n_chunks + c) * p.vdim + d] * Typed<T>::exp_(ml[2 * c] - m);
    Typed<T>::store(out + (long long)h * p.vdim + d, t * inv);
  }
  if (h == 0)
    for (int c = p.H * p.vdim + lane; c < p.ldo; c += 32) Typed<T>::store(out + c, 0.f);
}

static int dynamic_smem(const void* kernel, size_t bytes) {
  if (bytes <= 48 * 1024) return 0;
  if (bytes > 227 * 1024) return 1010;
  return int(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, int(bytes)));
}

template <typename T>
static int launch_prepare(const GqaPrepArgs& p, cudaStream_t s) {
  const bool kv = p.k_col >= 0;
  uintptr_t at = reinterpret_cast<uintptr_t>(p.proj) | reinterpret_cast<uintptr_t>(p.q) | reinterpret_cast<uintptr_t>(p.q_w);
  long long n = p.ld | p.ldq | p.dim | p.dims;
  at |= reinterpret_cast<uintptr_t>(p.cos) | reinterpret_cast<uintptr_t>(p.sin);
  if (kv) {
    at |= reinterpret_cast<uintptr_t>(p.k) | reinterpret_cast<uintptr_t>(p.v) | reinterpret_cast<uintptr_t>(p.k_w);
    n |= p.k_col | p.v_col | p.ldk | p.ldv | p.k_bs | p.v_bs | (long long)p.G * p.vdim;
  }
  const long long units = (long long)p.B * p.L * (kv ? 2 : 1);
  const bool vec = !(at & 15) && !(n & 7), few = units <= 1024;
  const dim3 grid{unsigned(few ? units : (units + 3) / 4)}, block(128);
  if (vec && few) launch_pdl(gqa_prepare_kernel<T, true, 4>, grid, block, 0, s, p);
  else if (vec) launch_pdl(gqa_prepare_kernel<T, true, 1>, grid, block, 0, s, p);
  else if (few) launch_pdl(gqa_prepare_kernel<T, false, 4>, grid, block, 0, s, p);
  else launch_pdl(gqa_prepare_kernel<T, false, 1>, grid, block, 0, s, p);
  return int(cudaGetLastError());
}

template <typename T>
static int launch_portion(const GqaArgs& p, cudaStream_t s) {
  const size_t smem = size_t(8) * p.dim * sizeof(float);
  int e = dynamic_smem(reinterpret_cast<const void*>(gqa_portion_kernel<T>), smem);
  if (e) return e;
  launch_pdl(gqa_portion_kernel<T>, dim3((p.L + 7) / 8, p.H, p.B), dim3(256), smem, s, p);
  return int(cudaGetLastError());
}

template <typename T>
static int launch_decode(const GqaArgs& p, cudaStream_t s) {
  const size_t smem = size_t(GD_R) * (((p.dim + 3) & ~3) + p.chunk) * sizeof(float);
  int e = dynamic_smem(reinterpret_cast<const void*>(gqa_decode_kernel<T>), smem);
  if (e) return e;
  launch_pdl(gqa_decode_kernel<T>, dim3(p.n_chunks, p.G, p.B), dim3(128), smem, s, p);
  launch_pdl(gqa_merge_kernel<T>, dim3((p.B * p.H + 7) / 8), dim3(256), 0, s, p);
  return int(cudaGetLastError());
}

}  // namespace ats

using namespace ats;

// Argument structs are passed by address (ctypes mirrors in ops/gqa.py); `fp32` selects the element type.
ATS_API int ats_gqa_prepare(const GqaPrepArgs* p, int fp32, void* stream) {
  if (p->B <= 0 || p->L <= 0) return 0;
  if ((p->lengths && p->L != 1) || (p->dims & 1) || p->dims > p->dim || p->G < 1 || p->H % p->G) return 1006;
  return fp32 ? launch_prepare<float>(*p, static_cast<cudaStream_t>(stream)) : launch_prepare<__nv_bfloat16>(*p, static_cast<cudaStream_t>(stream));
}

ATS_API int ats_gqa_portion(const GqaArgs* p, int fp32, void* stream) {
  if (p->B <= 0 || p->L <= 0) return 0;
  if (p->G < 1 || p->H % p->G || p->vdim > 32 * GA_MAX_V) return 1006;
  return fp32 ? launch_portion<float>(*p, static_cast<cudaStream_t>(stream)) : launch_portion<__nv_bfloat16>(*p, static_cast<cudaStream_t>(stream));
}

ATS_API int ats_gqa_decode(const GqaArgs* p, int fp32, void* stream) {
  if (p->B <= 0) return 0;
  if (!p->lengths || p->L != 1 || p->G < 1 || p->H % p->G || p->chunk < 1 || p->n_chunks < 1) return 1006;
  return fp32 ? launch_decode<float>(*p, static_cast<cudaStream_t>(stream)) : launch_decode<__nv_bfloat16>(*p, static_cast<cudaStream_t>(stream));
}
