// Lightning attention: linear attention with one constant decay per head over a per-head matrix state S [dim, vdim] (fp32)
//
//   S <- decay S + k_t v_t^T;   o_t = S^T q_t
//
// q, k and v arrive activated in one projection buffer (head h at its column + h * dim, h * vdim).
//
// * lightning_scan: portions of a prompt for any sizes and both element types, token by token on the fp32 lanes, eight tokens per
//   round of loads (lightning_tcgen05.cu is the chunked tensor-core form for bf16).
// * lightning_step: one decoded token per sequence, state read once and written once.
//
// A sequence at position 0 starts from a zero state whatever its buffer holds.
#include "typed.cuh"

namespace ats {

struct LightningArgs {
  const void* qkv;         // [B * L, ld]
  long long ld;
  int q_col, k_col, v_col;
  const float* decay;      // [H]
  float* state;            // [B, H, dim, vdim]
  long long state_bs;      // elements between sequences
  void* o;                 // [B * L, ldo], head h at h * vdim
  long long ldo;
  int B, L, H, dim, vdim, fresh;
  const int* lengths;      // decoding: position per sequence
  const int* active;       // decoding: rows with 0 leave the state alone
};

constexpr int LT = 8;      // tokens per round
constexpr int LROWS = 8;   // row groups: thread (row group, column) holds RPT consecutive state rows of one column

// CTA = 8 row groups x 32 columns of one head.
template <typename T, int RPT>
__global__ void __launch_bounds__(256) lightning_scan_kernel(const LightningArgs p) {
  pdl_prologue();
  constexpr int DK = LROWS * RPT;
  __shared__ __align__(16) float s_q[LT][DK], s_k[LT][DK];
  __shared__ float s_v[LT][32], s_o[LT][LROWS][32];
  const int tid = threadIdx.x, c = tid & 31, rg = tid >> 5, h = blockIdx.y, b = blockIdx.z, v0 = blockIdx.x * 32, col = v0 + c;
  const float decay = p.decay[h];
  float* st = p.state + (long long)b * p.state_bs + (long long)h * p.dim * p.vdim;
  const T* base = static_cast<const T*>(p.qkv) + (long long)b * p.L * p.ld;
  T* out = static_cast<T*>(p.o) + (long long)b * p.L * p.ldo + (long long)h * p.vdim;
  float S[RPT];
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int d = rg * RPT + i;
    S[i] = (!p.fresh && d < p.dim && col < p.vdim) ? st[(long long)d * p.vdim + col] : 0.f;
  }
  for (int t0 = 0; t0 < p.L; t0 += LT) {
    const int n = min(LT, p.L - t0);
    for (int i = tid; i < LT * DK; i += 256) {
      const int t = i / DK, d = i % DK;
      const bool ok = t < n && d < p.dim;
      const T* row = base + (long long)(t0 + t) * p.ld + (long long)h * p.dim + d;
      s_q[t][d] = ok ? Typed<T>::load(row + p.q_col) : 0.f;
      s_k[t][d] = ok ? Typed<T>::load(row + p.k_col) : 0.f;
    }
    {
      const int t = tid >> 5;
      s_v[t][c] = (t < n && col < p.vdim) ? Typed<T>::load(base + (long long)(t0 + t) * p.ld + p.v_col + (long long)h * p.vdim + col) : 0.f;
    }
    __syncthreads();
    for (int t = 0; t < n; ++t) {
      const float v = s_v[t][c];
      float o = 0.f;
#pragma unroll
      for (int i = 0; i < RPT; i += 4) {
        const float4 q = *reinterpret_cast<const float4*>(&s_q[t][rg * RPT + i]), k = *reinterpret_cast<const float4*>(&s_k[t][rg * RPT + i]);
        S[i] = S[i] * decay + k.x * v;
        S[i + 1] = S[i + 1] * decay + k.y * v;
        S[i + 2] = S[i + 2] * decay + k.z * v;
        S[i + 3] = S[i + 3] * decay + k.w * v;
        o += S[i] * q.x + S[i + 1] * q.y + S[i + 2] * q.z + S[i + 3] * q.w;
      }
      s_o[t][rg][c] = o;
    }
    __syncthreads();
    {
      const int t = tid >> 5;  // eight warps: one token each
      if (t < n && col < p.vdim) {
        float o = 0.f;
#pragma unroll
        for (int r = 0; r < LROWS; ++r) o += s_o[t][r][c];
        Typed<T>::store(out + (long long)(t0 + t) * p.ldo + col, o);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int d = rg * RPT + i;
    if (d < p.dim && col < p.vdim) st[(long long)d * p.vdim + col] = S[i];
  }
}

// One CTA per (head, sequence): four columns per access, 32 column quads x 8 row groups (vdim a multiple of 4).
template <typename T>
__global__ void __launch_bounds__(256) lightning_step_vec_kernel(const LightningArgs p) {
  pdl_prologue();
  extern __shared__ __align__(16) float lsm[];
  float4* s_r = reinterpret_cast<float4*>(lsm);     // [8][32]
  float* s_q = lsm + 8 * 32 * 4;                    // [dim]
  float* s_k = s_q + p.dim;
  const int tid = threadIdx.x, c = tid & 31, rg = tid >> 5, h = blockIdx.x, b = blockIdx.y;
  const bool fresh = p.lengths[b] == 0, keep = !(p.active && !p.active[b]);
  const float decay = fresh ? 0.f : p.decay[h];
  const T* row = static_cast<const T*>(p.qkv) + (long long)b * p.ld;
  float* st = p.state + (long long)b * p.state_bs + (long long)h * p.dim * p.vdim;
  T* out = static_cast<T*>(p.o) + (long long)b * p.ldo + (long long)h * p.vdim;
  for (int d = tid; d < p.dim; d += 256) {
    s_q[d] = Typed<T>::load(row + p.q_col + (long long)h * p.dim + d);
    s_k[d] = Typed<T>::load(row + p.k_col + (long long)h * p.dim + d);
  }
  __syncthreads();
  for (int v0 = 0; v0 < p.vdim; v0 += 128) {
    const int v = v0 + c * 4;
    const bool ok = v < p.vdim;
    float4 val = make_float4(0.f, 0.f, 0.f, 0.f), o = make_float4(0.f, 0.f, 0.f, 0.f);
    if (ok) {
      const T* vp = row + p.v_col + (long long)h * p.vdim + v;
      val = make_float4(Typed<T>::load(vp), Typed<T>::load(vp + 1), Typed<T>::load(vp + 2), Typed<T>::load(vp + 3));
      constexpr int U = 8;  // rows in flight
      for (int d0 = rg; d0 < p.dim; d0 += 8 * U) {
        float4 S[U];
#pragma unroll
        for (int u = 0; u < U; ++u) {
          const int d = d0 + 8 * u;
          S[u] = (d < p.dim && !fresh) ? __ldcs(reinterpret_cast<const float4*>(st + (long long)d * p.vdim + v)) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
#pragma unroll
        for (int u = 0; u < U; ++u) {
          const int d = d0 + 8 * u;
          if (d >= p.dim) break;
          const float k = s_k[d], q = s_q[d];
          S[u].x = S[u].x * decay + k * val.x; S[u].y = S[u].y * decay + k * val.y;
          S[u].z = S[u].z * decay + k * val.z; S[u].w = S[u].w * decay + k * val.w;
          o.x += S[u].x * q; o.y += S[u].y * q; o.z += S[u].z * q; o.w += S[u].w * q;
          if (keep) __stcs(reinterpret_cast<float4*>(st + (long long)d * p.vdim + v), S[u]);
        }
      }
    }
    s_r[rg * 32 + c] = o;
    __syncthreads();
    if (rg == 0 && ok) {
      float4 t = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int r = 0; r < 8; ++r) {
        const float4 x = s_r[r * 32 + c];
        t.x += x.x; t.y += x.y; t.z += x.z; t.w += x.w;
      }
      Typed<T>::store(out + v, t.x); Typed<T>::store(out + v + 1, t.y); Typed<T>::store(out + v + 2, t.z); Typed<T>::store(out + v + 3, t.w);
    }
    __syncthreads();
  }
}

// The same element by element, for any vdim.
template <typename T>
__global__ void __launch_bounds__(256) lightning_step_kernel(const LightningArgs p) {
  pdl_prologue();
  extern __shared__ __align__(16) float lsm[];
  float* s_r = lsm;                                 // [8][32]
  float* s_q = lsm + 8 * 32;                        // [dim]
  float* s_k = s_q + p.dim;
  const int tid = threadIdx.x, c = tid & 31, rg = tid >> 5, h = blockIdx.x, b = blockIdx.y;
  const bool fresh = p.lengths[b] == 0, keep = !(p.active && !p.active[b]);
  const float decay = p.decay[h];
  const T* row = static_cast<const T*>(p.qkv) + (long long)b * p.ld;
  float* st = p.state + (long long)b * p.state_bs + (long long)h * p.dim * p.vdim;
  T* out = static_cast<T*>(p.o) + (long long)b * p.ldo + (long long)h * p.vdim;
  for (int d = tid; d < p.dim; d += 256) {
    s_q[d] = Typed<T>::load(row + p.q_col + (long long)h * p.dim + d);
    s_k[d] = Typed<T>::load(row + p.k_col + (long long)h * p.dim + d);
  }
  __syncthreads();
  for (int v0 = 0; v0 < p.vdim; v0 += 32) {
    const int v = v0 + c;
    float o = 0.f;
    if (v < p.vdim) {
      const float val = Typed<T>::load(row + p.v_col + (long long)h * p.vdim + v);
      for (int d = rg; d < p.dim; d += 8) {
        float S = fresh ? 0.f : st[(long long)d * p.vdim + v] * decay;
        S += s_k[d] * val;
        o += S * s_q[d];
        if (keep) st[(long long)d * p.vdim + v] = S;
      }
    }
    s_r[rg * 32 + c] = o;
    __syncthreads();
    if (rg == 0 && v < p.vdim) {
      float t = 0.f;
#pragma unroll
      for (int r = 0; r < 8; ++r) t += s_r[r * 32 + c];
      Typed<T>::store(out + v, t);
    }
    __syncthreads();
  }
}

template <typename T>
static int launch_scan(const LightningArgs& p, cudaStream_t s) {
  const dim3 grid((p.vdim + 31) / 32, p.H, p.B);
  if (p.dim <= 32) launch_pdl(lightning_scan_kernel<T, 4>, grid, dim3(256), 0, s, p);
  else if (p.dim <= 64) launch_pdl(lightning_scan_kernel<T, 8>, grid, dim3(256), 0, s, p);
  else if (p.dim <= 128) launch_pdl(lightning_scan_kernel<T, 16>, grid, dim3(256), 0, s, p);
  else if (p.dim <= 256) launch_pdl(lightning_scan_kernel<T, 32>, grid, dim3(256), 0, s, p);
  else return 1006;
  return int(cudaGetLastError());
}

template <typename T>
static int launch_step(const LightningArgs& p, cudaStream_t s) {
  if (p.dim > 2048) return 1006;
  const dim3 grid(p.H, p.B);
  if ((p.vdim & 3) == 0 && (p.state_bs & 3) == 0 && (reinterpret_cast<uintptr_t>(p.state) & 15) == 0)
    launch_pdl(lightning_step_vec_kernel<T>, grid, dim3(256), size_t(8 * 32 * 4 + 2 * p.dim) * sizeof(float), s, p);
  else
    launch_pdl(lightning_step_kernel<T>, grid, dim3(256), size_t(8 * 32 + 2 * p.dim) * sizeof(float), s, p);
  return int(cudaGetLastError());
}

}  // namespace ats

using namespace ats;

// The argument struct is passed by address (ctypes mirror in ops/lightning.py); `fp32` selects the element type.
ATS_API int ats_lightning_scan(const LightningArgs* p, int fp32, void* stream) {
  if (p->B <= 0 || p->L <= 0) return 0;
  return fp32 ? launch_scan<float>(*p, static_cast<cudaStream_t>(stream)) : launch_scan<__nv_bfloat16>(*p, static_cast<cudaStream_t>(stream));
}

ATS_API int ats_lightning_step(const LightningArgs* p, int fp32, void* stream) {
  if (p->B <= 0) return 0;
  if (!p->lengths || p->L != 1) return 1006;
  return fp32 ? launch_step<float>(*p, static_cast<cudaStream_t>(stream)) : launch_step<__nv_bfloat16>(*p, static_cast<cudaStream_t>(stream));
}
