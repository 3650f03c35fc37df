// Gated delta rule with one decay per state row (per head and key channel): portions of a prompt
//
//   S <- diag(g_t) S;   u = beta_t (v_t - S^T k_t);   S <- S + k_t u^T;   o_t = S^T q_t,     g_t = exp(-exp(A) softplus(a_t + dt))
//
// The convolutions, lengths and step sizes come from delta_prep, the output norm and gate from delta_output, decoding from delta_step
// (all delta_rule.cu).  As there, the recurrence advances in groups of DC = 8 tokens.  With P_i = g_1 .. g_i (per row) and S the state
// before the group
//
//   u_i = beta_i (v_i - S^T (P_i k_i) - sum_{j < i} kk_ij u_j),  kk_ij = sum_d k_i k_j g_{j+1} .. g_i   (unit lower triangular),
//   o_i = S^T (P_i q_i) + sum_{j <= i} kq_ij u_j,               kq_ij = sum_d q_i k_j g_{j+1} .. g_i,
//   S   <- P_C S + sum_j (k_j g_{j+1} .. g_C) u_j^T
//
// channel_pairs computes, for all groups in parallel, the 8 x 8 inverse (times beta), kq, and the decayed rows P_i k_i, P_i q_i,
// k_j g_{j+1} .. g_C, P_C in fp32; all decay products are running products of factors in (0, 1], so nothing overflows however fast a
// channel decays.  channel_scan does three products with the state per token: sixteen lanes share eight columns, fp32 with packed
// fma.f32x2, the next group's rows arriving in shared memory by asynchronous copies.
#include "delta_common.cuh"

namespace ats {

struct ChannelArgs {
  const void* mixed;       // [B * L, ldm] convolved q, k, v
  long long ldm;
  const float* rlen;       // [B * L, 2 * KH] dim^-1/2 / |q|, 1 / |k|
  const float* gb;         // [B * L, 2 * H]: step size at H + h
  const void* a;           // [B * L, lda]: decay input of head h at h * dim
  long long lda;
  const float* neg_rate;   // [H] -exp(A)
  const float* dt_bias;    // [H * dim]
  float* coef;             // [B, groups, H, size()]
  float* state;            // [B, H, dim, vdim]
  long long state_bs;
  void* o;                 // [B * L, H * vdim]
  long long ldo;
  int B, L, H, KH, dim, vdim, groups, fresh;
  // Per group and head: [DC][2 * DC] inverse (times beta) and kq, then rows of DK floats: DC times P_i k_i, DC times P_i q_i, DC times
  // k_j g_{j+1} .. g_C, P_C; DK = 64, 128 or 256 (the state rows the scan kernel is built for), zero beyond dim.
  int DK;
  __host__ __device__ int size() const { return 2 * DC * DC + (3 * DC + 1) * DK; }
};

// One warp per (group, head, sequence).  VC channels per lane side by side, so that all of a warp's loads of a pass are in flight together
// and are whole lines; DK = 32 * VC * passes.
template <typename T, int VC, bool VEC>
__global__ void __launch_bounds__(128, 3) channel_pairs_kernel(const ChannelArgs p) {
  pdl_prologue();
  __shared__ float s_kk[4][DC][DC + 1], s_kq[4][DC][DC + 1];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long w = blockIdx.x * 4ll + warp;
  if (w >= (long long)p.B * p.groups * p.H) return;  // whole warp; only __syncwarp below
  const int h = int(w % p.H), grp = int((w / p.H) % p.groups), b = int(w / p.H / p.groups), kh = h / (p.H / p.KH);
  const int t0 = grp * DC, n = min(DC, p.L - t0);
  const long long row0 = (long long)b * p.L + t0;
  const T* q = static_cast<const T*>(p.mixed) + row0 * p.ldm + (long long)kh * p.dim;
  const T* k = static_cast<const T*>(p.mixed) + row0 * p.ldm + (long long)(p.KH + kh) * p.dim;
  const T* a = static_cast<const T*>(p.a) + row0 * p.lda + (long long)h * p.dim;
  const float* rl = p.rlen + row0 * 2 * p.KH;
  float* co = p.coef + w * p.size();
  float* rows = co + 2 * DC * DC;
  const float rate = p.neg_rate[h];
  // sums[8 i + j]: i >= j: kq_ij; i < j: kk_ji
  float sums[DC * DC];
#pragma unroll
  for (int i = 0; i < DC * DC; ++i) sums[i] = 0.f;
  using Bits_ = typename Bits<VC * int(sizeof(T))>::type;
  for (int d0 = lane * VC; d0 < p.DK; d0 += 32 * VC) {
    union Piece { Bits_ bits; T v[VC]; };
    Piece pk[DC], pq[DC], pa[DC];
    float dt[VC];
    auto fetch = [&](Piece& x, const T* src, bool in) {
#pragma unroll
      for (int c = 0; c < VC; ++c) Typed<T>::store(&x.v[c], 0.f);
      if (!in) return;
      if constexpr (VEC) {
        if (d0 < p.dim) x.bits = *reinterpret_cast<const Bits_*>(src + d0);
      } else {
#pragma unroll
        for (int c = 0; c < VC; ++c)
          if (d0 + c < p.dim) x.v[c] = src[d0 + c];
      }
    };
#pragma unroll
    for (int i = 0; i < DC; ++i) {
      fetch(pk[i], k + i * p.ldm, i < n);
      fetch(pq[i], q + i * p.ldm, i < n);
      fetch(pa[i], a + i * p.lda, i < n);
    }
#pragma unroll
    for (int c = 0; c < VC; ++c) dt[c] = d0 + c < p.dim ? p.dt_bias[(long long)h * p.dim + d0 + c] : 0.f;
    float kv[DC][VC], qv[DC][VC], g[DC][VC], P[VC];
#pragma unroll
    for (int i = 0; i < DC; ++i) {
      const float rk = i < n ? rl[(long long)i * 2 * p.KH + p.KH + kh] : 0.f, rq = i < n ? rl[(long long)i * 2 * p.KH + kh] : 0.f;
#pragma unroll
      for (int c = 0; c < VC; ++c) {
        kv[i][c] = Typed<T>::load(&pk[i].v[c]) * rk;
        qv[i][c] = Typed<T>::load(&pq[i].v[c]) * rq;
        g[i][c] = i < n && d0 + c < p.dim ? decay_of<T>(Typed<T>::load(&pa[i].v[c]) + dt[c], rate) : 1.f;
      }
    }
    auto put = [&](int row, const float (&x)[VC]) {
      static_assert(VC == 2, "one access per row");
      *reinterpret_cast<float2*>(rows + row * p.DK + d0) = make_float2(x[0], x[1]);
    };
#pragma unroll
    for (int c = 0; c < VC; ++c) P[c] = 1.f;
#pragma unroll
    for (int i = 0; i < DC; ++i) {
      float x[VC], y[VC];
#pragma unroll
      for (int c = 0; c < VC; ++c) {
        P[c] *= g[i][c];
        x[c] = kv[i][c] * P[c];
        y[c] = qv[i][c] * P[c];
      }
      put(i, x);
      put(DC + i, y);
    }
    put(3 * DC, P);
#pragma unroll
    for (int j = 0; j < DC; ++j) {
      float r[VC];
#pragma unroll
      for (int c = 0; c < VC; ++c) {
        r[c] = kv[j][c];
        sums[j * DC + j] += qv[j][c] * r[c];
      }
#pragma unroll
      for (int i = j + 1; i < DC; ++i)
#pragma unroll
        for (int c = 0; c < VC; ++c) {
          r[c] *= g[i][c];
          sums[i * DC + j] += qv[i][c] * r[c];
          sums[j * DC + i] += kv[i][c] * r[c];
        }
      put(2 * DC + j, r);
    }
  }
  // transposing reduction: after the steps, lane l holds the sums 2 l and 2 l + 1 over all lanes
#pragma unroll
  for (int i = 0; i < 32; ++i) sums[i] = keep_add(sums[i], sums[i + 32], lane, 16);
#pragma unroll
  for (int i = 0; i < 16; ++i) sums[i] = keep_add(sums[i], sums[i + 16], lane, 8);
#pragma unroll
  for (int i = 0; i < 8; ++i) sums[i] = keep_add(sums[i], sums[i + 8], lane, 4);
#pragma unroll
  for (int i = 0; i < 4; ++i) sums[i] = keep_add(sums[i], sums[i + 4], lane, 2);
#pragma unroll
  for (int i = 0; i < 2; ++i) sums[i] = keep_add(sums[i], sums[i + 2], lane, 1);
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int i = lane >> 2, j = 2 * (lane & 3) + e;
    if (i >= j) s_kq[warp][i][j] = sums[e];
    else s_kk[warp][j][i] = sums[e];
  }
  __syncwarp();
  if (lane < DC) {  // lane = column of the 8 x 8 inverse
    float beta[DC], y[DC];
#pragma unroll
    for (int i = 0; i < DC; ++i) beta[i] = i < n ? p.gb[(row0 + i) * 2 * p.H + p.H + h] : 0.f;
    inverse_column(beta, s_kk[warp], lane, y);
    const float bc = lane < n ? p.gb[(row0 + lane) * 2 * p.H + p.H + h] : 0.f;
#pragma unroll
    for (int i = 0; i < DC; ++i) {
      co[i * 2 * DC + lane] = y[i] * bc;
      co[i * 2 * DC + DC + lane] = i >= lane ? s_kq[warp][i][lane] : 0.f;
    }
  }
}

__device__ __forceinline__ void cp_async_16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void cp_async_wait_all() { asm volatile("cp.async.wait_group 0;" ::: "memory"); }

// Sixteen lanes share CPL value columns: lane l holds EPL state rows (DK = 16 * EPL) of each, rows 64 c + 4 l .. + 3 of every 64-row
// piece c.  CTA = 4 warps of 2 lane groups -> 8 * CPL columns of one head.  After a product, lane l holds token l % 8, columns
// (l / 8) * CPL / 2 ...
template <typename T, int EPL, int CPL, int OCC>
__global__ void __launch_bounds__(128, OCC) channel_scan_kernel(const ChannelArgs p) {
  pdl_prologue();
  constexpr int DK = 16 * EPL, HC = CPL / 2, CF = 2 * DC * DC, SIZE = CF + (3 * DC + 1) * DK;
  extern __shared__ __align__(16) float s_coef[];      // [2][SIZE]
  __shared__ __align__(16) float s_u[8][2][DC][CPL];   // [lane group][right-hand side, u]
  const int tid = threadIdx.x, lane = tid & 31, l16 = lane & 15, grp16 = tid >> 4, tok = l16 & 7, half = l16 >> 3;
  const int h = blockIdx.y, b = blockIdx.z;
  const int col0 = (blockIdx.x * 8 + grp16) * CPL, colh = col0 + half * HC;
  float2 S[CPL][EPL / 2];
  float* st = p.state + (long long)b * p.state_bs + (long long)h * p.dim * p.vdim;
  auto state_row = [&](int e) { return (e / 2) * 64 + l16 * 4 + 2 * (e & 1); };  // first row of pair e
#pragma unroll
  for (int c = 0; c < CPL; ++c)
#pragma unroll
    for (int e = 0; e < EPL / 2; ++e) {
      const int d = state_row(e);
      const bool ok = !p.fresh && col0 + c < p.vdim;
      S[c][e].x = (ok && d < p.dim) ? st[(long long)d * p.vdim + col0 + c] : 0.f;
      S[c][e].y = (ok && d + 1 < p.dim) ? st[(long long)(d + 1) * p.vdim + col0 + c] : 0.f;
    }
  const T* vbase = static_cast<const T*>(p.mixed) + (long long)b * p.L * p.ldm + 2 * p.KH * p.dim + (long long)h * p.vdim + colh;
  T* obase = static_cast<T*>(p.o) + (long long)b * p.L * p.ldo + (long long)h * p.vdim + colh;
  const float* cbase = p.coef + ((long long)b * p.groups * p.H + h) * SIZE;
  // the lane's HC values of a token are one aligned access when every head starts at a multiple of HC columns
  using VBits = typename Bits<HC * int(sizeof(T))>::type;
  const bool vecv = (p.vdim % HC) == 0 && ((2 * p.KH * p.dim) % HC) == 0 && (p.ldo % HC) == 0;
  const bool inside = colh < p.vdim;  // with vecv: all HC columns or none
  union { VBits bits; T v[HC]; } vnext;  // as loaded: converting here would wait for the load
  auto request = [&](int grp, int buf) {
    const int t0 = grp * DC, n = min(DC, p.L - t0);
    const float* src = cbase + (long long)grp * p.H * SIZE;
    for (int i = tid * 4; i < SIZE; i += 512) cp_async_16(s_coef + buf * SIZE + i, src + i);
    cp_async_commit();
#pragma unroll
    for (int c = 0; c < HC; ++c) Typed<T>::store(&vnext.v[c], 0.f);
    if (tok < n) {
      const T* vs = vbase + (long long)(t0 + tok) * p.ldm;
      if (vecv) {
        if (inside) vnext.bits = *reinterpret_cast<const VBits*>(vs);
      } else {
#pragma unroll
        for (int c = 0; c < HC; ++c)
          if (colh + c < p.vdim) vnext.v[c] = vs[c];
      }
    }
  };
  auto load_row = [&](const float* row, float2 (&k)[EPL / 2]) {
#pragma unroll
    for (int c = 0; c < EPL / 4; ++c) {
      const float4 v = *reinterpret_cast<const float4*>(row + c * 64 + l16 * 4);
      k[2 * c] = make_float2(v.x, v.y);
      k[2 * c + 1] = make_float2(v.z, v.w);
    }
  };
  // sums over the state rows of S times eight rows in shared memory
  auto products = [&](const float* rows, float (&out)[HC]) {
    float r2[2][CPL];
#pragma unroll
    for (int y = 0; y < 2; ++y) {      // tokens y, y + 4, y + 2, y + 6
      float r4[2][CPL];
#pragma unroll
      for (int z = 0; z < 2; ++z) {
        float r8[2][CPL];
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          const int i = y + 2 * z + 4 * x;
          float2 a[CPL];
#pragma unroll
          for (int c = 0; c < CPL; ++c) a[c] = make_float2(0.f, 0.f);
          float2 k[EPL / 2];
          load_row(rows + i * DK, k);
#pragma unroll
          for (int e = 0; e < EPL / 2; ++e)
#pragma unroll
            for (int c = 0; c < CPL; ++c) a[c] = fma2(S[c][e], k[e], a[c]);
#pragma unroll
          for (int c = 0; c < CPL; ++c) r8[x][c] = a[c].x + a[c].y;
        }
#pragma unroll
        for (int c = 0; c < CPL; ++c) r4[z][c] = keep_add(r8[0][c], r8[1][c], lane, 4);
        pace();
      }
#pragma unroll
      for (int c = 0; c < CPL; ++c) r2[y][c] = keep_add(r4[0][c], r4[1][c], lane, 2);
    }
#pragma unroll
    for (int c = 0; c < CPL; ++c) r2[0][c] = keep_add(r2[0][c], r2[1][c], lane, 1);
#pragma unroll
    for (int c = 0; c < HC; ++c) out[c] = keep_add(r2[0][c], r2[0][c + HC], lane, 8);
  };
  request(0, 0);
  for (int grp = 0; grp < p.groups; ++grp) {
    const int buf = grp & 1, t0 = grp * DC, n = min(DC, p.L - t0);
    cp_async_wait_all();
    __syncthreads();  // this group's rows are there for everyone, and everyone is done with the other buffer
    const float* co = s_coef + buf * SIZE;
    const float* rows = co + CF;
    float v[HC], sk[HC], o[HC];
#pragma unroll
    for (int c = 0; c < HC; ++c) v[c] = Typed<T>::load(&vnext.v[c]);
    if (grp + 1 < p.groups) request(grp + 1, buf ^ 1);
    products(rows, sk);
#pragma unroll
    for (int c = 0; c < HC; ++c) s_u[grp16][0][tok][half * HC + c] = v[c] - sk[c];
    __syncwarp();
    {
      float u[HC];
#pragma unroll
      for (int c = 0; c < HC; ++c) u[c] = 0.f;
#pragma unroll
      for (int j = 0; j < DC; ++j) {
        const float m = co[tok * 2 * DC + j];
#pragma unroll
        for (int c = 0; c < HC; ++c) u[c] += m * s_u[grp16][0][j][half * HC + c];
      }
#pragma unroll
      for (int c = 0; c < HC; ++c) s_u[grp16][1][tok][half * HC + c] = u[c];
    }
    __syncwarp();
#pragma unroll
    for (int c = 0; c < HC; ++c) o[c] = 0.f;
#pragma unroll
    for (int j = 0; j < DC; ++j) {
      const float m = co[tok * 2 * DC + DC + j];
#pragma unroll
      for (int c = 0; c < HC; ++c) o[c] += m * s_u[grp16][1][j][half * HC + c];
    }
    products(rows + DC * DK, sk);
    if (tok < n) {
      union { VBits bits; T v[HC]; } ov;
#pragma unroll
      for (int c = 0; c < HC; ++c) Typed<T>::store(&ov.v[c], o[c] + sk[c]);
      T* dst = obase + (long long)(t0 + tok) * p.ldo;
      if (vecv) {
        if (inside) *reinterpret_cast<VBits*>(dst) = ov.bits;
      } else {
#pragma unroll
        for (int c = 0; c < HC; ++c)
          if (colh + c < p.vdim) dst[c] = ov.v[c];
      }
    }
    {
      float2 P[EPL / 2];
      load_row(rows + 3 * DC * DK, P);
#pragma unroll
      for (int c = 0; c < CPL; ++c)
#pragma unroll
        for (int e = 0; e < EPL / 2; ++e) S[c][e] = make_float2(S[c][e].x * P[e].x, S[c][e].y * P[e].y);
    }
#pragma unroll
    for (int j = 0; j < DC; ++j) {
      float w[CPL];
#pragma unroll
      for (int c = 0; c < CPL; c += 4) {
        const float4 q = *reinterpret_cast<const float4*>(&s_u[grp16][1][j][c]);
        w[c] = q.x; w[c + 1] = q.y; w[c + 2] = q.z; w[c + 3] = q.w;
      }
      float2 k[EPL / 2];
      load_row(rows + (2 * DC + j) * DK, k);
#pragma unroll
      for (int e = 0; e < EPL / 2; ++e)
#pragma unroll
        for (int c = 0; c < CPL; ++c) S[c][e] = fma2(k[e], make_float2(w[c], w[c]), S[c][e]);
      if (j & 1) pace();
    }
  }
#pragma unroll
  for (int c = 0; c < CPL; ++c) {
    if (col0 + c >= p.vdim) continue;
#pragma unroll
    for (int e = 0; e < EPL / 2; ++e) {
      const int d = state_row(e);
      if (d < p.dim) st[(long long)d * p.vdim + col0 + c] = S[c][e].x;
      if (d + 1 < p.dim) st[(long long)(d + 1) * p.vdim + col0 + c] = S[c][e].y;
    }
  }
}

template <typename T, int EPL, int CPL>
static int launch_channel_scan(const ChannelArgs& p, cudaStream_t s) {
  const int smem = 2 * p.size() * int(sizeof(float));
  auto kernel = channel_scan_kernel<T, EPL, CPL, 2>;
  if (smem > 48 * 1024) {
    cudaError_t ce = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (ce != cudaSuccess) return int(ce);
  }
  launch_pdl(kernel, dim3((p.vdim + 8 * CPL - 1) / (8 * CPL), p.H, p.B), dim3(128), size_t(smem), s, p);
  return int(cudaGetLastError());
}

template <typename T>
static int launch_channel(const ChannelArgs& p, cudaStream_t s) {
  const long long warps = (long long)p.B * p.groups * p.H;
  const dim3 grid(unsigned((warps + 3) / 4)), block(128);
  // pairs of channels: one aligned access when every head and row starts at an even element
  const bool even = !((p.dim | p.ldm | p.lda) & 1);
  if (even) launch_pdl(channel_pairs_kernel<T, 2, true>, grid, block, 0, s, p);
  else launch_pdl(channel_pairs_kernel<T, 2, false>, grid, block, 0, s, p);
  if (p.DK == 64) return launch_channel_scan<T, 4, 8>(p, s);
  if (p.DK == 128) return launch_channel_scan<T, 8, 8>(p, s);
  return launch_channel_scan<T, 16, 4>(p, s);
}

}  // namespace ats

using namespace ats;

// The argument struct is passed by address (ctypes mirror in ops/delta.py); `fp32` selects the element type of mixed, a and o.
ATS_API int ats_channel_delta(const ChannelArgs* p, int fp32, void* stream) {
  if (p->B <= 0 || p->L <= 0) return 0;
  if (p->groups != (p->L + DC - 1) / DC || p->KH < 1 || p->H % p->KH || (p->DK != 64 && p->DK != 128 && p->DK != 256) || p->dim > p->DK ||
      (reinterpret_cast<uintptr_t>(p->coef) & 15))
    return 1006;
  return fp32 ? launch_channel<float>(*p, static_cast<cudaStream_t>(stream)) : launch_channel<__nv_bfloat16>(*p, static_cast<cudaStream_t>(stream));
}
