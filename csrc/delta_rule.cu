// Gated delta rule: a linear recurrence over a per-head matrix state S [dim, vdim] (fp32)
//
//   S <- g_t S;   u = beta_t (v_t - S^T k_t);   S <- S + k_t u^T;   o_t = S^T q_t
//
// with short causal convolutions (+ silu) on q, k, v, unit-length q and k, and an output norm with a silu gate.  `heads` value heads,
// `kv_heads` query / key heads (head h uses query / key head h / (heads / kv_heads)).
//
// * delta_prep: convolutions and activations, reciprocal lengths of q and k (kept apart in fp32, the vectors stay in the element
//   type), decay g and step size beta.  One warp per (token, head).
// * delta_pairs + delta_scan: portions of a prompt.  The recurrence is advanced in groups of DC = 8 tokens: with S the state before the
//   group, u_i = beta_i (v_i - G_i S^T k_i - sum_{j < i} D_ij (k_j . k_i) u_j), D_ij = g_{j+1} .. g_i, G_i = g_1 .. g_i, a unit lower
//   triangular system whose 8 x 8 inverse does not depend on the value column; delta_pairs computes it (and the read-out
//   coefficients) for all groups in parallel, so that the sequential kernel only does three products with the state per token.
//   Columns of S are independent: sixteen lanes share eight columns, everything in fp32 with packed fma.f32x2.
// * delta_output: output norm over vdim, weight, silu gate.
// * delta_step: one decoded token per sequence: state read once and written once, output norm and gate in the same launch.
//
// channel_delta.cu holds the portion kernels of the form with one decay per state row; it shares delta_prep (without the decays),
// delta_output and delta_step.
//
// A sequence at position 0 starts from a zero state and zero convolution inputs whatever its buffers hold.
#include "delta_common.cuh"

namespace ats {

struct DeltaArgs {
  const void* proj;        // [B * L, ld]: q at 0, k at kv_heads * dim, v at 2 * kv_heads * dim; gate / a / b at the columns below
  long long ld;
  int g_col, a_col, b_col;
  int B, L, H, KH, dim, vdim, taps, C;   // C = 2 * KH * dim + H * vdim convolved channels
  const float* conv;       // [taps, C], last row = current token
  const float* neg_rate;   // [H] -exp(A_log), or null: step sizes only (the decays come from elsewhere)
  const float* dt_bias;    // [H]
  void* tail;              // [B, taps - 1, C] last inputs of the convolutions (oldest first)
  long long tail_bs;
  int pos0;
  const int* lengths;      // decoding: position per sequence
  const int* active;       // decoding: rows with 0 leave tail and state alone
  void* mixed;             // [B * L, Cp] convolved q, k, v
  long long ldm;
  float* rlen;             // [B * L, 2 * KH] 1 / |q| (times dim^-1/2), 1 / |k|
  float* gb;               // [B * L, 2 * H] decay, step size
};

template <typename T>
__device__ __forceinline__ void delta_gate(const DeltaArgs& p, long long row, int h) {
  const T* in = static_cast<const T*>(p.proj) + row * p.ld;
  const float bt = Typed<T>::load(in + p.b_col + h);
  if (p.neg_rate) p.gb[row * 2 * p.H + h] = decay_of<T>(Typed<T>::load(in + p.a_col + h) + p.dt_bias[h], p.neg_rate[h]);
  p.gb[row * 2 * p.H + p.H + h] = 1.f / (1.f + expf(-bt));
}

template <typename T>
__global__ void __launch_bounds__(256) delta_prep_kernel(const DeltaArgs p) {
  pdl_prologue();
  const int units = 2 * p.KH + p.H + 1, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long w = blockIdx.x * 8ll + warp;
  if (w >= (long long)p.B * p.L * units) return;
  const long long row = w / units;
  const int unit = int(w % units), b = int(row / p.L), t = int(row % p.L);
  const int pos0 = p.lengths ? p.lengths[b] : p.pos0;
  const T* in = static_cast<const T*>(p.proj) + row * p.ld;
  if (unit == units - 1) {  // decay and step size of every head
    for (int h = lane; h < p.H; h += 32) delta_gate<T>(p, row, h);
    return;
  }
  const int width = unit < 2 * p.KH ? p.dim : p.vdim;
  const int c0 = unit < 2 * p.KH ? unit * p.dim : 2 * p.KH * p.dim + (unit - 2 * p.KH) * p.vdim;
  T* tail = static_cast<T*>(p.tail) + (long long)b * p.tail_bs;
  T* out = static_cast<T*>(p.mixed) + row * p.ldm;
  const bool keep = p.lengths && !(p.active && !p.active[b]);
  float ss = 0.f;
  for (int i = lane; i < width; i += 32) {
    const int c = c0 + i;
    const float* cw = p.conv + c;
    const T cur = in[c];
    float acc = Typed<T>::load(&cur) * cw[(long long)(p.taps - 1) * p.C];
    for (int j = 1; j < p.taps; ++j) {  // j tokens back
      float x = 0.f;
      if (t - j >= 0) x = Typed<T>::load(in - j * p.ld + c);
      else if (pos0 > 0) x = Typed<T>::load(tail + (long long)(p.taps - 1 + t - j) * p.C + c);
      acc += x * cw[(long long)(p.taps - 1 - j) * p.C];
    }
    if (keep) {  // decoding: shift the channel's inputs (this thread is the only one that touches them)
      for (int j = 0; j < p.taps - 2; ++j) {
        T v = tail[(long long)(j + 1) * p.C + c];
        if (pos0 == 0) Typed<T>::store(&v, 0.f);
        tail[(long long)j * p.C + c] = v;
      }
      if (p.taps > 1) tail[(long long)(p.taps - 2) * p.C + c] = cur;
    }
    const float y = acc * Typed<T>::sigmoid_(acc);
    T yt;
    Typed<T>::store(&yt, y);
    out[c] = yt;
    const float yr = Typed<T>::load(&yt);
    ss += yr * yr;
  }
  if (unit < 2 * p.KH) {
    ss = warp_sum(ss);
    if (lane == 0) p.rlen[row * 2 * p.KH + unit] = (unit < p.KH ? 1.f / sqrtf(float(p.dim)) : 1.f) / sqrtf(ss + 1e-6f);
  }
}

// The same when heads are whole 16-byte pieces: a thread owns eight channels and walks PT consecutive tokens with the convolution's
// inputs in registers; the lanes of a head (dim / 8 of them, a power of two) add up its length with shuffles.  The blocks after
// `conv_blocks` compute decays and step sizes.
constexpr int PT = 32, PV_THREADS = 128;
template <typename T, int TAPS>
__global__ void __launch_bounds__(PV_THREADS, 4) delta_prep_vec_kernel(const DeltaArgs p, int conv_blocks) {
  pdl_prologue();
  if (int(blockIdx.x) >= conv_blocks) {
    const long long i = (blockIdx.x - conv_blocks) * (long long)PV_THREADS + threadIdx.x;
    if (i < (long long)p.B * p.L * p.H) delta_gate<T>(p, i / p.H, int(i % p.H));
    return;
  }
  const int pieces = p.C >> 3, per_block = (pieces + PV_THREADS - 1) / PV_THREADS, blocks_t = (p.L + PT - 1) / PT;
  const int piece = (blockIdx.x % per_block) * PV_THREADS + threadIdx.x;
  const int tb = (blockIdx.x / per_block) % blocks_t, b = blockIdx.x / per_block / blocks_t;
  const int t0 = tb * PT, t1 = min(p.L, t0 + PT);
  const bool live = piece < pieces;  // C / 8 need not fill the last block: idle lanes still take part in the shuffles
  const int c = live ? piece * 8 : 0;
  const T* in = static_cast<const T*>(p.proj) + (long long)b * p.L * p.ld + c;
  const T* tail = static_cast<const T*>(p.tail) + (long long)b * p.tail_bs + c;
  T* out = static_cast<T*>(p.mixed) + (long long)b * p.L * p.ldm + c;
  constexpr int PB = 4;
  float w[TAPS][8], x[TAPS - 1 + PB][8];
#pragma unroll
  for (int j = 0; j < TAPS; ++j) Typed<float>::load8(p.conv + (long long)j * p.C + c, w[j]);
  const int pos0 = p.lengths ? p.lengths[b] : p.pos0;
#pragma unroll
  for (int j = 0; j < TAPS - 1; ++j) {
    const int t = t0 - (TAPS - 1) + j;
    if (t >= 0) Typed<T>::load8(in + (long long)t * p.ld, x[j]);
    else if (pos0 > 0) Typed<T>::load8(tail + (long long)(TAPS - 1 + t) * p.C, x[j]);
    else
#pragma unroll
      for (int e = 0; e < 8; ++e) x[j][e] = 0.f;
  }
  const int lanes = p.dim >> 3, kd = p.KH * p.dim;
  const bool qk = live && c < 2 * kd, warp_qk = __any_sync(0xffffffffu, qk);
  const int head = piece / lanes;
  // tokens come in batches of PB whose loads are issued one batch ahead; x[0 .. TAPS - 2] is the history, oldest first
  typename Typed<T>::Raw8 nx[PB];
#pragma unroll
  for (int u = 0; u < PB; ++u) nx[u] = Typed<T>::raw8(in + (long long)min(t0 + u, t1 - 1) * p.ld);
  for (int tb0 = t0; tb0 < t1; tb0 += PB) {
#pragma unroll
    for (int u = 0; u < PB; ++u) Typed<T>::unpack8(nx[u], x[TAPS - 1 + u]);
    if (tb0 + PB < t1)
#pragma unroll
      for (int u = 0; u < PB; ++u) nx[u] = Typed<T>::raw8(in + (long long)min(tb0 + PB + u, t1 - 1) * p.ld);
#pragma unroll
    for (int u = 0; u < PB; ++u) {
      const int t = tb0 + u;
      float y[8], ss = 0.f;
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        float acc = x[u][e] * w[0][e];
#pragma unroll
        for (int j = 1; j < TAPS; ++j) acc += x[u + j][e] * w[j][e];
        y[e] = acc * Typed<T>::sigmoid_(acc);
      }
      const typename Typed<T>::Raw8 packed = Typed<T>::pack8(y);
      if (live && t < t1) Typed<T>::store_raw8(out + (long long)t * p.ldm, packed);
      if (warp_qk) {
        Typed<T>::unpack8(packed, y);
#pragma unroll
        for (int e = 0; e < 8; ++e) ss += y[e] * y[e];
        for (int off = lanes >> 1; off > 0; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
        if (qk && t < t1 && (piece & (lanes - 1)) == 0)
          p.rlen[((long long)b * p.L + t) * 2 * p.KH + head] = (head < p.KH ? 1.f / sqrtf(float(p.dim)) : 1.f) / sqrtf(ss + 1e-6f);
      }
    }
    // the batch's last tokens are the next history (in decoding, the one token of the batch sits at x[TAPS - 1])
    if (tb0 + PB < t1)
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j)
#pragma unroll
        for (int e = 0; e < 8; ++e) x[j][e] = x[PB + j][e];
  }
  if (p.lengths && live && !(p.active && !p.active[b])) {  // decoding: this thread's channels move on by the token
    T* tw = static_cast<T*>(p.tail) + (long long)b * p.tail_bs + c;
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) Typed<T>::store8(tw + (long long)j * p.C, x[j + 1]);
  }
}

// After a portion: the last taps - 1 inputs of every channel (one thread per channel, oldest first, in place).
template <typename T>
__global__ void __launch_bounds__(256) delta_tail_kernel(const DeltaArgs p) {
  pdl_prologue();
  const int c = blockIdx.x * 256 + threadIdx.x, b = blockIdx.y, n = p.taps - 1;
  if (c >= p.C) return;
  T* tail = static_cast<T*>(p.tail) + (long long)b * p.tail_bs + c;
  const T* in = static_cast<const T*>(p.proj) + (long long)b * p.L * p.ld + c;
  for (int j = 0; j < n; ++j) {
    const int t = p.L - n + j;
    T v;
    Typed<T>::store(&v, 0.f);
    if (t >= 0) v = in[t * p.ld];
    else if (p.pos0 > 0) v = tail[(long long)(n + t) * p.C];
    tail[(long long)j * p.C] = v;
  }
}

// ------------------------------------------------------------------------------------------------ portions
// Per group and head: [DC][2 * DC] inverse of the triangular system (times beta) and read-out coefficients, then per token
// G_i / |k_i|, G_i dim^-1/2 / |q_i|, D_Ci / |k_i| (G_i = g_1 .. g_i, D_Ci = g_{i+1} .. g_C), then G_C: with the lengths folded in
// here, the sequential kernel works on the raw q and k.
constexpr int CO = 2 * DC * DC + 3 * DC + 8;

struct ScanArgs {
  const void* mixed;
  long long ldm;
  const float* rlen;
  const float* gb;
  float* coef;             // [B, groups, H, CO]: see CO
  float* state;            // [B, H, dim, vdim]
  long long state_bs;
  void* o;                 // [B * L, H * vdim]
  long long ldo;
  int B, L, H, KH, dim, vdim, groups, fresh;
};

// 16 x 8 products of one group: rows 0..7 k_i . k_j, rows 8..15 q_i . k_j, sums over dim.  bf16 values: exact products accumulated in
// fp32 by a warp-level MMA, whose B fragment is the same registers as the upper half of A (the order of the reduction is
// permuted so that a lane's 16-byte piece serves two steps).
__device__ __forceinline__ void group_products_mma(const __nv_bfloat16* q, const __nv_bfloat16* k, long long ldm, int dim, int n, int lane, float (&c)[4]) {
  const int g = lane >> 2, t = lane & 3;
  c[0] = c[1] = c[2] = c[3] = 0.f;
  for (int d = 8 * t; d < ((dim + 31) & ~31); d += 32) {
    uint4 kv = make_uint4(0, 0, 0, 0), qv = make_uint4(0, 0, 0, 0);
    if (g < n && d < dim) {
      kv = *reinterpret_cast<const uint4*>(k + g * ldm + d);
      qv = *reinterpret_cast<const uint4*>(q + g * ldm + d);
    }
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(kv.x), "r"(qv.x), "r"(kv.y), "r"(qv.y), "r"(kv.x), "r"(kv.y));
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(kv.z), "r"(qv.z), "r"(kv.w), "r"(qv.w), "r"(kv.z), "r"(kv.w));
  }
}

// One warp per (group, kv head, sequence): 8 x 8 products of the keys with keys and queries, then per value head the inverse.
template <typename T, bool MMA>
__global__ void __launch_bounds__(128) delta_pairs_kernel(const ScanArgs p) {
  pdl_prologue();
  __shared__ float s_kk[4][DC][DC + 1], s_kq[4][DC][DC + 1];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, rep = p.H / p.KH;
  const long long w = blockIdx.x * 4ll + warp;
  if (w >= (long long)p.B * p.groups * p.KH) return;  // whole warp; only __syncwarp below
  const int kh = int(w % p.KH), grp = int((w / p.KH) % p.groups), b = int(w / p.KH / p.groups);
  const int t0 = grp * DC, n = min(DC, p.L - t0);
  const long long row0 = (long long)b * p.L + t0;
  const T* base = static_cast<const T*>(p.mixed) + row0 * p.ldm;
  const T* q = base + (long long)kh * p.dim;
  const T* k = base + (long long)(p.KH + kh) * p.dim;
  const float* rl = p.rlen + row0 * 2 * p.KH;
  if constexpr (MMA) {
    float c[4];
    group_products_mma(q, k, p.ldm, p.dim, n, lane, c);
    const int i = lane >> 2, j = 2 * (lane & 3);
    const float rki = i < n ? rl[(long long)i * 2 * p.KH + p.KH + kh] : 0.f, rqi = i < n ? rl[(long long)i * 2 * p.KH + kh] : 0.f;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const float rkj = j + e < n ? rl[(long long)(j + e) * 2 * p.KH + p.KH + kh] : 0.f;
      s_kk[warp][i][j + e] = c[e] * rki * rkj;
      s_kq[warp][i][j + e] = c[2 + e] * rqi * rkj;
    }
  } else {
  float kk[DC][DC], kq[DC][DC];
#pragma unroll
  for (int i = 0; i < DC; ++i)
#pragma unroll
    for (int j = 0; j < DC; ++j) kk[i][j] = kq[i][j] = 0.f;
  for (int d = lane; d < p.dim; d += 32) {
    float kv[DC], qv[DC];
#pragma unroll
    for (int i = 0; i < DC; ++i) {
      kv[i] = i < n ? Typed<T>::load(k + i * p.ldm + d) : 0.f;
      qv[i] = i < n ? Typed<T>::load(q + i * p.ldm + d) : 0.f;
    }
#pragma unroll
    for (int i = 0; i < DC; ++i)
#pragma unroll
      for (int j = 0; j <= i; ++j) {
        kk[i][j] += kv[i] * kv[j];
        kq[i][j] += qv[i] * kv[j];
      }
  }
#pragma unroll
  for (int i = 0; i < DC; ++i)
#pragma unroll
    for (int j = 0; j <= i; ++j) {
      const float a = warp_sum(kk[i][j]), c = warp_sum(kq[i][j]);
      if (lane == 0) {
        const float rkj = j < n ? rl[(long long)j * 2 * p.KH + p.KH + kh] : 0.f;
        const float rki = i < n ? rl[(long long)i * 2 * p.KH + p.KH + kh] : 0.f, rqi = i < n ? rl[(long long)i * 2 * p.KH + kh] : 0.f;
        s_kk[warp][i][j] = a * rki * rkj;
        s_kq[warp][i][j] = c * rqi * rkj;
      }
    }
  }
  __syncwarp();
  // lane = (value head of the group r, column c of the 8 x 8 inverse)
  for (int x = lane; x < rep * DC; x += 32) {
    const int h = kh * rep + x / DC, c = x % DC;
    float g[DC], beta[DC];
#pragma unroll
    for (int i = 0; i < DC; ++i) {
      g[i] = i < n ? p.gb[(row0 + i) * 2 * p.H + h] : 1.f;
      beta[i] = i < n ? p.gb[(row0 + i) * 2 * p.H + p.H + h] : 0.f;
    }
    // column c of (1 + M)^-1, M_ij = beta_i D_ij kk_ij: forward substitution; the result is multiplied by beta_c (the right-hand
    // side of the system is beta_c (v_c - G_c S^T k_c))
    float y[DC];
    float* co = p.coef + (((long long)b * p.groups + grp) * p.H + h) * CO;
#pragma unroll
    for (int i = 0; i < DC; ++i) {
      float acc = i == c ? 1.f : 0.f, dec = 1.f;
#pragma unroll
      for (int j = i - 1; j >= 0; --j) {
        dec *= g[j + 1];
        acc -= beta[i] * dec * s_kk[warp][i][j] * y[j];
      }
      y[i] = acc;
      co[i * 2 * DC + c] = acc * beta[c];
    }
    // read-out coefficients of write c: D_ic (k_c . q_i) for i >= c
    float dec = 1.f;
#pragma unroll
    for (int i = 0; i < DC; ++i) {
      if (i > c) dec *= g[i];
      co[i * 2 * DC + DC + c] = i >= c ? dec * s_kq[warp][i][c] : 0.f;
    }
    float G = 1.f, GC = 1.f;
#pragma unroll
    for (int i = 0; i < DC; ++i) {
      if (i <= c) G *= g[i];
      GC *= g[i];
    }
    const float rk = c < n ? rl[(long long)c * 2 * p.KH + p.KH + kh] : 0.f, rq = c < n ? rl[(long long)c * 2 * p.KH + kh] : 0.f;
    co += 2 * DC * DC;
    co[c] = G * rk;
    co[DC + c] = G * rq;
    co[2 * DC + c] = dec * rk;  // dec has become g_{c+1} .. g_C
    if (c == 0) co[3 * DC] = GC;
  }
}

// A lane's EPL values of a k or q row in shared memory: pieces of up to eight consecutive elements, sixteen lanes side by side.
template <typename T, int EPL>
struct RowPiece {
  static constexpr int W = EPL < 8 ? EPL : 8;
  static __device__ __forceinline__ int index(int pair, int l16) {  // first state row of pair `pair` (two rows) of lane l16
    return ((2 * pair) / W * 16 + l16) * W + (2 * pair) % W;
  }
  static __device__ __forceinline__ void load(const T* row, int l16, float2 (&k)[EPL / 2]) {
#pragma unroll
    for (int c = 0; c < EPL / W; ++c) {
      const T* p = row + (c * 16 + l16) * W;
      if constexpr (sizeof(T) == 2) {
        uint32_t u[W / 2];
        if constexpr (W == 8) *reinterpret_cast<uint4*>(u) = *reinterpret_cast<const uint4*>(p);
        else *reinterpret_cast<uint2*>(u) = *reinterpret_cast<const uint2*>(p);
#pragma unroll
        for (int x = 0; x < W / 2; ++x) k[c * W / 2 + x] = unpack_bf16x2(u[x]);
      } else {
#pragma unroll
        for (int x = 0; x < W / 4; ++x) {
          const float4 v = *reinterpret_cast<const float4*>(p + 4 * x);
          k[c * W / 2 + 2 * x] = make_float2(v.x, v.y);
          k[c * W / 2 + 2 * x + 1] = make_float2(v.z, v.w);
        }
      }
    }
  }
};

// Sixteen lanes share CPL value columns: lane l holds EPL state rows (dim <= 16 * EPL) of each.  CTA = 4 warps of 2 lane groups ->
// 8 * CPL columns of one head.  k and q rows stay in the element type in shared memory: with the state spread over sixteen lanes and
// 16-byte reads of eight bf16 values the load pipe stays below the FMA pipe.  The next group's q, k, v and constants are requested before this group's products
// and stored to the other half of shared memory after them.  After a product, lane l holds token l % 8, columns (l / 8) * CPL / 2 ...
template <typename T, int EPL, int CPL, int OCC>
__global__ void __launch_bounds__(128, OCC) delta_scan_kernel(const ScanArgs p) {
  pdl_prologue();
  constexpr int DK = 16 * EPL, HC = CPL / 2;
  constexpr int VEC = 16 / int(sizeof(T));             // elements per 16-byte piece
  constexpr int NP = (2 * DC * DK / VEC + 127) / 128;  // pieces of q and k per thread and group
  using Row = RowPiece<T, EPL>;
  __shared__ __align__(16) T s_kq[2][2][DC][DK];       // [buffer][k, q]
  __shared__ __align__(16) float s_c[2][CO];
  __shared__ __align__(16) float s_u[8][3][DC][CPL];   // [lane group][right-hand side, u, D_Cj u_j / |k_j|]
  const int tid = threadIdx.x, lane = tid & 31, l16 = lane & 15, grp16 = tid >> 4, tok = l16 & 7, half = l16 >> 3;
  const int h = blockIdx.y, b = blockIdx.z, kh = h / (p.H / p.KH);
  const int col0 = (blockIdx.x * 8 + grp16) * CPL, colh = col0 + half * HC;
  float2 S[CPL][EPL / 2];
  float* st = p.state + (long long)b * p.state_bs + (long long)h * p.dim * p.vdim;
#pragma unroll
  for (int c = 0; c < CPL; ++c)
#pragma unroll
    for (int e = 0; e < EPL / 2; ++e) {
      const int d = Row::index(e, l16);
      const bool ok = !p.fresh && col0 + c < p.vdim;
      S[c][e].x = (ok && d < p.dim) ? st[(long long)d * p.vdim + col0 + c] : 0.f;
      S[c][e].y = (ok && d + 1 < p.dim) ? st[(long long)(d + 1) * p.vdim + col0 + c] : 0.f;
    }
  const T* base = static_cast<const T*>(p.mixed) + (long long)b * p.L * p.ldm;
  const T* vbase = base + 2 * p.KH * p.dim + (long long)h * p.vdim + colh;
  T* obase = static_cast<T*>(p.o) + (long long)b * p.L * p.ldo + (long long)h * p.vdim + colh;
  const float* cbase = p.coef + ((long long)b * p.groups * p.H + h) * CO;
  const bool vec = (p.dim % VEC) == 0;  // rows are whole 16-byte pieces (p.ldm is a multiple of 8)
  // the lane's HC values of a token are one aligned access when every head starts at a multiple of HC columns
  using VBits = typename Bits<HC * int(sizeof(T))>::type;
  const bool vecv = (p.vdim % HC) == 0 && ((2 * p.KH * p.dim) % HC) == 0 && (p.ldo % HC) == 0;
  const bool inside = colh < p.vdim;  // with vecv: all HC columns or none
  uint4 piece[NP];
  float4 cpiece;
  union { VBits bits; T v[HC]; } vnext;  // as loaded: converting here would wait for the load
  auto request = [&](int grp) {
    const int t0 = grp * DC, n = min(DC, p.L - t0);
#pragma unroll
    for (int u = 0; u < NP; ++u) {
      const int i = (u * 128 + tid) * VEC, which = i / (DC * DK), t = (i / DK) % DC, d = i % DK;
      const T* src = base + (long long)(t0 + t) * p.ldm + (long long)(which ? kh : p.KH + kh) * p.dim + d;
      piece[u] = make_uint4(0, 0, 0, 0);
      if (which < 2 && t < n && d < p.dim) {
        if (vec) piece[u] = *reinterpret_cast<const uint4*>(src);
        else {
          T* e = reinterpret_cast<T*>(&piece[u]);
          for (int x = 0; x < VEC && d + x < p.dim; ++x) e[x] = src[x];
        }
      }
    }
    if (tid < CO / 4) cpiece = *reinterpret_cast<const float4*>(cbase + (long long)grp * p.H * CO + tid * 4);
#pragma unroll
    for (int c = 0; c < HC; ++c) Typed<T>::store(&vnext.v[c], 0.f);
    if (tok < n) {
      const T* src = vbase + (long long)(t0 + tok) * p.ldm;
      if (vecv) {
        if (inside) vnext.bits = *reinterpret_cast<const VBits*>(src);
      } else {
#pragma unroll
        for (int c = 0; c < HC; ++c)
          if (colh + c < p.vdim) vnext.v[c] = src[c];
      }
    }
  };
  auto deposit = [&](int buf) {
#pragma unroll
    for (int u = 0; u < NP; ++u) {
      if ((u * 128 + tid) * VEC >= 2 * DC * DK) continue;
      *reinterpret_cast<uint4*>(&s_kq[buf][0][0][0] + (u * 128 + tid) * VEC) = piece[u];
    }
    if (tid < CO / 4) *reinterpret_cast<float4*>(&s_c[buf][tid * 4]) = cpiece;
  };
  // sums over the state rows of S times the eight k (which = 0) or q (1) vectors of the group
  auto products = [&](int buf, int which, float (&out)[HC]) {
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
          Row::load(s_kq[buf][which][i], l16, k);
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
  request(0);
  deposit(0);
  __syncthreads();
  for (int grp = 0; grp < p.groups; ++grp) {
    const int buf = grp & 1, t0 = grp * DC, n = min(DC, p.L - t0);
    const float* co = s_c[buf];
    float sk[HC], o[HC];
    {
      float v[HC];
#pragma unroll
      for (int c = 0; c < HC; ++c) v[c] = Typed<T>::load(&vnext.v[c]);
      if (grp + 1 < p.groups) request(grp + 1);
      products(buf, 0, sk);
      const float gk = co[2 * DC * DC + tok];
#pragma unroll
      for (int c = 0; c < HC; ++c) s_u[grp16][0][tok][half * HC + c] = v[c] - gk * sk[c];
    }
    __syncwarp();
    {
      const float dk = co[2 * DC * DC + 2 * DC + tok];
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
      for (int c = 0; c < HC; ++c) {
        s_u[grp16][1][tok][half * HC + c] = u[c];
        s_u[grp16][2][tok][half * HC + c] = u[c] * dk;
      }
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
    products(buf, 1, sk);
    const float gq = co[2 * DC * DC + DC + tok], GC = co[2 * DC * DC + 3 * DC];
    if (tok < n) {
      union { VBits bits; T v[HC]; } ov;
#pragma unroll
      for (int c = 0; c < HC; ++c) Typed<T>::store(&ov.v[c], o[c] + gq * sk[c]);
      T* dst = obase + (long long)(t0 + tok) * p.ldo;
      if (vecv) {
        if (inside) *reinterpret_cast<VBits*>(dst) = ov.bits;
      } else {
#pragma unroll
        for (int c = 0; c < HC; ++c)
          if (colh + c < p.vdim) dst[c] = ov.v[c];
      }
    }
#pragma unroll
    for (int c = 0; c < CPL; ++c)
#pragma unroll
      for (int e = 0; e < EPL / 2; ++e) S[c][e] = make_float2(S[c][e].x * GC, S[c][e].y * GC);
#pragma unroll
    for (int j = 0; j < DC; ++j) {
      float w[CPL];
#pragma unroll
      for (int c = 0; c < CPL; c += 4) {
        const float4 q = *reinterpret_cast<const float4*>(&s_u[grp16][2][j][c]);
        w[c] = q.x; w[c + 1] = q.y; w[c + 2] = q.z; w[c + 3] = q.w;
      }
      float2 k[EPL / 2];
      Row::load(s_kq[buf][0][j], l16, k);
#pragma unroll
      for (int e = 0; e < EPL / 2; ++e)
#pragma unroll
        for (int c = 0; c < CPL; ++c) S[c][e] = fma2(k[e], make_float2(w[c], w[c]), S[c][e]);
      if (j & 1) pace();
    }
    if (grp + 1 < p.groups) deposit(buf ^ 1);  // the other half was last read one group ago
    __syncthreads();
  }
#pragma unroll
  for (int c = 0; c < CPL; ++c) {
    if (col0 + c >= p.vdim) continue;
#pragma unroll
    for (int e = 0; e < EPL / 2; ++e) {
      const int d = Row::index(e, l16);
      if (d < p.dim) st[(long long)d * p.vdim + col0 + c] = S[c][e].x;
      if (d + 1 < p.dim) st[(long long)(d + 1) * p.vdim + col0 + c] = S[c][e].y;
    }
  }
}

struct DeltaOutArgs {
  const void* o;           // [rows, ldo] read-out of the recurrence
  long long ldo;
  const void* gate;        // [rows, ldg] + h * vdim
  long long ldg;
  const float* w;          // [vdim]
  float eps;
  void* out;               // [rows, ldout]; columns H * vdim .. ldout are zeroed
  long long ldout;
  long long rows;
  int H, vdim;
  int gate_sigmoid;        // gate activation: 0 silu, 1 sigmoid
};

template <typename T>
__global__ void __launch_bounds__(256) delta_output_kernel(const DeltaOutArgs p) {
  pdl_prologue();
  const long long w = blockIdx.x * 8ll + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (w >= p.rows * p.H) return;
  const long long row = w / p.H;
  const int h = int(w % p.H);
  const T* o = static_cast<const T*>(p.o) + row * p.ldo + (long long)h * p.vdim;
  const T* g = static_cast<const T*>(p.gate) + row * p.ldg + (long long)h * p.vdim;
  T* out = static_cast<T*>(p.out) + row * p.ldout;
  float ss = 0.f;
  for (int c = lane; c < p.vdim; c += 32) {
    const float v = Typed<T>::load(o + c);
    ss += v * v;
  }
  const float r = 1.f / sqrtf(warp_sum(ss) / float(p.vdim) + p.eps);
  for (int c = lane; c < p.vdim; c += 32) {
    const float z = Typed<T>::load(g + c);
    Typed<T>::store(out + (long long)h * p.vdim + c, Typed<T>::load(o + c) * r * p.w[c] * (p.gate_sigmoid ? 1.f : z) * Typed<T>::sigmoid_(z));
  }
  if (h == 0)
    for (int c = p.H * p.vdim + lane; c < p.ldout; c += 32) Typed<T>::store(out + c, 0.f);
}

// The same with eight values per thread: vdim / 8 lanes (a power of two) per head.
template <typename T>
__global__ void __launch_bounds__(256) delta_output_vec_kernel(const DeltaOutArgs p) {
  pdl_prologue();
  const int lanes = p.vdim >> 3;
  const long long i = blockIdx.x * 256ll + threadIdx.x, total = p.rows * p.H * lanes;
  const bool live = i < total;
  const long long hr = (live ? i : 0) / lanes, row = hr / p.H;
  const int h = int(hr % p.H), c = int((live ? i : 0) % lanes) * 8;
  float v[8], z[8], ss = 0.f;
  Typed<T>::load8(static_cast<const T*>(p.o) + row * p.ldo + (long long)h * p.vdim + c, v);
  Typed<T>::load8(static_cast<const T*>(p.gate) + row * p.ldg + (long long)h * p.vdim + c, z);
#pragma unroll
  for (int e = 0; e < 8; ++e) ss += v[e] * v[e];
  for (int off = lanes >> 1; off > 0; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
  const float r = 1.f / sqrtf(ss / float(p.vdim) + p.eps);
#pragma unroll
  for (int e = 0; e < 8; ++e) v[e] *= r * p.w[c + e] * (p.gate_sigmoid ? 1.f : z[e]) * Typed<T>::sigmoid_(z[e]);
  if (live) Typed<T>::store8(static_cast<T*>(p.out) + row * p.ldout + (long long)h * p.vdim + c, v);
}

// ------------------------------------------------------------------------------------------------ decoding
struct StepArgs {
  const void* mixed;       // [B, ldm]
  long long ldm;
  const float* rlen;
  const float* gb;
  float* state;
  long long state_bs;
  const int* lengths;
  const int* active;
  const void* gate;        // [B, ldg] + h * vdim
  long long ldg;
  const float* w;          // [vdim]
  float eps;
  void* out;               // [B, ldout]
  long long ldout;
  int B, H, KH, dim, vdim;
  int gate_sigmoid;        // gate activation: 0 silu, 1 sigmoid
  // one decay per state row instead of one per head: exp(neg_rate[h] softplus(a[b, h * dim + d] + dt_bias[h * dim + d])); a null: gb's
  const void* a;           // [B, lda]
  long long lda;
  const float* neg_rate;   // [H]
  const float* dt_bias;    // [H * dim]
};

// Decays of the state rows of head h -> s_g [dim].
template <typename T>
__device__ __forceinline__ void row_decays(const StepArgs& p, int b, int h, float* s_g, int threads) {
  const T* a = p.a ? static_cast<const T*>(p.a) + (long long)b * p.lda + (long long)h * p.dim : nullptr;
  const float g = p.a ? 0.f : p.gb[(long long)b * 2 * p.H + h], rate = p.a ? p.neg_rate[h] : 0.f;
  for (int d = threadIdx.x; d < p.dim; d += threads) s_g[d] = a ? decay_of<T>(Typed<T>::load(a + d) + p.dt_bias[(long long)h * p.dim + d], rate) : g;
}

constexpr int ST_THREADS = 512;
// One CTA per (head, sequence).  Threads are (row group, column): CW columns, 512 / CW row groups, RPT rows per thread in registers.
template <typename T, int RPT>
__global__ void __launch_bounds__(ST_THREADS) delta_step_kernel(const StepArgs p, int CW) {
  pdl_prologue();
  extern __shared__ float sm[];
  const int RG = ST_THREADS / CW, tid = threadIdx.x, c = tid % CW, rg = tid / CW, h = blockIdx.x, b = blockIdx.y;
  float* s_k = sm;                 // [dim]
  float* s_q = s_k + p.dim;        // [dim]
  float* s_g = s_q + p.dim;        // [dim]
  float* s_o = s_g + p.dim;        // [vdim]
  float* s_r = s_o + p.vdim;       // [RG][CW]
  float* s_red = s_r + ST_THREADS; // [40]
  const int kh = h / (p.H / p.KH);
  const bool fresh = p.lengths[b] == 0, keep = !(p.active && !p.active[b]);
  const T* mixed = static_cast<const T*>(p.mixed) + (long long)b * p.ldm;
  const float rq = p.rlen[(long long)b * 2 * p.KH + kh], rk = p.rlen[(long long)b * 2 * p.KH + p.KH + kh];
  for (int d = tid; d < p.dim; d += ST_THREADS) {
    s_k[d] = Typed<T>::load(mixed + (long long)(p.KH + kh) * p.dim + d) * rk;
    s_q[d] = Typed<T>::load(mixed + (long long)kh * p.dim + d) * rq;
  }
  row_decays<T>(p, b, h, s_g, ST_THREADS);
  const float beta = p.gb[(long long)b * 2 * p.H + p.H + h];
  float* st = p.state + (long long)b * p.state_bs + (long long)h * p.dim * p.vdim;
  __syncthreads();
  float ss = 0.f;
  for (int v0 = 0; v0 < p.vdim; v0 += CW) {
    const int v = v0 + c;
    const bool ok = v < p.vdim;
    float S[RPT], a = 0.f;
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
      const int d = rg + i * RG;
      S[i] = (ok && d < p.dim && !fresh) ? st[(long long)d * p.vdim + v] * s_g[d] : 0.f;
    }
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
      const int d = rg + i * RG;
      if (d < p.dim) a += S[i] * s_k[d];
    }
    s_r[tid] = a;
    __syncthreads();
    float sk = 0.f;
    for (int r = 0; r < RG; ++r) sk += s_r[r * CW + c];
    __syncthreads();
    const float u = ok ? beta * (Typed<T>::load(mixed + 2ll * p.KH * p.dim + (long long)h * p.vdim + v) - sk) : 0.f;
    float o = 0.f;
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
      const int d = rg + i * RG;
      if (d < p.dim) {
        S[i] += s_k[d] * u;
        o += S[i] * s_q[d];
        if (ok && keep) st[(long long)d * p.vdim + v] = S[i];
      }
    }
    s_r[tid] = o;
    __syncthreads();
    if (rg == 0 && ok) {
      float t = 0.f;
      for (int r = 0; r < RG; ++r) t += s_r[r * CW + c];
      s_o[v] = t;
      ss += t * t;
    }
    __syncthreads();
  }
  ss = block_sum(ss, s_red);
  const float r = 1.f / sqrtf(ss / float(p.vdim) + p.eps);
  T* out = static_cast<T*>(p.out) + (long long)b * p.ldout;
  const T* gt = static_cast<const T*>(p.gate) + (long long)b * p.ldg + (long long)h * p.vdim;
  for (int v = tid; v < p.vdim; v += ST_THREADS) {
    const float z = Typed<T>::load(gt + v);
    Typed<T>::store(out + (long long)h * p.vdim + v, s_o[v] * r * p.w[v] * (p.gate_sigmoid ? 1.f : z) * Typed<T>::sigmoid_(z));
  }
  if (h == 0)
    for (int v = p.H * p.vdim + tid; v < p.ldout; v += ST_THREADS) Typed<T>::store(out + v, 0.f);
}

// The same with four columns per access (vdim a multiple of 4, up to 128 per pass): 32 column quads x 8 row groups, RPT rows per thread.
constexpr int SV_THREADS = 256;
template <typename T, int RPT>
__global__ void __launch_bounds__(SV_THREADS, RPT <= 8 ? 4 : RPT <= 16 ? 2 : 1) delta_step_vec_kernel(const StepArgs p) {
  pdl_prologue();
  extern __shared__ __align__(16) float smv[];
  const int tid = threadIdx.x, c = tid & 31, rg = tid >> 5, h = blockIdx.x, b = blockIdx.y;
  float4* s_r = reinterpret_cast<float4*>(smv);                   // [8][32]
  float* s_k = smv + 8 * 32 * 4;                                  // [dim]
  float* s_q = s_k + p.dim;                                       // [dim]
  float* s_g = s_q + p.dim;                                       // [dim]
  float* s_o = s_g + p.dim;                                       // [vdim]
  float* s_red = s_o + p.vdim;                                    // [40]
  const int kh = h / (p.H / p.KH);
  const bool fresh = p.lengths[b] == 0, keep = !(p.active && !p.active[b]);
  const T* mixed = static_cast<const T*>(p.mixed) + (long long)b * p.ldm;
  float* st = p.state + (long long)b * p.state_bs + (long long)h * p.dim * p.vdim;
  const float rq = p.rlen[(long long)b * 2 * p.KH + kh], rk = p.rlen[(long long)b * 2 * p.KH + p.KH + kh];
  const float beta = p.gb[(long long)b * 2 * p.H + p.H + h];
  float ss = 0.f;
  for (int v0 = 0; v0 < p.vdim; v0 += 128) {
    const int v = v0 + c * 4;
    const bool ok = v < p.vdim;
    float4 S[RPT];
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
      const int d = rg + i * 8;
      S[i] = (ok && d < p.dim && !fresh) ? __ldcs(reinterpret_cast<const float4*>(st + (long long)d * p.vdim + v)) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    if (v0 == 0) {
      for (int d = tid; d < p.dim; d += SV_THREADS) {
        s_k[d] = Typed<T>::load(mixed + (long long)(p.KH + kh) * p.dim + d) * rk;
        s_q[d] = Typed<T>::load(mixed + (long long)kh * p.dim + d) * rq;
      }
      row_decays<T>(p, b, h, s_g, SV_THREADS);
      __syncthreads();
    }
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
      const int d = rg + i * 8;
      const float g = d < p.dim ? s_g[d] : 0.f, k = d < p.dim ? s_k[d] : 0.f;
      S[i].x *= g; S[i].y *= g; S[i].z *= g; S[i].w *= g;
      a.x += S[i].x * k; a.y += S[i].y * k; a.z += S[i].z * k; a.w += S[i].w * k;
    }
    s_r[rg * 32 + c] = a;
    __syncthreads();
    float4 t = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int r = 0; r < 8; ++r) {
      const float4 x = s_r[r * 32 + c];
      t.x += x.x; t.y += x.y; t.z += x.z; t.w += x.w;
    }
    __syncthreads();
    float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
    if (ok) {
      const T* vp = mixed + 2ll * p.KH * p.dim + (long long)h * p.vdim + v;
      u = make_float4(beta * (Typed<T>::load(vp) - t.x), beta * (Typed<T>::load(vp + 1) - t.y), beta * (Typed<T>::load(vp + 2) - t.z),
                      beta * (Typed<T>::load(vp + 3) - t.w));
    }
    a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
      const int d = rg + i * 8;
      if (d < p.dim) {
        const float k = s_k[d], q = s_q[d];
        S[i].x += k * u.x; S[i].y += k * u.y; S[i].z += k * u.z; S[i].w += k * u.w;
        a.x += S[i].x * q; a.y += S[i].y * q; a.z += S[i].z * q; a.w += S[i].w * q;
        if (ok && keep) __stcs(reinterpret_cast<float4*>(st + (long long)d * p.vdim + v), S[i]);
      }
    }
    s_r[rg * 32 + c] = a;
    __syncthreads();
    if (rg == 0 && ok) {
      t = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int r = 0; r < 8; ++r) {
        const float4 x = s_r[r * 32 + c];
        t.x += x.x; t.y += x.y; t.z += x.z; t.w += x.w;
      }
      s_o[v] = t.x; s_o[v + 1] = t.y; s_o[v + 2] = t.z; s_o[v + 3] = t.w;
      ss += t.x * t.x + t.y * t.y + t.z * t.z + t.w * t.w;
    }
    __syncthreads();
  }
  ss = block_sum(ss, s_red);
  const float r = 1.f / sqrtf(ss / float(p.vdim) + p.eps);
  T* out = static_cast<T*>(p.out) + (long long)b * p.ldout;
  const T* gt = static_cast<const T*>(p.gate) + (long long)b * p.ldg + (long long)h * p.vdim;
  for (int v = tid; v < p.vdim; v += SV_THREADS) {
    const float z = Typed<T>::load(gt + v);
    Typed<T>::store(out + (long long)h * p.vdim + v, s_o[v] * r * p.w[v] * (p.gate_sigmoid ? 1.f : z) * Typed<T>::sigmoid_(z));
  }
  if (h == 0)
    for (int v = p.H * p.vdim + tid; v < p.ldout; v += SV_THREADS) Typed<T>::store(out + v, 0.f);
}

template <typename T>
static int launch_scan(const ScanArgs& p, cudaStream_t s) {
  const long long pw = (long long)p.B * p.groups * p.KH;
  const dim3 pgrid(unsigned((pw + 3) / 4));
  if constexpr (sizeof(T) == 2) {
    if ((p.dim & 7) == 0 && (p.ldm & 7) == 0) launch_pdl(delta_pairs_kernel<T, true>, pgrid, dim3(128), 0, s, p);
    else launch_pdl(delta_pairs_kernel<T, false>, pgrid, dim3(128), 0, s, p);
  } else {
    launch_pdl(delta_pairs_kernel<T, false>, pgrid, dim3(128), 0, s, p);
  }
  auto grid = [&](int cpl) { return dim3((p.vdim + 8 * cpl - 1) / (8 * cpl), p.H, p.B); };
  if (p.dim <= 64) launch_pdl(delta_scan_kernel<T, 4, 8, 2>, grid(8), dim3(128), 0, s, p);
  else if (p.dim <= 128) launch_pdl(delta_scan_kernel<T, 8, 8, 2>, grid(8), dim3(128), 0, s, p);
  else if (p.dim <= 256) launch_pdl(delta_scan_kernel<T, 16, 4, 2>, grid(4), dim3(128), 0, s, p);
  else return 1006;
  return int(cudaGetLastError());
}

template <typename T>
static int launch_step(const StepArgs& p, cudaStream_t s) {
  if ((p.vdim & 3) == 0 && p.dim <= 256 && (p.state_bs & 3) == 0 && (reinterpret_cast<uintptr_t>(p.state) & 15) == 0) {
    const size_t sm = size_t(8 * 32 * 4 + 3 * p.dim + p.vdim + 40) * sizeof(float);
    if (sm <= 48 * 1024) {
      const dim3 vgrid(p.H, p.B);
      if (p.dim <= 64) launch_pdl(delta_step_vec_kernel<T, 8>, vgrid, dim3(SV_THREADS), sm, s, p);
      else if (p.dim <= 128) launch_pdl(delta_step_vec_kernel<T, 16>, vgrid, dim3(SV_THREADS), sm, s, p);
      else launch_pdl(delta_step_vec_kernel<T, 32>, vgrid, dim3(SV_THREADS), sm, s, p);
      return int(cudaGetLastError());
    }
  }
  int CW = 32;
  while (CW < p.vdim && CW < 128) CW *= 2;
  const int rg = ST_THREADS / CW, rows = (p.dim + rg - 1) / rg;
  const size_t smem = size_t(3 * p.dim + p.vdim + ST_THREADS + 40) * sizeof(float);
  if (smem > 48 * 1024) return 1010;
  const dim3 grid(p.H, p.B);
  if (rows <= 8) launch_pdl(delta_step_kernel<T, 8>, grid, dim3(ST_THREADS), smem, s, p, CW);
  else if (rows <= 16) launch_pdl(delta_step_kernel<T, 16>, grid, dim3(ST_THREADS), smem, s, p, CW);
  else if (rows <= 32) launch_pdl(delta_step_kernel<T, 32>, grid, dim3(ST_THREADS), smem, s, p, CW);
  else if (rows <= 64) launch_pdl(delta_step_kernel<T, 64>, grid, dim3(ST_THREADS), smem, s, p, CW);
  else return 1006;
  return int(cudaGetLastError());
}

}  // namespace ats

using namespace ats;

// Every entry point takes its argument struct by address (the ctypes mirror is in ops/delta.py); `fp32` selects the element type.
static bool pow2_lanes(int width) { return (width & 7) == 0 && width <= 256 && ((width >> 3) & ((width >> 3) - 1)) == 0; }

template <typename T>
static int launch_prep(const DeltaArgs& p, cudaStream_t s) {
  const bool aligned = (p.ld & 7) == 0 && (p.ldm & 7) == 0 && (p.C & 7) == 0 && (reinterpret_cast<uintptr_t>(p.proj) & 15) == 0 &&
                       (reinterpret_cast<uintptr_t>(p.tail) & 15) == 0 && (p.tail_bs & 7) == 0;
  if (aligned && pow2_lanes(p.dim) && (p.vdim & 7) == 0 && p.taps >= 2 && p.taps <= 4) {
    const int conv = p.B * ((p.L + PT - 1) / PT) * (((p.C >> 3) + PV_THREADS - 1) / PV_THREADS);
    const dim3 grid(unsigned(conv + ((long long)p.B * p.L * p.H + PV_THREADS - 1) / PV_THREADS));
    if (p.taps == 2) launch_pdl(delta_prep_vec_kernel<T, 2>, grid, dim3(PV_THREADS), 0, s, p, conv);
    else if (p.taps == 3) launch_pdl(delta_prep_vec_kernel<T, 3>, grid, dim3(PV_THREADS), 0, s, p, conv);
    else launch_pdl(delta_prep_vec_kernel<T, 4>, grid, dim3(PV_THREADS), 0, s, p, conv);
  } else {
    const long long warps = (long long)p.B * p.L * (2 * p.KH + p.H + 1);
    launch_pdl(delta_prep_kernel<T>, dim3(unsigned((warps + 7) / 8)), dim3(256), 0, s, p);
  }
  if (!p.lengths && p.taps > 1) launch_pdl(delta_tail_kernel<T>, dim3((p.C + 255) / 256, p.B), dim3(256), 0, s, p);
  return int(cudaGetLastError());
}

template <typename T>
static int launch_output(const DeltaOutArgs& p, cudaStream_t s) {
  const bool aligned = ((p.ldo | p.ldg | p.ldout) & 7) == 0 && ((reinterpret_cast<uintptr_t>(p.o) | reinterpret_cast<uintptr_t>(p.gate) | reinterpret_cast<uintptr_t>(p.out)) & 15) == 0;
  if (aligned && pow2_lanes(p.vdim)) {  // heads x vdim is a multiple of 8: no padded columns
    launch_pdl(delta_output_vec_kernel<T>, dim3(unsigned((p.rows * p.H * (p.vdim >> 3) + 255) / 256)), dim3(256), 0, s, p);
  } else {
    launch_pdl(delta_output_kernel<T>, dim3(unsigned((p.rows * p.H + 7) / 8)), dim3(256), 0, s, p);
  }
  return int(cudaGetLastError());
}

ATS_API int ats_delta_prep(const DeltaArgs* p, int fp32, void* stream) {
  if (p->taps < 1 || (p->lengths && p->L != 1) || p->KH < 1 || p->H % p->KH) return 1006;
  if (p->B <= 0 || p->L <= 0) return 0;
  return fp32 ? launch_prep<float>(*p, static_cast<cudaStream_t>(stream)) : launch_prep<__nv_bfloat16>(*p, static_cast<cudaStream_t>(stream));
}

ATS_API int ats_delta_scan(const ScanArgs* p, int fp32, void* stream) {
  if (p->B <= 0 || p->L <= 0) return 0;
  if (p->groups != (p->L + DC - 1) / DC) return 1006;
  return fp32 ? launch_scan<float>(*p, static_cast<cudaStream_t>(stream)) : launch_scan<__nv_bfloat16>(*p, static_cast<cudaStream_t>(stream));
}

ATS_API int ats_delta_output(const DeltaOutArgs* p, int fp32, void* stream) {
  if (p->rows <= 0) return 0;
  return fp32 ? launch_output<float>(*p, static_cast<cudaStream_t>(stream)) : launch_output<__nv_bfloat16>(*p, static_cast<cudaStream_t>(stream));
}

ATS_API int ats_delta_step(const StepArgs* p, int fp32, void* stream) {
  if (p->B <= 0) return 0;
  return fp32 ? launch_step<float>(*p, static_cast<cudaStream_t>(stream)) : launch_step<__nv_bfloat16>(*p, static_cast<cudaStream_t>(stream));
}
