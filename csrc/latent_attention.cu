// Latent attention over a sliding window (every head attends to one shared low-rank latent plus one shared rotated key part).
//
// A token's cache entry is [latent c (rank, RMS-normed), rotated key part (rot)], `cw` = rank + rot values in rows of `cwp` (a multiple
// of 8).  The cache of a sequence is a ring of R rows: the token at position p lives in row p % R.  R = min(window, longest sequence),
// so a decoded token overwrites exactly the entry that has just left the window, and "rows 0 .. min(p + 1, R) - 1" is the visible set.
//
// * Portions of a prompt: latent_context gathers the window that precedes the portion from the ring and appends the portion's own
//   entries (norms, rotation) -> ctx [n_old + L rows]; a GEMM expands ctx to per-head keys and values; window_attn attends; latent_finish
//   rotates the queries before that and puts the portion's last R entries into the ring.
// * Decoding works on the latents themselves: the query's unrotated part is multiplied by the key expansion (latent_absorb), scores and
//   weighted sums run over the ring (latent_decode), and the merged latent is multiplied by the value expansion (latent_expand, with the
//   output gate), so the per-head keys and values of the window never exist.
//
// bf16 and fp32 forms of every kernel; arithmetic is fp32 in both.
#include "typed.cuh"

namespace ats {

struct LatentArgs {
  const void* proj;      // [B * L, ld]: query latent at q_col, [latent, rotated key part] at kv_col
  long long ld;
  int q_col, kv_col, q_rank, q_pad, rank, rot, cwp;
  const float* q_w;      // [q_rank] norm weights
  const float* kv_w;     // [rank]
  float eps;
  const float* cos;      // [positions, rot / 2]
  const float* sin;
  void* cq;              // [B * L, q_pad]
  void* ctx;             // portions: [B, n_old + L, cwp]; decoding: unused
  void* ring;            // [B, R, cwp]
  long long ring_bs;     // elements between sequences
  int B, L, R, n_old, pos0;
  const int* lengths;    // decoding: position per sequence (L == 1), entries go straight to the ring
  const int* active;     // decoding: rows with 0 leave the ring alone (nullptr: all rows are live)
};

// One CTA per context row.
template <typename T>
__global__ void __launch_bounds__(128) latent_context_kernel(const LatentArgs p) {
  pdl_prologue();
  __shared__ float red[40];
  const int rows = p.n_old + p.L, b = blockIdx.x / rows, j = blockIdx.x % rows, tid = threadIdx.x;
  T* ring = static_cast<T*>(p.ring) + (long long)b * p.ring_bs;
  if (j < p.n_old) {
    const int src = (p.pos0 - p.n_old + j) % p.R;
    T* dst = static_cast<T*>(p.ctx) + ((long long)b * rows + j) * p.cwp;
    for (int c = tid; c < p.cwp; c += blockDim.x) dst[c] = ring[(long long)src * p.cwp + c];
    return;
  }
  const int t = j - p.n_old;
  const long long row = (long long)b * p.L + t;
  const T* in = static_cast<const T*>(p.proj) + row * p.ld;
  const int pos = p.lengths ? p.lengths[b] : p.pos0 + t;
  T* dst;
  if (p.lengths) dst = (p.active && !p.active[b]) ? nullptr : ring + (long long)(pos % p.R) * p.cwp;
  else dst = static_cast<T*>(p.ctx) + ((long long)b * rows + j) * p.cwp;
  float sq = 0.f, sc = 0.f;
  for (int c = tid; c < p.q_rank; c += blockDim.x) {
    const float v = Typed<T>::load(in + p.q_col + c);
    sq += v * v;
  }
  for (int c = tid; c < p.rank; c += blockDim.x) {
    const float v = Typed<T>::load(in + p.kv_col + c);
    sc += v * v;
  }
  sq = block_sum(sq, red);
  sc = block_sum(sc, red);
  const float rq = 1.f / sqrtf(sq / float(p.q_rank) + p.eps), rc = 1.f / sqrtf(sc / float(p.rank) + p.eps);
  T* cq = static_cast<T*>(p.cq) + row * p.q_pad;
  for (int c = tid; c < p.q_pad; c += blockDim.x)
    Typed<T>::store(cq + c, c < p.q_rank ? Typed<T>::load(in + p.q_col + c) * rq * p.q_w[c] : 0.f);
  if (dst == nullptr) return;
  const int half = p.rot >> 1;
  for (int c = tid; c < p.cwp; c += blockDim.x) {
    float v = 0.f;
    if (c < p.rank) {
      v = Typed<T>::load(in + p.kv_col + c) * rc * p.kv_w[c];
    } else if (c < p.rank + p.rot) {
      const int i = c - p.rank, m = i < half ? i : i - half;
      const float u = Typed<T>::load(in + p.kv_col + p.rank + m), w = Typed<T>::load(in + p.kv_col + p.rank + m + half);
      const float cs = p.cos[(long long)pos * half + m], sn = p.sin[(long long)pos * half + m];
      v = i < half ? u * cs - w * sn : w * cs + u * sn;
    }
    Typed<T>::store(dst + c, v);
  }
}

// The same when every part is whole 16-byte pieces: one warp per row, eight values per access.
template <typename T>
__global__ void __launch_bounds__(128) latent_context_vec_kernel(const LatentArgs p) {
  pdl_prologue();
  const int rows = p.n_old + p.L, lane = threadIdx.x & 31;
  const long long r = blockIdx.x * 4ll + (threadIdx.x >> 5);
  if (r >= (long long)p.B * rows) return;  // whole warp; no CTA barrier below
  const int b = int(r / rows), j = int(r % rows), half = p.rot >> 1;
  T* ring = static_cast<T*>(p.ring) + (long long)b * p.ring_bs;
  float v[8], w[8];
  if (j < p.n_old) {
    const T* src = ring + (long long)((p.pos0 - p.n_old + j) % p.R) * p.cwp;
    T* dst = static_cast<T*>(p.ctx) + r * p.cwp;
    for (int c = lane * 8; c < p.cwp; c += 256) {
      Typed<T>::load8(src + c, v);
      Typed<T>::store8(dst + c, v);
    }
    return;
  }
  const long long row = (long long)b * p.L + j - p.n_old;
  const T* in = static_cast<const T*>(p.proj) + row * p.ld;
  const int pos = p.lengths ? p.lengths[b] : p.pos0 + j - p.n_old;
  T* dst;
  if (p.lengths) dst = (p.active && !p.active[b]) ? nullptr : ring + (long long)(pos % p.R) * p.cwp;
  else dst = static_cast<T*>(p.ctx) + r * p.cwp;
  float sq = 0.f, sc = 0.f;
#pragma unroll 4
  for (int c = lane * 8; c < p.q_rank; c += 256) {
    Typed<T>::load8(in + p.q_col + c, v);
#pragma unroll
    for (int e = 0; e < 8; ++e) sq += v[e] * v[e];
  }
#pragma unroll 2
  for (int c = lane * 8; c < p.rank; c += 256) {
    Typed<T>::load8(in + p.kv_col + c, v);
#pragma unroll
    for (int e = 0; e < 8; ++e) sc += v[e] * v[e];
  }
  const float rq = 1.f / sqrtf(warp_sum(sq) / float(p.q_rank) + p.eps), rc = 1.f / sqrtf(warp_sum(sc) / float(p.rank) + p.eps);
  T* cq = static_cast<T*>(p.cq) + row * p.q_pad;
#pragma unroll 4
  for (int c = lane * 8; c < p.q_rank; c += 256) {  // second read: from L1
    Typed<T>::load8(in + p.q_col + c, v);
    Typed<float>::load8(p.q_w + c, w);
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] *= rq * w[e];
    Typed<T>::store8(cq + c, v);
  }
  if (dst == nullptr) return;
#pragma unroll 2
  for (int c = lane * 8; c < p.rank; c += 256) {
    Typed<T>::load8(in + p.kv_col + c, v);
    Typed<float>::load8(p.kv_w + c, w);
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] *= rc * w[e];
    Typed<T>::store8(dst + c, v);
  }
  for (int m = lane * 8; m < half; m += 256) {
    float u[8], x[8], cs[8], sn[8];
    Typed<T>::load8(in + p.kv_col + p.rank + m, u);
    Typed<T>::load8(in + p.kv_col + p.rank + half + m, x);
    Typed<float>::load8(p.cos + (long long)pos * half + m, cs);
    Typed<float>::load8(p.sin + (long long)pos * half + m, sn);
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      v[e] = u[e] * cs[e] - x[e] * sn[e];
      w[e] = x[e] * cs[e] + u[e] * sn[e];
    }
    Typed<T>::store8(dst + p.rank + m, v);
    Typed<T>::store8(dst + p.rank + half + m, w);
  }
}

struct FinishArgs {
  void* q;               // [B * L, ldq], head h at h * (dim + rot): its last `rot` values are rotated in place
  long long ldq;
  int H, dim, rot;
  const float* cos;
  const float* sin;
  const void* ctx;
  void* ring;
  long long ring_bs;
  int cwp, B, L, R, n_old, pos0;
};

// One CTA per token: rotate the query heads; the last R tokens of the portion also go into the ring.
template <typename T>
__global__ void __launch_bounds__(128) latent_finish_kernel(const FinishArgs p) {
  pdl_prologue();
  const int b = blockIdx.x / p.L, t = blockIdx.x % p.L, half = p.rot >> 1;
  const long long pos = p.pos0 + t;
  T* q = static_cast<T*>(p.q) + (long long)blockIdx.x * p.ldq;
  for (int i = threadIdx.x; i < p.H * half; i += blockDim.x) {
    const int h = i / half, m = i % half;
    T* d = q + (long long)h * (p.dim + p.rot) + p.dim + m;
    const float u = Typed<T>::load(d), w = Typed<T>::load(d + half);
    const float cs = p.cos[pos * half + m], sn = p.sin[pos * half + m];
    Typed<T>::store(d, u * cs - w * sn);
    Typed<T>::store(d + half, w * cs + u * sn);
  }
  if (t >= p.L - p.R) {
    const T* src = static_cast<const T*>(p.ctx) + ((long long)b * (p.n_old + p.L) + p.n_old + t) * p.cwp;
    T* dst = static_cast<T*>(p.ring) + (long long)b * p.ring_bs + (pos % p.R) * p.cwp;
    for (int c = threadIdx.x; c < p.cwp; c += blockDim.x) dst[c] = src[c];
  }
}

// The same when the halves of the rotated part are whole 16-byte pieces: a thread rotates eight pairs or copies eight values.
template <typename T>
__global__ void __launch_bounds__(256) latent_finish_vec_kernel(const FinishArgs p) {
  pdl_prologue();
  const int half = p.rot >> 1, per_head = half >> 3, keep = min(p.L, p.R), cp = p.cwp >> 3;
  const long long rot_n = (long long)p.B * p.L * p.H * per_head, total = rot_n + (long long)p.B * keep * cp;
  for (long long i = blockIdx.x * 256ll + threadIdx.x; i < total; i += (long long)gridDim.x * 256) {
    if (i < rot_n) {
      const int m = int(i % per_head) * 8, h = int((i / per_head) % p.H);
      const long long row = i / per_head / p.H, pos = p.pos0 + row % p.L;
      T* d = static_cast<T*>(p.q) + row * p.ldq + (long long)h * (p.dim + p.rot) + p.dim + m;
      float u[8], x[8], cs[8], sn[8], v[8], w[8];
      Typed<T>::load8(d, u);
      Typed<T>::load8(d + half, x);
      Typed<float>::load8(p.cos + pos * half + m, cs);
      Typed<float>::load8(p.sin + pos * half + m, sn);
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        v[e] = u[e] * cs[e] - x[e] * sn[e];
        w[e] = x[e] * cs[e] + u[e] * sn[e];
      }
      Typed<T>::store8(d, v);
      Typed<T>::store8(d + half, w);
    } else {
      const long long k = i - rot_n;
      const int c = int(k % cp) * 8, t = p.L - keep + int((k / cp) % keep), b = int(k / cp / keep);
      float v[8];
      Typed<T>::load8(static_cast<const T*>(p.ctx) + ((long long)b * (p.n_old + p.L) + p.n_old + t) * p.cwp + c, v);
      Typed<T>::store8(static_cast<T*>(p.ring) + (long long)b * p.ring_bs + ((p.pos0 + t) % p.R) * (long long)p.cwp + c, v);
    }
  }
}

struct WindowArgs {
  const void* q;         // [B * L, ldq], head h at h * (dim + rot): [unrotated, rotated]
  long long ldq;
  const void* kv;        // [B, n_old + L, ldkv]: key of head h at h * dim, value at v_col + h * vdim
  long long ldkv;
  int v_col;
  const void* kr;        // [B, n_old + L, ldkr]: the shared rotated key part
  long long ldkr;
  const void* gate;      // [B * L, ldg] + h * vdim: the output is multiplied by its sigmoid (nullptr: no gate)
  long long ldg;
  void* out;             // [B * L, ldo], head h at h * vdim; columns H * vdim .. ldo are zeroed
  long long ldo;
  int B, L, n_old, H, dim, rot, vdim, window;
  float scale;
};

// General form, any sizes: one warp per (query, head), lanes over keys for the scores and over value dimensions for the sum.
constexpr int WA_MAX_V = 16;  // value dimensions per lane: vdim <= 512
template <typename T>
__global__ void __launch_bounds__(256) window_attn_kernel(const WindowArgs p) {
  pdl_prologue();
  extern __shared__ float s_q[];
  const int dq = p.dim + p.rot, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x * 8 + warp, h = blockIdx.y, b = blockIdx.z, rows = p.n_old + p.L;
  if (t >= p.L) return;  // whole warp; no CTA barrier below
  const long long row = (long long)b * p.L + t;
  float* q = s_q + warp * dq;
  const T* qg = static_cast<const T*>(p.q) + row * p.ldq + (long long)h * dq;
  for (int c = lane; c < dq; c += 32) q[c] = Typed<T>::load(qg + c) * p.scale;
  __syncwarp();
  const T* kbase = static_cast<const T*>(p.kv) + (long long)b * rows * p.ldkv + (long long)h * p.dim;
  const T* vbase = static_cast<const T*>(p.kv) + (long long)b * rows * p.ldkv + p.v_col + (long long)h * p.vdim;
  const T* rbase = static_cast<const T*>(p.kr) + (long long)b * rows * p.ldkr;
  const int hi = p.n_old + t, lo = max(0, hi - p.window + 1);
  float m = -INFINITY, l = 0.f, o[WA_MAX_V];
#pragma unroll
  for (int e = 0; e < WA_MAX_V; ++e) o[e] = 0.f;
  for (int k0 = lo; k0 <= hi; k0 += 32) {
    const int key = k0 + lane;
    float s = -INFINITY;
    if (key <= hi) {
      const T* kk = kbase + key * p.ldkv;
      const T* kr = rbase + key * p.ldkr;
      float acc = 0.f;
      for (int c = 0; c < p.dim; ++c) acc += q[c] * Typed<T>::load(kk + c);
      for (int c = 0; c < p.rot; ++c) acc += q[p.dim + c] * Typed<T>::load(kr + c);
      s = acc;
    }
    const float mn = fmaxf(m, warp_max(s)), f = Typed<T>::exp_(m - mn);
    const float pr = key <= hi ? Typed<T>::exp_(s - mn) : 0.f;
    m = mn;
    l = l * f + pr;  // per lane; summed at the end
#pragma unroll
    for (int e = 0; e < WA_MAX_V; ++e) o[e] *= f;
    const int n = min(32, hi - k0 + 1);
    for (int j = 0; j < n; ++j) {
      const float pj = __shfl_sync(0xffffffffu, pr, j);
      const T* vv = vbase + (k0 + j) * p.ldkv;
#pragma unroll
      for (int e = 0; e < WA_MAX_V; ++e)
        if (e * 32 + lane < p.vdim) o[e] += pj * Typed<T>::load(vv + e * 32 + lane);
    }
  }
  const float inv = 1.f / warp_sum(l);
  T* out = static_cast<T*>(p.out) + row * p.ldo;
  const T* g = p.gate ? static_cast<const T*>(p.gate) + row * p.ldg + (long long)h * p.vdim : nullptr;
#pragma unroll
  for (int e = 0; e < WA_MAX_V; ++e) {
    const int c = e * 32 + lane;
    if (c < p.vdim) Typed<T>::store(out + (long long)h * p.vdim + c, o[e] * inv * (g ? Typed<T>::sigmoid_(Typed<T>::load(g + c)) : 1.f));
  }
  if (h == 0)
    for (int c = p.H * p.vdim + lane; c < p.ldo; c += 32) Typed<T>::store(out + c, 0.f);
}

// ------------------------------------------------------------------------------------------------ decoding
struct AbsorbArgs {
  const void* q;         // [B, ldq], head h at h * (dim + rot)
  long long ldq;
  const void* wk;        // [H * dim, ldw] key expansion
  long long ldw;
  const float* cos;
  const float* sin;
  const int* lengths;    // position of the new token per sequence
  void* qa;              // [B, H, cwp]: [query in latent space, rotated part], zero padded
  int B, H, dim, rot, rank, cwp;
};
constexpr int HM_B = 8;  // sequences per CTA: a weight element read once serves all of them

template <typename T>
__global__ void __launch_bounds__(128) latent_absorb_kernel(const AbsorbArgs p) {
  pdl_prologue();
  extern __shared__ float xs[];  // [HM_B][dim]
  const int h = blockIdx.x, r = blockIdx.y * 128 + threadIdx.x, b0 = blockIdx.z * HM_B, nb = min(HM_B, p.B - b0), dq = p.dim + p.rot;
  const T* q = static_cast<const T*>(p.q) + (long long)h * dq;
  for (int i = threadIdx.x; i < HM_B * p.dim; i += 128) {
    const int j = i / p.dim, d = i % p.dim;
    xs[i] = j < nb ? Typed<T>::load(q + (b0 + j) * p.ldq + d) : 0.f;
  }
  __syncthreads();
  if (r >= p.cwp) return;
  float acc[HM_B];
#pragma unroll
  for (int j = 0; j < HM_B; ++j) acc[j] = 0.f;
  if (r < p.rank) {
    const T* w = static_cast<const T*>(p.wk) + (long long)h * p.dim * p.ldw + r;
#pragma unroll 4
    for (int d = 0; d < p.dim; ++d) {
      const float wv = Typed<T>::load(w + d * p.ldw);
#pragma unroll
      for (int j = 0; j < HM_B; ++j) acc[j] += wv * xs[j * p.dim + d];
    }
  } else if (r < p.rank + p.rot) {
    const int half = p.rot >> 1, i = r - p.rank, m = i < half ? i : i - half;
    for (int j = 0; j < nb; ++j) {
      const T* d = q + (b0 + j) * p.ldq + p.dim + m;
      const long long pos = p.lengths[b0 + j];
      const float u = Typed<T>::load(d), w = Typed<T>::load(d + half), cs = p.cos[pos * half + m], sn = p.sin[pos * half + m];
      acc[j] = i < half ? u * cs - w * sn : w * cs + u * sn;
    }
  }
  for (int j = 0; j < nb; ++j) Typed<T>::store(static_cast<T*>(p.qa) + ((long long)(b0 + j) * p.H + h) * p.cwp + r, acc[j]);
}

struct LatentDecodeArgs {
  const void* qa;        // [B, H, cwp]
  const void* ring;      // [B, R, cwp]
  long long ring_bs;
  const int* lengths;
  int B, H, R, rank, cw, cwp, chunk, n_chunks;
  float scale;
  float* part_o;         // [B, H, n_chunks, rank]
  float* part_ml;        // [B, H, n_chunks, 2]
};

// General form: CTA per (chunk of ring rows, up to 8 heads, sequence); a warp scores one row at a time for all its heads.
constexpr int LD_H = 8, LD_THREADS = 256;
template <typename T>
__global__ void __launch_bounds__(LD_THREADS) latent_decode_kernel(const LatentDecodeArgs p) {
  pdl_prologue();
  extern __shared__ float sm[];
  float* s_q = sm;                       // [LD_H][cw]
  float* s_p = sm + LD_H * p.cw;         // [LD_H][chunk]
  const int chunk = blockIdx.x, h0 = blockIdx.y * LD_H, b = blockIdx.z, nh = min(LD_H, p.H - h0);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int n = min(p.lengths[b] + 1, p.R), k0 = chunk * p.chunk, nk = min(p.chunk, n - k0);
  float* ml = p.part_ml + (((long long)b * p.H + h0) * p.n_chunks + chunk) * 2;
  if (nk <= 0) {
    if (tid < nh) {
      ml[(long long)tid * p.n_chunks * 2] = -INFINITY;
      ml[(long long)tid * p.n_chunks * 2 + 1] = 0.f;
    }
    return;
  }
  const T* qa = static_cast<const T*>(p.qa) + ((long long)b * p.H + h0) * p.cwp;
  for (int i = tid; i < LD_H * p.cw; i += LD_THREADS) s_q[i] = (i / p.cw) < nh ? Typed<T>::load(qa + (i / p.cw) * p.cwp + i % p.cw) * p.scale : 0.f;
  __syncthreads();
  const T* ring = static_cast<const T*>(p.ring) + (long long)b * p.ring_bs + (long long)k0 * p.cwp;
  for (int k = warp; k < nk; k += LD_THREADS / 32) {
    float acc[LD_H];
#pragma unroll
    for (int e = 0; e < LD_H; ++e) acc[e] = 0.f;
    for (int c = lane; c < p.cw; c += 32) {
      const float v = Typed<T>::load(ring + (long long)k * p.cwp + c);
#pragma unroll
      for (int e = 0; e < LD_H; ++e) acc[e] += v * s_q[e * p.cw + c];
    }
#pragma unroll
    for (int e = 0; e < LD_H; ++e) {
      acc[e] = warp_sum(acc[e]);
      if (lane == 0) s_p[e * p.chunk + k] = acc[e];
    }
  }
  __syncthreads();
  if (warp < nh) {
    float m = -INFINITY, l = 0.f;
    for (int k = lane; k < nk; k += 32) m = fmaxf(m, s_p[warp * p.chunk + k]);
    m = warp_max(m);
    for (int k = lane; k < nk; k += 32) {
      const float e = Typed<T>::exp_(s_p[warp * p.chunk + k] - m);
      s_p[warp * p.chunk + k] = e;
      l += e;
    }
    l = warp_sum(l);
    if (lane == 0) {
      ml[(long long)warp * p.n_chunks * 2] = m;
      ml[(long long)warp * p.n_chunks * 2 + 1] = l;
    }
  }
  __syncthreads();
  for (int r = tid; r < p.rank; r += LD_THREADS) {
    float o[LD_H];
#pragma unroll
    for (int e = 0; e < LD_H; ++e) o[e] = 0.f;
#pragma unroll 4
    for (int k = 0; k < nk; ++k) {
      const float v = Typed<T>::load(ring + (long long)k * p.cwp + r);
#pragma unroll
      for (int e = 0; e < LD_H; ++e) o[e] += v * s_p[e * p.chunk + k];
    }
    for (int e = 0; e < nh; ++e) p.part_o[(((long long)b * p.H + h0 + e) * p.n_chunks + chunk) * p.rank + r] = o[e];
  }
}

struct ExpandArgs {
  const float* part_o;
  const float* part_ml;
  const void* wv;        // [H, rank, ldv] value expansion, transposed per head
  int ldv;
  const void* gate;      // [B, ldg] + h * vdim or nullptr
  long long ldg;
  void* out;             // [B, ldo]
  long long ldo;
  int B, H, rank, vdim, n_chunks;
};

template <typename T>
__global__ void __launch_bounds__(128) latent_expand_kernel(const ExpandArgs p) {
  pdl_prologue();
  extern __shared__ float xs[];  // [HM_B][rank] merged latent outputs
  __shared__ float s_f[HM_B];
  const int h = blockIdx.x, v = blockIdx.y * 128 + threadIdx.x, b0 = blockIdx.z * HM_B, nb = min(HM_B, p.B - b0);
  for (int j = 0; j < nb; ++j) {
    const long long w = (long long)(b0 + j) * p.H + h;
    const float* ml = p.part_ml + w * p.n_chunks * 2;
    float m = -INFINITY, l = 0.f;
    for (int c = 0; c < p.n_chunks; ++c) m = fmaxf(m, ml[2 * c]);
    for (int c = 0; c < p.n_chunks; ++c)
      if (ml[2 * c + 1] > 0.f) l += ml[2 * c + 1] * Typed<T>::exp_(ml[2 * c] - m);
    for (int r = threadIdx.x; r < p.rank; r += 128) {
      float t = 0.f;
      for (int c = 0; c < p.n_chunks; ++c)
        if (ml[2 * c + 1] > 0.f) t += p.part_o[(w * p.n_chunks + c) * p.rank + r] * Typed<T>::exp_(ml[2 * c] - m);
      xs[j * p.rank + r] = t;
    }
    if (threadIdx.x == 0) s_f[j] = 1.f / l;
  }
  for (int i = nb * p.rank + threadIdx.x; i < HM_B * p.rank; i += 128) xs[i] = 0.f;
  __syncthreads();
  if (v < p.vdim) {
    float acc[HM_B];
#pragma unroll
    for (int j = 0; j < HM_B; ++j) acc[j] = 0.f;
    const T* w = static_cast<const T*>(p.wv) + (long long)h * p.rank * p.ldv + v;
#pragma unroll 4
    for (int r = 0; r < p.rank; ++r) {
      const float wv = Typed<T>::load(w + (long long)r * p.ldv);
#pragma unroll
      for (int j = 0; j < HM_B; ++j) acc[j] += wv * xs[j * p.rank + r];
    }
#pragma unroll
    for (int j = 0; j < HM_B; ++j) {
      if (j >= nb) break;
      float o = acc[j] * s_f[j];
      if (p.gate) o *= Typed<T>::sigmoid_(Typed<T>::load(static_cast<const T*>(p.gate) + (b0 + j) * p.ldg + (long long)h * p.vdim + v));
      Typed<T>::store(static_cast<T*>(p.out) + (b0 + j) * p.ldo + (long long)h * p.vdim + v, o);
    }
  }
  if (h == 0 && blockIdx.y == 0)
    for (int j = 0; j < nb; ++j)
      for (int c = p.H * p.vdim + threadIdx.x; c < p.ldo; c += 128) Typed<T>::store(static_cast<T*>(p.out) + (b0 + j) * p.ldo + c, 0.f);
}

template <typename K>
static int big_smem(K kernel, size_t bytes) {
  if (bytes > 227 * 1024) return 1010;
  if (bytes > 48 * 1024) return int(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, int(bytes)));
  return 0;
}

}  // namespace ats

using namespace ats;

static bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

template <typename T>
static int launch_context(const LatentArgs& p, cudaStream_t s) {
  const int rows = p.B * (p.n_old + p.L);
  const bool vec = ((p.q_rank | p.rank | p.q_col | p.kv_col | p.q_pad | p.cwp) & 7) == 0 && (p.rot & 15) == 0 && p.rot > 0 && (p.ld & 7) == 0 && (p.ring_bs & 7) == 0 &&
                   p.q_pad == p.q_rank && p.cwp == p.rank + p.rot && aligned16(p.proj) && aligned16(p.ring);
  if (vec) launch_pdl(latent_context_vec_kernel<T>, dim3((rows + 3) / 4), dim3(128), 0, s, p);
  else launch_pdl(latent_context_kernel<T>, dim3(rows), dim3(128), 0, s, p);
  return int(cudaGetLastError());
}

template <typename T>
static int launch_finish(const FinishArgs& p, cudaStream_t s) {
  const bool vec = (p.rot & 15) == 0 && p.rot > 0 && (p.dim & 7) == 0 && (p.ldq & 7) == 0 && (p.cwp & 7) == 0 && (p.ring_bs & 7) == 0 && aligned16(p.q) && aligned16(p.ring);
  if (vec) {
    const long long n = (long long)p.B * p.L * p.H * (p.rot >> 4) + (long long)p.B * (p.L < p.R ? p.L : p.R) * (p.cwp >> 3);
    const long long blocks = (n + 255) / 256;
    launch_pdl(latent_finish_vec_kernel<T>, dim3(unsigned(blocks < 148 * 64 ? blocks : 148 * 64)), dim3(256), 0, s, p);
  } else {
    launch_pdl(latent_finish_kernel<T>, dim3(p.B * p.L), dim3(128), 0, s, p);
  }
  return int(cudaGetLastError());
}

// Every entry point takes its argument struct by address (the ctypes mirror is in ops/latent.py); `fp32` selects the element type.
ATS_API int ats_latent_context(const LatentArgs* p, int fp32, void* stream) {
  if (p->R < 1 || p->rot < 0 || (p->rot & 1) || (p->lengths && p->L != 1) || p->n_old < 0 || p->n_old > p->R) return 1006;
  if (p->B <= 0 || p->n_old + p->L <= 0) return 0;
  return fp32 ? launch_context<float>(*p, static_cast<cudaStream_t>(stream)) : launch_context<__nv_bfloat16>(*p, static_cast<cudaStream_t>(stream));
}

ATS_API int ats_latent_finish(const FinishArgs* p, int fp32, void* stream) {
  if (p->R < 1 || (p->rot & 1)) return 1006;
  if (p->B <= 0 || p->L <= 0) return 0;
  return fp32 ? launch_finish<float>(*p, static_cast<cudaStream_t>(stream)) : launch_finish<__nv_bfloat16>(*p, static_cast<cudaStream_t>(stream));
}

ATS_API int ats_window_attn(const WindowArgs* p, int fp32, void* stream) {
  if (p->vdim > 32 * WA_MAX_V || p->vdim < 1 || p->window < 1) return 1006;
  const size_t smem = size_t(8) * (p->dim + p->rot) * sizeof(float);
  const dim3 grid((p->L + 7) / 8, p->H, p->B);
  if (p->L <= 0 || p->B <= 0) return 0;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  int e;
  if (fp32) {
    if ((e = big_smem(window_attn_kernel<float>, smem))) return e;
    launch_pdl(window_attn_kernel<float>, grid, dim3(256), smem, s, *p);
  } else {
    if ((e = big_smem(window_attn_kernel<__nv_bfloat16>, smem))) return e;
    launch_pdl(window_attn_kernel<__nv_bfloat16>, grid, dim3(256), smem, s, *p);
  }
  return int(cudaGetLastError());
}

ATS_API int ats_latent_absorb(const AbsorbArgs* p, int fp32, void* stream) {
  if (p->B <= 0) return 0;
  const size_t smem = size_t(HM_B) * p->dim * sizeof(float);
  const dim3 grid(p->H, (p->cwp + 127) / 128, (p->B + HM_B - 1) / HM_B);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  int e;
  if (fp32) {
    if ((e = big_smem(latent_absorb_kernel<float>, smem))) return e;
    launch_pdl(latent_absorb_kernel<float>, grid, dim3(128), smem, s, *p);
  } else {
    if ((e = big_smem(latent_absorb_kernel<__nv_bfloat16>, smem))) return e;
    launch_pdl(latent_absorb_kernel<__nv_bfloat16>, grid, dim3(128), smem, s, *p);
  }
  return int(cudaGetLastError());
}

ATS_API int ats_latent_decode(const LatentDecodeArgs* p, int fp32, void* stream) {
  if (p->B <= 0) return 0;
  if (p->chunk < 1 || p->n_chunks < 1 || (long long)p->chunk * p->n_chunks < p->R) return 1006;
  const size_t smem = size_t(LD_H) * (p->cw + p->chunk) * sizeof(float);
  const dim3 grid(p->n_chunks, (p->H + LD_H - 1) / LD_H, p->B);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  int e;
  if (fp32) {
    if ((e = big_smem(latent_decode_kernel<float>, smem))) return e;
    launch_pdl(latent_decode_kernel<float>, grid, dim3(LD_THREADS), smem, s, *p);
  } else {
    if ((e = big_smem(latent_decode_kernel<__nv_bfloat16>, smem))) return e;
    launch_pdl(latent_decode_kernel<__nv_bfloat16>, grid, dim3(LD_THREADS), smem, s, *p);
  }
  return int(cudaGetLastError());
}

ATS_API int ats_latent_expand(const ExpandArgs* p, int fp32, void* stream) {
  if (p->B <= 0) return 0;
  const size_t smem = size_t(HM_B) * p->rank * sizeof(float);
  const dim3 grid(p->H, (p->vdim + 127) / 128, (p->B + HM_B - 1) / HM_B);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  int e;
  if (fp32) {
    if ((e = big_smem(latent_expand_kernel<float>, smem))) return e;
    launch_pdl(latent_expand_kernel<float>, grid, dim3(128), smem, s, *p);
  } else {
    if ((e = big_smem(latent_expand_kernel<__nv_bfloat16>, smem))) return e;
    launch_pdl(latent_expand_kernel<__nv_bfloat16>, grid, dim3(128), smem, s, *p);
  }
  return int(cudaGetLastError());
}
