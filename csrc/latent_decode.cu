// Decoding with latent attention on tensor cores (bf16): one query token per sequence against its ring of latents.  The general
// form for any sizes and for fp32, and the layout of the ring, are in latent_attention.cu.
//
//   latent_head_mm<absorb>   qa[b, h, :] = W_uk[h]^T q_u[b, h, :]               per head: [16 sequences x dim] x [dim x rank]
//   latent_ring              scores of 16 heads against the ring rows (one shared row serves all heads, so the heads are the 16 rows of
//                            the MMA), soft-max, weighted sum of the latents; chunks of the ring are merged by the next kernel
//   latent_head_mm<expand>   out[b, h, :] = sigmoid(gate) * W_uv[h] (merged latent)   [16 sequences x rank] x [rank x vdim]
//
// A decode step is bound by the bytes of the ring, so warp-level MMAs are enough; a tile of 32 or 64 ring rows is fetched once with
// cp.async (later ones while this one is used) and serves both products (plain and transposing ldmatrix; rows are padded by 16 bytes against bank conflicts).  Weights
// stream straight from global memory into B fragments: the order of the reduction index is permuted so that the 16-byte piece a lane
// loads is its fragment for two consecutive steps, and the A fragments are read with the same permutation.
#include "common.cuh"

namespace ats {

__device__ __forceinline__ void mma_bf16_16816(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldmatrix_x4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
// 16 bytes global -> shared; zeros when `ok` is false
__device__ __forceinline__ void cp_async_16(uint32_t dst, const void* src, bool ok) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(ok ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

struct HeadMmArgs {
  const __nv_bfloat16* x;   // absorb: q, head h at h * x_hs, rows x_ld apart
  long long x_ld;
  int x_hs;
  const float* part_o;      // expand: [B, H, n_chunks, K] partial latents and [B, H, n_chunks, 2] (max, sum)
  const float* part_ml;
  int n_chunks;
  const __nv_bfloat16* w;   // [H, N, ldw], reduction index contiguous
  long long w_hs;
  int ldw;
  __nv_bfloat16* out;       // row b, head h, column n at b * out_ld + h * out_hs + n
  long long out_ld;
  int out_hs;
  const __nv_bfloat16* gate;  // same columns as out, rows ldg apart (expand; may be null)
  long long ldg;
  int B, H, N, K;
};
constexpr int HM_EXPAND_ROWS = 8;  // sequences per CTA of the expand form: its time is the gathering of the partial latents, not the MMAs
constexpr int HM_MAX_CHUNKS = 64;  // two per lane in the merge

// CTA: 16 (expand: 8) sequences x (WARPS * NT * 8) output columns of one head.
template <int WARPS, int NT, bool EXPAND>
__global__ void __launch_bounds__(WARPS * 32, EXPAND ? 2 : 3) latent_head_mm_kernel(const HeadMmArgs p) {
  pdl_prologue();
  extern __shared__ __align__(16) uint8_t smem_raw[];
  __nv_bfloat16* sx = reinterpret_cast<__nv_bfloat16*>(smem_raw);  // [16][K + 32]
  __shared__ float s_f[EXPAND ? 16 : 1][EXPAND ? HM_MAX_CHUNKS : 1];
  const int ldx = p.K + 32, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  constexpr int ROWS = EXPAND ? HM_EXPAND_ROWS : 16;
  const int h = blockIdx.y, b0 = blockIdx.z * ROWS, nb = min(ROWS, p.B - b0);
  const int n0 = (blockIdx.x * WARPS + warp) * NT * 8;
  // the first PRE steps of this lane's weights, requested before the inputs are gathered
  constexpr int PRE = EXPAND ? 4 : 3;
  const __nv_bfloat16* w = p.w + h * p.w_hs + 8 * t;
  uint4 pre[PRE][NT];
#pragma unroll
  for (int u = 0; u < PRE; ++u)
#pragma unroll
    for (int i = 0; i < NT; ++i) {
      const int n = n0 + i * 8 + g;
      pre[u][i] = (n < p.N && u * 32 < p.K) ? *reinterpret_cast<const uint4*>(w + (long long)n * p.ldw + u * 32) : make_uint4(0, 0, 0, 0);
    }
  if (EXPAND) {
    for (int j = warp; j < nb; j += WARPS) {  // merge factors of the chunks: one warp per sequence, lanes over chunks
      const float2* ml = reinterpret_cast<const float2*>(p.part_ml) + ((long long)(b0 + j) * p.H + h) * p.n_chunks;
      const float2 x0 = lane < p.n_chunks ? ml[lane] : make_float2(-INFINITY, 0.f), x1 = lane + 32 < p.n_chunks ? ml[lane + 32] : make_float2(-INFINITY, 0.f);
      const float m = warp_max(fmaxf(x0.x, x1.x));
      const float f0 = x0.y > 0.f ? __expf(x0.x - m) : 0.f, f1 = x1.y > 0.f ? __expf(x1.x - m) : 0.f;
      const float inv = 1.f / warp_sum(f0 * x0.y + f1 * x1.y);
      s_f[j][lane] = f0 * inv;
      s_f[j][lane + 32] = f1 * inv;
    }
    __syncthreads();
    // four rows of a column quad at a time: with the chunk loop unrolled, up to eight loads are in flight per thread
    const int quads = p.K >> 2;
    const long long row = (long long)p.H * p.n_chunks * p.K;  // elements between sequences
    for (int i = tid; i < (ROWS / 4) * quads; i += WARPS * 32) {
      const int j = (i / quads) * 4, r = (i % quads) * 4;
      float4 a[4];
#pragma unroll
      for (int u = 0; u < 4; ++u) a[u] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (j < nb) {
        const float* po = p.part_o + ((long long)(b0 + j) * p.H + h) * p.n_chunks * p.K + r;
#pragma unroll 2
        for (int c = 0; c < p.n_chunks; ++c)
#pragma unroll
          for (int u = 0; u < 4; ++u) {
            const float f = j + u < nb ? s_f[j + u][c] : 0.f;
            // (a chunk beyond a short sequence was not written: its factor is zero and its values are not used)
            const float4 v = f > 0.f ? *reinterpret_cast<const float4*>(po + u * row + (long long)c * p.K) : make_float4(0.f, 0.f, 0.f, 0.f);
            a[u].x += f * v.x; a[u].y += f * v.y; a[u].z += f * v.z; a[u].w += f * v.w;
          }
      }
#pragma unroll
      for (int u = 0; u < 4; ++u)
        *reinterpret_cast<uint2*>(sx + (j + u) * ldx + r) = make_uint2(pack_bf16x2(a[u].x, a[u].y), pack_bf16x2(a[u].z, a[u].w));
    }
  } else {
    const int pieces = p.K >> 3;
    for (int i = tid; i < 16 * pieces; i += WARPS * 32) {
      const int j = i / pieces, c = (i % pieces) * 8;
      *reinterpret_cast<uint4*>(sx + j * ldx + c) =
          j < nb ? *reinterpret_cast<const uint4*>(p.x + (b0 + j) * p.x_ld + (long long)h * p.x_hs + c) : make_uint4(0, 0, 0, 0);
    }
  }
  __syncthreads();
  if (n0 >= p.N) return;
  float acc[NT][4];
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[i][e] = 0.f;
  // blocks of PRE steps: the next block's weights are in flight while this one is multiplied
  for (int k0 = 0; k0 < p.K; k0 += 32 * PRE) {
    uint4 cur[PRE][NT];
#pragma unroll
    for (int u = 0; u < PRE; ++u)
#pragma unroll
      for (int i = 0; i < NT; ++i) {
        cur[u][i] = pre[u][i];
        const int n = n0 + i * 8 + g, k = k0 + 32 * (PRE + u);
        pre[u][i] = (n < p.N && k < p.K) ? *reinterpret_cast<const uint4*>(w + (long long)n * p.ldw + k) : make_uint4(0, 0, 0, 0);
      }
#pragma unroll
    for (int u = 0; u < PRE; ++u) {
      const int k = k0 + 32 * u;
      if (k >= p.K) break;
      const uint4 lo = *reinterpret_cast<const uint4*>(sx + g * ldx + k + 8 * t);
      const uint4 hi = ROWS > 8 ? *reinterpret_cast<const uint4*>(sx + (g + 8) * ldx + k + 8 * t) : make_uint4(0, 0, 0, 0);
#pragma unroll
      for (int i = 0; i < NT; ++i) {
        mma_bf16_16816(acc[i], lo.x, hi.x, lo.y, hi.y, cur[u][i].x, cur[u][i].y);
        mma_bf16_16816(acc[i], lo.z, hi.z, lo.w, hi.w, cur[u][i].z, cur[u][i].w);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < NT; ++i) {
    const int n = n0 + i * 8 + 2 * t;
    if (n >= p.N) continue;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int j = g + 8 * e;
      if (j >= nb) continue;
      float v0 = acc[i][2 * e], v1 = acc[i][2 * e + 1];
      const long long at = (long long)h * p.out_hs + n;
      if (EXPAND && p.gate) {
        const float2 gt = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(p.gate + (b0 + j) * p.ldg + at));
        v0 = __fdividef(v0, 1.f + __expf(-gt.x));
        v1 = __fdividef(v1, 1.f + __expf(-gt.y));
      }
      *reinterpret_cast<uint32_t*>(p.out + (b0 + j) * p.out_ld + at) = pack_bf16x2(v0, v1);
    }
  }
}

struct RingArgs {
  const __nv_bfloat16* qa;    // [B, H, rank] absorbed queries
  const __nv_bfloat16* q;     // [B, ldq]: rotated part of head h at h * dq + dim (not yet rotated)
  long long ldq;
  int dim, dq;
  const float* cos;           // [positions, rot / 2]
  const float* sin;
  const __nv_bfloat16* ring;  // [B, R, cwp]
  long long ring_bs;
  const int* lengths;
  int H, R, rank, rot, cwp, chunk, n_chunks;
  float scale;
  float* part_o;              // [B, H, n_chunks, rank]
  float* part_ml;             // [B, H, n_chunks, 2]
};
constexpr int LR_THREADS = 256;

struct RingSmem {
  int ldt, qa, s, pr, al, total;  // row pitch of tile and queries (elements), byte offsets
  __host__ __device__ RingSmem(int cw, int groups, int stages, int keys) {
    ldt = cw + 8;
    qa = stages * keys * ldt * 2;
    s = qa + groups * 16 * ldt * 2;
    pr = s + groups * 4 * 16 * (keys + 4) * 4;
    al = pr + groups * 16 * (keys + 8) * 2;
    total = al + groups * 16 * 4;
  }
};

// NTW: 8-column tiles of the latent per warp (rank = 64 * NTW).  HG: groups of 16 heads that share the CTA's ring tiles, eight warps each.
// STAGES: ring tiles in shared memory.
// LR_KEYS: rows of a tile (32 or 64; more rows spread the barriers and the soft-max reductions over more keys).
template <int NTW, int HG, int STAGES, int LR_KEYS>
__global__ void __launch_bounds__(LR_THREADS * HG, 2 / HG) latent_ring_kernel(const RingArgs p) {
  pdl_prologue();
  extern __shared__ __align__(16) uint8_t smem_raw[];
  const int cw = p.rank + p.rot;
  const RingSmem L(cw, HG, STAGES, LR_KEYS);
  const int tid = threadIdx.x % LR_THREADS, group = threadIdx.x / LR_THREADS, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  __nv_bfloat16* tile = reinterpret_cast<__nv_bfloat16*>(smem_raw);
  __nv_bfloat16* sq = reinterpret_cast<__nv_bfloat16*>(smem_raw + L.qa) + group * 16 * L.ldt;
  float* ss = reinterpret_cast<float*>(smem_raw + L.s) + group * 4 * 16 * (LR_KEYS + 4);                  // [quarter of the reduction][16][LR_KEYS + 4]
  __nv_bfloat16* sp = reinterpret_cast<__nv_bfloat16*>(smem_raw + L.pr) + group * 16 * (LR_KEYS + 8);     // [16][LR_KEYS + 8]
  float* sal = reinterpret_cast<float*>(smem_raw + L.al) + group * 16;                                   // [16]
  const int chunk = blockIdx.x, h0 = (blockIdx.y * HG + group) * 16, b = blockIdx.z, nh = max(0, min(16, p.H - h0));
  const int pos = p.lengths[b], n = min(pos + 1, p.R), k0 = chunk * p.chunk, k1 = min(n, k0 + p.chunk);
  float* ml = p.part_ml + (((long long)b * p.H + h0) * p.n_chunks + chunk) * 2;
  if (k0 >= k1) {
    if (tid < nh) {
      ml[(long long)tid * p.n_chunks * 2] = -INFINITY;
      ml[(long long)tid * p.n_chunks * 2 + 1] = 0.f;
    }
    return;
  }
  const __nv_bfloat16* ring = p.ring + (long long)b * p.ring_bs;
  // every warp of the CTA copies its own rows of a tile: no divisions in the copy loop
  auto fetch = [&](int first, int buf) {
#pragma unroll
    for (int x = 0; x < LR_KEYS / (8 * HG); ++x) {
      const int r = (group * 8 + warp) * (LR_KEYS / (8 * HG)) + x;
      const bool ok = first + r < k1;
      const __nv_bfloat16* src = ring + (long long)(ok ? first + r : k0) * p.cwp;
      __nv_bfloat16* dst = tile + (buf * LR_KEYS + r) * L.ldt;
      for (int c = lane * 8; c < cw; c += 256) cp_async_16(smem_u32(dst + c), src + c, ok);
    }
  };
#pragma unroll
  for (int x = 0; x < STAGES - 1; ++x) {
    if (k0 + x * LR_KEYS < k1) fetch(k0 + x * LR_KEYS, x);
    cp_async_commit();  // (possibly empty: the number of groups in flight stays the same)
  }
  // absorbed queries (rows of heads that do not exist are zero), rotated parts
  for (int i = tid; i < 16 * (p.rank >> 3); i += LR_THREADS) {
    const int r = i / (p.rank >> 3), c = (i % (p.rank >> 3)) * 8;
    *reinterpret_cast<uint4*>(sq + r * L.ldt + c) =
        r < nh ? *reinterpret_cast<const uint4*>(p.qa + ((long long)b * p.H + h0 + r) * p.rank + c) : make_uint4(0, 0, 0, 0);
  }
  const int half = p.rot >> 1;
  for (int i = tid; i < 16 * half; i += LR_THREADS) {
    const int r = i / half, m = i % half;
    float u = 0.f, v = 0.f;
    if (r < nh) {
      const __nv_bfloat16* qr = p.q + b * p.ldq + (long long)(h0 + r) * p.dq + p.dim + m;
      const float x = __bfloat162float(qr[0]), y = __bfloat162float(qr[half]);
      const float cs = p.cos[(long long)pos * half + m], sn = p.sin[(long long)pos * half + m];
      u = x * cs - y * sn;
      v = y * cs + x * sn;
    }
    sq[r * L.ldt + p.rank + m] = __float2bfloat16(u);
    sq[r * L.ldt + p.rank + half + m] = __float2bfloat16(v);
  }
  float acc[NTW][4];
#pragma unroll
  for (int i = 0; i < NTW; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[i][e] = 0.f;
  float m_[2] = {-INFINITY, -INFINITY}, l_[2] = {0.f, 0.f};  // soft-max state of heads 2 * warp, + 1
  // score phase: warp w takes keys 16 (w & 1) .. + 15 of every 32 keys of a tile and a quarter of the reduction, whose query fragments stay in registers
  const int steps = cw >> 4, per = (steps + 3) >> 2, q_lo = (warp >> 1) * per, q_n = max(0, min(per, steps - q_lo));
  __syncthreads();  // queries are complete
  uint32_t aq[NTW + 2][4];
#pragma unroll
  for (int x = 0; x < NTW + 2; ++x)
    if (x < q_n) ldmatrix_x4(smem_u32(sq + (lane & 15) * L.ldt + (q_lo + x) * 16 + (lane >> 4) * 8), aq[x]);
  // (matrices: keys 0..7 and 8..15, each with the two halves of the 16 reduction columns)
  const uint32_t b_addr = smem_u32(tile + ((warp & 1) * 16 + (lane >> 4) * 8 + (lane & 7)) * L.ldt + q_lo * 16 + ((lane >> 3) & 1) * 8);
  const uint32_t p_addr = smem_u32(sp + (lane & 15) * (LR_KEYS + 8) + (lane >> 4) * 8);
  const uint32_t v_addr = smem_u32(tile + (lane & 15) * L.ldt + warp * NTW * 8 + (lane >> 4) * 8);
  int buf = 0;
  for (int first = k0; first < k1; first += LR_KEYS) {
    cp_async_wait<STAGES - 2>();
    __syncthreads();  // this tile is complete, and every warp is done with the one before it: its stage takes the next fetch
    const int ahead = first + (STAGES - 1) * LR_KEYS, into = buf == 0 ? STAGES - 1 : buf - 1;
    if (ahead < k1) fetch(ahead, into);
    cp_async_commit();
    const uint32_t stage = uint32_t(buf * LR_KEYS * L.ldt * 2);
    // ---- scores
    {
#pragma unroll
      for (int kg = 0; kg < LR_KEYS / 32; ++kg) {
        float c0[4] = {0.f, 0.f, 0.f, 0.f}, c1[4] = {0.f, 0.f, 0.f, 0.f};  // keys 0..7 / 8..15 of the sixteen
#pragma unroll
        for (int x = 0; x < NTW + 2; ++x)
          if (x < q_n) {
            uint32_t bb[4];
            ldmatrix_x4(b_addr + stage + (kg * 32 * L.ldt + x * 16) * 2, bb);
            mma_bf16_16816(c0, aq[x][0], aq[x][1], aq[x][2], aq[x][3], bb[0], bb[1]);
            mma_bf16_16816(c1, aq[x][0], aq[x][1], aq[x][2], aq[x][3], bb[2], bb[3]);
          }
        float* s0 = ss + ((warp >> 1) * 16 + g) * (LR_KEYS + 4) + kg * 32 + (warp & 1) * 16 + 2 * t;
        *reinterpret_cast<float2*>(s0) = make_float2(c0[0], c0[1]);
        *reinterpret_cast<float2*>(s0 + 8) = make_float2(c1[0], c1[1]);
        *reinterpret_cast<float2*>(s0 + 8 * (LR_KEYS + 4)) = make_float2(c0[2], c0[3]);
        *reinterpret_cast<float2*>(s0 + 8 * (LR_KEYS + 4) + 8) = make_float2(c1[2], c1[3]);
      }
    }
    __syncthreads();
    // ---- soft-max: two heads per warp, LR_KEYS / 32 keys per lane
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int r = warp * 2 + e;
      float x[LR_KEYS / 32], mt = -INFINITY, sum = 0.f;
#pragma unroll
      for (int kg = 0; kg < LR_KEYS / 32; ++kg) {
        const int key = kg * 32 + lane;
        const float* s0 = ss + r * (LR_KEYS + 4) + key;
        constexpr int Q = 16 * (LR_KEYS + 4);
        x[kg] = first + key < k1 ? ((s0[0] + s0[Q]) + (s0[2 * Q] + s0[3 * Q])) * p.scale : -INFINITY;
        mt = fmaxf(mt, x[kg]);
      }
      const float mn = fmaxf(m_[e], warp_max(mt));  // the tile has at least one key: finite
      const float al = __expf(m_[e] - mn);
#pragma unroll
      for (int kg = 0; kg < LR_KEYS / 32; ++kg) {
        const float pr = __expf(x[kg] - mn);
        sum += pr;
        sp[r * (LR_KEYS + 8) + kg * 32 + lane] = __float2bfloat16(pr);
      }
      m_[e] = mn;
      l_[e] = l_[e] * al + warp_sum(sum);
      if (lane == 0) sal[r] = al;
    }
    __syncthreads();
    // ---- weighted sum of the latents: warp w, columns w * NTW * 8 ..
    const float al0 = sal[g], al1 = sal[g + 8];
#pragma unroll
    for (int i = 0; i < NTW; ++i) {
      acc[i][0] *= al0; acc[i][1] *= al0;
      acc[i][2] *= al1; acc[i][3] *= al1;
    }
#pragma unroll
    for (int k = 0; k < LR_KEYS; k += 16) {
      uint32_t a[4];
      ldmatrix_x4(p_addr + k * 2, a);
#pragma unroll
      for (int i = 0; i < NTW; i += 2) {
        uint32_t v[4];
        ldmatrix_x4_trans(v_addr + stage + (k * L.ldt + i * 8) * 2, v);
        mma_bf16_16816(acc[i], a[0], a[1], a[2], a[3], v[0], v[1]);
        mma_bf16_16816(acc[i + 1], a[0], a[1], a[2], a[3], v[2], v[3]);
      }
    }
    buf = buf + 1 == STAGES ? 0 : buf + 1;
  }
#pragma unroll
  for (int i = 0; i < NTW; ++i) {
    const int c = (warp * NTW + i) * 8 + 2 * t;
    float* o = p.part_o + (((long long)b * p.H + h0 + g) * p.n_chunks + chunk) * p.rank + c;
    if (g < nh) *reinterpret_cast<float2*>(o) = make_float2(acc[i][0], acc[i][1]);
    if (g + 8 < nh) *reinterpret_cast<float2*>(o + 8ll * p.n_chunks * p.rank) = make_float2(acc[i][2], acc[i][3]);
  }
  if (lane == 0)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int r = warp * 2 + e;
      if (r < nh) {
        ml[(long long)r * p.n_chunks * 2] = m_[e];
        ml[(long long)r * p.n_chunks * 2 + 1] = l_[e];
      }
    }
}

template <int NTW, int HG, int STAGES, int KEYS>
static cudaError_t launch_ring_groups(const RingArgs& p, int B, cudaStream_t s) {
  const RingSmem L(p.rank + p.rot, HG, STAGES, KEYS);
  cudaError_t e = cudaFuncSetAttribute(latent_ring_kernel<NTW, HG, STAGES, KEYS>, cudaFuncAttributeMaxDynamicSharedMemorySize, L.total);
  if (e != cudaSuccess) return e;
  return launch_pdl(latent_ring_kernel<NTW, HG, STAGES, KEYS>, dim3(p.n_chunks, (p.H + 16 * HG - 1) / (16 * HG), B), dim3(LR_THREADS * HG), size_t(L.total), s, p);
}
template <int NTW>
static cudaError_t launch_ring(const RingArgs& p, int B, cudaStream_t s) {
  const bool wide = p.H > 16 && RingSmem(p.rank + p.rot, 2, 2, 64).total <= 227 * 1024;
  return wide ? launch_ring_groups<NTW, 2, 2, 64>(p, B, s) : launch_ring_groups<NTW, 1, 2, 32>(p, B, s);
}

}  // namespace ats

using namespace ats;

// One decoded token per sequence (see the head of the file).  q [B, ldq] head h at h * (dim + rot), not rotated; w_ukt [H, rank, dim],
// w_uv [H, vdim, ldv], ring [B, R, cwp].  qa [B, H, rank], part_o, part_ml: scratch.  Returns 1003 for shapes this form does not cover.
ATS_API int ats_latent_decode_mma(const void* q, long long ldq, const void* w_ukt, const void* w_uv, int ldv, const void* ring, long long ring_bs,
                                  const int* lengths, const float* cos, const float* sin, const void* gate, long long ldg, void* qa, float* part_o,
                                  float* part_ml, void* out, long long ldo, int B, int H, int dim, int rot, int rank, int vdim, int cwp, int R, int chunk,
                                  int n_chunks, float scale, void* stream) {
  if (B < 1) return 0;
  const bool rank_ok = rank == 128 || rank == 256 || rank == 384 || rank == 512;
  if (!rank_ok || (dim & 31) || dim > 512 || (rot & 31) || rot < 32 || rot > 128 || (vdim & 7) || (ldq & 7) || (ldv & 7) || (cwp & 7) || (ring_bs & 7) || (ldo & 1) ||
      (gate && (ldg & 1)) || chunk < 64 || (chunk % 64) || n_chunks < 1 || n_chunks > HM_MAX_CHUNKS || (long long)chunk * n_chunks < R)
    return 1003;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  HeadMmArgs a = {};
  a.x = static_cast<const __nv_bfloat16*>(q); a.x_ld = ldq; a.x_hs = dim + rot;
  a.w = static_cast<const __nv_bfloat16*>(w_ukt); a.w_hs = (long long)rank * dim; a.ldw = dim;
  a.out = static_cast<__nv_bfloat16*>(qa); a.out_ld = (long long)H * rank; a.out_hs = rank;
  a.B = B; a.H = H; a.N = rank; a.K = dim;
  const int bt = (B + 15) / 16;
  cudaError_t e = launch_pdl(latent_head_mm_kernel<4, 4, false>, dim3(rank / 128, H, bt), dim3(128), size_t(16) * (dim + 32) * 2, s, a);
  if (e != cudaSuccess) return int(e);
  RingArgs r;
  r.qa = static_cast<const __nv_bfloat16*>(qa); r.q = static_cast<const __nv_bfloat16*>(q); r.ldq = ldq; r.dim = dim; r.dq = dim + rot;
  r.cos = cos; r.sin = sin; r.ring = static_cast<const __nv_bfloat16*>(ring); r.ring_bs = ring_bs; r.lengths = lengths;
  r.H = H; r.R = R; r.rank = rank; r.rot = rot; r.cwp = cwp; r.chunk = chunk; r.n_chunks = n_chunks; r.scale = scale;
  r.part_o = part_o; r.part_ml = part_ml;
  e = rank == 128 ? launch_ring<2>(r, B, s) : rank == 256 ? launch_ring<4>(r, B, s) : rank == 384 ? launch_ring<6>(r, B, s) : launch_ring<8>(r, B, s);
  if (e != cudaSuccess) return int(e);
  HeadMmArgs x = {};
  x.part_o = part_o; x.part_ml = part_ml; x.n_chunks = n_chunks;
  x.w = static_cast<const __nv_bfloat16*>(w_uv); x.w_hs = (long long)vdim * ldv; x.ldw = ldv;
  x.out = static_cast<__nv_bfloat16*>(out); x.out_ld = ldo; x.out_hs = vdim;
  x.gate = static_cast<const __nv_bfloat16*>(gate); x.ldg = ldg;
  x.B = B; x.H = H; x.N = vdim; x.K = rank;
  e = launch_pdl(latent_head_mm_kernel<8, 2, true>, dim3((vdim + 127) / 128, H, (B + HM_EXPAND_ROWS - 1) / HM_EXPAND_ROWS), dim3(256), size_t(16) * (rank + 32) * 2, s, x);
  return int(e != cudaSuccess ? e : cudaGetLastError());
}
