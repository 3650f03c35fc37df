// Causal grouped-query attention of a portion of a prompt against a key / value cache, for sm_100a on tcgen05 tensor cores, with capped
// scores and one output gate per head:
//
//   out[i, h] = sigmoid(gate[i, h]) softmax_{j <= pos0 + i}( cap tanh(scale q[i, h] . k[j] / cap) ) v[j],   key head h / (H / G)
//
// The portion's own keys and values are in the cache already.  The general form for any sizes and for fp32 is gqa_portion_kernel in
// gqa_attention.cu; this one takes bf16 heads of up to 128 dimensions (multiples of 8; a head's last 64-column piece is zero-filled by
// the tensor map, so heads need not be whole pieces).
//
// Structure as in attention_window_tcgen05.cu: a CTA owns 256 consecutive queries of one head as two 128-row tiles A, B that ping-pong on
// the tensor cores and share the K / V stream; one query row per soft-max thread; P overwrites S in tensor memory and is the A operand
// of P V; O stays in tensor memory.
// Capped scores lie in [-cap, cap], so for moderate caps the soft-max needs no running maximum: p = 2^(c (tanh(x) - 1)), c = cap log2(e),
// and where all scores of a warp's rows are moderate, tanh is an odd polynomial on the FMA pipe.
// Every wait is bounded (status word + clean unwind); no load uses cluster multicast.
#include "common.cuh"

namespace ats {

constexpr int GT_THREADS = 320;  // soft-max A (warps 0-3), soft-max B (4-7), TMA (8), MMA (9)

struct GqaTcArgs {
  int L, pos0, H, G, vdim, max_len;   // max_len: cache rows per sequence
  const __nv_bfloat16* gate;          // [B * L, ldg] + h, or null
  long long ldg;
  __nv_bfloat16* out;                 // [B * L, ldo], head h at h * vdim
  long long ldo;
  float scale_log2;                   // scale log2(e): uncapped scores in units of log2
  float x_scale;                      // scale / cap
  float cap_log2;                     // cap log2(e)
  int* status;
};

enum GqaMode : int { kPlain = 0, kCapStatic = 1, kCapOnline = 2 };

template <int DQC, int DVC>  // 64-column pieces of a query / key row and of a value row
struct GqaTcSmem {
  static constexpr int TQ = DQC * 16384, TV = DVC * 16384;
  static constexpr int Q_OFF = 0;
  static constexpr int K_OFF = 2 * TQ;
  static constexpr int V_OFF = K_OFF + 2 * TQ;
  static constexpr int BAR_OFF = V_OFF + 2 * TV;
  static constexpr int TOTAL = BAR_OFF + 512 + 1024;
};

template <int DQC, int DVC, int MODE>
__global__ void __launch_bounds__(GT_THREADS, 1)
gqa_attn_tc_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_v,
                   const GqaTcArgs p) {
  using SM = GqaTcSmem<DQC, DVC>;
  constexpr int DV = DVC * 64;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sQ = smem + SM::Q_OFF;
  uint8_t* sK = smem + SM::K_OFF;
  uint8_t* sV = smem + SM::V_OFF;
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + SM::BAR_OFF);
  uint64_t* q_full = bars;         // 1
  uint64_t* k_full = bars + 1;     // [2]
  uint64_t* k_empty = bars + 3;    // [2]
  uint64_t* v_full = bars + 5;     // [2]
  uint64_t* v_empty = bars + 7;    // [2]
  uint64_t* s_full = bars + 9;     // [2] per tile
  uint64_t* p_full = bars + 11;    // [2] per tile, 4 arrivals
  uint64_t* o_done = bars + 13;    // [2] per tile: last P V finished
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 15);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.x, b = blockIdx.y, q0 = int(gridDim.z - 1 - blockIdx.z) * 256;  // the longest rows first
  const int g = h / (p.H / p.G);
  // key blocks of 128 rows: tile A uses blocks [0, nA), tile B blocks [0, nB)
  const int last = p.pos0 + p.L - 1;
  const int nA = min(p.pos0 + q0 + 127, last) / 128 + 1;
  const bool has_b = q0 + 128 < p.L;
  const int nB = has_b ? min(p.pos0 + q0 + 255, last) / 128 + 1 : 0;
  const int nb = max(nA, nB);

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int x = 0; x < 2; ++x) {
      mbar_init(&k_full[x], 1);
      mbar_init(&k_empty[x], 1);
      mbar_init(&v_full[x], 1);
      mbar_init(&v_empty[x], 1);
      mbar_init(&s_full[x], 1);
      mbar_init(&p_full[x], 4);
      mbar_init(&o_done[x], 1);
    }
    *abort_flag = 0;
    mbar_fence_init();
    tma_prefetch_desc(&map_q);
    tma_prefetch_desc(&map_k);
    tma_prefetch_desc(&map_v);
  }
  if (warp == 9) {
    tmem_alloc(tmem_slot, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  // columns: S_A [0,128)  S_B [128,256)  O_A [256, 256 + DV)  O_B [256 + DV, 256 + 2 DV)

  if (warp == 8) {
    if (lane == 0) {
      // ------------------------------------------------------------------ producer
      mbar_expect_tx(q_full, (has_b ? 2 : 1) * SM::TQ);
      for (int x = 0; x < (has_b ? 2 : 1); ++x)
#pragma unroll
        for (int c = 0; c < DQC; ++c) tma_load_3d(sQ + x * SM::TQ + c * 16384, &map_q, q_full, 64 * c, h, b * p.L + q0 + x * 128);
      for (int j = 0; j < nb; ++j) {
        const int krow = b * p.max_len + j * 128, st = j & 1;
        if (!mbar_wait_bounded(&k_empty[st], ((j >> 1) & 1) ^ 1, abort_flag, p.status, kTimeoutEmpty)) break;
        mbar_expect_tx(&k_full[st], SM::TQ);
#pragma unroll
        for (int c = 0; c < DQC; ++c) tma_load_3d(sK + st * SM::TQ + c * 16384, &map_k, &k_full[st], 64 * c, g, krow);
        if (!mbar_wait_bounded(&v_empty[st], ((j >> 1) & 1) ^ 1, abort_flag, p.status, kTimeoutEmpty)) break;
        mbar_expect_tx(&v_full[st], SM::TV);
#pragma unroll
        for (int c = 0; c < DVC; ++c) tma_load_3d(sV + st * SM::TV + c * 16384, &map_v, &v_full[st], 64 * c, g, krow);
      }
      if (*abort_flag) {  // give copies already in flight time to land before the CTA exits
        const uint64_t t0 = globaltimer_ns();
        while (globaltimer_ns() - t0 < 20000ull) {
        }
      }
    }
  } else if (warp == 9) {
    if (lane == 0) {
      // ------------------------------------------------------------------ MMA issuer
      const uint32_t idesc_s = make_idesc(128, 128, 1, 1, 0, 0);
      const uint32_t idesc_o = make_idesc(128, DV, 1, 1, 0, 1);
      const uint64_t q_k = make_smem_desc_sw128(smem_u32(sQ), 16, 1024), k_k = make_smem_desc_sw128(smem_u32(sK), 16, 1024);
      const uint64_t v_mn = make_smem_desc_sw128(smem_u32(sV), 16384, 1024);
      auto issue_s = [&](int x, int j) {
        const uint64_t q_d = desc_advance(q_k, uint32_t(x) * SM::TQ), k_d = desc_advance(k_k, uint32_t(j & 1) * SM::TQ);
#pragma unroll
        for (int k = 0; k < DQC * 4; ++k) {
          const uint32_t off = (k >> 2) * 16384 + (k & 3) * 32;
          tc_mma_f16(tmem_base + x * 128, desc_advance(q_d, off), desc_advance(k_d, off), idesc_s, k != 0);
        }
        tc_commit(&s_full[x]);
      };
      auto issue_pv = [&](int x, int j) {
        const uint64_t v_d = desc_advance(v_mn, uint32_t(j & 1) * SM::TV);  // MN-major: value dimension contiguous
#pragma unroll
        for (int k = 0; k < 8; ++k)
          tc_mma_f16_ts(tmem_base + 256 + x * DV, tmem_base + x * 128 + k * 8, desc_advance(v_d, k * 2048), idesc_o, !(j == 0 && k == 0));
      };
      bool ok = mbar_wait_bounded(q_full, 0, abort_flag, p.status, kTimeoutFull);
      ok = ok && mbar_wait_bounded(&k_full[0], 0, abort_flag, p.status, kTimeoutFull);
      if (ok) {
        tc_fence_after();
        issue_s(0, 0);
        if (nB > 0) issue_s(1, 0);
        tc_commit(&k_empty[0]);
      }
      for (int j = 0; ok && j < nb; ++j) {
        const int nk = (j + 1) & 1;
        const bool a_now = j < nA, a_next = j + 1 < nA, b_now = j < nB, b_next = j + 1 < nB;
        if (!mbar_wait_bounded(&v_full[j & 1], (j >> 1) & 1, abort_flag, p.status, kTimeoutFull)) break;
        if (a_now) {
          if (!mbar_wait_bounded(&p_full[0], j & 1, abort_flag, p.status, kTimeoutTmemFull)) break;
          tc_fence_after();
          issue_pv(0, j);
          if (!a_next) tc_commit(&o_done[0]);
        }
        if (j + 1 < nb) {
          if (!mbar_wait_bounded(&k_full[nk], ((j + 1) >> 1) & 1, abort_flag, p.status, kTimeoutFull)) break;
          tc_fence_after();
          if (a_next) issue_s(0, j + 1);
        }
        if (b_now) {
          if (!mbar_wait_bounded(&p_full[1], j & 1, abort_flag, p.status, kTimeoutTmemFull)) break;
          tc_fence_after();
          issue_pv(1, j);
          if (!b_next) tc_commit(&o_done[1]);
        }
        tc_commit(&v_empty[j & 1]);
        if (j + 1 < nb) {
          if (b_next) issue_s(1, j + 1);
          tc_commit(&k_empty[nk]);
        }
      }
    }
  } else if (warp < 8) {
    // -------------------------------------------------------------------- soft-max groups
    const int x = warp >> 2;        // 0 = tile A, 1 = tile B
    const int quad = warp & 3;      // TMEM lane quadrant this warp may touch
    const int r = quad * 32 + lane;
    const uint32_t lane_base = uint32_t(quad * 32) << 16;
    const uint32_t tmem_S = tmem_base + x * 128 + lane_base;
    const uint32_t tmem_O = tmem_base + 256 + x * DV + lane_base;
    const int n = x ? nB : nA;      // no blocks when tile B does not exist
    const int tile_q = p.pos0 + q0 + x * 128;  // position of the tile's first query
    float m = -1e30f, l = 0.f;
    bool ok = true;
    for (int j = 0; j < n; ++j) {
      if (!mbar_wait_bounded(&s_full[x], j & 1, abort_flag, p.status, kTimeoutTmemFull)) {
        ok = false;
        break;
      }
      tc_fence_after();
      uint32_t v[128];
#pragma unroll
      for (int c = 0; c < 4; ++c) tmem_ld_32x32(tmem_S + c * 32, reinterpret_cast<uint32_t(&)[32]>(v[c * 32]));
      tmem_ld_wait();
      const bool masked = j * 128 + 127 > tile_q;       // the block crosses the diagonal for some row
      const int hi = tile_q + r - j * 128;              // last visible column of this row
      float2 rsa = make_float2(0.f, 0.f), rsb = make_float2(0.f, 0.f);
      if constexpr (MODE == kCapStatic) {
        // p = 2^(cap_log2 (tanh(x) - 1)).  |x| <= 1/2 in all of the warp's scores: tanh(x) = x P(x^2) on the FMA pipe (the special-function
        // pipe would have to do three functions per score); else tanh(x) - 1 = -2 / (1 + e^2x).
        float m0 = 0.f, m1 = 0.f, m2 = 0.f, m3 = 0.f;
#pragma unroll
        for (int c = 0; c < 128; c += 8) {
          m0 = fmaxf(m0, fmaxf(fabsf(__uint_as_float(v[c])), fabsf(__uint_as_float(v[c + 1]))));
          m1 = fmaxf(m1, fmaxf(fabsf(__uint_as_float(v[c + 2])), fabsf(__uint_as_float(v[c + 3]))));
          m2 = fmaxf(m2, fmaxf(fabsf(__uint_as_float(v[c + 4])), fabsf(__uint_as_float(v[c + 5]))));
          m3 = fmaxf(m3, fmaxf(fabsf(__uint_as_float(v[c + 6])), fabsf(__uint_as_float(v[c + 7]))));
        }
        const bool large = __any_sync(0xffffffffu, !(fmaxf(fmaxf(m0, m1), fmaxf(m2, m3)) * p.x_scale <= 0.5f));
        auto finish = [&](int c, int e, float2 pr, uint32_t (&pk)[16]) {
          const int col = c * 32 + 2 * e;
          if (masked) {
            if (col > hi) pr.x = 0.f;
            if (col + 1 > hi) pr.y = 0.f;
          }
          pk[e] = pack_bf16x2(pr.x, pr.y);
          if (e & 1) rsb = __fadd2_rn(rsb, pr);
          else rsa = __fadd2_rn(rsa, pr);
        };
        if (large) {
          const float e_scale = 2.f * 1.4426950408889634f * p.x_scale, neg2c = -2.f * p.cap_log2;
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            uint32_t pk[16];
#pragma unroll
            for (int e = 0; e < 16; ++e) {
              const float s0 = __uint_as_float(v[c * 32 + 2 * e]), s1 = __uint_as_float(v[c * 32 + 2 * e + 1]);
              finish(c, e, make_float2(exp2f(neg2c * __fdividef(1.f, 1.f + exp2f(fminf(e_scale * s0, 120.f)))),
                                       exp2f(neg2c * __fdividef(1.f, 1.f + exp2f(fminf(e_scale * s1, 120.f))))), pk);
            }
            tmem_st_32x16(tmem_S + c * 16, pk);
          }
        } else {
          // tanh(x) / x in x^2 on [0, 1/4], least maximum of the error of tanh (3e-9)
          constexpr float T0 = 0.99999993162241f, T1 = -0.3333277617736538f, T2 = 0.13320570675304483f, T3 = -0.05276213064741831f, T4 = 0.016737566997775927f;
          const float2 xs = make_float2(p.x_scale, p.x_scale), cs = make_float2(p.x_scale * p.cap_log2, p.x_scale * p.cap_log2),
                       nc = make_float2(-p.cap_log2, -p.cap_log2), zero = make_float2(0.f, 0.f);
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            uint32_t pk[16];
#pragma unroll
            for (int e = 0; e < 16; ++e) {
              const float2 s2 = make_float2(__uint_as_float(v[c * 32 + 2 * e]), __uint_as_float(v[c * 32 + 2 * e + 1]));
              const float2 x = __ffma2_rn(s2, xs, zero), t = __ffma2_rn(x, x, zero), w = __ffma2_rn(s2, cs, zero);
              float2 y = __ffma2_rn(t, make_float2(T4, T4), make_float2(T3, T3));
              y = __ffma2_rn(t, y, make_float2(T2, T2));
              y = __ffma2_rn(t, y, make_float2(T1, T1));
              y = __ffma2_rn(t, y, make_float2(T0, T0));
              y = __ffma2_rn(w, y, nc);
              finish(c, e, make_float2(exp2f(y.x), exp2f(y.y)), pk);
            }
            tmem_st_32x16(tmem_S + c * 16, pk);
          }
        }
      } else {
        float to_log2 = p.scale_log2;
        if constexpr (MODE == kCapOnline) {
#pragma unroll
          for (int c = 0; c < 128; ++c) v[c] = __float_as_uint(tanh_fast(__uint_as_float(v[c]) * p.x_scale));
          to_log2 = p.cap_log2;
        }
        if (masked) {
#pragma unroll
          for (int c = 0; c < 128; ++c)
            if (c > hi) v[c] = 0xff800000u;  // -inf
        }
        float mx0 = -INFINITY, mx1 = -INFINITY, mx2 = -INFINITY, mx3 = -INFINITY;
#pragma unroll
        for (int c = 0; c < 128; c += 8) {
          mx0 = fmaxf(mx0, fmaxf(__uint_as_float(v[c]), __uint_as_float(v[c + 1])));
          mx1 = fmaxf(mx1, fmaxf(__uint_as_float(v[c + 2]), __uint_as_float(v[c + 3])));
          mx2 = fmaxf(mx2, fmaxf(__uint_as_float(v[c + 4]), __uint_as_float(v[c + 5])));
          mx3 = fmaxf(mx3, fmaxf(__uint_as_float(v[c + 6]), __uint_as_float(v[c + 7])));
        }
        const float mnew = fmaxf(m, fmaxf(fmaxf(mx0, mx1), fmaxf(mx2, mx3)) * to_log2);
        if (j == 0) {
          m = mnew;
        } else if (__any_sync(0xffffffffu, mnew > m + 8.f)) {
          const float alpha = exp2f(m - mnew);  // the previous P V of this tile has completed: S(j) was computed after it
          m = mnew;
          l *= alpha;
#pragma unroll 1
          for (int c = 0; c < DV / 16; ++c) {
            uint32_t o[16];
            tmem_ld_32x16(tmem_O + c * 16, o);
            tmem_ld_wait();
#pragma unroll
            for (int e = 0; e < 16; ++e) o[e] = __float_as_uint(__uint_as_float(o[e]) * alpha);
            tmem_st_32x16(tmem_O + c * 16, o);
          }
          tmem_st_wait();
        }
        const float2 sc2 = make_float2(to_log2, to_log2), nm2 = make_float2(-m, -m);
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          uint32_t pk[16];
#pragma unroll
          for (int e = 0; e < 16; ++e) {
            const float2 xs = __ffma2_rn(make_float2(__uint_as_float(v[c * 32 + 2 * e]), __uint_as_float(v[c * 32 + 2 * e + 1])), sc2, nm2);
            const float2 pr = make_float2(exp2f(xs.x), exp2f(xs.y));
            pk[e] = pack_bf16x2(pr.x, pr.y);
            if (e & 1) rsb = __fadd2_rn(rsb, pr);
            else rsa = __fadd2_rn(rsa, pr);
          }
          tmem_st_32x16(tmem_S + c * 16, pk);
        }
      }
      l += (rsa.x + rsa.y) + (rsb.x + rsb.y);
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_full[x]);
    }
    if (ok && n > 0 && mbar_wait_bounded(&o_done[x], 0, abort_flag, p.status, kTimeoutTmemFull)) {
      tc_fence_after();
      const int qi = q0 + x * 128 + r;
      const bool live = qi < p.L;
      const long long tok = (long long)b * p.L + qi;
      float inv = 1.f / l;
      if (p.gate && live) inv = __fdividef(inv, 1.f + __expf(-__bfloat162float(p.gate[tok * p.ldg + h])));
      __nv_bfloat16* orow = p.out + tok * p.ldo + (long long)h * p.vdim;
#pragma unroll
      for (int c = 0; c < DV / 32; ++c) {
        uint32_t o[32];
        tmem_ld_32x32(tmem_O + c * 32, o);
        tmem_ld_wait();
        if (!live) continue;
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          if (c * 32 + e * 8 >= p.vdim) break;
          float f[8];
#pragma unroll
          for (int i = 0; i < 8; ++i) f[i] = __uint_as_float(o[8 * e + i]) * inv;
          *reinterpret_cast<uint4*>(orow + c * 32 + e * 8) =
              make_uint4(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]), pack_bf16x2(f[4], f[5]), pack_bf16x2(f[6], f[7]));
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 9) {
    tc_fence_after();
    tmem_dealloc(tmem_base, 512);
  }
}

template <int DQC, int DVC, int MODE>
static int launch_gqa_tc(const CUtensorMap& mq, const CUtensorMap& mk, const CUtensorMap& mv, const GqaTcArgs& p, int B, cudaStream_t s) {
  using SM = GqaTcSmem<DQC, DVC>;
  static_assert(SM::TOTAL <= 227 * 1024, "does not fit an SM");
  cudaError_t ce = cudaFuncSetAttribute(gqa_attn_tc_kernel<DQC, DVC, MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize, SM::TOTAL);
  if (ce != cudaSuccess) return int(ce);
  gqa_attn_tc_kernel<DQC, DVC, MODE><<<dim3(p.H, B, (p.L + 255) / 256), GT_THREADS, SM::TOTAL, s>>>(mq, mk, mv, p);
  return int(cudaGetLastError());
}

template <int MODE>
static int pick_gqa_tc(const CUtensorMap& mq, const CUtensorMap& mk, const CUtensorMap& mv, const GqaTcArgs& p, int dim, int B, cudaStream_t s) {
  if (dim <= 64) return p.vdim <= 64 ? launch_gqa_tc<1, 1, MODE>(mq, mk, mv, p, B, s) : launch_gqa_tc<1, 2, MODE>(mq, mk, mv, p, B, s);
  return p.vdim <= 64 ? launch_gqa_tc<2, 1, MODE>(mq, mk, mv, p, B, s) : launch_gqa_tc<2, 2, MODE>(mq, mk, mv, p, B, s);
}

}  // namespace ats

using namespace ats;

// q [B * L, ldq] (head h at h * dim, normed and rotated); k [B, max_len, ldk], v [B, max_len, ldv], sequences back to back.  cap = 0: scores
// are not capped.  Returns 1003 for shapes this kernel does not cover.
ATS_API int ats_gqa_attn_tc(const void* q, long long ldq, const void* k, long long ldk, const void* v, long long ldv, const void* gate, long long ldg, void* out,
                            long long ldo, int B, int L, int pos0, int max_len, int H, int G, int dim, int vdim, float scale, float cap, int* status,
                            void* stream) {
  if (B < 1 || L < 1 || pos0 < 0 || pos0 + L > max_len || G < 1 || H % G || !(scale > 0.f) || cap < 0.f || (dim & 7) || dim < 8 || dim > 128 || (vdim & 7) ||
      vdim < 8 || vdim > 128 || (ldo & 7) || (reinterpret_cast<uintptr_t>(out) & 15))
    return 1003;
  static thread_local bool ctx_bound = false;
  if (!ctx_bound) {
    cudaFree(0);
    ctx_bound = true;
  }
  CUtensorMap mq, mk, mv;
  int e;
  if ((e = make_tmap_heads(&mq, q, (uint64_t)B * L, H, dim, ldq))) return e;
  if ((e = make_tmap_heads(&mk, k, (uint64_t)B * max_len, G, dim, ldk))) return e;
  if ((e = make_tmap_heads(&mv, v, (uint64_t)B * max_len, G, vdim, ldv))) return e;
  GqaTcArgs p;
  p.L = L; p.pos0 = pos0; p.H = H; p.G = G; p.vdim = vdim; p.max_len = max_len;
  p.gate = static_cast<const __nv_bfloat16*>(gate); p.ldg = ldg; p.out = static_cast<__nv_bfloat16*>(out); p.ldo = ldo;
  const float log2e = 1.4426950408889634f;
  p.scale_log2 = scale * log2e; p.x_scale = cap > 0.f ? scale / cap : 0.f; p.cap_log2 = cap * log2e; p.status = status;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (cap == 0.f) return pick_gqa_tc<kPlain>(mq, mk, mv, p, dim, B, s);
  // probabilities relative to the cap go down to 2^(-2 cap_log2): normal numbers in bf16 and fp32 up to here
  if (p.cap_log2 <= 58.f) return pick_gqa_tc<kCapStatic>(mq, mk, mv, p, dim, B, s);
  return pick_gqa_tc<kCapOnline>(mq, mk, mv, p, dim, B, s);
}
