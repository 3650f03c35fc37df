// Sliding-window attention over a portion of a prompt for sm_100a on tcgen05 tensor cores, for heads whose query and key are an
// unrotated part (own key per head) followed by a rotated part (one key shared by all heads): latent attention.
//
//   out[i, h, :] = sigmoid(gate[i, h, :]) * softmax_{0 <= i - j < window}( scale (q_u . k_u[j, h] + q_r . k_r[j]) ) v[j, h, :]
//
// The portion's L queries follow n_old context rows (the window before the portion), so key row n_old + i is query i's own.  The general
// form for any sizes and for fp32 is window_attn_kernel in latent_attention.cu; this one takes bf16 with dim a multiple of 64,
// rot a multiple of 8 up to 64, and vdim 64 or 128.
//
// Structure as in attention_fwd2_tcgen05.cu: a CTA owns 256 consecutive queries of one head as two 128-row tiles A, B that ping-pong on
// the tensor cores and share the K / V stream; one query row per soft-max thread; P overwrites S in tensor memory and is the A
// operand of P V; O stays in tensor memory and is rescaled only when the running maximum grows by more than 2^8.
// Differences: the key tile is assembled from two tensors, 64 columns at a time (the last chunk of a narrow rotated part is zero-filled by
// the tensor map's bound, which also cancels the query columns beside it); key blocks start at the first key that the CTA's first
// query sees, so tile A starts at block 0 and tile B at block 0 or 1, and only blocks that cross an edge of the window are masked;
// the output gate is applied before the store.
// Every wait is bounded (status word + clean unwind); no load uses cluster multicast.
#include "common.cuh"

namespace ats {

constexpr int WT_THREADS = 320;  // soft-max A (warps 0-3), soft-max B (4-7), TMA (8), MMA (9)

struct WinTcArgs {
  int L, n_old, rows;          // rows = n_old + L context rows per sequence
  int H, dim, dq, vdim, v_col, window;
  const __nv_bfloat16* gate;   // [B * L, ldg] + h * vdim or null
  long long ldg;
  __nv_bfloat16* out;          // [B * L, ldo], head h at h * vdim
  long long ldo;
  float scale_log2;
  int* status;
};

template <int DQC, int DVC>  // 64-column chunks of a query / key row and of a value row
struct WinTcSmem {
  static constexpr int TQ = DQC * 16384, TV = DVC * 16384;
  static constexpr int KST = 2, VST = (DQC == 3 && DVC == 2) ? 1 : 2;
  static constexpr int Q_OFF = 0;
  static constexpr int K_OFF = 2 * TQ;
  static constexpr int V_OFF = K_OFF + KST * TQ;
  static constexpr int BAR_OFF = V_OFF + VST * TV;
  static constexpr int TOTAL = BAR_OFF + 512 + 1024;
};

template <int DQC, int DVC>
__global__ void __launch_bounds__(WT_THREADS, 1)
window_attn_tc_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_r,
                      const __grid_constant__ CUtensorMap map_v, const WinTcArgs p) {
  using SM = WinTcSmem<DQC, DVC>;
  constexpr int KST = SM::KST, VST = SM::VST, DV = DVC * 64;
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
  const int h = blockIdx.x, b = blockIdx.y, q0 = blockIdx.z * 256;
  const int last_row = p.rows - 1;
  // key blocks of 128 rows start at kb0; tile A uses blocks [0, nA), tile B blocks [jB, nB)
  const int kb0 = max(0, p.n_old + q0 - p.window + 1);
  const int nA = (min(p.n_old + q0 + 127, last_row) - kb0) / 128 + 1;
  const bool has_b = q0 + 128 < p.L;
  const int jB = has_b ? (max(0, p.n_old + q0 + 128 - p.window + 1) - kb0) / 128 : 0;
  const int nB = has_b ? (min(p.n_old + q0 + 255, last_row) - kb0) / 128 + 1 : 0;
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
    tma_prefetch_desc(&map_r);
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
      const int own = p.dim >> 6;  // chunks of the head's own key part
      mbar_expect_tx(q_full, (has_b ? 2 : 1) * SM::TQ);
      for (int x = 0; x < (has_b ? 2 : 1); ++x)
#pragma unroll
        for (int c = 0; c < DQC; ++c) tma_load_2d(sQ + x * SM::TQ + c * 16384, &map_q, q_full, h * p.dq + 64 * c, b * p.L + q0 + x * 128);
      for (int j = 0; j < nb; ++j) {
        const int krow = b * p.rows + kb0 + j * 128;
        const int sk = j % KST, sv = j % VST;
        if (!mbar_wait_bounded(&k_empty[sk], ((j / KST) & 1) ^ 1, abort_flag, p.status, kTimeoutEmpty)) break;
        mbar_expect_tx(&k_full[sk], SM::TQ);
#pragma unroll
        for (int c = 0; c < DQC; ++c) {
          uint8_t* dst = sK + sk * SM::TQ + c * 16384;
          if (c < own) tma_load_2d(dst, &map_k, &k_full[sk], h * p.dim + 64 * c, krow);
          else tma_load_2d(dst, &map_r, &k_full[sk], 64 * (c - own), krow);
        }
        if (!mbar_wait_bounded(&v_empty[sv], ((j / VST) & 1) ^ 1, abort_flag, p.status, kTimeoutEmpty)) break;
        mbar_expect_tx(&v_full[sv], SM::TV);
#pragma unroll
        for (int c = 0; c < DVC; ++c) tma_load_2d(sV + sv * SM::TV + c * 16384, &map_v, &v_full[sv], p.v_col + h * p.vdim + 64 * c, krow);
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
        const uint64_t q_d = desc_advance(q_k, uint32_t(x) * SM::TQ), k_d = desc_advance(k_k, uint32_t(j % KST) * SM::TQ);
#pragma unroll
        for (int k = 0; k < DQC * 4; ++k) {
          const uint32_t off = (k >> 2) * 16384 + (k & 3) * 32;
          tc_mma_f16(tmem_base + x * 128, desc_advance(q_d, off), desc_advance(k_d, off), idesc_s, k != 0);
        }
        tc_commit(&s_full[x]);
      };
      auto issue_pv = [&](int x, int j, bool first) {
        const uint64_t v_d = desc_advance(v_mn, uint32_t(j % VST) * SM::TV);  // MN-major: value dimension contiguous
#pragma unroll
        for (int k = 0; k < 8; ++k)
          tc_mma_f16_ts(tmem_base + 256 + x * DV, tmem_base + x * 128 + k * 8, desc_advance(v_d, k * 2048), idesc_o, !(first && k == 0));
      };
      bool ok = mbar_wait_bounded(q_full, 0, abort_flag, p.status, kTimeoutFull);
      ok = ok && mbar_wait_bounded(&k_full[0], 0, abort_flag, p.status, kTimeoutFull);
      if (ok) {
        tc_fence_after();
        issue_s(0, 0);
        if (jB == 0 && nB > 0) issue_s(1, 0);
        tc_commit(&k_empty[0]);
      }
      for (int j = 0; ok && j < nb; ++j) {
        const int nk = (j + 1) % KST;
        const bool a_now = j < nA, a_next = j + 1 < nA, b_now = j >= jB && j < nB, b_next = j + 1 >= jB && j + 1 < nB;
        if (!mbar_wait_bounded(&v_full[j % VST], (j / VST) & 1, abort_flag, p.status, kTimeoutFull)) break;
        if (a_now) {
          if (!mbar_wait_bounded(&p_full[0], j & 1, abort_flag, p.status, kTimeoutTmemFull)) break;
          tc_fence_after();
          issue_pv(0, j, j == 0);
          if (!a_next) tc_commit(&o_done[0]);
        }
        if (j + 1 < nb) {
          if (!mbar_wait_bounded(&k_full[nk], ((j + 1) / KST) & 1, abort_flag, p.status, kTimeoutFull)) break;
          tc_fence_after();
          if (a_next) issue_s(0, j + 1);
        }
        if (b_now) {
          if (!mbar_wait_bounded(&p_full[1], (j - jB) & 1, abort_flag, p.status, kTimeoutTmemFull)) break;
          tc_fence_after();
          issue_pv(1, j, j == jB);
          if (!b_next) tc_commit(&o_done[1]);
        }
        tc_commit(&v_empty[j % VST]);
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
    const int j0 = x ? jB : 0, n = x ? nB - jB : nA;  // no blocks when tile B does not exist
    const int tile_q = p.n_old + q0 + x * 128;        // context row of the tile's first query
    float m = -1e30f, l = 0.f;
    bool ok = true;
    for (int i = 0; i < n; ++i) {
      if (!mbar_wait_bounded(&s_full[x], i & 1, abort_flag, p.status, kTimeoutTmemFull)) {
        ok = false;
        break;
      }
      tc_fence_after();
      uint32_t v[128];
#pragma unroll
      for (int c = 0; c < 4; ++c) tmem_ld_32x32(tmem_S + c * 32, reinterpret_cast<uint32_t(&)[32]>(v[c * 32]));
      tmem_ld_wait();
      const int kb = kb0 + (j0 + i) * 128;
      if (kb + 127 > tile_q || kb < tile_q + 127 - p.window + 1) {  // the block crosses the diagonal or the window's far edge for some row
        const int hi = tile_q + r - kb, lo = hi - p.window + 1;
#pragma unroll
        for (int c = 0; c < 128; ++c)
          if (c > hi || c < lo) v[c] = 0xff800000u;  // -inf
      }
      float mx0 = -INFINITY, mx1 = -INFINITY, mx2 = -INFINITY, mx3 = -INFINITY;
#pragma unroll
      for (int c = 0; c < 128; c += 8) {
        mx0 = fmaxf(mx0, fmaxf(__uint_as_float(v[c]), __uint_as_float(v[c + 1])));
        mx1 = fmaxf(mx1, fmaxf(__uint_as_float(v[c + 2]), __uint_as_float(v[c + 3])));
        mx2 = fmaxf(mx2, fmaxf(__uint_as_float(v[c + 4]), __uint_as_float(v[c + 5])));
        mx3 = fmaxf(mx3, fmaxf(__uint_as_float(v[c + 6]), __uint_as_float(v[c + 7])));
      }
      // a row none of whose keys has come yet keeps m = -1e30: its probabilities are exp2(-inf) = 0
      const float mnew = fmaxf(m, fmaxf(fmaxf(mx0, mx1), fmaxf(mx2, mx3)) * p.scale_log2);
      if (i == 0) {
        m = mnew;
      } else if (__any_sync(0xffffffffu, mnew > m + 8.f)) {
        const float alpha = exp2f(m - mnew);  // the previous P V of this tile has completed: S(i) was computed after it
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
      float2 rsa = make_float2(0.f, 0.f), rsb = make_float2(0.f, 0.f);
      const float2 sc2 = make_float2(p.scale_log2, p.scale_log2), nm2 = make_float2(-m, -m);
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
      l += (rsa.x + rsa.y) + (rsb.x + rsb.y);
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_full[x]);
    }
    if (ok && n > 0 && mbar_wait_bounded(&o_done[x], 0, abort_flag, p.status, kTimeoutTmemFull)) {
      tc_fence_after();
      const int qi = q0 + x * 128 + r;
      const float inv = 1.f / l;
      const long long tok = (long long)b * p.L + qi;
      const bool live = qi < p.L;
      __nv_bfloat16* orow = p.out + tok * p.ldo + (long long)h * DV;
      const __nv_bfloat16* grow = p.gate ? p.gate + tok * p.ldg + (long long)h * DV : nullptr;
#pragma unroll
      for (int c = 0; c < DV / 32; ++c) {
        uint32_t o[32];
        tmem_ld_32x32(tmem_O + c * 32, o);
        tmem_ld_wait();
        if (!live) continue;
#pragma unroll
        for (int g = 0; g < 4; ++g) {
          float f[8];
#pragma unroll
          for (int e = 0; e < 8; ++e) f[e] = __uint_as_float(o[8 * g + e]) * inv;
          if (grow) {
            const uint4 gq = *reinterpret_cast<const uint4*>(grow + c * 32 + g * 8);
            const float2 g0 = unpack_bf16x2(gq.x), g1 = unpack_bf16x2(gq.y), g2 = unpack_bf16x2(gq.z), g3 = unpack_bf16x2(gq.w);
            const float gs[8] = {g0.x, g0.y, g1.x, g1.y, g2.x, g2.y, g3.x, g3.y};
#pragma unroll
            for (int e = 0; e < 8; ++e) f[e] = __fdividef(f[e], 1.f + __expf(-gs[e]));
          }
          *reinterpret_cast<uint4*>(orow + c * 32 + g * 8) =
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

template <int DQC, int DVC>
static int launch_window_tc(const CUtensorMap& mq, const CUtensorMap& mk, const CUtensorMap& mr, const CUtensorMap& mv, const WinTcArgs& p, int B, cudaStream_t s) {
  using SM = WinTcSmem<DQC, DVC>;
  static_assert(SM::TOTAL <= 227 * 1024, "does not fit an SM");
  cudaError_t ce = cudaFuncSetAttribute(window_attn_tc_kernel<DQC, DVC>, cudaFuncAttributeMaxDynamicSharedMemorySize, SM::TOTAL);
  if (ce != cudaSuccess) return int(ce);
  window_attn_tc_kernel<DQC, DVC><<<dim3(p.H, B, (p.L + 255) / 256), WT_THREADS, SM::TOTAL, s>>>(mq, mk, mr, mv, p);
  return int(cudaGetLastError());
}

}  // namespace ats

using namespace ats;

// q [B * L, ldq] (head h at h * (dim + rot), rotated); kv [B * (n_old + L), ldkv] (key of head h at h * dim, value at v_col + h * vdim);
// kr [B * (n_old + L), ldkr] (rot columns from the base pointer).  Returns 1003 for shapes this kernel does not cover.
ATS_API int ats_window_attn_tc(const void* q, long long ldq, const void* kv, long long ldkv, int v_col, const void* kr, long long ldkr, const void* gate,
                               long long ldg, void* out, long long ldo, int B, int L, int n_old, int H, int dim, int rot, int vdim, int window, float scale,
                               int* status, void* stream) {
  const int dqc = dim / 64 + 1;
  if (B < 1 || L < 1 || n_old < 0 || window < 1 || !(scale > 0.f) || (dim & 63) || (dqc != 2 && dqc != 3) || (rot & 7) || rot < 8 || rot > 64 ||
      (vdim != 64 && vdim != 128) || (v_col & 7) || (ldo & 7) || (gate && ((ldg & 7) || (reinterpret_cast<uintptr_t>(gate) & 15))) ||
      (reinterpret_cast<uintptr_t>(out) & 15))
    return 1003;
  static thread_local bool ctx_bound = false;
  if (!ctx_bound) {
    cudaFree(0);
    ctx_bound = true;
  }
  const unsigned long long qrows = (unsigned long long)B * L, krows = (unsigned long long)B * (n_old + L);
  CUtensorMap mq, mk, mr, mv;
  int e;
  if ((e = make_tmap_2d(&mq, q, qrows, (unsigned long long)H * (dim + rot), ldq, 2, 64, 128))) return e;
  if ((e = make_tmap_2d(&mk, kv, krows, (unsigned long long)H * dim, ldkv, 2, 64, 128))) return e;
  if ((e = make_tmap_2d(&mr, kr, krows, rot, ldkr, 2, 64, 128))) return e;
  if ((e = make_tmap_2d(&mv, kv, krows, (unsigned long long)v_col + (unsigned long long)H * vdim, ldkv, 2, 64, 128))) return e;
  WinTcArgs p;
  p.L = L; p.n_old = n_old; p.rows = n_old + L; p.H = H; p.dim = dim; p.dq = dim + rot; p.vdim = vdim; p.v_col = v_col; p.window = window;
  p.gate = static_cast<const __nv_bfloat16*>(gate); p.ldg = ldg; p.out = static_cast<__nv_bfloat16*>(out); p.ldo = ldo;
  p.scale_log2 = scale * 1.4426950408889634f; p.status = status;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dqc == 3) return vdim == 128 ? launch_window_tc<3, 2>(mq, mk, mr, mv, p, B, s) : launch_window_tc<3, 1>(mq, mk, mr, mv, p, B, s);
  return vdim == 128 ? launch_window_tc<2, 2>(mq, mk, mr, mv, p, B, s) : launch_window_tc<2, 1>(mq, mk, mr, mv, p, B, s);
}
