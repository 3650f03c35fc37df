// Lightning attention over a portion of a prompt for sm_100a on tcgen05 tensor cores, 128 tokens at a time.  With S the state before a
// chunk of n tokens and a the head's decay (i, j count inside the chunk)
//
//   o_i = a^(i+1) S^T q_i + sum_{j <= i} a^(i-j) (q_i . k_j) v_j;     S <- a^n S + sum_j a^(n-1-j) k_j v_j^T
//
// A CTA walks the chunks of one (head, 64 value columns, sequence).  q, k and v are bf16 and enter the products exactly; everything else
// that enters a product -- the state, the decayed scores and the decayed values -- goes in as the sum of two bf16 numbers (16 bits of
// mantissa).  The state itself stays in fp32 accumulators in tensor memory from the first chunk to the last.
//
// Per chunk: Q K^T and Q S (first products) | group A (warps 0-3) decays and masks the scores, block of 32 keys by block, while group B (warps
// 4-7) writes the decayed values and decays the read-out | K^T V' as soon as the values are there, then P V | B rewrites the state as the
// next chunk's operand (and leaves it decayed in tensor memory) while P V runs, A stores the outputs.  The next chunk's tiles are
// prefetched into L2 from the start of a chunk.  Two CTAs share an SM, so one's products run under the other's arithmetic.
//
// Tensor memory (256 columns): scores / P 128, read-out 64, state 64 (lanes = state rows).  The P of 32 keys overwrites their scores: 16
// packed columns of high parts, 16 of low parts.  The state operand and the decayed values share one buffer in turn.
// Every wait is bounded (status word + clean unwind); no load uses cluster multicast.
#include "common.cuh"

namespace ats {

constexpr int LC = 128;            // tokens per chunk
constexpr int LC_THREADS = 288;    // group A (warps 0-3), group B (4-7), TMA + MMA (8)

struct LightningTcArgs {
  const float* powers;   // [H, LC + 1] a^n
  float* state;          // [B, H, dim, vdim] fp32
  long long state_bs;
  __nv_bfloat16* o;      // [B * L, ldo], head h at h * vdim
  long long ldo;
  int L, H, dim, vdim, fresh;
  int* status;
};

constexpr int LS_Q = 0, LS_K = 32768, LS_V = 65536, LS_S = 81920;  // Q, K: two 64-column pieces of 128 rows; V, S hi, S lo: one
constexpr int LS_AUX = 114688;                                     // powers, barriers
constexpr int LS_TOTAL = LS_AUX + 1024;

__device__ __forceinline__ void prefetch_3d(const CUtensorMap* map, int c0, int c1, int c2) {  // into L2
  asm volatile("cp.async.bulk.prefetch.tensor.3d.L2.global [%0, {%1, %2, %3}];" ::"l"(reinterpret_cast<uint64_t>(map)), "r"(c0), "r"(c1), "r"(c2) : "memory");
}
// Two values as bf16 pairs hi + lo.
__device__ __forceinline__ void split_bf16x2(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(a, b);
  const float2 r = unpack_bf16x2(hi);
  lo = pack_bf16x2(a - r.x, b - r.y);
}

__global__ void __launch_bounds__(LC_THREADS, 2)
lightning_tc_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_v,
                    const LightningTcArgs p) {
  extern __shared__ __align__(1024) uint8_t smem[];
  uint8_t* sQ = smem + LS_Q;
  uint8_t* sK = smem + LS_K;
  uint8_t* sV = smem + LS_V;
  uint8_t* sS = smem + LS_S;
  float* s_pow = reinterpret_cast<float*>(smem + LS_AUX);   // [LC + 1]
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + LS_AUX + 768);
  uint64_t* in_full = bars;       // Q, K, V of a chunk
  uint64_t* s_done = bars + 1;    // scores
  uint64_t* r_done = bars + 2;    // read-out of the state
  uint64_t* v_ready = bars + 3;   // 4 arrivals: decayed values
  uint64_t* p_ready = bars + 4;   // 8 arrivals: P, decayed read-out
  uint64_t* u_done = bars + 5;    // K^T V'
  uint64_t* o_done = bars + 6;    // P V (and everything before it)
  uint64_t* s_ready = bars + 7;   // 8 arrivals: state operand written, state decayed, outputs taken
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 8);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int v0 = blockIdx.x * 64, h = blockIdx.y, b = blockIdx.z;
  const int chunks = (p.L + LC - 1) / LC;
  if (smem_u32(smem) & 1023) {  // the swizzled tiles need it
    if (threadIdx.x == 0) atomicCAS(p.status, 0, kBadArgument);
    return;
  }
  if (threadIdx.x == 0) {
    mbar_init(in_full, 1);
    mbar_init(s_done, 1);
    mbar_init(r_done, 1);
    mbar_init(v_ready, 4);
    mbar_init(p_ready, 8);
    mbar_init(o_done, 1);
    mbar_init(u_done, 1);
    mbar_init(s_ready, 8);
    *abort_flag = 0;
    mbar_fence_init();
    tma_prefetch_desc(&map_q);
    tma_prefetch_desc(&map_k);
    tma_prefetch_desc(&map_v);
  }
  for (int i = threadIdx.x; i <= LC; i += LC_THREADS) s_pow[i] = p.powers[(long long)h * (LC + 1) + i];
  if (warp == 8) {
    tmem_alloc(tmem_slot, 256);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  const uint32_t t_scores = tmem, t_out = tmem + 128, t_state = tmem + 192;

  if (warp == 8) {
    if (lane == 0) {
      // ------------------------------------------------------------------ loads and products
      const uint32_t id_s = make_idesc(128, 128, 1, 1, 0, 0);   // Q K^T: both K-major
      const uint32_t id_r = make_idesc(128, 64, 1, 1, 0, 1);    // Q S, P V: B contiguous along the value columns
      const uint32_t id_u = make_idesc(128, 64, 1, 1, 1, 1);    // K^T V': A contiguous along the state rows
      const uint64_t q_k = make_smem_desc_sw128(smem_u32(sQ), 16, 1024), k_k = make_smem_desc_sw128(smem_u32(sK), 16, 1024);
      const uint64_t k_mn = make_smem_desc_sw128(smem_u32(sK), 16384, 1024), v_mn = make_smem_desc_sw128(smem_u32(sV), 16384, 1024);
      const uint64_t s_mn = make_smem_desc_sw128(smem_u32(sS), 16384, 1024);
      auto load_q = [&](int c) {
        const int row = b * p.L + c * LC;
        tma_load_3d(sQ, &map_q, in_full, 0, h, row);
        tma_load_3d(sQ + 16384, &map_q, in_full, 64, h, row);
      };
      auto load_kv = [&](int c) {
        const int row = b * p.L + c * LC;
        tma_load_3d(sK, &map_k, in_full, 0, h, row);
        tma_load_3d(sK + 16384, &map_k, in_full, 64, h, row);
        tma_load_3d(sV, &map_v, in_full, v0, h, row);
      };
      mbar_expect_tx(in_full, 81920);
      load_q(0);
      load_kv(0);
      for (int c = 0; c < chunks; ++c) {
        if (!mbar_wait_bounded(in_full, c & 1, abort_flag, p.status, kTimeoutFull)) break;
        const bool more = c + 1 < chunks;
        if (more) {
          const int row = b * p.L + (c + 1) * LC;
          prefetch_3d(&map_q, 0, h, row);
          prefetch_3d(&map_q, 64, h, row);
          prefetch_3d(&map_k, 0, h, row);
          prefetch_3d(&map_k, 64, h, row);
          prefetch_3d(&map_v, v0, h, row);
        }
        if (!mbar_wait_bounded(s_ready, c & 1, abort_flag, p.status, kTimeoutTmemEmpty)) break;
        tc_fence_after();
#pragma unroll
        for (int k = 0; k < 8; ++k) {
          const uint32_t off = (k >> 2) * 16384 + (k & 3) * 32;
          tc_mma_f16(t_scores, desc_advance(q_k, off), desc_advance(k_k, off), id_s, k != 0);
        }
        tc_commit(s_done);
#pragma unroll
        for (int part = 0; part < 2; ++part)
#pragma unroll
          for (int k = 0; k < 8; ++k)
            tc_mma_f16(t_out, desc_advance(q_k, (k >> 2) * 16384 + (k & 3) * 32), desc_advance(s_mn, part * 16384 + k * 2048), id_r, part | k);
        tc_commit(r_done);
        if (!mbar_wait_bounded(v_ready, c & 1, abort_flag, p.status, kTimeoutTmemFull)) break;
        tc_fence_after();
        if (more) {  // the products that read Q have completed: group B waited for them
          mbar_expect_tx(in_full, 81920);
          load_q(c + 1);
        }
#pragma unroll
        for (int part = 0; part < 2; ++part)
#pragma unroll
          for (int k = 0; k < 8; ++k) tc_mma_f16(t_state, desc_advance(k_mn, k * 2048), desc_advance(s_mn, part * 16384 + k * 2048), id_u, 1);
        tc_commit(u_done);
        if (!mbar_wait_bounded(p_ready, c & 1, abort_flag, p.status, kTimeoutTmemFull)) break;
        tc_fence_after();
#pragma unroll
        for (int part = 0; part < 2; ++part)
#pragma unroll
          for (int k = 0; k < 8; ++k) tc_mma_f16_ts(t_out, t_scores + (k >> 1) * 32 + part * 16 + (k & 1) * 8, desc_advance(v_mn, k * 2048), id_r, 1);
        tc_commit(o_done);
        if (more) {
          if (!mbar_wait_bounded(o_done, c & 1, abort_flag, p.status, kTimeoutTmemFull)) break;
          load_kv(c + 1);
        }
      }
      if (*abort_flag) {  // give copies already in flight time to land before the CTA exits
        const uint64_t t0 = globaltimer_ns();
        while (globaltimer_ns() - t0 < 20000ull) {
        }
      }
    }
  } else {
    const int r = (warp & 3) * 32 + lane;                         // TMEM lane: token of the chunk, or state row
    const uint32_t lane_base = uint32_t((warp & 3) * 32) << 16;
    const uint32_t swz = uint32_t(r & 7) << 4;
    uint8_t* my_hi = sS + r * 128;                                // this row of the operand buffer, and of its low parts
    uint8_t* my_lo = my_hi + 16384;
    float* st = p.state + (long long)b * p.state_bs + (long long)h * p.dim * p.vdim + (long long)r * p.vdim + v0;
    const int cols = min(64, p.vdim - v0);                        // a multiple of 8
    // 16 values of this row (columns 16 q ..) -> operand buffer
    auto put16 = [&](int q, const float (&f)[16]) {
      uint32_t hi[8], lo[8];
#pragma unroll
      for (int e = 0; e < 8; ++e) split_bf16x2(f[2 * e], f[2 * e + 1], hi[e], lo[e]);
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        const uint32_t at = (uint32_t(2 * q + u) << 4) ^ swz;
        *reinterpret_cast<uint4*>(my_hi + at) = make_uint4(hi[4 * u], hi[4 * u + 1], hi[4 * u + 2], hi[4 * u + 3]);
        *reinterpret_cast<uint4*>(my_lo + at) = make_uint4(lo[4 * u], lo[4 * u + 1], lo[4 * u + 2], lo[4 * u + 3]);
      }
    };
    if (warp >= 4) {  // the state before the portion
#pragma unroll 1
      for (int q = 0; q < 4; ++q) {
        float f[16];
#pragma unroll
        for (int e = 0; e < 16; e += 4) {
          const float4 t = (!p.fresh && r < p.dim && 16 * q + e < cols) ? *reinterpret_cast<const float4*>(st + 16 * q + e) : make_float4(0.f, 0.f, 0.f, 0.f);
          f[e] = t.x; f[e + 1] = t.y; f[e + 2] = t.z; f[e + 3] = t.w;
        }
        put16(q, f);
        const float fs = s_pow[min(LC, p.L)];
#pragma unroll
        for (int e = 0; e < 16; ++e) f[e] *= fs;
        tmem_st_32x16(t_state + lane_base + 16 * q, reinterpret_cast<uint32_t(&)[16]>(f));
      }
      tmem_st_wait();
      tc_fence_before();
      fence_proxy_async_smem();
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(s_ready);
    bool ok = true;
    for (int c = 0; ok && c < chunks; ++c) {
      const int n = min(LC, p.L - c * LC);
      if (warp < 4) {
        // ---------------------------------------------------------------- group A: P = decayed, masked scores
        if (!mbar_wait_bounded(s_done, c & 1, abort_flag, p.status, kTimeoutTmemFull)) break;
        tc_fence_after();
#pragma unroll 1
        for (int k = 0; k < 4; ++k) {   // 32 keys
          const uint32_t at = t_scores + lane_base + 32 * k;
          uint32_t pk[32];              // 16 high, 16 low
          if (k > warp) {  // all keys after all of this warp's queries
#pragma unroll
            for (int e = 0; e < 32; ++e) pk[e] = 0u;
          } else {
            uint32_t s[32];
            tmem_ld_32x32(at, s);
            tmem_ld_wait();
            if (k < warp) {
              const float f = s_pow[r - 32 * k - 31];
#pragma unroll
              for (int e = 0; e < 16; ++e)
                split_bf16x2(__uint_as_float(s[2 * e]) * (f * s_pow[31 - 2 * e]), __uint_as_float(s[2 * e + 1]) * (f * s_pow[30 - 2 * e]), pk[e], pk[16 + e]);
            } else {
#pragma unroll
              for (int e = 0; e < 16; ++e)
                split_bf16x2(2 * e <= lane ? __uint_as_float(s[2 * e]) * s_pow[max(lane - 2 * e, 0)] : 0.f,
                             2 * e + 1 <= lane ? __uint_as_float(s[2 * e + 1]) * s_pow[max(lane - 2 * e - 1, 0)] : 0.f, pk[e], pk[16 + e]);
            }
          }
          tmem_st_32x32(at, pk);
        }
        tmem_st_wait();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(p_ready);
        // ---------------------------------------------------------------- outputs
        if (!mbar_wait_bounded(o_done, c & 1, abort_flag, p.status, kTimeoutTmemFull)) break;
        tc_fence_after();
        __nv_bfloat16* orow = p.o + ((long long)b * p.L + c * LC + r) * p.ldo + (long long)h * p.vdim + v0;
        uint32_t f[64];
        tmem_ld_32x32(t_out + lane_base, reinterpret_cast<uint32_t(&)[32]>(f[0]));
        tmem_ld_32x32(t_out + lane_base + 32, reinterpret_cast<uint32_t(&)[32]>(f[32]));
        tmem_ld_wait();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(s_ready);
        if (r < n) {
#pragma unroll
          for (int e = 0; e < 64; e += 8)
            if (e < cols)
              *reinterpret_cast<uint4*>(orow + e) =
                  make_uint4(pack_bf16x2(__uint_as_float(f[e]), __uint_as_float(f[e + 1])), pack_bf16x2(__uint_as_float(f[e + 2]), __uint_as_float(f[e + 3])),
                             pack_bf16x2(__uint_as_float(f[e + 4]), __uint_as_float(f[e + 5])), pack_bf16x2(__uint_as_float(f[e + 6]), __uint_as_float(f[e + 7])));
        }
      } else {
        // ---------------------------------------------------------------- group B: values
        if (!mbar_wait_bounded(in_full, c & 1, abort_flag, p.status, kTimeoutFull)) break;
        const float fo = s_pow[r + 1], fv = r < n ? s_pow[n - 1 - r] : 0.f;
        const uint8_t* vrow = sV + r * 128;
        {
          uint32_t hi[32], lo[32];
#pragma unroll
          for (int u = 0; u < 8; ++u) {
            const uint4 w = *reinterpret_cast<const uint4*>(vrow + ((uint32_t(u) << 4) ^ swz));
            const uint32_t x[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const float2 t = unpack_bf16x2(x[e]);
              split_bf16x2(r < n ? t.x * fv : 0.f, r < n ? t.y * fv : 0.f, hi[4 * u + e], lo[4 * u + e]);
            }
          }
          // the buffer is free once the read-out of the state is done
          if (!mbar_wait_bounded(r_done, c & 1, abort_flag, p.status, kTimeoutTmemFull)) break;
#pragma unroll
          for (int u = 0; u < 8; ++u) {
            const uint32_t at = (uint32_t(u) << 4) ^ swz;
            *reinterpret_cast<uint4*>(my_hi + at) = make_uint4(hi[4 * u], hi[4 * u + 1], hi[4 * u + 2], hi[4 * u + 3]);
            *reinterpret_cast<uint4*>(my_lo + at) = make_uint4(lo[4 * u], lo[4 * u + 1], lo[4 * u + 2], lo[4 * u + 3]);
          }
          fence_proxy_async_smem();
          __syncwarp();
          if (lane == 0) mbar_arrive(v_ready);
        }
        // ---------------------------------------------------------------- read-out
        tc_fence_after();
        {
          uint32_t x[64];
          tmem_ld_32x32(t_out + lane_base, reinterpret_cast<uint32_t(&)[32]>(x[0]));
          tmem_ld_32x32(t_out + lane_base + 32, reinterpret_cast<uint32_t(&)[32]>(x[32]));
          tmem_ld_wait();
#pragma unroll
          for (int e = 0; e < 64; ++e) x[e] = __float_as_uint(__uint_as_float(x[e]) * fo);
          tmem_st_32x32(t_out + lane_base, reinterpret_cast<uint32_t(&)[32]>(x[0]));
          tmem_st_32x32(t_out + lane_base + 32, reinterpret_cast<uint32_t(&)[32]>(x[32]));
          tmem_st_wait();
        }
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(p_ready);
        // ---------------------------------------------------------------- the state as the next chunk's operand
        if (!mbar_wait_bounded(u_done, c & 1, abort_flag, p.status, kTimeoutTmemFull)) break;
        tc_fence_after();
        const bool end = c + 1 == chunks;
        const float fs = end ? 1.f : s_pow[min(LC, p.L - (c + 1) * LC)];
#pragma unroll
        for (int q = 0; q < 2; ++q) {
          uint32_t x[32];
          tmem_ld_32x32(t_state + lane_base + 32 * q, x);
          tmem_ld_wait();
          if (!end) {
#pragma unroll
            for (int u = 0; u < 2; ++u) put16(2 * q + u, reinterpret_cast<float(&)[16]>(x[16 * u]));
#pragma unroll
            for (int e = 0; e < 32; ++e) x[e] = __float_as_uint(__uint_as_float(x[e]) * fs);
            tmem_st_32x32(t_state + lane_base + 32 * q, x);
          } else if (r < p.dim) {
#pragma unroll
            for (int e = 0; e < 32; e += 4)
              if (32 * q + e < cols)
                *reinterpret_cast<float4*>(st + 32 * q + e) =
                    make_float4(__uint_as_float(x[e]), __uint_as_float(x[e + 1]), __uint_as_float(x[e + 2]), __uint_as_float(x[e + 3]));
          }
        }
        tmem_st_wait();
        tc_fence_before();
        fence_proxy_async_smem();
        __syncwarp();
        if (lane == 0) mbar_arrive(s_ready);
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 8) {
    tc_fence_after();
    tmem_dealloc(tmem, 256);
  }
}

}  // namespace ats

using namespace ats;

// qkv [B * L, ld] bf16, activated, head h at q_col + h * dim, k_col + h * dim, v_col + h * vdim; powers [H, 129] fp32 (decay^n); state
// [B, H, dim, vdim] fp32, updated in place; o [B * L, ldo].  Returns 1003 for shapes this kernel does not cover.
ATS_API int ats_lightning_tc(const void* qkv, long long ld, int q_col, int k_col, int v_col, const float* powers, float* state, long long state_bs, void* o,
                             long long ldo, int B, int L, int H, int dim, int vdim, int fresh, int* status, void* stream) {
  if (B < 1 || L < 1 || H < 1 || (dim & 7) || dim < 8 || dim > 128 || (vdim & 7) || vdim < 8 || ((q_col | k_col | v_col) & 7) || (ldo & 7) ||
      (state_bs & 3) || ((reinterpret_cast<uintptr_t>(state) | reinterpret_cast<uintptr_t>(o)) & 15) || !status)
    return 1003;
  static thread_local bool ctx_bound = false;
  if (!ctx_bound) {
    cudaFree(0);
    ctx_bound = true;
  }
  const __nv_bfloat16* base = static_cast<const __nv_bfloat16*>(qkv);
  CUtensorMap mq, mk, mv;
  int e;
  if ((e = make_tmap_heads(&mq, base + q_col, (uint64_t)B * L, H, dim, ld))) return e;
  if ((e = make_tmap_heads(&mk, base + k_col, (uint64_t)B * L, H, dim, ld))) return e;
  if ((e = make_tmap_heads(&mv, base + v_col, (uint64_t)B * L, H, vdim, ld))) return e;
  LightningTcArgs p;
  p.powers = powers; p.state = state; p.state_bs = state_bs; p.o = static_cast<__nv_bfloat16*>(o); p.ldo = ldo;
  p.L = L; p.H = H; p.dim = dim; p.vdim = vdim; p.fresh = fresh; p.status = status;
  cudaError_t ce = cudaFuncSetAttribute(lightning_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, LS_TOTAL);
  if (ce != cudaSuccess) return int(ce);
  lightning_tc_kernel<<<dim3((vdim + 63) / 64, H, B), LC_THREADS, LS_TOTAL, static_cast<cudaStream_t>(stream)>>>(mq, mk, mv, p);
  return int(cudaGetLastError());
}
