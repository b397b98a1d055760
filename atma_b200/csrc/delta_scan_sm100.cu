// The gated delta rule over packed prompt rows on the 5th-generation tensor cores (sm_100a), 64 rows a chunk, at fp32
// accuracy: whatever stands between the 16-bit q, k, v and the fp32 state enters the 16-bit products as two terms
// (rounded value and remainder), and everything that is a scalar per row - unit-norm factors, decays, step sizes - is
// applied to fp32 accumulators instead of to 16-bit operands.
//
// With S the state before a chunk, a_s the inclusive decay prefix inside it, k^ = k k_inv, q^ = q q_inv:
//
//   R_s = v_s - a_s k_inv_s (S^T k_s)                                 residual against the old state
//   U   = M1 R,          M1 = (I + A)^-1 diag(beta),  A[p][s] = beta_p (a_p / a_s) k^_p.k^_s   (s < p)
//   O_p = a_p q_inv_p (S^T q_p) + (M2 R)_p,   M2 = Rq M1,  Rq[p][s] = (a_p / a_s) q^_p.k^_s    (s <= p)
//   S'  = a_C S + sum_s (a_C / a_s) k_inv_s k_s u_s^T
//
// factors (delta_factors_kernel): M1, M2 and the row scalars of every chunk and head, side by side.  A persistent CTA
//   takes two chunks of a head as one 128-row tile: Gram matrices K K^T and Q K^T by tcgen05.mma (exact products of the
//   16-bit rows), A and Rq in fp32, the inverse by 16 x 16 blocks - substitution on the diagonal, mma.sync tf32 with
//   split operands below it - and M2 the same way.  Two CTAs share an SM, so one's serial chain runs under the other's.
// recurrence (delta_recur_kernel): one CTA per (sequence, head, 128 value channels) holds S^T in fp32 registers and walks
//   the chunks.  v is on the 128 TMEM lanes of every accumulator; the A operands S^T, R^T, U^T sit in TMEM as two 16-bit
//   terms, the B operands are the K and Q rows exactly as TMA delivers them and M1, M2 as two terms.  Issue order per
//   chunk: P = S^T K^T | first half of S^T Q^T | U^T = R^T M1^T | second half of S^T Q^T | dS^T = U^T K | R^T M2^T, so that
//   the products the next step does not wait for run under the thread phases.
//     warp 0 TMA producer (two stages), warp 1 MMA issuer, warps 2-17 state warps (TMEM lanes 32 (warp % 4) .. + 31, column
//     quarter (warp - 2) / 4); what a thread phase reads from shared memory is fetched while the product before it runs.
//     TMEM: S hi/lo [0,128) | P, U [128,192) | dS [192,320) | R hi/lo [320,384) | U hi/lo, then R M2 [384,448) | S Q [448,512)
// Every mbarrier wait is bounded; on expiry a CTA frees its TMEM, returns and leaves a status word for the host.
#include "delta_rule.cuh"
#include "sm100.cuh"

namespace atma {

using namespace sm100;

namespace {

__device__ int g_delta_status = 0;

constexpr int kC = 64, kD = 128;
constexpr int kRecBytes = 4 * kC * kC * 2;          // M1 hi, M2 hi, M1 lo, M2 lo: [64 p][64 s] 16-bit each
constexpr int kScal = 256;                          // floats per record: a k_inv [64] | a q_inv [64] | (a_C/a) k_inv [64] | a_C
constexpr int kThreads = 320;

struct Params {
  const float *q_inv, *k_inv, *log_decay, *beta;
  const int32_t *cu_rows, *start_pos, *cu_chunks;
  const int64_t* slots;
  uint8_t* recs; float* scal;
  float* state; int64_t state_ss;
  void* o;
  int n_seqs, NC, H, G, vdim;
};

__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
  __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&h);
}
// two fp32 values as a pair of rounded 16-bit values and the pair of their remainders
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16(x, y);
  lo = pack_bf16(x - __uint_as_float(hi << 16), y - __uint_as_float(hi & 0xffff0000u));
}
__device__ __forceinline__ void bulk_load(void* smem_dst, const void* src, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
               ::"r"(smem_u32(smem_dst)), "l"(reinterpret_cast<uint64_t>(src)), "r"(bytes), "r"(smem_u32(bar)) : "memory");
}
__device__ __forceinline__ void worker_sync() { asm volatile("bar.sync 1, 256;" ::: "memory"); }

// ---- chunk offsets of the sequences ------------------------------------------------------------------------------------
__global__ void chunk_offsets_kernel(const int32_t* __restrict__ cu_rows, const int32_t* __restrict__ start_pos, int n_seqs,
                                     int32_t* __restrict__ cu_chunks) {
  if (threadIdx.x == 0) {
    int at = 0;
    cu_chunks[0] = 0;
    for (int s = 0; s < n_seqs; ++s) {
      if (start_pos[s] >= 0) at += (cu_rows[s + 1] - cu_rows[s] + kC - 1) / kC;
      cu_chunks[s + 1] = at;
    }
  }
}

// ======================================= factors =========================================================================
constexpr int kLd = 68;                              // fp32 row stride of A, T and Rq
constexpr int kMat = 128 * kLd * 4;
constexpr int kOffQ = 32768, kOffT = 0, kOffR = kMat, kOffA = 2 * kMat, kFactorSmem = 3 * kMat + 1024;   // T and Rq over the K, Q tiles

struct FactorBarriers { uint64_t kq_full, g_done, tile_free; };
struct Meta { int64_t t0[2]; int rows[2]; int64_t rec[2]; int h, g; };

__device__ __forceinline__ void tile_meta(const Params& p, int64_t tile, Meta& m) {
  m.h = (int)(tile % p.H);
  m.g = m.h / (p.H / p.G);
  const int j = (int)(tile / p.H);
  const int total = p.cu_chunks[p.n_seqs];
#pragma unroll
  for (int ci = 0; ci < 2; ++ci) {
    const int c = 2 * j + ci;
    m.t0[ci] = 0; m.rows[ci] = 0; m.rec[ci] = -1;
    if (c < total) {
      int lo = 0, hi = p.n_seqs;                     // largest s with cu_chunks[s] <= c
      while (hi - lo > 1) {
        const int mid = (lo + hi) >> 1;
        if (p.cu_chunks[mid] <= c) lo = mid; else hi = mid;
      }
      m.t0[ci] = (int64_t)p.cu_rows[lo] + (int64_t)(c - p.cu_chunks[lo]) * kC;
      m.rows[ci] = (int)min((int64_t)kC, (int64_t)p.cu_rows[lo + 1] - m.t0[ci]);
      m.rec[ci] = (int64_t)m.h * p.NC + c;
    }
  }
}

__device__ __forceinline__ void mma_tf32(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void split_tf32(float x, uint32_t& hi, uint32_t& lo) {
  hi = __float_as_uint(x) & 0xffffe000u;
  lo = __float_as_uint(x - __uint_as_float(hi));
}
// acc (16 x 16 as two 8-column tiles) += A (16 x 16) * B (16 x 16), both row-major with stride kLd, operands split in two
__device__ __forceinline__ void block_mma(float (&acc)[2][4], const float* A, const float* B, int lane) {
  const int g = lane >> 2, t = lane & 3;
#pragma unroll
  for (int ks = 0; ks < 2; ++ks) {
    uint32_t ah[4], al[4];
    split_tf32(A[g * kLd + 8 * ks + t], ah[0], al[0]);
    split_tf32(A[(g + 8) * kLd + 8 * ks + t], ah[1], al[1]);
    split_tf32(A[g * kLd + 8 * ks + t + 4], ah[2], al[2]);
    split_tf32(A[(g + 8) * kLd + 8 * ks + t + 4], ah[3], al[3]);
#pragma unroll
    for (int nt = 0; nt < 2; ++nt) {
      uint32_t bh[2], bl[2];
      split_tf32(B[(8 * ks + t) * kLd + 8 * nt + g], bh[0], bl[0]);
      split_tf32(B[(8 * ks + t + 4) * kLd + 8 * nt + g], bh[1], bl[1]);
      mma_tf32(acc[nt], al, bh[0], bh[1]);
      mma_tf32(acc[nt], ah, bl[0], bl[1]);
      mma_tf32(acc[nt], ah, bh[0], bh[1]);
    }
  }
}
__device__ __forceinline__ void block_store(float* C, const float (&acc)[2][4], int lane, float sign) {
  const int g = lane >> 2, t = lane & 3;
#pragma unroll
  for (int nt = 0; nt < 2; ++nt) {
    *reinterpret_cast<float2*>(C + g * kLd + 8 * nt + 2 * t) = make_float2(sign * acc[nt][0], sign * acc[nt][1]);
    *reinterpret_cast<float2*>(C + (g + 8) * kLd + 8 * nt + 2 * t) = make_float2(sign * acc[nt][2], sign * acc[nt][3]);
  }
}

__global__ void __launch_bounds__(kThreads, 2)
delta_factors_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_k, const Params p) {
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* Ks = smem;
  uint8_t* Qs = smem + kOffQ;
  float* Tf = reinterpret_cast<float*>(smem + kOffT);
  float* Rf = reinterpret_cast<float*>(smem + kOffR);
  float* Af = reinterpret_cast<float*>(smem + kOffA);
  __shared__ FactorBarriers bar;
  __shared__ uint32_t s_tmem_base;
  __shared__ int s_abort;
  __shared__ float s_lg[128], s_bt[128], s_kinv[128], s_wsum[4];

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  if (tid == 0) {
    mbar_init(&bar.kq_full, 1); mbar_init(&bar.g_done, 1); mbar_init(&bar.tile_free, 8);
    s_abort = 0;
    fence_barrier_init();
  }
  if (warp == 1) tmem_alloc(&s_tmem_base, 256);
  if (warp == 0 && lane == 0) { prefetch_tensormap(&tmap_q); prefetch_tensormap(&tmap_k); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tbase = s_tmem_base;
  volatile int* abort_flag = &s_abort;
  const int64_t n_tiles = (int64_t)((p.cu_chunks[p.n_seqs] + 1) / 2) * p.H;

  if (warp == 0) {
    // ---- TMA producer ------------------------------------------------------------------------------------------
    if (lane == 0) {
      uint32_t it = 0;
      for (int64_t tile = blockIdx.x; tile < n_tiles; tile += gridDim.x, ++it) {
        if (it > 0 && !mbar_wait(&bar.tile_free, (it - 1) & 1u, abort_flag)) break;
        Meta m;
        tile_meta(p, tile, m);
        mbar_arrive_expect_tx(&bar.kq_full, 4 * 16384);
#pragma unroll
        for (int ci = 0; ci < 2; ++ci)
#pragma unroll
          for (int cb = 0; cb < 2; ++cb) {
            const int t0 = (int)(ci ? m.t0[1] : m.t0[0]);
            tma_load_4d(Ks + cb * 16384 + ci * 8192, &tmap_k, &bar.kq_full, cb * 64, m.g, t0, 0);
            tma_load_4d(Qs + cb * 16384 + ci * 8192, &tmap_q, &bar.kq_full, cb * 64, m.g, t0, 0);
          }
      }
    }
    __syncwarp();
  } else if (warp == 1) {
    // ---- MMA issuer --------------------------------------------------------------------------------------------
    if (lane == 0) {
      constexpr uint32_t idesc = make_idesc(128, 128, 1, 0, 0);
      const uint64_t hi_k = (uint64_t(1024 >> 4) << 32) | (uint64_t(1) << 46) | (uint64_t(2) << 61) | (uint64_t(16 >> 4) << 16);
      const uint64_t kd = hi_k | uint64_t((smem_u32(Ks) >> 4) & 0x3FFFu), qd = hi_k | uint64_t((smem_u32(Qs) >> 4) & 0x3FFFu);
      uint32_t it = 0;
      for (int64_t tile = blockIdx.x; tile < n_tiles; tile += gridDim.x, ++it) {
        if (!mbar_wait(&bar.kq_full, it & 1u, abort_flag)) break;
        tc_fence_after();
#pragma unroll
        for (int kk = 0; kk < 8; ++kk) {
          const uint64_t off = uint64_t(((kk >> 2) * 16384 + (kk & 3) * 32) >> 4);
          mma_ss(tbase, kd + off, kd + off, idesc, kk > 0);
        }
#pragma unroll
        for (int kk = 0; kk < 8; ++kk) {
          const uint64_t off = uint64_t(((kk >> 2) * 16384 + (kk & 3) * 32) >> 4);
          mma_ss(tbase + 128, qd + off, kd + off, idesc, kk > 0);
        }
        tc_commit(&bar.g_done);
      }
    }
    __syncwarp();
  } else {
    // ---- workers -----------------------------------------------------------------------------------------------
    const int wtid = tid - 64, w = warp - 2;
    const int quad = warp & 3, half = w >> 2;
    const int row = 32 * quad + lane;                  // tile row (and TMEM lane)
    const int ci = row >> 6, pr = row & 63;            // chunk of the tile, row inside the chunk
    const uint32_t lane_base = tbase + (uint32_t(32 * quad) << 16);
    uint32_t it = 0;
    for (int64_t tile = blockIdx.x; tile < n_tiles; tile += gridDim.x, ++it) {
      Meta m;
      tile_meta(p, tile, m);
      const bool valid = pr < (ci ? m.rows[1] : m.rows[0]);
      const int64_t rec = ci ? m.rec[1] : m.rec[0];
      const int64_t t = (ci ? m.t0[1] : m.t0[0]) + pr;
      const float bt_p = valid ? p.beta[t * p.H + m.h] : 0.f;
      const float kinv_p = valid ? p.k_inv[t * p.G + m.g] : 0.f;
      const float qinv_p = valid ? p.q_inv[t * p.G + m.g] : 0.f;
      float run = valid ? p.log_decay[t * p.H + m.h] : 0.f;
      // decay prefix over the chunk's 64 rows (two warps)
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float up = __shfl_up_sync(0xffffffffu, run, o);
        if (lane >= o) run += up;
      }
      worker_sync();                                   // every warp is done with the previous tile's arrays
      if (half == 0 && lane == 31) s_wsum[quad] = run;
      worker_sync();
      if (quad & 1) run += s_wsum[quad - 1];
      if (half == 0) { s_lg[row] = run; s_bt[row] = bt_p; s_kinv[row] = kinv_p; }
      worker_sync();
      const float lg_p = run, lg_C = s_lg[64 * ci + 63];
      if (half == 0 && rec >= 0) {
        float* sc = p.scal + rec * kScal;
        sc[pr] = expf(lg_p) * kinv_p;
        sc[64 + pr] = expf(lg_p) * qinv_p;
        sc[128 + pr] = expf(lg_C - lg_p) * kinv_p;
        if (pr == kC - 1) sc[192] = expf(lg_C);
      }
      // ---- A and Rq from the Gram matrices ----
      mbar_wait(&bar.g_done, it & 1u, abort_flag);      // after a timeout every later wait returns at once
      __syncwarp();
      tc_fence_after();
      if (half == 1 && (quad & 1) == 0) {               // rows 0-31 see no column of the second half
#pragma unroll
        for (int j = 0; j < 32; j += 4) {
          *reinterpret_cast<float4*>(Af + row * kLd + 32 + j) = make_float4(0.f, 0.f, 0.f, 0.f);
          *reinterpret_cast<float4*>(Rf + row * kLd + 32 + j) = make_float4(0.f, 0.f, 0.f, 0.f);
        }
      } else {
#pragma unroll 1
        for (int which = 0; which < 2; ++which) {
          uint32_t gm[32];
          tmem_ld32(lane_base + 128 * which + 64 * ci + 32 * half, gm);
          float* dst = (which ? Rf : Af) + row * kLd + 32 * half;
          const float f = which ? qinv_p : bt_p * kinv_p;
#pragma unroll
          for (int j = 0; j < 32; j += 4) {
            float x[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const int s = 32 * half + j + e;
              const bool seen = which ? s <= pr : s < pr;
              x[e] = seen ? f * (__expf(lg_p - s_lg[64 * ci + s]) * s_kinv[64 * ci + s]) * __uint_as_float(gm[j + e]) : 0.f;
            }
            *reinterpret_cast<float4*>(dst + j) = make_float4(x[0], x[1], x[2], x[3]);
          }
        }
      }
      tc_fence_before();
      worker_sync();
      // ---- T = (I + A)^-1: diagonal 16 x 16 blocks by substitution ----
      if (wtid < 128) {
        const int cc = wtid >> 6, blk = (wtid >> 4) & 3, j = wtid & 15;
        const float* Ab = Af + (64 * cc + 16 * blk) * kLd + 16 * blk;
        float* Tb = Tf + (64 * cc + 16 * blk) * kLd + 16 * blk;
        float x[16];
#pragma unroll
        for (int r = 0; r < 16; ++r) {
          float acc = (r == j) ? 1.f : 0.f;
#pragma unroll
          for (int s = 0; s < r; ++s) acc = fmaf(-Ab[r * kLd + s], x[s], acc);
          x[r] = acc;
          Tb[r * kLd + j] = acc;
        }
      }
      worker_sync();
      // G_il = -T_ii A_il below the diagonal (in place over A_il), then T_ij = sum_l G_il T_lj level by level
      for (int blk = w; blk < 12; blk += 8) {
        const int cc = blk / 6, e = blk % 6;
        const int bi = (e == 0) ? 1 : (e < 3 ? 2 : 3), bl = (e == 0) ? 0 : (e < 3 ? e - 1 : e - 3);
        float acc[2][4] = {};
        float* Ail = Af + (64 * cc + 16 * bi) * kLd + 16 * bl;
        block_mma(acc, Tf + (64 * cc + 16 * bi) * kLd + 16 * bi, Ail, lane);
        __syncwarp();
        block_store(Ail, acc, lane, -1.f);
      }
      worker_sync();
#pragma unroll 1
      for (int d = 1; d <= 3; ++d) {
        const int per = 4 - d;
        for (int blk = w; blk < 2 * per; blk += 8) {
          const int cc = blk / per, bj = blk % per, bi = bj + d;
          float acc[2][4] = {};
          for (int l = bj; l < bi; ++l)
            block_mma(acc, Af + (64 * cc + 16 * bi) * kLd + 16 * l, Tf + (64 * cc + 16 * l) * kLd + 16 * bj, lane);
          block_store(Tf + (64 * cc + 16 * bi) * kLd + 16 * bj, acc, lane, 1.f);
        }
        worker_sync();
      }
      // ---- M1 = T diag(beta): this thread's row, 32 columns, as two terms; zeros of M2 above the diagonal blocks ----
      if (rec >= 0) {
        uint8_t* r1 = p.recs + rec * (int64_t)kRecBytes + pr * 128 + half * 64;
#pragma unroll
        for (int c4 = 0; c4 < 4; ++c4) {
          uint32_t hi[4], lo[4];
          const bool above = ((32 * half + 8 * c4) >> 4) > (pr >> 4);
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int s = 32 * half + 8 * c4 + 2 * e;
            float x = 0.f, y = 0.f;
            if (!above) {
              const float2 tt = *reinterpret_cast<const float2*>(Tf + row * kLd + s);
              x = s <= pr ? tt.x * s_bt[64 * ci + s] : 0.f;
              y = s + 1 <= pr ? tt.y * s_bt[64 * ci + s + 1] : 0.f;
            }
            split2(x, y, hi[e], lo[e]);
          }
          *reinterpret_cast<uint4*>(r1 + c4 * 16) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
          *reinterpret_cast<uint4*>(r1 + 16384 + c4 * 16) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
          if (above) {
            *reinterpret_cast<uint4*>(r1 + 8192 + c4 * 16) = make_uint4(0u, 0u, 0u, 0u);
            *reinterpret_cast<uint4*>(r1 + 24576 + c4 * 16) = make_uint4(0u, 0u, 0u, 0u);
          }
        }
      }
      // ---- M2 = Rq T diag(beta): ten blocks per chunk, five block products per warp ----
      {
        const int cc = w >> 2, q = w & 3;
        const int64_t rc = cc ? m.rec[1] : m.rec[0];
        const int n_blk = q == 0 || q == 1 || q == 2 ? 2 : 4;
#pragma unroll 1
        for (int b = 0; b < n_blk; ++b) {
          int bi, bj;                                  // q=0: (3,0) (0,0)   1: (2,0) (1,0)   2: (3,1) (2,1)   3: (3,2) (1,1) (2,2) (3,3)
          if (q == 0) { bi = b ? 0 : 3; bj = 0; }
          else if (q == 1) { bi = b ? 1 : 2; bj = 0; }
          else if (q == 2) { bi = b ? 2 : 3; bj = 1; }
          else { bi = b == 0 ? 3 : b; bj = b == 0 ? 2 : b; }
          float acc[2][4] = {};
          for (int l = bj; l <= bi; ++l)
            block_mma(acc, Rf + (64 * cc + 16 * bi) * kLd + 16 * l, Tf + (64 * cc + 16 * l) * kLd + 16 * bj, lane);
          if (rc >= 0) {
            const int g = lane >> 2, t2 = 2 * (lane & 3);
            uint8_t* r2 = p.recs + rc * (int64_t)kRecBytes + 8192;
#pragma unroll
            for (int nt = 0; nt < 2; ++nt) {
              const int s = 16 * bj + 8 * nt + t2;
              const float b0 = s_bt[64 * cc + s], b1 = s_bt[64 * cc + s + 1];
#pragma unroll
              for (int e = 0; e < 2; ++e) {
                uint32_t hi, lo;
                split2(acc[nt][2 * e] * b0, acc[nt][2 * e + 1] * b1, hi, lo);
                uint8_t* dst = r2 + (16 * bi + g + 8 * e) * 128 + s * 2;
                *reinterpret_cast<uint32_t*>(dst) = hi;
                *reinterpret_cast<uint32_t*>(dst + 16384) = lo;
              }
            }
          }
        }
      }
      fence_proxy_async();                             // the next tile's TMA writes over T and Rq
      __syncwarp();
      if (lane == 0) mbar_arrive(&bar.tile_free);
    }
  }
  tc_fence_before();
  __syncthreads();
  if (tid == 0 && s_abort) atomicExch(&g_delta_status, 1);
  if (warp == 1) tmem_dealloc(tbase, 256);
}

// ======================================= recurrence =======================================================================
constexpr int kStages = 2, kStateWarps = 16, kRecurThreads = 64 + 32 * kStateWarps;
// a stage: [K rows; Q rows] as two boxes of 64 channels x 128 rows | V, two boxes of 64 channels x 64 rows | [M1; M2] rounded,
// [M1; M2] remainders | scalars
constexpr int kOffKQ = 0, kOffRV = 32768, kOffRM = 49152, kOffRS = 81920, kStageBytes = 82944;
constexpr int kRecurSmem = kStages * kStageBytes + 1024;
constexpr uint32_t kColS = 0, kColP = 128, kColQ = 192, kColD = 128, kColX = 256, kColX2 = 320, kColR = 384, kColU = 448;

struct RecurBarriers {
  uint64_t in_full[kStages], m_full[kStages], empty[kStages];
  uint64_t s_ready, pq_full, r_ready, uo_full, us_ready, s_done;
};

__global__ void __launch_bounds__(kRecurThreads, 1)
delta_recur_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_k,
                   const __grid_constant__ CUtensorMap tmap_v, const __grid_constant__ CUtensorMap tmap_m, const Params p) {
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  __shared__ RecurBarriers bar;
  __shared__ uint32_t s_tmem_base;
  __shared__ int s_abort;

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int vblocks = p.vdim / kD;
  const int hv = blockIdx.x, h = hv / vblocks, b = blockIdx.y, g = h / (p.H / p.G);
  const int c0 = p.cu_chunks[b], n_chunks = p.cu_chunks[b + 1] - c0;
  const int64_t slot = p.slots[b];
  if (n_chunks <= 0 || slot < 0) return;              // the whole CTA, before anything is allocated
  const int row_begin = p.cu_rows[b], row_end = p.cu_rows[b + 1];
  const int64_t rec0 = (int64_t)h * p.NC + c0;

  if (tid == 0) {
    for (int i = 0; i < kStages; ++i) { mbar_init(&bar.in_full[i], 1); mbar_init(&bar.m_full[i], 1); mbar_init(&bar.empty[i], 1 + kStateWarps); }
    mbar_init(&bar.s_ready, kStateWarps); mbar_init(&bar.r_ready, kStateWarps); mbar_init(&bar.us_ready, kStateWarps);
    mbar_init(&bar.pq_full, 1); mbar_init(&bar.uo_full, 1); mbar_init(&bar.s_done, 1);
    s_abort = 0;
    fence_barrier_init();
  }
  if (warp == 1) tmem_alloc(&s_tmem_base, 512);
  if (warp == 0 && lane == 0) { prefetch_tensormap(&tmap_q); prefetch_tensormap(&tmap_k); prefetch_tensormap(&tmap_v); prefetch_tensormap(&tmap_m); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tbase = s_tmem_base;
  volatile int* abort_flag = &s_abort;

  if (warp == 0) {
    // ---- TMA producer ------------------------------------------------------------------------------------------
    if (lane == 0) {
      for (int i = 0; i < n_chunks; ++i) {
        const int s = i % kStages;
        uint8_t* st = smem + s * kStageBytes;
        const int t0 = row_begin + i * kC;
        const int64_t rec = rec0 + i;
        if (!mbar_wait(&bar.empty[s], ((uint32_t)(i / kStages) & 1u) ^ 1u, abort_flag)) break;
        mbar_arrive_expect_tx(&bar.in_full[s], 3 * 16384 + 1024);
#pragma unroll
        for (int cb = 0; cb < 2; ++cb) {
          tma_load_4d(st + kOffKQ + cb * 16384, &tmap_k, &bar.in_full[s], cb * 64, g, t0, 0);
          tma_load_4d(st + kOffKQ + cb * 16384 + 8192, &tmap_q, &bar.in_full[s], cb * 64, g, t0, 0);
          tma_load_4d(st + kOffRV + cb * 8192, &tmap_v, &bar.in_full[s], cb * 64, hv, t0, 0);
        }
        bulk_load(st + kOffRS, p.scal + rec * kScal, kScal * 4, &bar.in_full[s]);
        mbar_arrive_expect_tx(&bar.m_full[s], kRecBytes);
#pragma unroll
        for (int q = 0; q < 4; ++q) tma_load_4d(st + kOffRM + q * 8192, &tmap_m, &bar.m_full[s], 0, (int)(rec * 256) + q * 64, 0, 0);
      }
    }
    __syncwarp();
  } else if (warp == 1) {
    // ---- MMA issuer --------------------------------------------------------------------------------------------
    if (lane == 0) {
      constexpr uint32_t idesc_k = make_idesc(128, 128, 1, 0, 0);      // B rows as they lie: [K; Q] or [M1; M2]
      constexpr uint32_t idesc_ds = make_idesc(128, 128, 1, 0, 1);     // B = K [s][k], MN-major
      const uint64_t hi_k = (uint64_t(1024 >> 4) << 32) | (uint64_t(1) << 46) | (uint64_t(2) << 61) | (uint64_t(16 >> 4) << 16);
      const uint64_t hi_mn = (uint64_t(1024 >> 4) << 32) | (uint64_t(1) << 46) | (uint64_t(2) << 61) | (uint64_t(16384 >> 4) << 16);
      bool ok = true;
      for (int i = 0; i < n_chunks && ok; ++i) {
        const int s = i % kStages;
        const uint32_t ph = (uint32_t)(i / kStages) & 1u, pi = (uint32_t)i & 1u;
        const uint32_t st = smem_u32(smem + s * kStageBytes);
        const uint64_t kq = hi_k | uint64_t(((st + kOffKQ) >> 4) & 0x3FFFu), kmn = hi_mn | uint64_t(((st + kOffKQ) >> 4) & 0x3FFFu);
        const uint64_t md = hi_k | uint64_t(((st + kOffRM) >> 4) & 0x3FFFu);
        ok = mbar_wait(&bar.s_ready, pi, abort_flag) && mbar_wait(&bar.in_full[s], ph, abort_flag);
        if (!ok) break;
        tc_fence_after();
#pragma unroll
        for (int term = 0; term < 2; ++term)
#pragma unroll
          for (int kk = 0; kk < 8; ++kk)
            mma_ts(tbase + kColP, tbase + kColS + term * 64 + kk * 8, kq + uint64_t(((kk >> 2) * 16384 + (kk & 3) * 32) >> 4), idesc_k,
                   (term > 0 || kk > 0) ? 1u : 0u);
        tc_commit(&bar.pq_full);
        ok = mbar_wait(&bar.r_ready, pi, abort_flag) && mbar_wait(&bar.m_full[s], ph, abort_flag);
        if (!ok) break;
        tc_fence_after();
        // (rounded, rounded), (remainder, rounded), (rounded, remainder)
#pragma unroll
        for (int term = 0; term < 3; ++term)
#pragma unroll
          for (int kk = 0; kk < 4; ++kk)
            mma_ts(tbase + kColX, tbase + kColR + (term == 1 ? 32 : 0) + kk * 8, md + uint64_t(((term == 2 ? 16384 : 0) + kk * 32) >> 4), idesc_k,
                   (term > 0 || kk > 0) ? 1u : 0u);
        tc_commit(&bar.uo_full);
        ok = mbar_wait(&bar.us_ready, pi, abort_flag);
        if (!ok) break;
        tc_fence_after();
#pragma unroll
        for (int term = 0; term < 2; ++term)
#pragma unroll
          for (int kk = 0; kk < 4; ++kk)
            mma_ts(tbase + kColD, tbase + kColU + term * 32 + kk * 8, kmn + uint64_t((kk * 2048) >> 4), idesc_ds, (term > 0 || kk > 0) ? 1u : 0u);
        tc_commit(&bar.s_done);
        tc_commit(&bar.empty[s]);
      }
    }
    __syncwarp();
  } else {
    // ---- state warps -------------------------------------------------------------------------------------------
    const int quad = warp & 3, qt = (warp - 2) >> 2;   // qt: 32 of the 128 state columns, 16 of a chunk's 64 rows
    const int v = 32 * quad + lane;                    // TMEM lane = value channel of this CTA's block
    const uint32_t lane_base = tbase + (uint32_t(32 * quad) << 16);
    const int vcol = (hv % vblocks) * kD + v;
    float* plane = p.state + slot * p.state_ss + ((int64_t)h * kD + 32 * qt) * p.vdim + vcol;   // element (k = 32 qt + j, v)
    const bool fresh = p.start_pos[b] == 0;
    float S[32];
    {
      const float* src = plane;
      int64_t step = p.vdim;
      asm volatile("" : "+l"(step));                    // not a loop invariant: its multiples would be kept in registers
#pragma unroll
      for (int j = 0; j < 32; ++j) { S[j] = fresh ? 0.f : *src; src += step; }
    }
    float gC = 0.f;                                    // decay over the chunk before
    bool ok = true;
    for (int i = 0; i <= n_chunks; ++i) {
      if (i > 0) {                                     // the state after chunk i - 1
        ok = mbar_wait(&bar.s_done, (uint32_t)(i - 1) & 1u, abort_flag);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        tc_fence_after();
        uint32_t d[32];
        tmem_ld32(lane_base + kColD + 32 * qt, d);
#pragma unroll
        for (int j = 0; j < 32; ++j) S[j] = fmaf(gC, S[j], __uint_as_float(d[j]));
      }
      if (i == n_chunks) break;
      // ---- S^T as two 16-bit terms (the dS columns have been read: the next products may overwrite them) ----
      {
        uint32_t hi[16], lo[16];
#pragma unroll
        for (int j = 0; j < 16; ++j) split2(S[2 * j], S[2 * j + 1], hi[j], lo[j]);
        tmem_st16(lane_base + kColS + 16 * qt, hi);
        tmem_st16(lane_base + kColS + 64 + 16 * qt, lo);
      }
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&bar.s_ready);

      const int s = i % kStages;
      const uint8_t* st = smem + s * kStageBytes;
      const float* sc = reinterpret_cast<const float*>(st + kOffRS) + 16 * qt;
      // ---- R^T = V^T - (a k_inv) P: this thread's value channel, rows 16 qt .. + 15 ----
      ok = mbar_wait(&bar.in_full[s], (uint32_t)(i / kStages) & 1u, abort_flag);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      float vv[16], ek[16];
      {
        const uint8_t* vb = st + kOffRV + (v >> 6) * 8192 + (v & 7) * 2;
        const int ch = (v & 63) >> 3;
#pragma unroll
        for (int j = 0; j < 16; ++j) {
          const int t = 16 * qt + j;
          vv[j] = __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(vb + t * 128 + ((ch ^ (t & 7)) << 4)));
        }
#pragma unroll
        for (int j = 0; j < 16; j += 4) {
          const float4 e = *reinterpret_cast<const float4*>(sc + j);
          ek[j] = e.x; ek[j + 1] = e.y; ek[j + 2] = e.z; ek[j + 3] = e.w;
        }
      }
      ok = mbar_wait(&bar.pq_full, (uint32_t)i & 1u, abort_flag);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      tc_fence_after();
      {
        uint32_t pr[16], hi[8], lo[8];
        tmem_ld16(lane_base + kColP + 16 * qt, pr);
#pragma unroll
        for (int j = 0; j < 16; j += 2)
          split2(fmaf(-ek[j], __uint_as_float(pr[j]), vv[j]), fmaf(-ek[j + 1], __uint_as_float(pr[j + 1]), vv[j + 1]), hi[j >> 1], lo[j >> 1]);
        tmem_st8(lane_base + kColR + 8 * qt, hi);
        tmem_st8(lane_base + kColR + 32 + 8 * qt, lo);
        tmem_st_wait();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(&bar.r_ready);
      }
      // ---- U^T scaled by (a_C / a) k_inv; S^T Q^T leaves the columns that dS will take ----
      float ed[16];
#pragma unroll
      for (int j = 0; j < 16; j += 4) {
        const float4 e = *reinterpret_cast<const float4*>(sc + 128 + j);
        ed[j] = e.x; ed[j + 1] = e.y; ed[j + 2] = e.z; ed[j + 3] = e.w;
      }
      uint32_t sq[16];
      tmem_ld16(lane_base + kColQ + 16 * qt, sq);
      ok = mbar_wait(&bar.uo_full, (uint32_t)i & 1u, abort_flag);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      tc_fence_after();
      {
        uint32_t u[16], hi[8], lo[8];
        tmem_ld16(lane_base + kColX + 16 * qt, u);
#pragma unroll
        for (int j = 0; j < 16; j += 2) split2(__uint_as_float(u[j]) * ed[j], __uint_as_float(u[j + 1]) * ed[j + 1], hi[j >> 1], lo[j >> 1]);
        tmem_st8(lane_base + kColU + 8 * qt, hi);
        tmem_st8(lane_base + kColU + 32 + 8 * qt, lo);
        tmem_st_wait();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(&bar.us_ready);
      }
      // ---- O = (a q_inv) S Q + R M2, under the last product ----
      {
        gC = reinterpret_cast<const float*>(st + kOffRS)[192];
        const int t0 = row_begin + i * kC + 16 * qt;
        const int n_ok = min(16, row_end - t0);
        uint16_t* oc = static_cast<uint16_t*>(p.o) + ((int64_t)t0 * p.H + h) * p.vdim + vcol;
        int64_t orow = (int64_t)p.H * p.vdim;
        asm volatile("" : "+l"(orow));
        uint32_t r[16];
        tmem_ld16(lane_base + kColX2 + 16 * qt, r);
#pragma unroll
        for (int j = 0; j < 16; j += 2) {
          const float2 e = *reinterpret_cast<const float2*>(sc + 64 + j);
          const uint32_t w = pack_bf16(fmaf(e.x, __uint_as_float(sq[j]), __uint_as_float(r[j])), fmaf(e.y, __uint_as_float(sq[j + 1]), __uint_as_float(r[j + 1])));
          if (j < n_ok) *oc = (uint16_t)(w & 0xffffu);
          oc += orow;
          if (j + 1 < n_ok) *oc = (uint16_t)(w >> 16);
          oc += orow;
        }
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(&bar.empty[s]);
      }
    }
    if (ok) {
      int64_t step = p.vdim;
      asm volatile("" : "+l"(step));
#pragma unroll
      for (int j = 0; j < 32; ++j) { *plane = S[j]; plane += step; }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (tid == 0 && s_abort) atomicExch(&g_delta_status, 1);
  if (warp == 1) tmem_dealloc(tbase, 512);
}

// (channel, head, row) view of a (rows, heads, 128) tensor; boxes of 64 channels x 64 rows of one head
int heads_map(CUtensorMap* out, const void* base, int heads, int64_t rows) {
  const uint64_t dims[4] = {128, (uint64_t)heads, (uint64_t)rows, 1};
  const int64_t strides[3] = {128, (int64_t)heads * 128, (int64_t)heads * 128 * rows};
  const uint32_t box[4] = {64, 1, 64, 1};
  return make_tmap_16bit_4d(out, base, 1, dims, strides, box);
}

int64_t max_chunks(const atma_delta_args& a) { return a.total_rows / kC + a.n_seqs; }
int64_t align_up(int64_t n) { return (n + 1023) & ~int64_t(1023); }

}  // namespace

bool delta_scan_sm100_supported(const atma_delta_args& a) {
  return a.dtype == ATMA_BF16 && a.dim == kD && a.vdim > 0 && a.vdim % kD == 0 && a.G > 0 && a.H > 0 &&
         max_chunks(a) * a.H * 256 < (int64_t(1) << 31);
}

int64_t delta_scan_sm100_scratch_bytes(const atma_delta_args& a) {
  const int64_t n = max_chunks(a) * a.H;
  return align_up(4 * ((int64_t)a.n_seqs + 1)) + n * kScal * 4 + n * kRecBytes + 1024;
}

int delta_scan_sm100(const atma_delta_args& a, const void* q, const void* k, const void* v, const float* q_inv, const float* k_inv,
                     const float* log_decay, const float* beta, void* o, void* scratch, cudaStream_t st) {
  ATMA_REQUIRE(scratch != nullptr, "delta_scan: scratch is required for this shape");
  auto al = [](const void* ptr) { return (reinterpret_cast<uintptr_t>(ptr) & 15) == 0; };
  ATMA_REQUIRE(al(q) && al(k) && al(v), "delta_scan: q, k and v must be 16-byte aligned");
  const int64_t NC = max_chunks(a);
  Params p{};
  uint8_t* base = reinterpret_cast<uint8_t*>(align_up((int64_t)reinterpret_cast<uintptr_t>(scratch)));
  int32_t* cu_chunks = reinterpret_cast<int32_t*>(base);
  p.scal = reinterpret_cast<float*>(base + align_up(4 * ((int64_t)a.n_seqs + 1)));
  p.recs = reinterpret_cast<uint8_t*>(p.scal + NC * a.H * kScal);
  p.q_inv = q_inv; p.k_inv = k_inv; p.log_decay = log_decay; p.beta = beta;
  p.cu_rows = a.cu_rows; p.start_pos = a.start_pos; p.cu_chunks = cu_chunks; p.slots = a.slots;
  p.state = a.state_table; p.state_ss = a.state_ss; p.o = o;
  p.n_seqs = a.n_seqs; p.NC = (int)NC; p.H = a.H; p.G = a.G; p.vdim = a.vdim;
  CUtensorMap mq, mk, mv, mm;
  int rc = heads_map(&mq, q, a.G, a.total_rows);
  if (rc == ATMA_OK) rc = heads_map(&mk, k, a.G, a.total_rows);
  if (rc == ATMA_OK) rc = heads_map(&mv, v, a.H * (a.vdim / kD), a.total_rows);
  if (rc == ATMA_OK) {
    const int64_t rows = NC * a.H * 256;
    const uint64_t dims[4] = {64, (uint64_t)rows, 1, 1};
    const int64_t strides[3] = {64, rows * 64, rows * 64};
    const uint32_t box[4] = {64, 64, 1, 1};
    rc = make_tmap_16bit_4d(&mm, p.recs, 1, dims, strides, box);
  }
  if (rc != ATMA_OK) return rc;
  chunk_offsets_kernel<<<1, 32, 0, st>>>(a.cu_rows, a.start_pos, a.n_seqs, cu_chunks);
  const int64_t tiles = (NC + 1) / 2 * a.H;
  const int sms = sm_count_of_current_device();
  ATMA_CUDA_OK(cudaFuncSetAttribute(delta_factors_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kFactorSmem));
  delta_factors_kernel<<<(unsigned)(tiles < 2 * sms ? tiles : 2 * sms), kThreads, kFactorSmem, st>>>(mq, mk, p);
  ATMA_CUDA_OK(cudaFuncSetAttribute(delta_recur_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kRecurSmem));
  delta_recur_kernel<<<dim3(a.H * (a.vdim / kD), a.n_seqs), kRecurThreads, kRecurSmem, st>>>(mq, mk, mv, mm, p);
  return launch_status("delta_scan (tcgen05)");
}

int delta_sm100_status_fetch_and_clear(int* out) {
  int v = 0, zero = 0;
  ATMA_CUDA_OK(cudaMemcpyFromSymbol(&v, g_delta_status, sizeof(int)));
  if (v != 0) ATMA_CUDA_OK(cudaMemcpyToSymbol(g_delta_status, &zero, sizeof(int)));
  *out = v;
  return ATMA_OK;
}

}  // namespace atma
