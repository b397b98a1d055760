// Softmax attention of prompt rows on the 5th-generation tensor cores (sm_100a), keys and values read from the paged
// cache by TMA; one map per head, or two with the differential combination.
//
// One CTA owns a 128-row query tile and two streams m = 0, 1 over its keys, S_m = Q_m K_m^T (SS) and O_m += P_m V_m (P
// from TMEM).  The streams ping-pong on the tensor pipe: while the softmax warps of one work on their scores the other's
// products run.  With two maps the streams are the maps of one head (K tiles apart, V tiles shared); with one map they are
// two neighbouring query heads, which share K and V tiles where they belong to the same key/value head (an odd last head
// runs alone).  A 128-key tile lies inside one page (the page size is a multiple of 128), so the producer turns a key tile
// into a cache row with one page-table lookup.  Key tiles that no row of the tile sees are left out.
//
//   warp 0      TMA producer: the Q tiles once, K and V tiles (stream 0, stream 1, stream 0, ... or shared) through rings,
//               with one map the output gate's tiles at the end
//   warp 1      MMA issuer (one lane)
//   warps 2-3   idle (they complete the first warpgroup, whose registers are handed over)
//   warps 4-7   softmax of stream 0, one thread per query row (= one TMEM lane), and its epilogue (two maps: half of the
//               epilogue's channels)
//   warps 8-11  softmax of stream 1; its epilogue or the other half
// TMEM (512 columns): S_0 [0,128) S_1 [128,256) O_0 [256,384) O_1 [384,512).  P_m overwrites S_m once the row is in
// registers, as two 16-bit terms - the rounded weight in the first 64 columns, the remainder in the second - so that the
// weights enter the product with 16 bits of mantissa; O_m += P_hi V + P_lo V.
// Rows stream (m, L = sum p, O = sum p v) in the log2 domain, starting from the sink (its score, 1, 0) if there is one; the
// maximum in use moves only when it grew by more than 2^8.  With two maps the epilogue forms o = O_0/L_0 - lambda O_1/L_1 over half of the channels per warpgroup, exchanges the sums of
// squares and writes o * out_scale / rms(o); with one map it writes O/L.  Both apply the output gate.
// Every mbarrier wait is bounded; on expiry the CTA frees its TMEM, returns and leaves a status word for the host.
#include "softmax_attention.cuh"
#include "sm100.cuh"

namespace atma {

using namespace sm100;

namespace {

constexpr int kBM = 128, kBN = 128, kThreads = 384, kVStages = 2;
constexpr float kLog2e = 1.4426950408889634f;
constexpr float kNegInit = -1.0e30f;
constexpr float kLazyThreshold = 8.0f;

__device__ int g_softmax_status = 0;

template <int DIM, int VD>
struct Cfg {
  static constexpr int kMapTile = kBM * DIM * 2;                 // a Q or K tile of one map
  static constexpr int kKSlots = DIM == 64 ? 4 : 3;
  static constexpr int kVTile = kBN * VD * 2;
  // one map: the gate tiles of both streams lie over the Q tiles (read once the last scores are there) or, where they are
  // larger, behind the rings
  static constexpr bool kGateOverQ = VD <= DIM;
  static constexpr int kRings = (2 + kKSlots) * kMapTile + kVStages * kVTile;
  template <int MAPS>
  static constexpr int bytes() { return kRings + (MAPS == 1 && !kGateOverQ ? 2 * kVTile : 0) + 1024; }
};

template <int KS>
struct Barriers {
  uint64_t q_full[2];
  uint64_t k_full[KS], k_empty[KS], v_full[kVStages], v_empty[kVStages];
  uint64_t s_full[2], p_full[2], o_final[2], g_full[2];
};

__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
  __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&h);
}
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float max3(float a, float b, float c) {
  float d;
  asm("max.f32 %0, %1, %2, %3;" : "=f"(d) : "f"(a), "f"(b), "f"(c));
  return d;
}
__device__ __forceinline__ void softmax_sync() { asm volatile("bar.sync 1, 256;" ::: "memory"); }

// WIN: a window is set (without one the key tiles are 0, 1, ... and only the last ones need a mask)
template <int MAPS, int DIM, int VD, bool WIN>
__global__ void __launch_bounds__(kThreads, 1)
softmax_prefill_sm100_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_k,
                             const __grid_constant__ CUtensorMap tmap_v, const __grid_constant__ CUtensorMap tmap_g,
                             const atma_softmax_args a) {
  using C = Cfg<DIM, VD>;
  constexpr int kMapTile = C::kMapTile, KS = C::kKSlots, kVTile = C::kVTile;
  constexpr int kBox = kBM * 128;                                // one 64-channel box of 128 rows
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sQ = smem;                                            // [2 maps]
  uint8_t* sK = sQ + 2 * kMapTile;                               // [KS]
  uint8_t* sV = sK + KS * kMapTile;                              // [kVStages]
  uint8_t* sG = C::kGateOverQ ? sQ : smem + C::kRings;           // [2 streams], one map
  __shared__ Barriers<KS> bar;
  __shared__ uint32_t s_tmem_base;
  __shared__ int s_abort;
  // row exchanges of the epilogue, over the Q tiles: written once every product has been read (o_final)
  float (*s_l)[kBM] = reinterpret_cast<float (*)[kBM]>(sQ);
  float (*s_ss)[kBM] = s_l + 2;

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int seq = a.tile_seq[blockIdx.x], row0 = a.tile_row[blockIdx.x];
  // head and key/value head of each stream; K and V tiles per key tile
  const int h0 = MAPS == 2 ? blockIdx.y : 2 * blockIdx.y, h1 = MAPS == 2 ? h0 : h0 + 1;
  const int n_streams = MAPS == 2 || h1 < a.H ? 2 : 1;
  const int g0 = h0 / (a.H / a.G), g1 = MAPS == 2 ? g0 : min(h1, a.H - 1) / (a.H / a.G);
  const int nv = MAPS == 2 || g0 == g1 ? 1 : 2, nk = MAPS == 2 ? 2 : nv;
  const int r_begin = a.cu_rows[seq], n_rows = a.cu_rows[seq + 1] - r_begin, start = a.start_pos[seq];
  const KeyTiles tiles(start + row0, start + min(row0 + kBM, n_rows) - 1, a.max_blocks * a.block_size, a.window, a.keep_first, kBN);
  const int n_kt = start < 0 || row0 >= n_rows ? 0 : tiles.n;

  if (tid == 0) {
    for (int i = 0; i < 2; ++i) {
      mbar_init(&bar.q_full[i], 1); mbar_init(&bar.s_full[i], 1);
      mbar_init(&bar.p_full[i], 4); mbar_init(&bar.o_final[i], 1); mbar_init(&bar.g_full[i], 1);
    }
    for (int i = 0; i < KS; ++i) { mbar_init(&bar.k_full[i], 1); mbar_init(&bar.k_empty[i], 1); }
    for (int i = 0; i < kVStages; ++i) { mbar_init(&bar.v_full[i], 1); mbar_init(&bar.v_empty[i], 1); }
    s_abort = 0;
    fence_barrier_init();
  }
  if (warp == 0) {
    if (lane == 0) { prefetch_tensormap(&tmap_q); prefetch_tensormap(&tmap_k); prefetch_tensormap(&tmap_v); }
    __syncwarp();
    tmem_alloc(&s_tmem_base, 512);
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tbase = s_tmem_base;
  volatile int* abort_flag = &s_abort;

  if (warp < 4) {
    // Register hand-over: 88 x 128 + 208 x 256 = 168 x 384, the pool this CTA is launched with.  The sum must not exceed
    // that pool, or the last setmaxnreg.inc never returns.
    asm volatile("setmaxnreg.dec.sync.aligned.u32 88;");
    if (warp == 0) {
      // ============================= TMA producer ==============================================
      if (lane == 0 && n_kt > 0) {
        const int32_t* bt = a.block_tables + seq * a.bt_stride;
        for (int m = 0; m < n_streams; ++m) {
          mbar_arrive_expect_tx(&bar.q_full[m], kMapTile);
#pragma unroll
          for (int cb = 0; cb < DIM / 64; ++cb)
            tma_load_4d(sQ + m * kMapTile + cb * kBox, &tmap_q, &bar.q_full[m], (MAPS == 2 ? h0 * 2 + m : h0 + m) * DIM + cb * 64,
                        r_begin + row0, 0, 0);
        }
        bool ok = true;
        for (int j = 0; j < n_kt && ok; ++j) {
          const int key0 = (WIN ? tiles[j] : j) * kBN, blk = key0 / a.block_size;
          const int row = min(max(bt[blk], 0), a.num_blocks - 1) * a.block_size + (key0 - blk * a.block_size);
          for (int m = 0; m < nk; ++m) {
            const int i = nk * j + m, s = i % KS;
            ok = ok && mbar_wait(&bar.k_empty[s], ((uint32_t)(i / KS) & 1u) ^ 1u, abort_flag);
            if (!ok) break;
            mbar_arrive_expect_tx(&bar.k_full[s], kMapTile);
#pragma unroll
            for (int cb = 0; cb < DIM / 64; ++cb)
              tma_load_4d(sK + s * kMapTile + cb * kBox, &tmap_k, &bar.k_full[s], (MAPS == 2 ? g0 * 2 + m : (m == 0 ? g0 : g1)) * DIM + cb * 64, row, 0, 0);
          }
          for (int m = 0; m < nv && ok; ++m) {
            const int i = nv * j + m, s = i % kVStages;
            ok = mbar_wait(&bar.v_empty[s], ((uint32_t)(i / kVStages) & 1u) ^ 1u, abort_flag);
            if (!ok) break;
            mbar_arrive_expect_tx(&bar.v_full[s], kVTile);
#pragma unroll
            for (int cb = 0; cb < VD / 64; ++cb)
              tma_load_4d(sV + s * kVTile + cb * kBox, &tmap_v, &bar.v_full[s], (m == 0 ? g0 : g1) * VD + cb * 64, row, 0, 0);
          }
        }
        if (MAPS == 1 && a.gate != nullptr) {
          const int i = nk * n_kt - 1;                            // once the last K tile is given back nobody reads Q any more
          ok = ok && (!C::kGateOverQ || mbar_wait(&bar.k_empty[i % KS], (uint32_t)(i / KS) & 1u, abort_flag));
          for (int m = 0; m < n_streams && ok; ++m) {
            mbar_arrive_expect_tx(&bar.g_full[m], kVTile);
#pragma unroll
            for (int cb = 0; cb < VD / 64; ++cb)
              tma_load_4d(sG + m * kVTile + cb * kBox, &tmap_g, &bar.g_full[m], (h0 + m) * VD + cb * 64, r_begin + row0, 0, 0);
          }
        }
      }
      __syncwarp();
    } else if (warp == 1) {
      // ============================= MMA issuer ================================================
      if (lane == 0 && n_kt > 0) {
        constexpr uint32_t idesc_qk = make_idesc(kBM, kBN, 1, 0, 0);
        constexpr uint32_t idesc_pv = make_idesc(kBM, VD, 1, 0, 1);
        const uint32_t q_addr = smem_u32(sQ), k_addr = smem_u32(sK), v_addr = smem_u32(sV);
        const uint64_t desc_hi_k = (uint64_t(1024 >> 4) << 32) | (uint64_t(1) << 46) | (uint64_t(2) << 61) | (uint64_t(16 >> 4) << 16);
        const uint64_t desc_hi_v = (uint64_t(1024 >> 4) << 32) | (uint64_t(1) << 46) | (uint64_t(2) << 61) | (uint64_t(kBox >> 4) << 16);
        auto issue_qk = [&](int m, int s) {
          const uint64_t a0 = desc_hi_k | uint64_t(((q_addr + m * kMapTile) >> 4) & 0x3FFFu);
          const uint64_t b0 = desc_hi_k | uint64_t(((k_addr + s * kMapTile) >> 4) & 0x3FFFu);
#pragma unroll
          for (int kk = 0; kk < DIM / 16; ++kk) {
            const uint64_t off = uint64_t(((kk >> 2) * kBox + (kk & 3) * 32) >> 4);
            mma_ss(tbase + m * 128, a0 + off, b0 + off, idesc_qk, kk > 0);
          }
        };
        auto issue_pv = [&](int m, int s, bool acc) {
          const uint64_t b0 = desc_hi_v | uint64_t(((v_addr + s * kVTile) >> 4) & 0x3FFFu);
          const uint32_t pa = tbase + m * 128, od = tbase + 256 + m * 128;
#pragma unroll
          for (int half = 0; half < 2; ++half)                   // rounded weights, then their remainders
#pragma unroll
            for (int kk = 0; kk < kBN / 16; ++kk)
              mma_ts(od, pa + half * 64 + kk * 8, b0 + uint64_t(kk * (2048 >> 4)), idesc_pv, (half > 0 || kk > 0 || acc) ? 1u : 0u);
        };
        bool ok = true;
        // a tile that both streams read is given back by the last of them
        const int last = n_streams - 1;
        auto next_qk = [&](int m, int j) {
          const int i = nk == 2 ? 2 * j + m : j, s = i % KS;
          if (!mbar_wait(&bar.k_full[s], (uint32_t)(i / KS) & 1u, abort_flag)) return false;
          tc_fence_after();
          issue_qk(m, s);
          tc_commit(&bar.s_full[m]);
          if (nk == 2 || m == last) tc_commit(&bar.k_empty[s]);
          return true;
        };
        for (int m = 0; m < n_streams && ok; ++m) ok = mbar_wait(&bar.q_full[m], 0, abort_flag) && next_qk(m, 0);
        for (int j = 0; j < n_kt && ok; ++j) {
          const bool more = j + 1 < n_kt;
#pragma unroll
          for (int m = 0; m < 2; ++m) {
            if (!ok || m >= n_streams) break;
            const int i = nv == 2 ? 2 * j + m : j, vs = i % kVStages;
            ok = mbar_wait(&bar.p_full[m], (uint32_t)j & 1u, abort_flag) && mbar_wait(&bar.v_full[vs], (uint32_t)(i / kVStages) & 1u, abort_flag);
            if (!ok) break;
            tc_fence_after();
            issue_pv(m, vs, j > 0);
            if (nv == 2 || m == last) tc_commit(&bar.v_empty[vs]);
            if (more) ok = next_qk(m, j + 1);
            else tc_commit(&bar.o_final[m]);
          }
        }
      }
      __syncwarp();
    }
  } else {
    asm volatile("setmaxnreg.inc.sync.aligned.u32 208;");
    // ============================= softmax + epilogue ===========================================
    const int m = warp >= 8 ? 1 : 0;
    const int r = 32 * (warp & 3) + lane;
    const bool row_ok = row0 + r < n_rows;
    const int pos = start + row0 + r;
    const uint32_t lane_base = tbase + (uint32_t(32 * (warp & 3)) << 16);
    const uint32_t tS = lane_base + m * 128, tO = lane_base + 256 + m * 128;
    const float sc2 = a.scale * kLog2e;
    const bool sink = a.sink > -INFINITY;
    float m_used = sink ? a.sink * kLog2e : kNegInit, m_run = m_used, L = sink ? 1.f : 0.f;
    bool ok = true;
    const int my_tiles = m < n_streams ? n_kt : 0;
    for (int j = 0; j < my_tiles; ++j) {
      ok = mbar_wait(&bar.s_full[m], (uint32_t)j & 1u, abort_flag);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      tc_fence_after();
      const int key0 = (WIN ? tiles[j] : j) * kBN;
      const int vis = row_ok ? pos + 1 - key0 : 0;                // key columns below this one are seen
      uint32_t s[kBN];
#pragma unroll
      for (int ch = 0; ch < 4; ++ch) tmem_ld32_nowait(tS + ch * 32, &s[ch * 32]);
      tmem_ld_wait();
#pragma unroll
      for (int i = 0; i < kBN; ++i) reg_fence(s[i]);
      if (vis < kBN) {
#pragma unroll
        for (int i = 0; i < kBN; ++i)
          if (i >= vis) s[i] = 0xff800000u;                       // -inf
      }
      if constexpr (WIN) {
        // and of those the ones from win on and the kept ones
        const int win = pos - a.window + 1 - key0, kept = a.keep_first - key0;
        if (win > 0 && kept < kBN) {
#pragma unroll
          for (int i = 0; i < kBN; ++i)
            if (i < win && i >= kept) s[i] = 0xff800000u;
        }
      }
      float mx0 = -INFINITY, mx1 = -INFINITY, mx2 = -INFINITY, mx3 = -INFINITY;
#pragma unroll
      for (int i = 0; i < kBN; i += 8) {
        mx0 = max3(mx0, __uint_as_float(s[i]), __uint_as_float(s[i + 1]));
        mx1 = max3(mx1, __uint_as_float(s[i + 2]), __uint_as_float(s[i + 3]));
        mx2 = max3(mx2, __uint_as_float(s[i + 4]), __uint_as_float(s[i + 5]));
        mx3 = max3(mx3, __uint_as_float(s[i + 6]), __uint_as_float(s[i + 7]));
      }
      // a negative scale would turn the maximum into a minimum: the host refuses it
      const float m_new = fmaxf(m_run, fmaxf(fmaxf(mx0, mx1), fmaxf(mx2, mx3)) * sc2);
      m_run = m_new;
      if (__any_sync(0xffffffffu, (m_new - m_used) > kLazyThreshold)) {
        const float alpha = ex2(m_used - m_new);
        L *= alpha;
        if (j > 0) {
#pragma unroll 1
          for (int ch = 0; ch < VD / 32; ++ch) {
            uint32_t o[32];
            tmem_ld32(tO + ch * 32, o);
#pragma unroll
            for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * alpha);
            tmem_st32(tO + ch * 32, o);
          }
        }
        m_used = m_new;
      }
      const float neg_m = -m_used;
      const float2 sc2v = make_float2(sc2, sc2), negv = make_float2(neg_m, neg_m);
      float2 la = make_float2(0.f, 0.f), lb = la;
#pragma unroll
      for (int ch = 0; ch < 4; ++ch) {
        uint32_t hi[16], lo[16];
#pragma unroll
        for (int i = 0; i < 32; i += 2) {
          const float2 x = __ffma2_rn(make_float2(__uint_as_float(s[ch * 32 + i]), __uint_as_float(s[ch * 32 + i + 1])), sc2v, negv);
          const float2 p = make_float2(ex2(x.x), ex2(x.y));
          if (i & 2) lb = __fadd2_rn(lb, p); else la = __fadd2_rn(la, p);
          const uint32_t w = pack_bf16(p.x, p.y);
          const float2 rem = __fadd2_rn(p, make_float2(-__uint_as_float(w << 16), -__uint_as_float(w & 0xffff0000u)));
          hi[i >> 1] = w;
          lo[i >> 1] = pack_bf16(rem.x, rem.y);
        }
        tmem_st16(tS + ch * 16, hi);
        tmem_st16(tS + 64 + ch * 16, lo);
      }
      L += (la.x + la.y) + (lb.x + lb.y);
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&bar.p_full[m]);
    }
    // ---- epilogue ----
    if constexpr (MAPS == 1) {                                    // each warpgroup its own head
      if (ok && my_tiles > 0) {
        ok = mbar_wait(&bar.o_final[m], 0, abort_flag) && (a.gate == nullptr || mbar_wait(&bar.g_full[m], 0, abort_flag));
        ok = __all_sync(0xffffffffu, ok);
        tc_fence_after();
      }
      const bool live = ok && my_tiles > 0;
      if (m < n_streams) {
        const float inv = L > 0.f ? 1.0f / L : 0.f;
        const int64_t row = r_begin + row0 + r;
        __nv_bfloat16* op = static_cast<__nv_bfloat16*>(a.out) + row * a.out_rs + (int64_t)(h0 + m) * VD;
        const uint8_t* gp = sG + m * kVTile + r * 128;            // this row in the first 64-channel box, 16-byte pieces swizzled
#pragma unroll 1
        for (int ch = 0; ch < VD; ch += 32) {
          uint32_t u[32];
          if (live) {
            tmem_ld32(tO + ch, u);
          } else {
#pragma unroll
            for (int i = 0; i < 32; ++i) u[i] = 0u;
          }
#pragma unroll
          for (int i = 0; i < 32; i += 8) {
            if (!row_ok) break;
            float o[8];
#pragma unroll
            for (int e = 0; e < 8; ++e) o[e] = __uint_as_float(u[i + e]) * inv;
            if (a.gate != nullptr && live) {
              const int c = ch + i;
              const uint4 z = *reinterpret_cast<const uint4*>(gp + (c >> 6) * kBox + ((((c & 63) >> 3) ^ (r & 7)) << 4));
              const uint32_t zw[4] = {z.x, z.y, z.z, z.w};
#pragma unroll
              for (int e = 0; e < 4; ++e) {
                o[2 * e] *= __fdividef(1.0f, 1.0f + __expf(-__uint_as_float(zw[e] << 16)));
                o[2 * e + 1] *= __fdividef(1.0f, 1.0f + __expf(-__uint_as_float(zw[e] & 0xffff0000u)));
              }
            }
            *reinterpret_cast<uint4*>(op + ch + i) = make_uint4(pack_bf16(o[0], o[1]), pack_bf16(o[2], o[3]), pack_bf16(o[4], o[5]), pack_bf16(o[6], o[7]));
          }
          __syncwarp();
        }
      }
    } else {                  // both maps' accumulators, half of the channels per warpgroup; the barriers are met on every path
      if (ok && n_kt > 0) {
        ok = mbar_wait(&bar.o_final[0], 0, abort_flag) && mbar_wait(&bar.o_final[1], 0, abort_flag);
        ok = __all_sync(0xffffffffu, ok);
        tc_fence_after();
      }
      s_l[m][r] = L;
      softmax_sync();
      const bool live = ok && n_kt > 0;
      const float i0 = s_l[0][r] > 0.f ? 1.0f / s_l[0][r] : 0.f, i1 = s_l[1][r] > 0.f ? a.lambda / s_l[1][r] : 0.f;
      constexpr int HC = VD / 2;
      float o[HC];
      float ss = 0.f;
#pragma unroll
      for (int ch = 0; ch < HC / 32; ++ch) {
        uint32_t u0[32], u1[32];
        if (live) {
          tmem_ld32(lane_base + 256 + m * HC + ch * 32, u0);
          tmem_ld32(lane_base + 384 + m * HC + ch * 32, u1);
        } else {
#pragma unroll
          for (int i = 0; i < 32; ++i) u0[i] = u1[i] = 0u;
        }
#pragma unroll
        for (int i = 0; i < 32; ++i) {
          o[ch * 32 + i] = __uint_as_float(u0[i]) * i0 - __uint_as_float(u1[i]) * i1;
          ss = fmaf(o[ch * 32 + i], o[ch * 32 + i], ss);
        }
      }
      s_ss[m][r] = ss;
      softmax_sync();
      const float f = a.out_scale / sqrtf((s_ss[0][r] + s_ss[1][r]) / (float)VD + a.eps);
      if (row_ok) {
        const int64_t row = r_begin + row0 + r, ch0 = (int64_t)h0 * VD + m * HC;
        __nv_bfloat16* op = static_cast<__nv_bfloat16*>(a.out) + row * a.out_rs + ch0;
        if (a.gate != nullptr) {
          const __nv_bfloat16* gp = static_cast<const __nv_bfloat16*>(a.gate) + row * a.gate_rs + ch0;
#pragma unroll
          for (int i = 0; i < HC; ++i) o[i] *= sigmoid_gate(gp[i]);
        }
#pragma unroll
        for (int i = 0; i < HC; i += 8) {
          uint4 w = make_uint4(0u, 0u, 0u, 0u);
          if (live) {
            w = make_uint4(pack_bf16(o[i] * f, o[i + 1] * f), pack_bf16(o[i + 2] * f, o[i + 3] * f), pack_bf16(o[i + 4] * f, o[i + 5] * f),
                           pack_bf16(o[i + 6] * f, o[i + 7] * f));
          }
          *reinterpret_cast<uint4*>(op + i) = w;
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (tid == 0 && s_abort) atomicExch(&g_softmax_status, 1);
  if (warp == 0) tmem_dealloc(tbase, 512);
}

int rows_map(CUtensorMap* out, const void* base, int64_t width, int64_t rows, int64_t row_stride) {
  const uint64_t dims[4] = {(uint64_t)width, (uint64_t)rows, 1, 1};
  const int64_t strides[3] = {row_stride, row_stride * rows, row_stride * rows};
  const uint32_t box[4] = {64, 128, 1, 1};
  return make_tmap_16bit_4d(out, base, 1, dims, strides, box);
}

template <int MAPS, int DIM, int VD>
int launch(const atma_softmax_args& a, cudaStream_t st) {
  CUtensorMap mq, mk, mv, mg;
  const int64_t slots = (int64_t)a.num_blocks * a.block_size, wq = (int64_t)a.H * MAPS * DIM, wk = (int64_t)a.G * MAPS * DIM, wv = (int64_t)a.G * VD;
  int rc = rows_map(&mq, a.q, wq, a.total_rows, wq);
  if (rc == ATMA_OK) rc = rows_map(&mk, a.k_cache, wk, slots, wk);
  if (rc == ATMA_OK) rc = rows_map(&mv, a.v_cache, wv, slots, wv);
  mg = mq;                                                       // not used without a gate
  if (rc == ATMA_OK && MAPS == 1 && a.gate != nullptr) rc = rows_map(&mg, a.gate, (int64_t)a.H * VD, a.total_rows, a.gate_rs);
  if (rc != ATMA_OK) return rc;
  constexpr int smem = Cfg<DIM, VD>::template bytes<MAPS>();
  // a window that no position of this cache outgrows is none
  const bool win = a.window < (int64_t)a.max_blocks * a.block_size;
  auto kern = win ? softmax_prefill_sm100_kernel<MAPS, DIM, VD, true> : softmax_prefill_sm100_kernel<MAPS, DIM, VD, false>;
  ATMA_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
  kern<<<dim3(a.n_tiles, MAPS == 2 ? a.H : (a.H + 1) / 2), kThreads, smem, st>>>(mq, mk, mv, mg, a);
  return launch_status("softmax_prefill (tcgen05)");
}

}  // namespace

bool softmax_prefill_sm100_supported(const atma_softmax_args& a) {
  auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  return a.dtype == ATMA_BF16 && (a.maps == 1 || a.maps == 2) && (a.dim == 64 || a.dim == 128) && (a.vdim == 64 || a.vdim == 128) && a.block_size % kBN == 0 &&
         a.scale >= 0.f && a.out_rs % 8 == 0 && al(a.q) && al(a.k_cache) && al(a.v_cache) && al(a.out) && a.gate_rs % 8 == 0 && al(a.gate) &&
         (int64_t)a.num_blocks * a.block_size < (int64_t(1) << 31);
}

int softmax_prefill_sm100(const atma_softmax_args& a, cudaStream_t st) {
  ATMA_REQUIRE(a.tile_seq != nullptr && a.tile_row != nullptr && a.n_tiles > 0, "softmax_prefill: the query tiles are required for this shape");
  if (a.maps == 1) {
    if (a.dim == 64) return a.vdim == 64 ? launch<1, 64, 64>(a, st) : launch<1, 64, 128>(a, st);
    return a.vdim == 64 ? launch<1, 128, 64>(a, st) : launch<1, 128, 128>(a, st);
  }
  if (a.dim == 64) return a.vdim == 64 ? launch<2, 64, 64>(a, st) : launch<2, 64, 128>(a, st);
  return a.vdim == 64 ? launch<2, 128, 64>(a, st) : launch<2, 128, 128>(a, st);
}

int softmax_sm100_status_fetch_and_clear(int* out) {
  int v = 0, zero = 0;
  ATMA_CUDA_OK(cudaMemcpyFromSymbol(&v, g_softmax_status, sizeof(int)));
  if (v != 0) ATMA_CUDA_OK(cudaMemcpyToSymbol(g_softmax_status, &zero, sizeof(int)));
  *out = v;
  return ATMA_OK;
}

}  // namespace atma
