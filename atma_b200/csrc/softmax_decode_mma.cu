// Paged softmax attention of one query row per sequence, 16-bit caches: key ranges side by side, then a merge that also
// adds the sink to the denominator and applies the differential combination and the output gate.  With one map and a
// single key range (short contexts and windows) the first kernel finishes by itself.  Key ranges are cut from the list of
// key tiles that the row sees at all.
//
// A CTA streams the K and V rows of one key range of one (sequence, key/value head) through a cp.async ring of 64-key
// tiles (16-byte copies, one page-table lookup per tile when tiles cannot straddle pages).  Keys are the rows of the
// tensor-core products: each of the four warps owns 16 keys of a tile and computes S^T = K_w Q^T with mma.sync m16n8k16.
// The eight columns are (map, query head) pairs of the group; a K row holds its head's maps side by side, so a column's
// Q^T is zero outside its own map's channels and one pass over the row serves both maps.  P^T goes back in as the B
// operand of O^T += V_w^T P^T through a register transpose, as two 16-bit terms (rounded weight and remainder), which
// keeps the weights at 16 bits of mantissa; both maps share the V fragments.  Where four columns are enough for the group
// the other four hold the same queries again and carry the remainders, so that both terms are one product (COLS = 4).
// The reference maximum of a column is raised
// only when a score exceeds it by more than 2^8.
#include "softmax_attention.cuh"
#include "mma_sync.cuh"

namespace atma {

using namespace mma;

namespace {

constexpr int kTileKeys = 64;
constexpr float kLog2e = 1.4426950408889634f;
constexpr float kNegBig = -1e30f;
constexpr float kRaise = 8.0f;

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ uint32_t movmatrix_trans(uint32_t a) {
  uint32_t d;
  asm volatile("movmatrix.sync.aligned.m8n8.trans.b16 %0, %1;" : "=r"(d) : "r"(a));
  return d;
}

template <int MAPS, int DIM, int VD, int STAGES, int COLS>
__global__ void __launch_bounds__(128, 2)
softmax_decode_split_kernel(const atma_softmax_args a) {
  constexpr int KD = MAPS * DIM;
  constexpr int KS = KD / 16, MT = VD / 16, CK = KD / 8, CV = VD / 8;
  constexpr int kKBytes = kTileKeys * KD * 2, kVBytes = kTileKeys * VD * 2, kStage = kKBytes + kVBytes;
  constexpr int GC = COLS / MAPS;             // query heads per CTA; a column is a (map, head) pair
  constexpr int OLD = VD + 4;
  extern __shared__ __align__(128) uint8_t sm[];
  const int rep = a.H / a.G, ngrp = (rep + GC - 1) / GC;
  const int split = blockIdx.x, g = blockIdx.y / ngrp, h0 = g * rep + (blockIdx.y % ngrp) * GC, b = blockIdx.z;
  const int nh = min(GC, (g + 1) * rep - h0);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int gq = lane >> 2, tq = lane & 3;

  const int pos = a.start_pos[b];
  const int n = max(0, min(pos + 1, a.max_blocks * a.block_size));
  const KeyTiles tiles(pos, pos, a.max_blocks * a.block_size, a.window, a.keep_first, kTileKeys);
  const int per_split = (tiles.n + a.n_splits - 1) / a.n_splits;
  const int tile0 = split * per_split, n_tiles = max(0, min(per_split, tiles.n - tile0));
  const bool direct = MAPS == 1 && a.n_splits == 1;
  float* stats = a.scratch;                   // [b][h][map][split]{m, l}, then [b][h][map][split][VD]
  float* sacc = a.scratch + (int64_t)a.n_seqs * a.H * MAPS * a.n_splits * 2;
  auto part = [&](int col) {                  // column (below COLS) = map * GC + head
    return (((int64_t)b * a.H + h0 + col % GC) * MAPS + col / GC) * a.n_splits + split;
  };
  auto finish = [&](int c, int d, float v) {    // direct form: gate and store channel d of head h0 + c
    const int64_t ch = (int64_t)(h0 + c) * VD + d;
    if (a.gate != nullptr) v *= sigmoid_gate(static_cast<const __nv_bfloat16*>(a.gate)[b * a.gate_rs + ch]);
    static_cast<__nv_bfloat16*>(a.out)[b * a.out_rs + ch] = __float2bfloat16_rn(v);
  };
  if (n_tiles == 0) {                         // nothing in this range: weight zero in the merge
    if (direct) {
      for (int i = tid; i < nh * VD; i += 128) static_cast<__nv_bfloat16*>(a.out)[b * a.out_rs + (int64_t)h0 * VD + i] = __float2bfloat16_rn(0.f);
      return;
    }
    for (int c = warp; c < MAPS * GC; c += 4) {
      if (c % GC >= nh) continue;
      const int64_t p = part(c);
      if (lane == 0) { stats[2 * p] = kNegBig; stats[2 * p + 1] = 0.f; }
      for (int d = lane; d < VD; d += 32) sacc[p * VD + d] = 0.f;
    }
    return;
  }
  const uint16_t* K = static_cast<const uint16_t*>(a.k_cache) + (int64_t)g * KD;
  const uint16_t* V = static_cast<const uint16_t*>(a.v_cache) + (int64_t)g * VD;
  const int64_t krow = (int64_t)a.G * KD, vrow = (int64_t)a.G * VD;
  const int32_t* bt = a.block_tables + b * a.bt_stride;
  const bool tile_in_page = a.block_size % kTileKeys == 0;

  auto row_of = [&](int pos) {
    const int blk = pos / a.block_size;
    return (int64_t)min(max(bt[blk], 0), a.num_blocks - 1) * a.block_size + (pos - blk * a.block_size);
  };
  // whether the row sees every key of the tile that starts at pos0 (nearly all of them)
  auto whole = [&](int pos0) { return pos0 + kTileKeys <= n && (pos - pos0 < a.window || pos0 + kTileKeys <= a.keep_first); };
  constexpr int kKStep = 128 / CK, kVStep = 128 / CV;            // rows between a thread's copies; its 16-byte column is fixed
  const int64_t k_off = (tid / CK) * krow + tid % CK * 8, v_off = (tid / CV) * vrow + tid % CV * 8;
  auto load_tile = [&](int it) {
    const uint32_t dst = smem_u32(sm + (it % STAGES) * kStage);
    const int pos0 = tiles[tile0 + it] * kTileKeys;
    const int64_t base = tile_in_page ? row_of(pos0) : 0;
    if (tile_in_page && whole(pos0)) {
      const uint16_t *kp = K + base * krow + k_off, *vp = V + base * vrow + v_off;
#pragma unroll
      for (int j = 0; j < kTileKeys / kKStep; ++j, kp += kKStep * krow) cp_async16(dst + tile_off(tid / CK + j * kKStep, tid % CK * 8, KD), kp);
#pragma unroll
      for (int j = 0; j < kTileKeys / kVStep; ++j, vp += kVStep * vrow)
        cp_async16(dst + kKBytes + tile_off(tid / CV + j * kVStep, tid % CV * 8, VD), vp);
      return;
    }
#pragma unroll
    for (int j = 0; j < kTileKeys * CK / 128; ++j) {
      const int i = tid + j * 128, r = i / CK, ch = i % CK;
      const bool ok = pos0 + r < n && key_visible(pos, pos0 + r, a.window, a.keep_first);
      const int64_t row = !ok ? 0 : (tile_in_page ? base + r : row_of(pos0 + r));
      cp_async16(dst + tile_off(r, ch * 8, KD), K + row * krow + ch * 8, ok);
    }
#pragma unroll
    for (int j = 0; j < kTileKeys * CV / 128; ++j) {
      const int i = tid + j * 128, r = i / CV, ch = i % CV;
      const bool ok = pos0 + r < n && key_visible(pos, pos0 + r, a.window, a.keep_first);
      const int64_t row = !ok ? 0 : (tile_in_page ? base + r : row_of(pos0 + r));
      cp_async16(dst + kKBytes + tile_off(r, ch * 8, VD), V + row * vrow + ch * 8, ok);
    }
  };
#pragma unroll
  for (int s = 0; s < STAGES - 1; ++s) {
    if (s < n_tiles) load_tile(s);
    cp_async_commit();
  }

  // Q^T as the B operand: column c = gq mod COLS = (map c / GC, head c % GC), zero outside its map's channels and past the
  // group
  uint32_t qb[KS][2];
  {
    const int m = gq % COLS / GC, hh = gq % GC;
    const bool on = hh < nh;
    const uint16_t* qrow = static_cast<const uint16_t*>(a.q) + ((int64_t)b * a.H + h0 + (on ? hh : 0)) * KD;
#pragma unroll
    for (int ks = 0; ks < KS; ++ks) {
      const bool mine = on && (16 * ks) / DIM == m;
      qb[ks][0] = mine ? *reinterpret_cast<const uint32_t*>(qrow + 16 * ks + 2 * tq) : 0u;
      qb[ks][1] = mine ? *reinterpret_cast<const uint32_t*>(qrow + 16 * ks + 8 + 2 * tq) : 0u;
    }
  }
  const float sc = a.scale * kLog2e;
  float mref[2] = {kNegBig, kNegBig}, L[2] = {0.f, 0.f};        // columns 2 tq + e; L: this thread's keys only
  float O[MT][4];
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int e = 0; e < 4; ++e) O[mt][e] = 0.f;
  int am, ak, vk, vm;
  a_rowmajor_lane(lane, am, ak);
  a_km_lane(lane, vk, vm);

  for (int it = 0; it < n_tiles; ++it) {
    cp_async_wait<STAGES - 2>();
    __syncthreads();
    if (it + STAGES - 1 < n_tiles) load_tile(it + STAGES - 1);
    cp_async_commit();
    const uint32_t Ksm = smem_u32(sm + (it % STAGES) * kStage), Vsm = Ksm + kKBytes;
    float S[4] = {0.f, 0.f, 0.f, 0.f}, S2[4] = {0.f, 0.f, 0.f, 0.f};      // two chains, half as long
#pragma unroll
    for (int ks = 0; ks < KS; ks += 2) {
      uint32_t af[4], ag[4];
      ldsm_x4(Ksm + tile_off(16 * warp + am, 16 * ks + ak, KD), af);
      ldsm_x4(Ksm + tile_off(16 * warp + am, 16 * ks + 16 + ak, KD), ag);
      mma16816<true>(S, af, qb[ks][0], qb[ks][1]);
      mma16816<true>(S2, ag, qb[ks + 1][0], qb[ks + 1][1]);
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) S[e] += S2[e];
    const int pos0 = tiles[tile0 + it] * kTileKeys;
    float x[4];                               // [key gq][e], [key gq + 8][e]
#pragma unroll
    for (int e = 0; e < 4; ++e) x[e] = S[e] * sc;
    if (!whole(pos0)) {
      const int key0 = pos0 + 16 * warp + gq;
      if (!(key0 < n && key_visible(pos, key0, a.window, a.keep_first))) x[0] = x[1] = -INFINITY;
      if (!(key0 + 8 < n && key_visible(pos, key0 + 8, a.window, a.keep_first))) x[2] = x[3] = -INFINITY;
    }
    const float mx[2] = {fmaxf(x[0], x[2]), fmaxf(x[1], x[3])};
    if (__any_sync(0xffffffffu, mx[0] > mref[0] + kRaise || mx[1] > mref[1] + kRaise)) {
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        float w = mx[e];
        w = fmaxf(w, __shfl_xor_sync(0xffffffffu, w, 4));
        w = fmaxf(w, __shfl_xor_sync(0xffffffffu, w, 8));
        w = fmaxf(w, __shfl_xor_sync(0xffffffffu, w, 16));
        const float m_new = fmaxf(mref[e], w);
        const float alpha = exp2f(mref[e] - m_new);
        L[e] *= alpha;
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) { O[mt][e] *= alpha; O[mt][2 + e] *= alpha; }
        mref[e] = m_new;
      }
    }
    float p[4];
    p[0] = ex2(x[0] - mref[0]); p[1] = ex2(x[1] - mref[1]);
    p[2] = ex2(x[2] - mref[0]); p[3] = ex2(x[3] - mref[1]);
    L[0] += p[0] + p[2]; L[1] += p[1] + p[3];
    const uint32_t h01 = pack2<true>(p[0], p[1]), h23 = pack2<true>(p[2], p[3]);
    const float2 f01 = unpack2<true>(h01), f23 = unpack2<true>(h23);
    const uint32_t l01 = pack2<true>(p[0] - f01.x, p[1] - f01.y), l23 = pack2<true>(p[2] - f23.x, p[3] - f23.y);
    const bool rem = COLS == 4 && tq >= 2;                       // this thread's columns 2 tq, 2 tq + 1 carry remainders
    const uint32_t pb0 = movmatrix_trans(rem ? l01 : h01), pb1 = movmatrix_trans(rem ? l23 : h23);
    uint32_t lb0 = 0u, lb1 = 0u;
    if constexpr (COLS == 8) { lb0 = movmatrix_trans(l01); lb1 = movmatrix_trans(l23); }
#pragma unroll
    for (int mt = 0; mt < MT; mt += 4) {
      uint32_t af[4][4];
#pragma unroll
      for (int q = 0; q < 4; ++q) ldsm_x4_trans(Vsm + tile_off(16 * warp + vk, 16 * (mt + q) + vm, VD), af[q]);
#pragma unroll
      for (int q = 0; q < 4; ++q) mma16816<true>(O[mt + q], af[q], pb0, pb1);
      if constexpr (COLS == 8) {
#pragma unroll
        for (int q = 0; q < 4; ++q) mma16816<true>(O[mt + q], af[q], lb0, lb1);
      }
    }
  }
  cp_async_wait<0>();
  __syncthreads();

  // merge the four warps (over the stage buffers)
  float* s_o = reinterpret_cast<float*>(sm);                     // [4][8][OLD]
  float* s_m = s_o + 4 * 8 * OLD;
  float* s_l = s_m + 32;
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    L[e] += __shfl_xor_sync(0xffffffffu, L[e], 4); L[e] += __shfl_xor_sync(0xffffffffu, L[e], 8);
    L[e] += __shfl_xor_sync(0xffffffffu, L[e], 16);
    if (gq == 0) s_m[warp * 8 + 2 * tq + e] = mref[e];
  }
  __syncthreads();
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int c = 2 * tq + e;
    const float M = fmaxf(fmaxf(s_m[c], s_m[8 + c]), fmaxf(s_m[16 + c], s_m[24 + c]));
    const float w = exp2f(mref[e] - M);
    if (gq == 0) s_l[warp * 8 + c] = L[e] * w;
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {
      s_o[(warp * 8 + c) * OLD + 16 * mt + gq] = O[mt][e] * w;
      s_o[(warp * 8 + c) * OLD + 16 * mt + gq + 8] = O[mt][2 + e] * w;
    }
  }
  __syncthreads();
  auto total = [&](int c, int d) {            // the four warps, both terms
    float v = 0.f;
#pragma unroll
    for (int t = 0; t < 8 / COLS; ++t)
#pragma unroll
      for (int w = 0; w < 4; ++w) v += s_o[(8 * w + COLS * t + c) * OLD + d];
    return v;
  };
  if (direct) {
    for (int i = tid; i < nh * VD; i += 128) {
      const int c = i / VD, d = i - c * VD;
      const float M = fmaxf(fmaxf(s_m[c], s_m[8 + c]), fmaxf(s_m[16 + c], s_m[24 + c])), s2 = a.sink * kLog2e;
      const float M2 = fmaxf(M, s2), w = exp2f(M - M2);
      const float l = (s_l[c] + s_l[8 + c] + s_l[16 + c] + s_l[24 + c]) * w + exp2f(s2 - M2);
      const float acc = total(c, d) * w;
      finish(c, d, l > 0.f ? acc / l : 0.f);
    }
    return;
  }
  for (int i = tid; i < MAPS * GC * VD; i += 128) {
    const int c = i / VD, d = i - c * VD;
    if (c % GC >= nh) continue;
    sacc[part(c) * VD + d] = total(c, d);
  }
  if (tid < MAPS * GC && tid % GC < nh) {
    const int c = tid;
    const int64_t p = part(c);
    stats[2 * p] = fmaxf(fmaxf(s_m[c], s_m[8 + c]), fmaxf(s_m[16 + c], s_m[24 + c]));
    stats[2 * p + 1] = s_l[c] + s_l[8 + c] + s_l[16 + c] + s_l[24 + c];
  }
}

// One CTA of VD threads per (sequence, head): the key ranges of both maps, then their combination.
template <int MAPS, int VD>
__global__ void __launch_bounds__(VD)
softmax_decode_merge_kernel(const atma_softmax_args a) {
  __shared__ float s_part[VD / 32];
  const int h = blockIdx.x, b = blockIdx.y, d = threadIdx.x;
  __nv_bfloat16* out = static_cast<__nv_bfloat16*>(a.out) + b * a.out_rs + (int64_t)h * VD + d;
  if (a.start_pos[b] < 0) { *out = __float2bfloat16_rn(0.f); return; }
  const float* stats = a.scratch;
  const float* sacc = a.scratch + (int64_t)a.n_seqs * a.H * MAPS * a.n_splits * 2;
  float o[MAPS];
#pragma unroll
  for (int m = 0; m < MAPS; ++m) {
    const int64_t p0 = (((int64_t)b * a.H + h) * MAPS + m) * a.n_splits;
    const float s2 = a.sink * kLog2e;
    float M = fmaxf(kNegBig, s2);
    for (int s = 0; s < a.n_splits; ++s) M = fmaxf(M, stats[2 * (p0 + s)]);
    float l = exp2f(s2 - M), acc = 0.f;
    for (int s = 0; s < a.n_splits; ++s) {
      const float w = exp2f(stats[2 * (p0 + s)] - M);
      l = fmaf(stats[2 * (p0 + s) + 1], w, l);
      acc = fmaf(sacc[(p0 + s) * VD + d], w, acc);
    }
    o[m] = l > 0.f ? acc / l : 0.f;
  }
  float v = o[0];
  if constexpr (MAPS == 2) {
    v = o[0] - a.lambda * o[MAPS - 1];
    float ss = warp_sum(v * v);
    if ((d & 31) == 0) s_part[d >> 5] = ss;
    __syncthreads();
    ss = 0.f;
#pragma unroll
    for (int i = 0; i < VD / 32; ++i) ss += s_part[i];
    v *= a.out_scale / sqrtf(ss / (float)VD + a.eps);
  }
  if (a.gate != nullptr) v *= sigmoid_gate(static_cast<const __nv_bfloat16*>(a.gate)[b * a.gate_rs + (int64_t)h * VD + d]);
  *out = __float2bfloat16_rn(v);
}

template <int MAPS, int DIM, int VD>
int launch(const atma_softmax_args& a, cudaStream_t st) {
  constexpr int kStage = kTileKeys * (MAPS * DIM + VD) * 2;
  constexpr int kStages = kStage * 3 * 2 <= 224 * 1024 ? 3 : 2;
  constexpr int kMerge = (4 * 8 * (VD + 4) + 64) * 4;
  constexpr int smem = kStages * kStage > kMerge ? kStages * kStage : kMerge;
  const int rep = a.H / a.G;
  const int cols = rep * MAPS <= 4 ? 4 : 8, gc = cols / MAPS;
  auto kern = cols == 4 ? softmax_decode_split_kernel<MAPS, DIM, VD, kStages, 4> : softmax_decode_split_kernel<MAPS, DIM, VD, kStages, 8>;
  ATMA_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
  kern<<<dim3(a.n_splits, a.G * ((rep + gc - 1) / gc), a.n_seqs), 128, smem, st>>>(a);
  if (MAPS == 2 || a.n_splits > 1) softmax_decode_merge_kernel<MAPS, VD><<<dim3(a.H, a.n_seqs), VD, 0, st>>>(a);
  return launch_status("softmax_decode (mma)");
}

}  // namespace

bool softmax_decode_mma_supported(const atma_softmax_args& a) {
  auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  return a.dtype == ATMA_BF16 && (a.dim == 64 || a.dim == 128) && (a.vdim == 64 || a.vdim == 128) && (a.maps == 1 || a.maps == 2) &&
         al(a.q) && al(a.k_cache) && al(a.v_cache);
}

int softmax_decode_mma(const atma_softmax_args& a, cudaStream_t st) {
  ATMA_REQUIRE(a.n_splits <= 65535 && (int64_t)a.G * ((a.H / a.G + 3) / 4 * 2) <= 65535, "softmax_decode: grid limits");
#define ATMA_SD(M, D, V) return launch<M, D, V>(a, st)
#define ATMA_SDV(M, D) do { if (a.vdim == 64) ATMA_SD(M, D, 64); else ATMA_SD(M, D, 128); } while (0)
  if (a.maps == 1) { if (a.dim == 64) ATMA_SDV(1, 64); else ATMA_SDV(1, 128); }
  if (a.dim == 64) ATMA_SDV(2, 64);
  ATMA_SDV(2, 128);
#undef ATMA_SDV
#undef ATMA_SD
}

}  // namespace atma
