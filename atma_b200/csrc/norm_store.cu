// RMS norms of whole q and k projections, value mixing and the K/V cache write: one pass over the projection rows.
//
// One CTA per row.  A thread holds up to NV groups of VEC channels between the sums of squares (q and k at once) and the
// results; a group belongs to one part of the row (the vector form needs part widths that are multiples of VEC).
#include "common.cuh"
#include "../../include/atma_decoder.h"

namespace atma {

namespace {

constexpr int kThreads = 256;

struct NormStoreArgs {
  const void* z; int64_t z_rs;
  const int64_t* slot_mapping;
  const void *wq, *wk, *v_first;
  int64_t v_first_rs;
  float lambda, eps;
  void *q_out, *k_cache, *v_cache;
  int nq, nk, nv;
};

template <typename T, int VEC, int NV>
__global__ void __launch_bounds__(kThreads)
norm_store_kernel(const NormStoreArgs a) {
  struct alignas(VEC * sizeof(T)) Pack { T e[VEC]; };
  __shared__ float s_q[kThreads / 32], s_k[kThreads / 32];
  const int64_t row = blockIdx.x;
  const int total = a.nq + a.nk + a.nv;
  const T* zr = static_cast<const T*>(a.z) + row * a.z_rs;
  Pack x[NV];
  float sq = 0.f, sk = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * (int)blockDim.x + (int)threadIdx.x) * VEC;
    if (c < total) x[i] = *reinterpret_cast<const Pack*>(zr + c);
  }
  const int64_t slot = a.slot_mapping[row];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * (int)blockDim.x + (int)threadIdx.x) * VEC;
    if (c >= a.nq + a.nk) continue;
    float ss = 0.f;
#pragma unroll
    for (int e = 0; e < VEC; ++e) { const float f = to_f32(x[i].e[e]); ss = fmaf(f, f, ss); }
    if (c < a.nq) sq += ss; else sk += ss;
  }
  sq = warp_sum(sq);
  sk = warp_sum(sk);
  if ((threadIdx.x & 31) == 0) { s_q[threadIdx.x >> 5] = sq; s_k[threadIdx.x >> 5] = sk; }
  __syncthreads();
  sq = sk = 0.f;
  for (int i = 0; i < (int)(blockDim.x >> 5); ++i) { sq += s_q[i]; sk += s_k[i]; }
  const float rq = 1.0f / sqrtf(sq / (float)a.nq + a.eps), rk = 1.0f / sqrtf(sk / (float)a.nk + a.eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * (int)blockDim.x + (int)threadIdx.x) * VEC;
    if (c >= total || (c >= a.nq && slot < 0)) continue;
    T* dst;
    if (c < a.nq + a.nk) {
      const bool is_q = c < a.nq;
      const int ch = is_q ? c : c - a.nq;
      const T* w = static_cast<const T*>(is_q ? a.wq : a.wk);
      if (w != nullptr) {
        const Pack wv = *reinterpret_cast<const Pack*>(w + ch);
        const float rs = is_q ? rq : rk;
#pragma unroll
        for (int e = 0; e < VEC; ++e) x[i].e[e] = from_f32<T>(to_f32(x[i].e[e]) * rs * to_f32(wv.e[e]));
      }
      dst = is_q ? static_cast<T*>(a.q_out) + row * a.nq + ch : static_cast<T*>(a.k_cache) + slot * a.nk + ch;
    } else {
      const int ch = c - a.nq - a.nk;
      if (a.v_first != nullptr) {
        const Pack f = *reinterpret_cast<const Pack*>(static_cast<const T*>(a.v_first) + row * a.v_first_rs + ch);
#pragma unroll
        for (int e = 0; e < VEC; ++e) x[i].e[e] = from_f32<T>((1.0f - a.lambda) * to_f32(x[i].e[e]) + a.lambda * to_f32(f.e[e]));
      }
      dst = static_cast<T*>(a.v_cache) + slot * a.nv + ch;
    }
    *reinterpret_cast<Pack*>(dst) = x[i];
  }
}

template <typename T, int VEC>
int launch(const NormStoreArgs& a, int rows, cudaStream_t st) {
  const int groups = (a.nq + a.nk + a.nv) / VEC;
  // many rows: two groups per thread, which halves what the sums and roots cost per channel; few rows: the shorter chain
  const int nv = max((groups + kThreads - 1) / kThreads, rows >= 2048 && groups >= 128 ? 2 : 1);
  ATMA_REQUIRE(nv <= 32, "norm_store: rows of %d channels", groups * VEC);
  const auto threads = [&](int n) { return min(kThreads, ((groups + n - 1) / n + 31) / 32 * 32); };
  if (nv <= 1) norm_store_kernel<T, VEC, 1><<<rows, threads(1), 0, st>>>(a);
  else if (nv <= 2) norm_store_kernel<T, VEC, 2><<<rows, threads(2), 0, st>>>(a);
  else if (nv <= 4) norm_store_kernel<T, VEC, 4><<<rows, threads(4), 0, st>>>(a);
  else if (nv <= 8) norm_store_kernel<T, VEC, 8><<<rows, threads(8), 0, st>>>(a);
  else norm_store_kernel<T, VEC, 32><<<rows, threads(32), 0, st>>>(a);
  return launch_status("norm_store");
}

}  // namespace
}  // namespace atma

using namespace atma;

extern "C" int atma_norm_store(const void* z, int64_t z_rs, const int64_t* slot_mapping, const void* wq, const void* wk,
                               const void* v_first, int64_t v_first_rs, float lambda, float eps, void* q_out, void* k_cache,
                               void* v_cache, int rows, int q_width, int k_width, int v_width, int dtype, void* stream) {
  ATMA_REQUIRE(dtype == ATMA_F32 || dtype == ATMA_BF16, "norm_store: unsupported dtype %d", dtype);
  ATMA_REQUIRE(q_width > 0 && k_width > 0 && v_width > 0, "norm_store: bad shape");
  if (rows <= 0) return ATMA_OK;
  const NormStoreArgs a{z, z_rs, slot_mapping, wq, wk, v_first, v_first_rs, lambda, eps, q_out, k_cache, v_cache, q_width, k_width, v_width};
  const int V = dtype == ATMA_F32 ? 4 : 8;
  auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  const bool vec = q_width % V == 0 && k_width % V == 0 && v_width % V == 0 && z_rs % V == 0 && v_first_rs % V == 0 && al(z) && al(wq) &&
                   al(wk) && al(v_first) && al(q_out) && al(k_cache) && al(v_cache);
  cudaStream_t st = (cudaStream_t)stream;
  if (dtype == ATMA_F32) return vec ? launch<float, 4>(a, rows, st) : launch<float, 1>(a, rows, st);
  return vec ? launch<__nv_bfloat16, 8>(a, rows, st) : launch<__nv_bfloat16, 1>(a, rows, st);
}
