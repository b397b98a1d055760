// Rotary positions on q and k and the K/V cache write, one pass over the projection rows.  The table holds
// (cos, sin) per position and channel pair, so scaled frequencies and amplitudes are the caller's business.
#include "common.cuh"
#include "../../include/atma_decoder.h"

namespace atma {

namespace {

struct RotArgs {
  const void* z; int64_t z_rs;
  const int32_t* positions; const int64_t* slot_mapping;
  const float2* cs; int table_rows;
  void *q_out, *k_cache, *v_cache;
  int rows, nq, nk, nv, dim, rot_dims;      // nq, nk, nv: channels of the q, k and v parts of a row
};

// One thread = VEC consecutive channels of one row (VEC even, or 1: the partner channel is read from the row).
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
rotary_store_kernel(const RotArgs a) {
  struct alignas(VEC * sizeof(T)) Vec { T e[VEC]; };
  const int per_row = (a.nq + a.nk + a.nv) / VEC;
  const int64_t i = (int64_t)blockIdx.x * 256 + threadIdx.x;
  const int64_t row = i / per_row;
  if (row >= a.rows) return;
  const int c = (int)(i - row * per_row) * VEC;
  const int64_t slot = a.slot_mapping[row];
  if (c >= a.nq && slot < 0) return;
  const T* zr = static_cast<const T*>(a.z) + row * a.z_rs;
  Vec x = *reinterpret_cast<const Vec*>(zr + c);
  if (c < a.nq + a.nk) {
    const int ch = (c < a.nq ? c : c - a.nq) % a.dim;       // channel inside its map
    if (ch < a.rot_dims) {
      const int pos = min(max(a.positions[row], 0), a.table_rows - 1);
      const float2* cs = a.cs + (int64_t)pos * (a.rot_dims / 2);
      if constexpr (VEC == 1) {
        const float2 t = cs[ch >> 1];
        const float self = to_f32(x.e[0]), other = to_f32(zr[(ch & 1) ? c - 1 : c + 1]);
        x.e[0] = from_f32<T>((ch & 1) ? self * t.x + other * t.y : self * t.x - other * t.y);
      } else {
#pragma unroll
        for (int e = 0; e < VEC; e += 2) {
          if (ch + e < a.rot_dims) {
            const float2 t = cs[(ch + e) >> 1];
            const float u = to_f32(x.e[e]), v = to_f32(x.e[e + 1]);
            x.e[e] = from_f32<T>(u * t.x - v * t.y);
            x.e[e + 1] = from_f32<T>(v * t.x + u * t.y);
          }
        }
      }
    }
  }
  T* dst;
  if (c < a.nq) dst = static_cast<T*>(a.q_out) + row * a.nq + c;
  else if (c < a.nq + a.nk) dst = static_cast<T*>(a.k_cache) + slot * a.nk + (c - a.nq);
  else dst = static_cast<T*>(a.v_cache) + slot * a.nv + (c - a.nq - a.nk);
  *reinterpret_cast<Vec*>(dst) = x;
}

}  // namespace
}  // namespace atma

using namespace atma;

extern "C" int atma_rotary_store(const void* z, int64_t z_rs, const int32_t* positions, const int64_t* slot_mapping,
                                 const float* cos_sin, int table_rows, void* q_out, void* k_cache, void* v_cache, int rows, int H,
                                 int G, int maps, int dim, int vdim, int rot_dims, int dtype, void* stream) {
  ATMA_REQUIRE(dtype == ATMA_F32 || dtype == ATMA_BF16, "rotary_store: unsupported dtype %d", dtype);
  ATMA_REQUIRE(H > 0 && G > 0 && H % G == 0 && maps > 0 && dim > 0 && vdim > 0, "rotary_store: bad shape");
  ATMA_REQUIRE(rot_dims >= 0 && rot_dims % 2 == 0 && rot_dims <= dim, "rotary_store: %d rotated channels of %d", rot_dims, dim);
  ATMA_REQUIRE(rot_dims == 0 || (cos_sin != nullptr && table_rows > 0), "rotary_store: empty table");
  if (rows <= 0) return ATMA_OK;
  RotArgs a{z, z_rs, positions, slot_mapping, (const float2*)cos_sin, table_rows, q_out, k_cache, v_cache,
            rows, H * maps * dim, G * maps * dim, G * vdim, dim, rot_dims};
  auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  const int V = dtype == ATMA_F32 ? 4 : 8;
  const bool vec = dim % V == 0 && vdim % V == 0 && z_rs % V == 0 && al(z) && al(q_out) && al(k_cache) && al(v_cache);
  const int64_t n = (int64_t)rows * ((a.nq + a.nk + a.nv) / (vec ? V : 1));
  const unsigned grid = (unsigned)((n + 255) / 256);
  cudaStream_t st = (cudaStream_t)stream;
  if (dtype == ATMA_F32) {
    if (vec) rotary_store_kernel<float, 4><<<grid, 256, 0, st>>>(a);
    else rotary_store_kernel<float, 1><<<grid, 256, 0, st>>>(a);
  } else {
    if (vec) rotary_store_kernel<__nv_bfloat16, 8><<<grid, 256, 0, st>>>(a);
    else rotary_store_kernel<__nv_bfloat16, 1><<<grid, 256, 0, st>>>(a);
  }
  return launch_status("rotary_store");
}
