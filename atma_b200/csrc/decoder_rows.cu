// Row operations of the decoder models: token + bigram and token + learned-position embeddings, the fp32 residual
// stream with RMS norms of the stream or of what a sublayer adds to it, the feed-forward activations and the per-head
// norm with a silu gate.  Everything is one pass over rows, 16 bytes per thread and access where the shapes allow it.
#include "common.cuh"
#include "../../include/atma_decoder.h"

namespace atma {

namespace {

// VEC values of type T as one access (VEC * sizeof(T) = 4, 8 or 16 bytes), or one scalar.
template <typename T, int VEC>
struct alignas(VEC * sizeof(T)) Pack { T e[VEC]; };

inline bool aligned(const void* p, int n) { return (reinterpret_cast<uintptr_t>(p) & (uintptr_t)(n - 1)) == 0; }

// ---- x = embed[id] + bigram[row] -----------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(128)
embed_bigram_kernel(const int32_t* __restrict__ ids, const int32_t* __restrict__ prev, const T* __restrict__ embed,
                    const T* __restrict__ bigram, float* __restrict__ x, int D, int vocab, int64_t mul_prev, int64_t mul_cur,
                    int64_t buckets) {
  const int row = blockIdx.x;
  const int64_t id = min(max(ids[row], 0), vocab - 1);
  const int64_t pv = prev[row];
  const T* e = embed + id * D;
  const T* g = nullptr;
  if (bigram != nullptr) {
    int64_t r = buckets;
    if (pv >= 0) {
      r = (pv * mul_prev + id * mul_cur) % buckets;
      if (r < 0) r += buckets;
    }
    g = bigram + r * D;
  }
  for (int c = threadIdx.x; c < D; c += 128) x[(int64_t)row * D + c] = to_f32(e[c]) + (g != nullptr ? to_f32(g[c]) : 0.f);
}

// ---- residual add and up to two norms of the sum ---------------------------------------------------
constexpr int kNormThreads = 256;

// One CTA per row; the row stays in registers between the sum of squares and the outputs.
template <typename T, int NV>
__global__ void __launch_bounds__(kNormThreads)
residual_norms_kernel(const float* __restrict__ x, const T* __restrict__ y, float* __restrict__ x_out, const T* __restrict__ w1,
                      T* __restrict__ h1, const T* __restrict__ w2, T* __restrict__ h2, int D, float eps, float offset) {
  __shared__ float s_part[kNormThreads / 32];
  const int64_t base = (int64_t)blockIdx.x * D;
  const int tid = threadIdx.x;
  float4 v[NV];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * kNormThreads + tid) * 4;
    v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < D) {
      v[i] = *reinterpret_cast<const float4*>(x + base + c);
      if (y != nullptr) {
        const Pack<T, 4> p = *reinterpret_cast<const Pack<T, 4>*>(y + base + c);
        v[i].x += to_f32(p.e[0]); v[i].y += to_f32(p.e[1]); v[i].z += to_f32(p.e[2]); v[i].w += to_f32(p.e[3]);
      }
    }
    ss = fmaf(v[i].x, v[i].x, fmaf(v[i].y, v[i].y, fmaf(v[i].z, v[i].z, fmaf(v[i].w, v[i].w, ss))));
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) s_part[tid >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
  for (int i = 0; i < (int)(blockDim.x >> 5); ++i) tot += s_part[i];
  const float rs = 1.0f / sqrtf(tot / (float)D + eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * kNormThreads + tid) * 4;
    if (c >= D) continue;
    if (x_out != nullptr) *reinterpret_cast<float4*>(x_out + base + c) = v[i];
    const float f[4] = {v[i].x * rs, v[i].y * rs, v[i].z * rs, v[i].w * rs};
    if (h1 != nullptr) {
      const Pack<T, 4> p = *reinterpret_cast<const Pack<T, 4>*>(w1 + c);
      Pack<T, 4> o;
#pragma unroll
      for (int e = 0; e < 4; ++e) o.e[e] = from_f32<T>(f[e] * (offset + to_f32(p.e[e])));
      *reinterpret_cast<Pack<T, 4>*>(h1 + base + c) = o;
    }
    if (h2 != nullptr) {
      const Pack<T, 4> p = *reinterpret_cast<const Pack<T, 4>*>(w2 + c);
      Pack<T, 4> o;
#pragma unroll
      for (int e = 0; e < 4; ++e) o.e[e] = from_f32<T>(f[e] * (offset + to_f32(p.e[e])));
      *reinterpret_cast<Pack<T, 4>*>(h2 + base + c) = o;
    }
  }
}

// Any width: the sum is recomputed in the second pass.
template <typename T>
__global__ void __launch_bounds__(kNormThreads)
residual_norms_any_kernel(const float* x, const T* __restrict__ y, float* x_out, const T* __restrict__ w1, T* __restrict__ h1,
                          const T* __restrict__ w2, T* __restrict__ h2, int D, float eps, float offset) {
  __shared__ float s_part[kNormThreads / 32];
  const int64_t base = (int64_t)blockIdx.x * D;
  const int tid = threadIdx.x;
  float ss = 0.f;
  for (int c = tid; c < D; c += kNormThreads) {
    const float v = x[base + c] + (y != nullptr ? to_f32(y[base + c]) : 0.f);
    ss = fmaf(v, v, ss);
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) s_part[tid >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
  for (int i = 0; i < kNormThreads / 32; ++i) tot += s_part[i];
  const float rs = 1.0f / sqrtf(tot / (float)D + eps);
  for (int c = tid; c < D; c += kNormThreads) {          // the same thread reads and writes column c: in place is fine
    const float v = x[base + c] + (y != nullptr ? to_f32(y[base + c]) : 0.f);
    if (x_out != nullptr) x_out[base + c] = v;
    if (h1 != nullptr) h1[base + c] = from_f32<T>(v * rs * (offset + to_f32(w1[c])));
    if (h2 != nullptr) h2[base + c] = from_f32<T>(v * rs * (offset + to_f32(w2[c])));
  }
}

// ---- rows that are normalised before they enter the residual stream -----------------------------------
// Sum over the CTA, the same value in every thread.  Two calls use different halves of s_part.
__device__ __forceinline__ float cta_sum(float v, float* s_part) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) s_part[threadIdx.x >> 5] = v;
  __syncthreads();
  float tot = 0.f;
  for (int i = 0; i < (int)(blockDim.x >> 5); ++i) tot += s_part[i];
  return tot;
}

// Loads and stores of VEC (4 or 1) consecutive channels as fp32.
template <int VEC>
__device__ __forceinline__ void load_f32(const float* p, float (&f)[VEC]) {
  const Pack<float, VEC> v = *reinterpret_cast<const Pack<float, VEC>*>(p);
#pragma unroll
  for (int e = 0; e < VEC; ++e) f[e] = v.e[e];
}
template <typename T, int VEC>
__device__ __forceinline__ void load_t(const T* p, float (&f)[VEC]) {
  const Pack<T, VEC> v = *reinterpret_cast<const Pack<T, VEC>*>(p);
#pragma unroll
  for (int e = 0; e < VEC; ++e) f[e] = to_f32(v.e[e]);
}
template <typename T, int VEC>
__device__ __forceinline__ void store_t(T* p, const float (&f)[VEC]) {
  Pack<T, VEC> v;
#pragma unroll
  for (int e = 0; e < VEC; ++e) v.e[e] = from_f32<T>(f[e]);
  *reinterpret_cast<Pack<T, VEC>*>(p) = v;
}

struct EmbedNormArgs {
  const int32_t *ids, *positions;
  const void *embed, *pos, *w;
  float* x;
  void* h;
  int D, vocab, max_positions;
  float scale, eps, offset;
};

// One CTA per row, up to NV groups of VEC channels per thread held between the sum of squares and the result.
template <typename T, int VEC, int NV>
__global__ void __launch_bounds__(kNormThreads)
embed_position_norm_kernel(const EmbedNormArgs a) {
  __shared__ float s_part[kNormThreads / 32];
  const int64_t row = blockIdx.x;
  const T* e = static_cast<const T*>(a.embed) + (int64_t)min(max(a.ids[row], 0), a.vocab - 1) * a.D;
  const T* p = a.pos == nullptr ? nullptr : static_cast<const T*>(a.pos) + (int64_t)min(max(a.positions[row], 0), a.max_positions - 1) * a.D;
  const T* w = static_cast<const T*>(a.w);
  float v[NV][VEC];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * (int)blockDim.x + (int)threadIdx.x) * VEC;
    if (c >= a.D) continue;
    load_t<T, VEC>(e + c, v[i]);
#pragma unroll
    for (int k = 0; k < VEC; ++k) v[i][k] *= a.scale;
    if (p != nullptr) {
      float q[VEC];
      load_t<T, VEC>(p + c, q);
#pragma unroll
      for (int k = 0; k < VEC; ++k) v[i][k] += q[k];
    }
#pragma unroll
    for (int k = 0; k < VEC; ++k) ss = fmaf(v[i][k], v[i][k], ss);
  }
  const float rs = 1.0f / sqrtf(cta_sum(ss, s_part) / (float)a.D + a.eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * (int)blockDim.x + (int)threadIdx.x) * VEC;
    if (c >= a.D) continue;
    float g[VEC];
    load_t<T, VEC>(w + c, g);
#pragma unroll
    for (int k = 0; k < VEC; ++k) v[i][k] = v[i][k] * rs * (a.offset + g[k]);
    store_t<float, VEC>(a.x + row * a.D + c, v[i]);
    if (a.h != nullptr) store_t<T, VEC>(static_cast<T*>(a.h) + row * a.D + c, v[i]);
  }
}

struct PostNormArgs {
  const float* x;
  const void *y, *bias, *w;
  float* x_out;
  void* h;
  const void* w_next;
  int D;
  float eps, offset;
};

template <typename T, int VEC, int NV>
__global__ void __launch_bounds__(kNormThreads)
residual_post_norm_kernel(const PostNormArgs a) {
  __shared__ float s_part[2][kNormThreads / 32];
  const int64_t base = (int64_t)blockIdx.x * a.D;
  const T *y = static_cast<const T*>(a.y) + base, *bias = static_cast<const T*>(a.bias), *w = static_cast<const T*>(a.w);
  float v[NV][VEC], x[NV][VEC];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * (int)blockDim.x + (int)threadIdx.x) * VEC;
    if (c >= a.D) continue;
    load_t<T, VEC>(y + c, v[i]);
    load_f32<VEC>(a.x + base + c, x[i]);
    if (bias != nullptr) {
      float b[VEC];
      load_t<T, VEC>(bias + c, b);
#pragma unroll
      for (int k = 0; k < VEC; ++k) v[i][k] += b[k];
    }
#pragma unroll
    for (int k = 0; k < VEC; ++k) ss = fmaf(v[i][k], v[i][k], ss);
  }
  const float rs = 1.0f / sqrtf(cta_sum(ss, s_part[0]) / (float)a.D + a.eps);
  ss = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * (int)blockDim.x + (int)threadIdx.x) * VEC;
    if (c >= a.D) continue;
    float g[VEC];
    load_t<T, VEC>(w + c, g);
#pragma unroll
    for (int k = 0; k < VEC; ++k) {
      x[i][k] = fmaf(v[i][k] * rs, a.offset + g[k], x[i][k]);
      ss = fmaf(x[i][k], x[i][k], ss);
    }
    if (a.x_out != nullptr) store_t<float, VEC>(a.x_out + base + c, x[i]);
    if (a.h != nullptr && a.w_next == nullptr) store_t<T, VEC>(static_cast<T*>(a.h) + base + c, x[i]);
  }
  if (a.h == nullptr || a.w_next == nullptr) return;               // the same for every thread
  const float rn = 1.0f / sqrtf(cta_sum(ss, s_part[1]) / (float)a.D + a.eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * (int)blockDim.x + (int)threadIdx.x) * VEC;
    if (c >= a.D) continue;
    float g[VEC];
    load_t<T, VEC>(static_cast<const T*>(a.w_next) + c, g);
#pragma unroll
    for (int k = 0; k < VEC; ++k) g[k] = x[i][k] * rn * (a.offset + g[k]);
    store_t<T, VEC>(static_cast<T*>(a.h) + base + c, g);
  }
}

// Groups per thread and threads of a row of D channels; 0 groups: the row is too wide.
template <int VEC>
inline int row_groups(int D, int* threads) {
  const int g = (D + VEC - 1) / VEC;
  const int nv = (g + kNormThreads - 1) / kNormThreads;
  for (int n = 1; n <= 16; n *= 2)
    if (nv <= n) {
      *threads = min(kNormThreads, ((g + n - 1) / n + 31) / 32 * 32);
      return n;
    }
  return 0;
}

// ---- relu(z + bias)^2 ---------------------------------------------------------------------------------
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
bias_squared_relu_kernel(const T* z, int64_t z_rs, const T* __restrict__ bias, T* out, int64_t out_rs, int rows, int width) {
  const int c = (blockIdx.x * 256 + threadIdx.x) * VEC;
  if (c >= width) return;
  float b[VEC] = {};
  if (bias != nullptr) load_t<T, VEC>(bias + c, b);
  // rows 4 at a time: their loads are in flight together
  for (int64_t row = (int64_t)blockIdx.y * 4; row < rows; row += (int64_t)gridDim.y * 4) {
    float f[4][VEC];
#pragma unroll
    for (int r = 0; r < 4; ++r)
      if (row + r < rows) load_t<T, VEC>(z + (row + r) * z_rs + c, f[r]);
#pragma unroll
    for (int r = 0; r < 4; ++r) {
      if (row + r >= rows) continue;
#pragma unroll
      for (int k = 0; k < VEC; ++k) {
        const float t = fmaxf(f[r][k] + b[k], 0.f);
        f[r][k] = t * t;
      }
      store_t<T, VEC>(out + (row + r) * out_rs + c, f[r]);
    }
  }
}

// ---- gelu_tanh(gate) * up ---------------------------------------------------------------------------
__device__ __forceinline__ float gelu_tanh(float z) {
  const float c = 0.7978845608028654f;                    // sqrt(2 / pi)
  return 0.5f * z * (1.0f + tanhf(c * fmaf(0.044715f * z * z, z, z)));
}

template <typename T, int VEC>
__global__ void gelu_gate_kernel(const T* __restrict__ gate, int64_t gate_rs, const T* __restrict__ up, int64_t up_rs,
                                 T* __restrict__ out, int64_t out_rs, int width) {
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * VEC;
  if (c >= width) return;
  const int64_t row = blockIdx.y;
  const Pack<T, VEC> g = *reinterpret_cast<const Pack<T, VEC>*>(gate + row * gate_rs + c);
  const Pack<T, VEC> u = *reinterpret_cast<const Pack<T, VEC>*>(up + row * up_rs + c);
  Pack<T, VEC> o;
#pragma unroll
  for (int e = 0; e < VEC; ++e) o.e[e] = from_f32<T>(gelu_tanh(to_f32(g.e[e])) * to_f32(u.e[e]));
  *reinterpret_cast<Pack<T, VEC>*>(out + row * out_rs + c) = o;
}

// ---- o / rms(o) * w * silu(gate), per head -----------------------------------------------------------
// LANES threads share a head row, VEC channels each; heads wider than LANES * VEC take several rounds.
template <typename T, int VEC, int LANES>
__global__ void __launch_bounds__(256)
head_norm_silu_gate_kernel(const T* __restrict__ o, const T* __restrict__ w, const T* __restrict__ gate, int64_t gate_rs,
                           T* __restrict__ out, int64_t out_rs, int64_t units, int H, int vdim, float eps) {
  const int64_t unit = ((int64_t)blockIdx.x * 256 + threadIdx.x) / LANES;
  const int l = threadIdx.x % LANES;
  const bool on = unit < units;
  const int64_t row = on ? unit / H : 0;
  const int h = on ? (int)(unit % H) : 0;
  const T* op = o + (row * H + h) * vdim;
  float ss = 0.f;
  if (on)
    for (int c = l * VEC; c < vdim; c += LANES * VEC) {
      const Pack<T, VEC> p = *reinterpret_cast<const Pack<T, VEC>*>(op + c);
#pragma unroll
      for (int e = 0; e < VEC; ++e) { const float f = to_f32(p.e[e]); ss = fmaf(f, f, ss); }
    }
#pragma unroll
  for (int s = LANES / 2; s > 0; s >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, s);
  if (!on) return;
  const float rs = 1.0f / sqrtf(ss / (float)vdim + eps);
  const T* gp = gate + row * gate_rs + (int64_t)h * vdim;
  T* outp = out + row * out_rs + (int64_t)h * vdim;
  for (int c = l * VEC; c < vdim; c += LANES * VEC) {
    const Pack<T, VEC> p = *reinterpret_cast<const Pack<T, VEC>*>(op + c);
    const Pack<T, VEC> g = *reinterpret_cast<const Pack<T, VEC>*>(gp + c);
    const Pack<T, VEC> wv = *reinterpret_cast<const Pack<T, VEC>*>(w + c);
    Pack<T, VEC> r;
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      const float gf = to_f32(g.e[e]);
      float sg;                                          // 16-bit results: the fast exponential and division
      if constexpr (sizeof(T) == 2) sg = __fdividef(gf, 1.0f + __expf(-gf));
      else sg = gf / (1.0f + expf(-gf));
      r.e[e] = from_f32<T>(to_f32(p.e[e]) * rs * to_f32(wv.e[e]) * sg);
    }
    *reinterpret_cast<Pack<T, VEC>*>(outp + c) = r;
  }
}

}  // namespace
}  // namespace atma

using namespace atma;

#define ATMA_DECODER_DISPATCH(dt, T, ...)                                    \
  do {                                                                      \
    if ((dt) == ATMA_F32) { using T = float; __VA_ARGS__; }                 \
    else { using T = __nv_bfloat16; __VA_ARGS__; }                          \
  } while (0)

#define ATMA_ROW_KERNEL(KERNEL, T, VEC, a)                                                                 \
  do {                                                                                                     \
    int threads = 0;                                                                                       \
    const int nv = row_groups<VEC>(a.D, &threads);                                                         \
    if (nv == 1) KERNEL<T, VEC, 1><<<rows, threads, 0, st>>>(a);                                           \
    else if (nv == 2) KERNEL<T, VEC, 2><<<rows, threads, 0, st>>>(a);                                      \
    else if (nv == 4) KERNEL<T, VEC, 4><<<rows, threads, 0, st>>>(a);                                      \
    else if (nv == 8) KERNEL<T, VEC, 8><<<rows, threads, 0, st>>>(a);                                      \
    else KERNEL<T, VEC, 16><<<rows, threads, 0, st>>>(a);                                                  \
  } while (0)

extern "C" int atma_decoder_abi_version(void) { return 2; }

extern "C" int atma_embed_position_norm(const int32_t* ids, const int32_t* positions, const void* embed, const void* pos, const void* w,
                                        float* x, void* h, int rows, int D, int vocab, int max_positions, float scale, float eps,
                                        float offset, int dtype, void* stream) {
  ATMA_REQUIRE(dtype == ATMA_F32 || dtype == ATMA_BF16, "embed_position_norm: unsupported dtype %d", dtype);
  ATMA_REQUIRE(D > 0 && vocab > 0 && w != nullptr && x != nullptr, "embed_position_norm: bad arguments");
  ATMA_REQUIRE(pos == nullptr || (positions != nullptr && max_positions > 0), "embed_position_norm: an empty position table");
  if (rows <= 0) return ATMA_OK;
  cudaStream_t st = (cudaStream_t)stream;
  const int vb = dtype == ATMA_F32 ? 16 : 8;
  const bool vec = D % 4 == 0 && aligned(x, 16) && aligned(embed, vb) && aligned(pos, vb) && aligned(w, vb) && aligned(h, vb);
  ATMA_REQUIRE(D <= kNormThreads * 16 * (vec ? 4 : 1), "embed_position_norm: rows of %d channels", D);
  const EmbedNormArgs a{ids, positions, embed, pos, w, x, h, D, vocab, max_positions, scale, eps, offset};
  ATMA_DECODER_DISPATCH(dtype, T, {
    if (vec) ATMA_ROW_KERNEL(embed_position_norm_kernel, T, 4, a);
    else ATMA_ROW_KERNEL(embed_position_norm_kernel, T, 1, a);
  });
  return launch_status("embed_position_norm");
}

extern "C" int atma_residual_post_norm(const float* x, const void* y, const void* bias, const void* w, float* x_out, void* h,
                                       const void* w_next, int rows, int D, float eps, float offset, int dtype, void* stream) {
  ATMA_REQUIRE(dtype == ATMA_F32 || dtype == ATMA_BF16, "residual_post_norm: unsupported dtype %d", dtype);
  ATMA_REQUIRE(D > 0 && x != nullptr && y != nullptr && w != nullptr, "residual_post_norm: bad arguments");
  if (rows <= 0) return ATMA_OK;
  cudaStream_t st = (cudaStream_t)stream;
  const int vb = dtype == ATMA_F32 ? 16 : 8;
  const bool vec = D % 4 == 0 && aligned(x, 16) && aligned(x_out, 16) && aligned(y, vb) && aligned(bias, vb) && aligned(w, vb) &&
                   aligned(h, vb) && aligned(w_next, vb);
  ATMA_REQUIRE(D <= kNormThreads * 16 * (vec ? 4 : 1), "residual_post_norm: rows of %d channels", D);
  const PostNormArgs a{x, y, bias, w, x_out, h, w_next, D, eps, offset};
  ATMA_DECODER_DISPATCH(dtype, T, {
    if (vec) ATMA_ROW_KERNEL(residual_post_norm_kernel, T, 4, a);
    else ATMA_ROW_KERNEL(residual_post_norm_kernel, T, 1, a);
  });
  return launch_status("residual_post_norm");
}

extern "C" int atma_bias_squared_relu(const void* z, int64_t z_rs, const void* bias, void* out, int64_t out_rs, int rows, int width,
                                      int dtype, void* stream) {
  ATMA_REQUIRE(dtype == ATMA_F32 || dtype == ATMA_BF16, "bias_squared_relu: unsupported dtype %d", dtype);
  if (rows <= 0 || width <= 0) return ATMA_OK;
  cudaStream_t st = (cudaStream_t)stream;
  ATMA_DECODER_DISPATCH(dtype, T, {
    constexpr int V = 16 / sizeof(T);
    const bool vec = width % V == 0 && z_rs % V == 0 && out_rs % V == 0 && aligned(z, 16) && aligned(bias, 16) && aligned(out, 16);
    const int per = 256 * (vec ? V : 1);
    const dim3 grid((width + per - 1) / per, min((rows + 3) / 4, 65535));
    const T *zp = (const T*)z, *bp = (const T*)bias;
    if (vec) bias_squared_relu_kernel<T, V><<<grid, 256, 0, st>>>(zp, z_rs, bp, (T*)out, out_rs, rows, width);
    else bias_squared_relu_kernel<T, 1><<<grid, 256, 0, st>>>(zp, z_rs, bp, (T*)out, out_rs, rows, width);
  });
  return launch_status("bias_squared_relu");
}

extern "C" int atma_embed_bigram(const int32_t* ids, const int32_t* prev, const void* embed, const void* bigram, float* x, int rows,
                                 int D, int vocab, int64_t mul_prev, int64_t mul_cur, int64_t buckets, int dtype, void* stream) {
  ATMA_REQUIRE(dtype == ATMA_F32 || dtype == ATMA_BF16, "embed_bigram: unsupported dtype %d", dtype);
  ATMA_REQUIRE(D > 0 && vocab > 0, "embed_bigram: bad shape");
  ATMA_REQUIRE(bigram == nullptr || buckets > 0, "embed_bigram: buckets must be positive");
  if (rows <= 0) return ATMA_OK;
  ATMA_DECODER_DISPATCH(dtype, T, {
    embed_bigram_kernel<T><<<rows, 128, 0, (cudaStream_t)stream>>>(ids, prev, (const T*)embed, (const T*)bigram, x, D, vocab,
                                                                   mul_prev, mul_cur, buckets);
  });
  return launch_status("embed_bigram");
}

extern "C" int atma_residual_norms(const float* x, const void* y, float* x_out, const void* w1, void* h1, const void* w2, void* h2,
                                   int rows, int D, float eps, float offset, int dtype, void* stream) {
  ATMA_REQUIRE(dtype == ATMA_F32 || dtype == ATMA_BF16, "residual_norms: unsupported dtype %d", dtype);
  ATMA_REQUIRE(D > 0 && x != nullptr, "residual_norms: bad arguments");
  ATMA_REQUIRE((h1 == nullptr || w1 != nullptr) && (h2 == nullptr || w2 != nullptr), "residual_norms: a norm without its weight");
  if (rows <= 0) return ATMA_OK;
  cudaStream_t st = (cudaStream_t)stream;
  const int vb = dtype == ATMA_F32 ? 16 : 8;
  const bool vec = D % 4 == 0 && D <= kNormThreads * 4 * 8 && aligned(x, 16) && aligned(x_out, 16) && aligned(y, vb) &&
                   aligned(w1, vb) && aligned(w2, vb) && aligned(h1, vb) && aligned(h2, vb);
  ATMA_DECODER_DISPATCH(dtype, T, {
    const T *yp = (const T*)y, *w1p = (const T*)w1, *w2p = (const T*)w2;
    T *h1p = (T*)h1, *h2p = (T*)h2;
    const int nv = (D / 4 + kNormThreads - 1) / kNormThreads;
    const int threads = min(kNormThreads, ((D / 4 + 31) / 32) * 32);
    if (!vec) residual_norms_any_kernel<T><<<rows, kNormThreads, 0, st>>>(x, yp, x_out, w1p, h1p, w2p, h2p, D, eps, offset);
    else if (nv <= 1) residual_norms_kernel<T, 1><<<rows, threads, 0, st>>>(x, yp, x_out, w1p, h1p, w2p, h2p, D, eps, offset);
    else if (nv <= 2) residual_norms_kernel<T, 2><<<rows, threads, 0, st>>>(x, yp, x_out, w1p, h1p, w2p, h2p, D, eps, offset);
    else if (nv <= 4) residual_norms_kernel<T, 4><<<rows, threads, 0, st>>>(x, yp, x_out, w1p, h1p, w2p, h2p, D, eps, offset);
    else residual_norms_kernel<T, 8><<<rows, threads, 0, st>>>(x, yp, x_out, w1p, h1p, w2p, h2p, D, eps, offset);
  });
  return launch_status("residual_norms");
}

extern "C" int atma_gelu_gate(const void* gate, int64_t gate_rs, const void* up, int64_t up_rs, void* out, int64_t out_rs, int rows,
                              int width, int dtype, void* stream) {
  ATMA_REQUIRE(dtype == ATMA_F32 || dtype == ATMA_BF16, "gelu_gate: unsupported dtype %d", dtype);
  if (rows <= 0 || width <= 0) return ATMA_OK;
  ATMA_REQUIRE(rows <= 65535 * 1024, "gelu_gate: too many rows");
  cudaStream_t st = (cudaStream_t)stream;
  ATMA_DECODER_DISPATCH(dtype, T, {
    constexpr int V = 16 / sizeof(T);
    const bool vec = width % V == 0 && gate_rs % V == 0 && up_rs % V == 0 && out_rs % V == 0 && aligned(gate, 16) && aligned(up, 16) &&
                     aligned(out, 16);
    for (int r0 = 0; r0 < rows; r0 += 65535) {             // grid.y limit
      const int nr = min(65535, rows - r0);
      const T *g = (const T*)gate + (int64_t)r0 * gate_rs, *u = (const T*)up + (int64_t)r0 * up_rs;
      T* o = (T*)out + (int64_t)r0 * out_rs;
      if (vec) gelu_gate_kernel<T, V><<<dim3((width / V + 127) / 128, nr), 128, 0, st>>>(g, gate_rs, u, up_rs, o, out_rs, width);
      else gelu_gate_kernel<T, 1><<<dim3((width + 127) / 128, nr), 128, 0, st>>>(g, gate_rs, u, up_rs, o, out_rs, width);
    }
  });
  return launch_status("gelu_gate");
}

extern "C" int atma_head_norm_silu_gate(const void* o, const void* w, const void* gate, int64_t gate_rs, void* out, int64_t out_rs,
                                        int rows, int H, int vdim, float eps, int dtype, void* stream) {
  ATMA_REQUIRE(dtype == ATMA_F32 || dtype == ATMA_BF16, "head_norm_silu_gate: unsupported dtype %d", dtype);
  ATMA_REQUIRE(H > 0 && vdim > 0, "head_norm_silu_gate: bad shape");
  if (rows <= 0) return ATMA_OK;
  cudaStream_t st = (cudaStream_t)stream;
  const int64_t units = (int64_t)rows * H;
  ATMA_DECODER_DISPATCH(dtype, T, {
    constexpr int V = 16 / sizeof(T);
    const T *op = (const T*)o, *wp = (const T*)w, *gp = (const T*)gate;
    T* outp = (T*)out;
    const bool vec = vdim % V == 0 && gate_rs % V == 0 && out_rs % V == 0 && aligned(o, 16) && aligned(w, 16) && aligned(gate, 16) &&
                     aligned(out, 16);
    if (vec) head_norm_silu_gate_kernel<T, V, 16><<<(unsigned)((units * 16 + 255) / 256), 256, 0, st>>>(op, wp, gp, gate_rs, outp, out_rs, units, H, vdim, eps);
    else head_norm_silu_gate_kernel<T, 1, 32><<<(unsigned)((units * 32 + 255) / 256), 256, 0, st>>>(op, wp, gp, gate_rs, outp, out_rs, units, H, vdim, eps);
  });
  return launch_status("head_norm_silu_gate");
}
