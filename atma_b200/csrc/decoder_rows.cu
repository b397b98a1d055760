// Row operations of the decoder models: token + bigram embedding, the fp32 residual stream with its zero-centred
// RMS norms, the gelu-gated feed-forward product and the per-head norm with a silu gate.  Everything is one pass
// over rows, 16 bytes per thread and access where the shapes allow it.
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

extern "C" int atma_decoder_abi_version(void) { return 1; }

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
