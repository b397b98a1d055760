// Causal softmax attention over a paged cache, fp32 arithmetic throughout: the path for fp32 models and for head sizes
// the tensor-core kernels do not serve, prompts and single tokens alike, with one or two maps per head, windows, a sink,
// the differential combination and the output gate.  Also the entry points that choose between the kernels.
//
// A CTA of eight warps holds 16 query rows of one head, two per warp.  Keys come in tiles of 32: a lane owns a key for
// the scores, and vdim / 32 value channels for the weighted sum, so the softmax statistics of a row are warp reductions.
#include "softmax_attention.cuh"

namespace atma {

namespace {

constexpr int kTK = 32, kWarps = 8, kRPW = 2, kTQ = kWarps * kRPW;

template <typename T, int M, int NC>
__global__ void __launch_bounds__(kWarps * 32)
softmax_rows_kernel(const atma_softmax_args a) {
  extern __shared__ float sm[];
  const int kd = M * a.dim, kld = kd + 1;
  float* sK = sm;                              // [32][kd + 1]
  float* sV = sK + kTK * kld;                  // [32][vdim]
  float* sQ = sV + kTK * a.vdim;               // [16][kd]
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int s = blockIdx.z, h = blockIdx.y;
  const int r_begin = a.cu_rows[s], n_rows = a.cu_rows[s + 1] - r_begin;
  const int q0 = blockIdx.x * kTQ;
  if (q0 >= n_rows) return;
  const int start = a.start_pos[s];
  const int g = h / (a.H / a.G);
  T* out = static_cast<T*>(a.out);
  if (start < 0) {                             // padded sequence
    for (int i = tid; i < min(kTQ, n_rows - q0) * a.vdim; i += kWarps * 32)
      out[(int64_t)(r_begin + q0 + i / a.vdim) * a.out_rs + (int64_t)h * a.vdim + i % a.vdim] = from_f32<T>(0.f);
    return;
  }
  const T* Q = static_cast<const T*>(a.q);
  const T* K = static_cast<const T*>(a.k_cache);
  const T* V = static_cast<const T*>(a.v_cache);
  for (int i = tid; i < kTQ * kd; i += kWarps * 32) {
    const int r = i / kd, c = i - r * kd;
    sQ[i] = (q0 + r < n_rows) ? to_f32(Q[((int64_t)(r_begin + q0 + r) * a.H + h) * kd + c]) * a.scale : 0.f;
  }
  const int last_pos = start + min(q0 + kTQ, n_rows) - 1;     // the last query's own position
  const int n_keys = min(last_pos + 1, a.max_blocks * a.block_size);
  const KeyTiles tiles(start + q0, last_pos, a.max_blocks * a.block_size, a.window, a.keep_first, kTK);
  const int32_t* bt = a.block_tables + s * a.bt_stride;

  float m[kRPW][M], l[kRPW][M], acc[kRPW][M][NC];
#pragma unroll
  for (int r = 0; r < kRPW; ++r)
#pragma unroll
    for (int t = 0; t < M; ++t) {
      m[r][t] = a.sink;                        // the sink is a key that was seen before the others
      l[r][t] = a.sink > -INFINITY ? 1.f : 0.f;
#pragma unroll
      for (int i = 0; i < NC; ++i) acc[r][t][i] = 0.f;
    }

  for (int kt = 0; kt < tiles.n; ++kt) {
    const int k0 = tiles[kt] * kTK;
    __syncthreads();
    for (int j = warp; j < kTK; j += kWarps) {                // a warp per key row
      const int pos = k0 + j;
      if (pos < n_keys) {
        const int blk = pos / a.block_size;
        const int phys = min(max(bt[blk], 0), a.num_blocks - 1);
        const int64_t slot = (int64_t)phys * a.block_size + (pos - blk * a.block_size);
        const T* kr = K + (slot * a.G + g) * kd;
        const T* vr = V + (slot * a.G + g) * a.vdim;
        for (int c = lane; c < kd; c += 32) sK[j * kld + c] = to_f32(kr[c]);
        for (int c = lane; c < a.vdim; c += 32) sV[j * a.vdim + c] = to_f32(vr[c]);
      } else {
        for (int c = lane; c < kd; c += 32) sK[j * kld + c] = 0.f;
        for (int c = lane; c < a.vdim; c += 32) sV[j * a.vdim + c] = 0.f;
      }
    }
    __syncthreads();
#pragma unroll
    for (int t = 0; t < M; ++t) {
      float sc[kRPW] = {};
      const float* kr = sK + lane * kld + t * a.dim;
      const float* qr = sQ + warp * kRPW * kd + t * a.dim;
      for (int c = 0; c < a.dim; ++c) {
        const float kv = kr[c];
#pragma unroll
        for (int r = 0; r < kRPW; ++r) sc[r] = fmaf(qr[r * kd + c], kv, sc[r]);
      }
#pragma unroll
      for (int r = 0; r < kRPW; ++r) {
        const int pos = start + q0 + warp * kRPW + r;
        const float v = (k0 + lane < n_keys && key_visible(pos, k0 + lane, a.window, a.keep_first)) ? sc[r] : -INFINITY;
        const float mn = fmaxf(m[r][t], warp_max(v));
        const float p = mn == -INFINITY ? 0.f : expf(v - mn);
        const float al = mn == -INFINITY ? 1.f : expf(m[r][t] - mn);
        l[r][t] = l[r][t] * al + warp_sum(p);
        m[r][t] = mn;
#pragma unroll
        for (int i = 0; i < NC; ++i) acc[r][t][i] *= al;
        sc[r] = p;
      }
      for (int j = 0; j < kTK; ++j) {
        float p[kRPW];
#pragma unroll
        for (int r = 0; r < kRPW; ++r) p[r] = __shfl_sync(0xffffffffu, sc[r], j);
#pragma unroll
        for (int i = 0; i < NC; ++i) {
          const int c = lane + 32 * i;
          const float v = c < a.vdim ? sV[j * a.vdim + c] : 0.f;
#pragma unroll
          for (int r = 0; r < kRPW; ++r) acc[r][t][i] = fmaf(p[r], v, acc[r][t][i]);
        }
      }
    }
  }
#pragma unroll
  for (int r = 0; r < kRPW; ++r) {
    const int row = q0 + warp * kRPW + r;
    if (row >= n_rows) continue;
    float o[NC];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NC; ++i) {
      o[i] = l[r][0] > 0.f ? acc[r][0][i] / l[r][0] : 0.f;
      if constexpr (M == 2) o[i] -= l[r][M - 1] > 0.f ? a.lambda * (acc[r][M - 1][i] / l[r][M - 1]) : 0.f;
      ss = fmaf(o[i], o[i], ss);
    }
    float f = 1.f;
    if constexpr (M == 2) {
      ss = warp_sum(ss);
      f = a.out_scale / sqrtf(ss / (float)a.vdim + a.eps);
    }
    T* op = out + (int64_t)(r_begin + row) * a.out_rs + (int64_t)h * a.vdim;
    const T* gp = a.gate == nullptr ? nullptr : static_cast<const T*>(a.gate) + (int64_t)(r_begin + row) * a.gate_rs + (int64_t)h * a.vdim;
#pragma unroll
    for (int i = 0; i < NC; ++i) {
      const int c = lane + 32 * i;
      if (c < a.vdim) op[c] = from_f32<T>(o[i] * f * (gp != nullptr ? sigmoid_gate(gp[c]) : 1.f));
    }
  }
}

int64_t rows_smem(const atma_softmax_args& a) {
  const int64_t kd = (int64_t)a.maps * a.dim;
  return 4 * (kTK * (kd + 1) + (int64_t)kTK * a.vdim + kTQ * kd);
}

template <typename T, int M, int NC>
int launch_rows(const atma_softmax_args& a, int max_rows, cudaStream_t st) {
  auto kern = softmax_rows_kernel<T, M, NC>;
  const int smem = (int)rows_smem(a);
  ATMA_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
  kern<<<dim3((max_rows + kTQ - 1) / kTQ, a.H, a.n_seqs), kWarps * 32, smem, st>>>(a);
  return launch_status("softmax attention (fp32 arithmetic)");
}

template <typename T>
int launch_rows_t(const atma_softmax_args& a, int max_rows, cudaStream_t st) {
  const int nc = (a.vdim + 31) / 32;
#define ATMA_ROWS(NCV) (a.maps == 1 ? launch_rows<T, 1, NCV>(a, max_rows, st) : launch_rows<T, 2, NCV>(a, max_rows, st))
  if (nc <= 1) return ATMA_ROWS(1);
  if (nc <= 2) return ATMA_ROWS(2);
  if (nc <= 4) return ATMA_ROWS(4);
  if (nc <= 8) return ATMA_ROWS(8);
  return ATMA_ROWS(16);
#undef ATMA_ROWS
}

int check(const atma_softmax_args* a, const char* what) {
  ATMA_REQUIRE(a != nullptr, "%s: null args", what);
  ATMA_REQUIRE(a->dtype == ATMA_F32 || a->dtype == ATMA_BF16, "%s: unsupported dtype %d", what, a->dtype);
  ATMA_REQUIRE(a->H > 0 && a->G > 0 && a->H % a->G == 0, "%s: %d query heads over %d key/value heads", what, a->H, a->G);
  ATMA_REQUIRE(a->maps == 1 || a->maps == 2, "%s: %d maps per head", what, a->maps);
  ATMA_REQUIRE(a->dim > 0 && a->vdim > 0 && a->vdim <= 512, "%s: head sizes %d / %d (value channels up to 512)", what, a->dim, a->vdim);
  ATMA_REQUIRE(a->block_size > 0 && a->num_blocks > 0 && a->max_blocks > 0, "%s: empty cache", what);
  ATMA_REQUIRE(rows_smem(*a) <= 227 * 1024, "%s: head sizes %d / %d do not fit shared memory", what, a->dim, a->vdim);
  ATMA_REQUIRE(a->n_seqs <= 65535 && a->H <= 65535, "%s: grid limits", what);
  return ATMA_OK;
}

// Window and kept first keys within what index arithmetic on positions takes without overflow.
atma_softmax_args bounded(const atma_softmax_args& a) {
  constexpr int kMost = 1 << 30;
  atma_softmax_args b = a;
  b.window = min(max(a.window, 0), kMost);
  b.keep_first = min(max(a.keep_first, 0), kMost);
  return b;
}

int rows_path(const atma_softmax_args& a, int max_rows, cudaStream_t st) {
  return a.dtype == ATMA_F32 ? launch_rows_t<float>(a, max_rows, st) : launch_rows_t<__nv_bfloat16>(a, max_rows, st);
}

}  // namespace
}  // namespace atma

using namespace atma;

extern "C" int atma_softmax_prefill_path(const atma_softmax_args* a) { return a != nullptr && softmax_prefill_sm100_supported(*a) ? 1 : 0; }
extern "C" int atma_softmax_decode_path(const atma_softmax_args* a) { return a != nullptr && softmax_decode_mma_supported(*a) ? 1 : 0; }

extern "C" int atma_softmax_prefill(const atma_softmax_args* a, void* stream) {
  int rc = check(a, "softmax_prefill");
  if (rc != ATMA_OK) return rc;
  if (a->n_seqs <= 0 || a->max_rows <= 0) return ATMA_OK;
  const atma_softmax_args b = bounded(*a);
  if (softmax_prefill_sm100_supported(b)) return softmax_prefill_sm100(b, (cudaStream_t)stream);
  return rows_path(b, b.max_rows, (cudaStream_t)stream);
}

extern "C" int atma_softmax_decode(const atma_softmax_args* a, void* stream) {
  int rc = check(a, "softmax_decode");
  if (rc != ATMA_OK) return rc;
  if (a->n_seqs <= 0) return ATMA_OK;
  if (softmax_decode_mma_supported(*a)) {
    ATMA_REQUIRE(a->scratch != nullptr && a->n_splits > 0, "softmax_decode: scratch and n_splits are required");
    return softmax_decode_mma(bounded(*a), (cudaStream_t)stream);
  }
  return rows_path(bounded(*a), 1, (cudaStream_t)stream);
}

extern "C" int64_t atma_softmax_decode_scratch_floats(int n_seqs, int H, int maps, int vdim, int n_splits) {
  return (int64_t)n_seqs * H * maps * n_splits * (2 + (int64_t)vdim);
}

extern "C" int atma_decoder_device_status(int* status) {
  ATMA_REQUIRE(status != nullptr, "decoder_device_status: null out pointer");
  int a = 0, b = 0;
  int rc = softmax_sm100_status_fetch_and_clear(&a);
  if (rc == ATMA_OK) rc = delta_sm100_status_fetch_and_clear(&b);
  *status = a | b;
  return rc;
}
