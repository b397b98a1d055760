// Shared between the softmax-attention kernels of the decoder models: which shapes the tensor-core kernels serve, which
// keys a row sees and which key tiles a block of rows needs.
#pragma once

#include "common.cuh"
#include "../../include/atma_decoder.h"

namespace atma {

bool softmax_prefill_sm100_supported(const atma_softmax_args& a);
int softmax_prefill_sm100(const atma_softmax_args& a, cudaStream_t st);
bool softmax_decode_mma_supported(const atma_softmax_args& a);
int softmax_decode_mma(const atma_softmax_args& a, cudaStream_t st);
int softmax_sm100_status_fetch_and_clear(int* out);
int delta_sm100_status_fetch_and_clear(int* out);

// A row at position pos sees key j <= pos if it is among the first `keep` or fewer than `window` positions back.
__device__ __forceinline__ bool key_visible(int pos, int key, int window, int keep) {
  return key <= pos && (pos - key < window || key < keep);
}

// Key tiles of `tile` keys that rows at positions first .. last need, in ascending order: those with kept first keys that
// lie before the first row's window, then from that window's first key to the last row's own.
struct KeyTiles {
  int n_kept, t_lo, n;
  __device__ __forceinline__ KeyTiles(int first, int last, int n_cached, int window, int keep, int tile) {
    const int n_keys = min(last + 1, n_cached);
    if (n_keys <= 0) { n_kept = t_lo = n = 0; return; }
    const int t_end = (n_keys - 1) / tile + 1;
    t_lo = min(max(first - window + 1, 0) / tile, t_end);
    n_kept = min((min(max(keep, 0), n_keys) + tile - 1) / tile, t_lo);
    n = n_kept + t_end - t_lo;
  }
  __device__ __forceinline__ int operator[](int j) const { return j < n_kept ? j : t_lo + (j - n_kept); }
};

template <typename T>
__device__ __forceinline__ float sigmoid_gate(T z) { return 1.0f / (1.0f + expf(-to_f32(z))); }

}  // namespace atma
