// Shared between the softmax-attention kernels of the decoder models: which shapes the tensor-core kernels serve.
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

}  // namespace atma
