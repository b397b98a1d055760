// The tensor-core path of the delta rule's recurrence (delta_scan_sm100.cu), as the entry points see it.
#pragma once

#include "common.cuh"
#include "../../include/atma_decoder.h"

namespace atma {

bool delta_scan_sm100_supported(const atma_delta_args& a);
int64_t delta_scan_sm100_scratch_bytes(const atma_delta_args& a);
int delta_scan_sm100(const atma_delta_args& a, const void* q, const void* k, const void* v, const float* q_inv, const float* k_inv,
                     const float* log_decay, const float* beta, void* o, void* scratch, cudaStream_t st);

}  // namespace atma
