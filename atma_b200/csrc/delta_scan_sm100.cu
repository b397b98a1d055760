#include "delta_rule.cuh"
namespace atma {
bool delta_scan_sm100_supported(const atma_delta_args& a) { return false; }
int64_t delta_scan_sm100_scratch_bytes(const atma_delta_args& a) { return 0; }
int delta_scan_sm100(const atma_delta_args& a, const void* q, const void* k, const void* v, const float* q_inv, const float* k_inv,
                     const float* log_decay, const float* beta, void* o, void* scratch, cudaStream_t st) { return ATMA_ERR_UNSUPPORTED; }
int delta_sm100_status_fetch_and_clear(int* out) { *out = 0; return ATMA_OK; }
}
