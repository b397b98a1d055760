#include "softmax_attention.cuh"
namespace atma {
bool softmax_prefill_sm100_supported(const atma_softmax_args& a) { return false; }
int softmax_prefill_sm100(const atma_softmax_args& a, cudaStream_t st) { return ATMA_ERR_UNSUPPORTED; }
int softmax_sm100_status_fetch_and_clear(int* out) { *out = 0; return ATMA_OK; }
}
