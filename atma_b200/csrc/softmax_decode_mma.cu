#include "softmax_attention.cuh"
namespace atma {
bool softmax_decode_mma_supported(const atma_softmax_args& a) { return false; }
int softmax_decode_mma(const atma_softmax_args& a, cudaStream_t st) { return ATMA_ERR_UNSUPPORTED; }
}
