#include "blocks.cuh"
namespace sk {
bool attn_decode_mma_applicable(const sk_attn_params& p) { return false; }
size_t attn_decode_mma_workspace(const sk_attn_params& p) { return 0; }
int launch_attn_decode_mma(const sk_attn_params& p, cudaStream_t st) { return SK_ERR_UNSUPPORTED; }
bool attn_prefill_tc_applicable(const sk_attn_params& p) { return false; }
int launch_attn_prefill_tc(const sk_attn_params& p, cudaStream_t st) { return SK_ERR_UNSUPPORTED; }
bool ssm_chunks_applicable(const sk_ssm_params& p) { return false; }
size_t ssm_chunks_workspace(const sk_ssm_params& p) { return 0; }
int launch_ssm_chunks(const sk_ssm_params& p, cudaStream_t st) { return SK_ERR_UNSUPPORTED; }
}
