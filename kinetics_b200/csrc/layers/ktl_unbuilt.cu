#include "ktl_common.cuh"
namespace ktk {
bool attn_decode_supported(const ktk_attn&) { return false; }
int32_t attn_decode_splits(const ktk_attn&, int, int64_t) { return 1; }
size_t attn_decode_workspace(const ktk_attn&, int64_t, int) { return 0; }
int launch_attn_decode(const AttnParams&, cudaStream_t) { return KTK_ERR_UNSUPPORTED; }
bool attn_umma_supported(const ktk_attn&) { return false; }
int launch_attn_umma(const AttnParams&, cudaStream_t) { return KTK_ERR_UNSUPPORTED; }
bool moe_umma_supported(const ktk_moe&) { return false; }
int launch_moe_umma(int, const MoeParams&, cudaStream_t) { return KTK_ERR_UNSUPPORTED; }
}
