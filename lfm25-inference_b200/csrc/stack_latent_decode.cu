#include "stack_latent.h"
namespace lfm25 {
bool latent_attention_umma_supports(const LatentAttentionLaunch&) { return false; }
cudaError_t launch_latent_attention_umma(cudaStream_t, const LatentAttentionLaunch&) { return cudaErrorInvalidValue; }
bool expanded_attention_supports(Activation, const LatentAttentionShape&, size_t, size_t, size_t) { return false; }
cudaError_t launch_expanded_attention(cudaStream_t, const ExpandedAttentionLaunch&) { return cudaErrorInvalidValue; }
}
