#include "mixer_attention.h"
namespace l3ci {
bool mixer_mma_applies(const l3ci_mixer_attn_args*) { return false; }
size_t mixer_mma_scratch_bytes(const l3ci_mixer_attn_args*) { return 0; }
int mixer_mma_launch(const l3ci_mixer_attn_args*) { return L3CI_ERR_UNSUPPORTED; }
}  // namespace l3ci
