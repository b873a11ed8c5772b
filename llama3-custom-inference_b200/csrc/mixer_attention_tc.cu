#include "mixer_attention.h"
namespace l3ci {
bool mixer_tc_applies(const l3ci_mixer_attn_args*) { return false; }
size_t mixer_tc_scratch_bytes(const l3ci_mixer_attn_args*) { return 0; }
int mixer_tc_launch(const l3ci_mixer_attn_args*) { return L3CI_ERR_UNSUPPORTED; }
}  // namespace l3ci
