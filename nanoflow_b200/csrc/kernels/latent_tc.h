// tcgen05 form of the latent attention kernel (latent_tc.cu), chosen by nfk_latent_attn.
#pragma once
#include "common.cuh"
#include "kernels.h"

namespace nf {
bool latent_tc_built(long long ld);      // row sizes it exists for
// Checked parameters, bf16, 16-token pages; with splits > 1 partial results go to the workspace.
int latent_tc_launch(const nfk_latent_attn_params& p, cudaStream_t stream);
}  // namespace nf
