// Latent attention, expanded form for long portions: not there yet, every portion takes the absorbed form.
#include "tlc_dense.cuh"

namespace tlc_dense {

bool latent_prefill_fits(int, int, int) { return false; }
int32_t launch_latent_prefill(tlc_ctx *, const LatentParams &) {
    return tlc_fail(TLC_ERR_INVALID_OPERATION, "latent attention: no expanded form");
}

}  // namespace tlc_dense
