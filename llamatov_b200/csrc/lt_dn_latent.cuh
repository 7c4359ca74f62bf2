// Host check of the description of a latent attention layer.
#pragma once
#include "lt_dn_common.cuh"

namespace lt {
namespace dn {

inline const char* latent_error(const lt_dn_latent* L) {
    if (L == nullptr) return "null description";
    if (L->H <= 0 || L->dp < 0 || L->rtp < 0 || L->dvp <= 0 || L->rp <= 0) return "sizes must be positive";
    if (L->dp % 8 || L->rtp % 8 || L->dvp % 8 || L->rp % 8) return "padded sizes must be multiples of 8";
    if (L->rot < 0 || L->rot % 2 || L->rot > L->rtp) return "rotated dimensions must be even and fit their padded size";
    if (L->rank <= 0 || L->rank > L->rp) return "latent size";
    if (L->window <= 0 || L->cap <= 0) return "window and ring must be positive";
    if (L->cnorm == nullptr || (L->rot > 0 && L->freq == nullptr)) return "null constants";
    return nullptr;
}

}  // namespace dn
}  // namespace lt
