// Recurrences over a prompt portion in chunks: what lt_dn_chunk.cu (decays per key channel or per head) and
// lt_dn_ssd_chunk.cu (state-space form) share.
#pragma once
#include "lt_dn_common.cuh"

namespace lt {
namespace dn {

constexpr int CH = 64;                         // tokens of a chunk
constexpr float LOG2E = 1.4426950408889634f;   // the kernels keep log decays to base 2

struct SsdChunkP {
    const bf16 *q, *k, *v;
    float *S, *o, *ws;               // ws [chunk][H][dvp][dp rounded up to 16]: states the chunks start from
    const float *hla, *hdt, *D;      // [T][ldh] log decays and step sizes, [H]
    int ld, ldo, T, H, dp, dvp, nchunk, ldh;
    int per;                         // consecutive heads that share q and k
    int hpc, nb;                     // heads of a CTA of the output pass, such CTAs of a group of heads
};
int launch_ssd_chunked(const SsdChunkP& P, cudaStream_t s);

}  // namespace dn
}  // namespace lt
