// The tensor-core tiles of b200_paged_attention for scores that carry a learned bias per distance and a learned sink per head.
// Two key widths and three value widths are built; sizes in between run on the next larger tile.
#include "common.cuh"
#include "paged_attention_tile.cuh"

namespace b200 {

template <int D>
static int biased_tile_v(const PA& a, cudaStream_t s) {
    if (a.vdim <= 64) return launch_tile<D, 64, true>(a, s);
    if (a.vdim <= 128) return launch_tile<D, 128, true>(a, s);
    if (a.vdim <= 256) return launch_tile<D, 256, true>(a, s);
    return -1;
}

int biased_tile(const PA& a, cudaStream_t s) {
    if (a.dim <= 64) return biased_tile_v<64>(a, s);
    if (a.dim <= 128) return biased_tile_v<128>(a, s);
    return -1;
}

}  // namespace b200
