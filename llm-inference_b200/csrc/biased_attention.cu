// The tensor-core tiles of b200_paged_attention for scores that carry a learned bias per distance and / or a learned sink per head:
// the usual head sizes without a mask exactly, everything else (up to 128 key and 256 value dimensions in multiples of 8, with or
// without a block mask or a window) on the next larger tile.
#include "common.cuh"
#include "paged_attention_tile.cuh"

namespace b200 {

template <int D>
static int biased_tile_padded(const PA& a, cudaStream_t s) {
    if (a.vdim <= 64) return launch_tile<D, 64, kBiasPadded>(a, s);
    if (a.vdim <= 128) return launch_tile<D, 128, kBiasPadded>(a, s);
    if (a.vdim <= 256) return launch_tile<D, 256, kBiasPadded>(a, s);
    return -1;
}

int biased_tile(const PA& a, cudaStream_t s) {
    if (a.chunk == 0 && a.window == 0) {
        if (a.dim == 64 && a.vdim == 64) return launch_tile<64, 64, kBias, false>(a, s);
        if (a.dim == 64 && a.vdim == 128) return launch_tile<64, 128, kBias, false>(a, s);
        if (a.dim == 128 && a.vdim == 128) return launch_tile<128, 128, kBias, false>(a, s);
        if (a.dim == 128 && a.vdim == 256) return launch_tile<128, 256, kBias, false>(a, s);
    }
    if (a.dim <= 64) return biased_tile_padded<64>(a, s);
    if (a.dim <= 128) return biased_tile_padded<128>(a, s);
    return -1;
}

}  // namespace b200
