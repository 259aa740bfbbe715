// What a query of the grouped-query attention kernels sees.
#pragma once
#include <cuda_runtime.h>

namespace seqmix {

// the first position that position i sees: at most `window` back, and (chunk > 0) not before its own aligned run of `chunk` positions
__device__ __forceinline__ int first_visible(int i, int window, int chunk) {
    const int lo = max(0, i - window + 1);
    return chunk > 0 ? max(lo, i / chunk * chunk) : lo;
}

}  // namespace seqmix
